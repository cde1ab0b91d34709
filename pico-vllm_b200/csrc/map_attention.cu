// What stands around the paged attention kernels when a head has several maps (differential attention): M attentions with
// queries and keys of their own over the same values, combined afterwards.
//
// The M key maps of a key/value head lie side by side in ONE cached key row [map 1 | map 2 | ...] of M * d numbers, and a
// query map becomes a row of that size which is zero everywhere but in its own map's place, so that its product with the key
// row is the product with its own map.  The attention kernels then see M * H query heads over G key/value heads: every
// key and value is cached once and read once for all maps.
//
// map_rope_store_kernel    from a projection row [q: H * M * d | k: G * M * d | v: G * dv]: rotation of the first rot_dim
//                          numbers of each map (i with i + rot_dim / 2, by position * inv_freq[i], cos and sin times `mult`),
//                          queries spread out into rows of `row` numbers, keys and values into the token's place of the pages
//                          [pages, G, page_size, row] (slot = page * page_size + offset; -1: not stored), zero-padded to `row`.
// map_difference_kernel    o = a_1 - lambda * a_2 per head, o <- o / sqrt(mean(o^2) + eps) * factor * sigmoid(gate_h): from the
//                          attention kernels' rows [T, H, 2, row] to [T, H * dv].
// All arithmetic in float32; inputs and outputs in the activation type.
#include "common.cuh"

struct MapArgs {
    int row_stride, q_off, k_off, v_off;
    int H, G, M, d, dv, row, page_size, rot_half;
    float mult;
    const int* positions;
    const int* slots;
    const float* inv_freq;
};

// A block per token, its cos and sin in shared memory; a thread takes W neighbouring numbers of an output row: 16 bytes
// (d, dv, row and all offsets multiples of W = 16 / sizeof(TA)) or one.
template <typename TA, int W>
__global__ void __launch_bounds__(256) map_rope_store_kernel(const TA* __restrict__ proj, TA* __restrict__ k_pages, TA* __restrict__ v_pages,
                                                             TA* __restrict__ q_out, const MapArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float mr_cs[];                     // cos[rot_half], sin[rot_half]
    const size_t t = blockIdx.x;
    const int pos = p.positions[t];
    const int slot = p.slots ? p.slots[t] : -1;
    if (pos >= 0)
        for (int i = threadIdx.x; i < p.rot_half; i += blockDim.x) {
            float s, c;
            sincosf((float)pos * p.inv_freq[i], &s, &c);
            mr_cs[i] = c * p.mult;
            mr_cs[p.rot_half + i] = s * p.mult;
        }
    __syncthreads();
    const int per = p.row / W, nq = p.H * p.M, rot = pos >= 0 ? 2 * p.rot_half : 0;
    const int total = (nq + (slot >= 0 ? 2 * p.G : 0)) * per;
    const TA* in = proj + t * p.row_stride;
    for (int idx = threadIdx.x; idx < total; idx += blockDim.x) {
        const int head = idx / per, e0 = (idx - head * per) * W;
        const TA* src;                                   // the map (or value head) this thread's numbers belong to; null: zeros
        int i0, n;                                       // first number within it, and how many it turns
        TA* dst;
        if (head < nq) {
            const int m = head % p.M;
            i0 = e0 - m * p.d;
            src = i0 >= 0 && i0 < p.d ? in + p.q_off + head * p.d : nullptr;
            n = rot;
            dst = q_out + (t * nq + head) * (size_t)p.row + e0;
        } else {
            const bool key = head < nq + p.G;
            const int g = head - nq - (key ? 0 : p.G);
            const int width = key ? p.M * p.d : p.dv;
            const int m = key ? e0 / p.d : 0;
            i0 = e0 - m * p.d;
            src = e0 < width ? in + (key ? p.k_off + (g * p.M + m) * p.d : p.v_off + g * p.dv) : nullptr;
            n = key ? rot : 0;
            dst = (key ? k_pages : v_pages) + (((size_t)(slot / p.page_size) * p.G + g) * p.page_size + slot % p.page_size) * (size_t)p.row + e0;
        }
        if constexpr (W == 1) {
            float y = 0.f;
            if (src) {
                y = to_f32(src[i0]);
                if (i0 < n) {
                    const bool low = i0 < p.rot_half;
                    const int i = low ? i0 : i0 - p.rot_half;
                    const float other = to_f32(src[low ? i0 + p.rot_half : i]);
                    y = low ? y * mr_cs[i] - other * mr_cs[p.rot_half + i] : y * mr_cs[i] + other * mr_cs[p.rot_half + i];
                }
            }
            *dst = from_f32<TA>(y);
        } else {
            uint4 raw = make_uint4(0u, 0u, 0u, 0u);
            if (src) {
                raw = *reinterpret_cast<const uint4*>(src + i0);
                if (i0 < n) {
                    TA* v = reinterpret_cast<TA*>(&raw);
                    if (p.rot_half % W == 0) {           // the partners are one vector too
                        const bool low = i0 < p.rot_half;
                        const int i1 = low ? i0 : i0 - p.rot_half;
                        const uint4 oraw = *reinterpret_cast<const uint4*>(src + (low ? i0 + p.rot_half : i1));
                        const TA* o = reinterpret_cast<const TA*>(&oraw);
                        const float sign = low ? -1.0f : 1.0f;
#pragma unroll
                        for (int k = 0; k < W; ++k)
                            v[k] = from_f32<TA>(to_f32(v[k]) * mr_cs[i1 + k] + sign * (to_f32(o[k]) * mr_cs[p.rot_half + i1 + k]));
                    } else {
#pragma unroll
                        for (int k = 0; k < W; ++k) {
                            const int e = i0 + k;
                            if (e < n) {
                                const bool low = e < p.rot_half;
                                const int i = low ? e : e - p.rot_half;
                                const float other = to_f32(src[low ? e + p.rot_half : i]), s = mr_cs[p.rot_half + i];
                                v[k] = from_f32<TA>(to_f32(v[k]) * mr_cs[i] + (low ? -other * s : other * s));
                            }
                        }
                    }
                }
            }
            *reinterpret_cast<uint4*>(dst) = raw;
        }
    }
}

template <typename TA>
static void launch_map_rope_store(const void* proj, void* k_pages, void* v_pages, void* q_out, const MapArgs& p, int T, cudaStream_t stream) {
    constexpr int W = 16 / (int)sizeof(TA);
    const bool vec = (((uintptr_t)proj | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_out) & 15) == 0 && p.d % W == 0 &&
                     p.dv % W == 0 && p.row % W == 0 && p.q_off % W == 0 && p.k_off % W == 0 && p.v_off % W == 0 && p.row_stride % W == 0;
    const size_t smem = (size_t)2 * p.rot_half * sizeof(float);
    const int items = (p.H * p.M + 2 * p.G) * (vec ? p.row / W : p.row);
    const int threads = items <= 128 ? 128 : 256;
    if (vec)
        pico_launch((map_rope_store_kernel<TA, W>), dim3(T), dim3(threads), smem, stream, (const TA*)proj, (TA*)k_pages, (TA*)v_pages, (TA*)q_out, p);
    else
        pico_launch((map_rope_store_kernel<TA, 1>), dim3(T), dim3(threads), smem, stream, (const TA*)proj, (TA*)k_pages, (TA*)v_pages, (TA*)q_out, p);
}

// proj rows of row_stride elements; inv_freq float32 [rot_half], 2 * rot_half <= d; slots int32 [T] or nullptr (queries only);
// q_out [T, H * M * row]; pages [pages, G, page_size, row] with row >= M * d and row >= dv.  A token of position -1 is not turned.
PICO_API int pico_map_rope_store(const void* proj, int row_stride, int q_off, int k_off, int v_off, const int* positions,
                                 const float* inv_freq, int rot_half, float mult, const int* slots, void* k_pages, void* v_pages,
                                 void* q_out, int T, int H, int G, int M, int d, int dv, int row, int page_size, int dtype,
                                 cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H < 1 || G < 1 || M < 1 || d < 1 || dv < 1 || row < M * d || row < dv || rot_half < 0 || 2 * rot_half > d || rot_half > 4096 ||
        page_size < 1 || !positions || !q_out || (rot_half > 0 && !inv_freq) || (slots && (!k_pages || !v_pages)))
        return PICO_ERR_SIZE;
    const MapArgs p = {row_stride, q_off, k_off, v_off, H, G, M, d, dv, row, page_size, rot_half, mult, positions, slots, inv_freq};
    if (dtype == PICO_F32) launch_map_rope_store<float>(proj, k_pages, v_pages, q_out, p, T, stream);
    else if (dtype == PICO_BF16) launch_map_rope_store<bf16>(proj, k_pages, v_pages, q_out, p, T, stream);
    else return PICO_ERR_DTYPE;
    return pico_launch_status();
}

// L lanes (a power of two, at least dv / W) take a head; heads of all tokens one after the other.  16 bytes per access.
template <typename TA, int L>
__global__ void __launch_bounds__(256) map_difference_vec_kernel(const TA* __restrict__ a, const TA* __restrict__ gate, int gate_stride,
                                                                 float lambda, float eps, float factor, TA* __restrict__ y, int heads,
                                                                 int row, int dv, int items) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int W = 16 / (int)sizeof(TA);
    const int item = blockIdx.x * (256 / L) + threadIdx.x / L;
    const bool live = item < items;                      // lanes of a warp stay together for the shuffles
    const int e0 = (threadIdx.x % L) * W;
    uint4 r1 = make_uint4(0u, 0u, 0u, 0u), r2 = r1;
    float z = 0.f;
    if (live && e0 < dv) {
        const TA* src = a + (size_t)item * 2 * row + e0;
        r1 = *reinterpret_cast<const uint4*>(src);
        r2 = *reinterpret_cast<const uint4*>(src + row);
        const int t = item / heads;
        if (gate) z = to_f32(gate[(size_t)t * gate_stride + item - t * heads]);
    }
    const TA* x1 = reinterpret_cast<const TA*>(&r1);
    const TA* x2 = reinterpret_cast<const TA*>(&r2);
    float v[W], ss = 0.f;
#pragma unroll
    for (int k = 0; k < W; ++k) {
        v[k] = fmaf(-lambda, to_f32(x2[k]), to_f32(x1[k]));
        ss = fmaf(v[k], v[k], ss);
    }
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live || e0 >= dv) return;
    float f = factor / sqrtf(ss / (float)dv + eps);
    if (gate) f /= 1.0f + expf(-z);
    uint4 res;
    TA* o = reinterpret_cast<TA*>(&res);
#pragma unroll
    for (int k = 0; k < W; ++k) o[k] = from_f32<TA>(v[k] * f);
    *reinterpret_cast<uint4*>(y + (size_t)item * dv + e0) = res;
}

// Any sizes: a warp per head.
template <typename TA>
__global__ void __launch_bounds__(256) map_difference_kernel(const TA* __restrict__ a, const TA* __restrict__ gate, int gate_stride,
                                                             float lambda, float eps, float factor, TA* __restrict__ y, int heads, int row,
                                                             int dv, int items) {
    pdl_launch_dependents();
    pdl_wait();
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= items) return;
    const TA* x1 = a + (size_t)item * 2 * row;
    const TA* x2 = x1 + row;
    float ss = 0.f;
    for (int e = lane; e < dv; e += 32) {
        const float v = fmaf(-lambda, to_f32(x2[e]), to_f32(x1[e]));
        ss = fmaf(v, v, ss);
    }
    float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
    if (gate) {
        const int t = item / heads;
        f /= 1.0f + expf(-to_f32(gate[(size_t)t * gate_stride + item - t * heads]));
    }
    for (int e = lane; e < dv; e += 32) y[(size_t)item * dv + e] = from_f32<TA>(fmaf(-lambda, to_f32(x2[e]), to_f32(x1[e])) * f);
}

template <typename TA>
static void launch_map_difference(const void* a, const void* gate, int gate_stride, float lambda, float eps, float factor, void* y, int heads,
                                  int row, int dv, int items, cudaStream_t stream) {
    constexpr int W = 16 / (int)sizeof(TA);
    if ((((uintptr_t)a | (uintptr_t)y) & 15) == 0 && row % W == 0 && dv % W == 0 && dv <= 32 * W) {
#define MD_LAUNCH(LN)                                                                                                          \
    pico_launch((map_difference_vec_kernel<TA, LN>), dim3((items + 256 / LN - 1) / (256 / LN)), dim3(256), 0, stream, (const TA*)a, \
                (const TA*)gate, gate_stride, lambda, eps, factor, (TA*)y, heads, row, dv, items)
        const int need = dv / W;
        if (need <= 4) MD_LAUNCH(4);
        else if (need <= 8) MD_LAUNCH(8);
        else if (need <= 16) MD_LAUNCH(16);
        else MD_LAUNCH(32);
#undef MD_LAUNCH
        return;
    }
    pico_launch((map_difference_kernel<TA>), dim3((items + 7) / 8), dim3(256), 0, stream, (const TA*)a, (const TA*)gate, gate_stride, lambda,
                eps, factor, (TA*)y, heads, row, dv, items);
}

// a [T, heads, 2, row]; gate (rows of gate_stride elements, one logit a head) or nullptr; y [T, heads * dv].
PICO_API int pico_map_difference(const void* a, const void* gate, int gate_stride, float lambda, float eps, float factor, void* y, int T,
                                 int heads, int row, int dv, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (heads < 1 || dv < 1 || row < dv || (long long)T * heads > 0x7fffffffLL) return PICO_ERR_SIZE;
    if (dtype == PICO_F32) launch_map_difference<float>(a, gate, gate_stride, lambda, eps, factor, y, heads, row, dv, T * heads, stream);
    else if (dtype == PICO_BF16) launch_map_difference<bf16>(a, gate, gate_stride, lambda, eps, factor, y, heads, row, dv, T * heads, stream);
    else return PICO_ERR_DTYPE;
    return pico_launch_status();
}
