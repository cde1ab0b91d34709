// Queries and keys on their way into paged attention when each head is divided by its own root mean square, and values that
// are moved towards another layer's values of the same token:
//
//   q_a <- q_a / sqrt(mean(q_a^2) + eps),  k_g likewise over the head's d numbers, no weight           (optional)
//   v_g <- (1 - lambda) v_g + lambda first_g                                                            (optional; lambda one number)
//
// q goes to a buffer of its own with heads of `row` elements (zeros beyond d: the attention kernels want one size for queries,
// keys and values), k and v to the token's place in the pages [pages, G, page_size, row] (slot = page * page_size + offset;
// -1: not stored).  No positions are encoded here.  Float32 arithmetic; inputs and outputs in the activation type.
#include "common.cuh"

struct HeadNormArgs {
    int row_stride, q_off, k_off, v_off, first_stride;
    int T, H, G, d, dv, row, page_size, norm;
    float eps;
    const float* lambda;      // one number on the device, or null: values pass
    const int* slots;
};

// Where head `a` of token t goes: null when it is not stored.  kind: 0 query, 1 key, 2 value.
template <typename TA>
__device__ __forceinline__ TA* head_dst(const HeadNormArgs& p, size_t t, int kind, int a, TA* q_out, TA* k_pages, TA* v_pages) {
    if (kind == 0) return q_out + (t * p.H + a) * (size_t)p.row;
    const int slot = p.slots ? p.slots[t] : -1;
    if (slot < 0) return nullptr;
    return (kind == 1 ? k_pages : v_pages) + (((size_t)(slot / p.page_size) * p.G + a) * p.page_size + slot % p.page_size) * (size_t)p.row;
}

// 16 bytes per access: d, dv, offsets and strides are multiples of W = 16 / sizeof(TA), row <= 32 W.  L lanes (a power of two,
// at least row / W) take a head; heads of all tokens are dealt out one after the other.
template <typename TA, int L>
__global__ void __launch_bounds__(256) head_norm_store_vec_kernel(const TA* __restrict__ proj, const TA* __restrict__ first,
                                                                  TA* __restrict__ k_pages, TA* __restrict__ v_pages,
                                                                  TA* __restrict__ q_out, const HeadNormArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int W = 16 / (int)sizeof(TA);
    const int heads = p.H + 2 * p.G;
    const long long item = (long long)blockIdx.x * (256 / L) + threadIdx.x / L;
    const bool live = item < (long long)p.T * heads;                      // lanes of a warp stay together for the shuffles
    const size_t t = live ? (size_t)(item / heads) : 0;
    const int head = live ? (int)(item - (long long)t * heads) : 0;
    const int kind = head < p.H ? 0 : head < p.H + p.G ? 1 : 2;
    const int a = kind == 0 ? head : kind == 1 ? head - p.H : head - p.H - p.G;
    const int n = kind == 2 ? p.dv : p.d, e0 = (threadIdx.x % L) * W;
    const int off = (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + a * n;
    float v[W];
    uint4 raw = make_uint4(0u, 0u, 0u, 0u), rf = raw;
    const bool mix = kind == 2 && p.lambda != nullptr;
    if (live && e0 < n) {
        raw = *reinterpret_cast<const uint4*>(proj + t * p.row_stride + off + e0);
        if (mix) rf = *reinterpret_cast<const uint4*>(first + t * p.first_stride + a * n + e0);
    }
    const TA* x = reinterpret_cast<const TA*>(&raw);
    const TA* f = reinterpret_cast<const TA*>(&rf);
    const float lam = mix ? *p.lambda : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < W; ++k) {
        v[k] = to_f32(x[k]);
        if (mix) v[k] = (1.0f - lam) * v[k] + lam * to_f32(f[k]);
        ss = fmaf(v[k], v[k], ss);
    }
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = p.norm && kind < 2 ? 1.0f / sqrtf(ss / (float)n + p.eps) : 1.0f;
    if (!live || e0 >= p.row) return;
    TA* dst = head_dst<TA>(p, t, kind, a, q_out, k_pages, v_pages);
    if (!dst) return;
    uint4 y;
    TA* yo = reinterpret_cast<TA*>(&y);
#pragma unroll
    for (int k = 0; k < W; ++k) yo[k] = from_f32<TA>(v[k] * inv);
    *reinterpret_cast<uint4*>(dst + e0) = y;
}

// Any sizes: a warp per head.
template <typename TA>
__global__ void __launch_bounds__(256) head_norm_store_kernel(const TA* __restrict__ proj, const TA* __restrict__ first,
                                                              TA* __restrict__ k_pages, TA* __restrict__ v_pages,
                                                              TA* __restrict__ q_out, const HeadNormArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    const int heads = p.H + 2 * p.G, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= (long long)p.T * heads) return;
    const size_t t = (size_t)(item / heads);
    const int head = (int)(item - (long long)t * heads);
    const int kind = head < p.H ? 0 : head < p.H + p.G ? 1 : 2;
    const int a = kind == 0 ? head : kind == 1 ? head - p.H : head - p.H - p.G;
    const int n = kind == 2 ? p.dv : p.d;
    TA* dst = head_dst<TA>(p, t, kind, a, q_out, k_pages, v_pages);
    if (!dst) return;
    const TA* x = proj + t * p.row_stride + (kind == 0 ? p.q_off : kind == 1 ? p.k_off : p.v_off) + a * n;
    float inv = 1.0f;
    if (p.norm && kind < 2) {
        float ss = 0.f;
        for (int e = lane; e < n; e += 32) { const float u = to_f32(x[e]); ss = fmaf(u, u, ss); }
        inv = 1.0f / sqrtf(warp_sum(ss) / (float)n + p.eps);
    }
    const bool mix = kind == 2 && p.lambda != nullptr;
    const float lam = mix ? *p.lambda : 0.f;
    for (int e = lane; e < p.row; e += 32) {
        float u = e < n ? to_f32(x[e]) : 0.f;
        if (mix && e < n) u = (1.0f - lam) * u + lam * to_f32(first[t * p.first_stride + a * n + e]);
        dst[e] = from_f32<TA>(u * inv);
    }
}

template <typename TA>
static void launch_head_norm(const void* proj, const void* first, void* k_pages, void* v_pages, void* q_out, const HeadNormArgs& p,
                             cudaStream_t stream) {
    constexpr int W = 16 / (int)sizeof(TA);
    const long long items = (long long)p.T * (p.H + 2 * p.G);
    const bool aligned = ((uintptr_t)proj & 15) == 0 && ((uintptr_t)first & 15) == 0 && ((uintptr_t)k_pages & 15) == 0 &&
                         ((uintptr_t)v_pages & 15) == 0 && ((uintptr_t)q_out & 15) == 0;
    if (aligned && p.d % W == 0 && p.dv % W == 0 && p.row % W == 0 && p.row <= 32 * W && p.q_off % W == 0 && p.k_off % W == 0 &&
        p.v_off % W == 0 && p.row_stride % W == 0 && (!first || p.first_stride % W == 0)) {
#define HNS(LN)                                                                                                            \
    pico_launch((head_norm_store_vec_kernel<TA, LN>), dim3((unsigned)((items + 256 / LN - 1) / (256 / LN))), dim3(256), 0, stream, \
                (const TA*)proj, (const TA*)first, (TA*)k_pages, (TA*)v_pages, (TA*)q_out, p)
        const int need = p.row / W;
        if (need <= 4) HNS(4);
        else if (need <= 8) HNS(8);
        else if (need <= 16) HNS(16);
        else HNS(32);
#undef HNS
        return;
    }
    pico_launch((head_norm_store_kernel<TA>), dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, (const TA*)proj, (const TA*)first,
                (TA*)k_pages, (TA*)v_pages, (TA*)q_out, p);
}

// proj rows [q heads | k heads | v heads] at the given offsets; slots int32 [T] or nullptr; q_out [T, H * row]; pages
// [pages, G, page_size, row]; norm 0/1: queries and keys to unit root mean square; lambda (one float32 on the device) and
// first (rows of first_stride elements, the token's G * dv values): the value mixing, or both nullptr.
PICO_API int pico_head_norm_store(const void* proj, int row_stride, int q_off, int k_off, int v_off, int norm, float eps,
                                  const int* slots, void* k_pages, void* v_pages, void* q_out, const float* lambda,
                                  const void* first, int first_stride, int T, int H, int G, int d, int dv, int row,
                                  int page_size, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H < 1 || G < 1 || d < 1 || dv < 1 || row < d || row < dv || page_size < 1 || !q_out || (slots && (!k_pages || !v_pages)) ||
        ((lambda != nullptr) != (first != nullptr)) || (long long)T * (H + 2 * G) > 0x7fffffffLL)
        return PICO_ERR_SIZE;
    HeadNormArgs p;
    p.row_stride = row_stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.first_stride = first_stride;
    p.T = T; p.H = H; p.G = G; p.d = d; p.dv = dv; p.row = row; p.page_size = page_size; p.norm = norm;
    p.eps = eps; p.lambda = lambda; p.slots = slots;
    if (dtype == PICO_F32) launch_head_norm<float>(proj, first, k_pages, v_pages, q_out, p, stream);
    else if (dtype == PICO_BF16) launch_head_norm<bf16>(proj, first, k_pages, v_pages, q_out, p, stream);
    else return PICO_ERR_DTYPE;
    return pico_launch_status();
}
