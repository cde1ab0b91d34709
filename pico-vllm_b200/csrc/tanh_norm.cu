// A squashing in the place of a norm, fused with the adds into the residual stream that precede it:
//
//   x <- x + sum_i s_i * d_i                    (up to three terms in the activation type; the stream is float32)
//   y  = tanh(alpha * x) * w + b                (alpha one number, w and b a number per coordinate; float32 arithmetic)
//
// No statistics of a row enter, so every coordinate stands alone: a thread takes eight neighbours of a row (or one, where the
// width is no multiple of eight) and nothing is reduced or kept in shared memory.
#include "common.cuh"

struct TanhTerms {
    const void* d0;
    const void* d1;
    const void* d2;
    float s0, s1, s2;
};

template <typename TA> struct Vec8;
template <> struct Vec8<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[8]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
};
template <> struct Vec8<bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[8]) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(h[k]);
            v[2 * k] = f.x;
            v[2 * k + 1] = f.y;
        }
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[8]) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};

// W: 8 (the width a multiple of 8, everything 16-byte aligned) or 1.  items = rows * width / W.
template <typename TA, int W>
__global__ void __launch_bounds__(256) tanh_norm_kernel(float* __restrict__ x, const TanhTerms tm, const float* __restrict__ alpha,
                                                        const float* __restrict__ w, const float* __restrict__ b,
                                                        TA* __restrict__ out, const int* __restrict__ rows, int width, int items) {
    pdl_launch_dependents();
    pdl_wait();
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= items) return;
    const int per_row = width / W;
    const int r = idx / per_row, c = (idx - r * per_row) * W;
    const size_t src = (size_t)(rows ? rows[r] : r) * width + c;
    const TA* d[3] = {(const TA*)tm.d0, (const TA*)tm.d1, (const TA*)tm.d2};
    const float s[3] = {tm.s0, tm.s1, tm.s2};
    const float a = out ? *alpha : 0.f;
    if constexpr (W == 8) {
        float v[8], t[3][8], wv[8], bv[8];
        Vec8<float>::load(x + src, v);
#pragma unroll
        for (int k = 0; k < 3; ++k)
            if (d[k]) Vec8<TA>::load(d[k] + src, t[k]);
        if (out) {
            Vec8<float>::load(w + c, wv);
            Vec8<float>::load(b + c, bv);
        }
#pragma unroll
        for (int k = 0; k < 3; ++k)
            if (d[k]) {
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = fmaf(s[k], t[k][e], v[e]);
            }
        if (!rows && d[0]) Vec8<float>::store(x + src, v);
        if (!out) return;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = fmaf(tanhf(a * v[e]), wv[e], bv[e]);
        Vec8<TA>::store(out + (size_t)r * width + c, v);
    } else {
        float v = x[src];
#pragma unroll
        for (int k = 0; k < 3; ++k)
            if (d[k]) v = fmaf(s[k], to_f32(d[k][src]), v);
        if (!rows && d[0]) x[src] = v;
        if (out) out[(size_t)r * width + c] = from_f32<TA>(fmaf(tanhf(a * v), w[c], b[c]));
    }
}

// x float32 [*, width]; d0..d2 [*, width] in the activation type (a term is given only when the ones before it are) or nullptr;
// alpha float32 [1], w and b float32 [width]; out [R, width] or nullptr (the adds alone); rows int32 [R] or nullptr: row r is
// made from row rows[r] and x is left alone.
PICO_API int pico_tanh_norm(float* x, const void* d0, float s0, const void* d1, float s1, const void* d2, float s2, const float* alpha,
                            const float* w, const float* b, void* out, const int* rows, int R, int width, int act_dtype,
                            cudaStream_t stream) {
    if (R <= 0) return 0;
    if (width < 1 || (long long)R * width > 0x7fffffffLL || (out && (!alpha || !w || !b)) || (!d0 && (d1 || d2)) || (!d1 && d2))
        return PICO_ERR_SIZE;
    const uintptr_t at = (uintptr_t)x | (uintptr_t)d0 | (uintptr_t)d1 | (uintptr_t)d2 | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out;
    const bool vec = width % 8 == 0 && (at & 15) == 0;
    const int items = R * (vec ? width / 8 : width);
    const int threads = items >= 256 * pico_num_sms() ? 256 : 64;      // few rows: more, smaller blocks
    const dim3 grid((items + threads - 1) / threads);
    const TanhTerms tm = {d0, d1, d2, s0, s1, s2};
#define TN_LAUNCH(TA, W)                                                                                                    \
    pico_launch((tanh_norm_kernel<TA, W>), grid, dim3(threads), 0, stream, x, tm, alpha, w, b, (TA*)out, rows, width, items)
    if (act_dtype == PICO_F32) { if (vec) TN_LAUNCH(float, 8); else TN_LAUNCH(float, 1); }
    else if (act_dtype == PICO_BF16) { if (vec) TN_LAUNCH(bf16, 8); else TN_LAUNCH(bf16, 1); }
    else
        return PICO_ERR_DTYPE;
#undef TN_LAUNCH
    return pico_launch_status();
}
