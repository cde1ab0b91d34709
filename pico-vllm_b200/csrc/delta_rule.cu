// The gated delta rule: a matrix memory per head and request whose rows decay and whose write is corrected by what the
// memory already holds under the key,
//
//   S <- diag(a_t) S ;   u = beta_t (v_t - S^T k_t) ;   S <- S + k_t u^T ;   o_t = S^T q_t          (S: [d, dv], float32)
//
// token by token, the read seeing the write; the decay a_t is one number per row of S, or one for the whole of it (PER_HEAD).
// With the decayed memory S' = diag(a_t) S both sums over rows are taken in one
// pass,  r1 = S'^T k_t  and  r2 = S'^T q_t :  u = beta_t (v_t - r1),  o_t = r2 + u (k_t . q_t),  so a token costs one pass
// over the registers, one reduction and one update.
//
// delta_prepare_kernel makes the float32 inputs of the recurrence from the projections: q and k as unit vectors per head
// (q times d^-1/2), beta = sigmoid, the decay a = exp(-exp(A_log) softplus(z + bias)) per head and row (or per head), and k . q.
// gated_delta_rule_kernel is the recurrence: the columns of S evolve independently of each other, so a block takes
// 16 columns of one head of one segment, eight or sixteen lanes a column with the rows dealt out among them in
// registers; the state is stored transposed [slot, head, dv, d].  A token's q, k and decay pass through shared
// memory, DR_TOK tokens at a time, the next ones' loads in flight (cp.async) while these are walked.  A segment of one token is a decode step; a
// portion of a prompt goes on from the state the portion before left.
//
// Everything here is float32 whatever the activation type; only the projections read are not.
#include "common.cuh"

#define DR_TOK 8

__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Grid (tokens, 1 + H): block y = 0 makes the unit vectors and k . q of all query/key heads (a warp a head), block y = h + 1
// the decays and beta of head h (PER_HEAD: block y = 0 makes those too, a thread a head, and there are no others).  xc float32 [T, >= q_off.. ] holds the convolved q and k (G heads of d each); proj
// (activation type) holds one beta logit per head at b_off; dt [T, H * d] (PER_HEAD: [T, H]; activation type) the
// decay's argument before its bias.  prep float32 [T, P] with P = 2 G d + H d + H + G:  q | k | a | beta | k . q.
// PER_HEAD: P = 2 G d + 4 H + 8 G:  q | k | four numbers a head: a, beta, two of no use | eight numbers a query/key head: q_t . k_(t-j) for
// j = 0 .. 3, k_t . k_(t-j) for j = 1 .. 3 (with `back`; else the first alone), one of no use; k_(t-j) is the row j before - of
// use where that is the same request's token.
template <typename TA, bool PER_HEAD>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const float* __restrict__ xc, int xc_stride, int q_off, int k_off, const TA* __restrict__ proj,
                     int proj_stride, int b_off, const TA* __restrict__ dt, int dt_stride, const float* __restrict__ dt_bias,
                     const float* __restrict__ a_log, float* __restrict__ prep, int P, int H, int G, int d, float q_scale,
                     float unit_eps, int back) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float* out = prep + t * P;
    if (PER_HEAD) {
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            const float z = to_f32(dt[t * dt_stride + h]) + (dt_bias ? dt_bias[h] : 0.f);
            out[2 * G * d + 4 * h] = expf(-expf(a_log[h]) * dr_softplus(z));
            out[2 * G * d + 4 * h + 1] = dr_sigmoid(to_f32(proj[t * proj_stride + b_off + h]));
        }
    } else if (blockIdx.y > 0) {
        const int h = blockIdx.y - 1;
        const float rate = expf(a_log[h]);
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            const float z = to_f32(dt[t * dt_stride + h * d + i]) + (dt_bias ? dt_bias[h * d + i] : 0.f);
            out[2 * G * d + h * d + i] = expf(-rate * dr_softplus(z));
        }
        if (threadIdx.x == 0) out[2 * G * d + H * d + h] = dr_sigmoid(to_f32(proj[t * proj_stride + b_off + h]));
        return;
    }
    const float* row = xc + t * xc_stride;
    for (int g = warp; g < G; g += nw) {
        float sq = 0.f, sk = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float a = row[q_off + g * d + i], b = row[k_off + g * d + i];
            sq += a * a;
            sk += b * b;
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        const float iq = q_scale / sqrtf(sq + unit_eps), ik = 1.0f / sqrtf(sk + unit_eps);
        float kq = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float a = row[q_off + g * d + i] * iq, b = row[k_off + g * d + i] * ik;
            out[g * d + i] = a;
            out[G * d + g * d + i] = b;
            kq += a * b;
        }
        kq = warp_sum(kq);
        float* dots = out + 2 * G * d + (PER_HEAD ? 4 * H + 8 * g : H * d + H + g);
        if (lane == 0) dots[0] = kq;
        if (PER_HEAD && back) {
            float n[3] = {0.f, 0.f, 0.f}, dq[3] = {0.f, 0.f, 0.f}, dk[3] = {0.f, 0.f, 0.f};
            for (int i = lane; i < d; i += 32) {
                const float a = row[q_off + g * d + i], b = row[k_off + g * d + i];
#pragma unroll
                for (int j = 0; j < 3; ++j)
                    if (t > j) {
                        const float c = (row - (size_t)(j + 1) * xc_stride)[k_off + g * d + i];
                        n[j] = fmaf(c, c, n[j]);
                        dq[j] = fmaf(a, c, dq[j]);
                        dk[j] = fmaf(b, c, dk[j]);
                    }
            }
#pragma unroll
            for (int j = 0; j < 3; ++j) {
                n[j] = warp_sum(n[j]);
                dq[j] = warp_sum(dq[j]);
                dk[j] = warp_sum(dk[j]);
            }
            if (lane == 0) {
#pragma unroll
                for (int j = 0; j < 3; ++j) {
                    const float in = 1.0f / sqrtf(n[j] + unit_eps);
                    dots[1 + j] = dq[j] * iq * in;
                    dots[4 + j] = dk[j] * ik * in;
                }
            }
        }
    }
}

PICO_API int pico_delta_prepare(const float* xc, int xc_stride, int q_off, int k_off, const void* proj, int proj_stride,
                                int b_off, const void* dt, int dt_stride, const float* dt_bias, const float* a_log,
                                float* prep, int T, int H, int G, int d, float q_scale, float unit_eps, int per_head,
                                int back, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H < 1 || G < 1 || H % G || d < 1 || H + 1 > 65535) return PICO_ERR_SIZE;
    const int P = 2 * G * d + (per_head ? 4 * H + 8 * G : H * d + H + G);
    const dim3 grid(T, per_head ? 1 : 1 + H);
#define DP_LAUNCH(TA, PH)                                                                                                   \
    pico_launch((delta_prepare_kernel<TA, PH>), grid, dim3(128), 0, stream, xc, xc_stride, q_off, k_off, (const TA*)proj,   \
                proj_stride, b_off, (const TA*)dt, dt_stride, dt_bias, a_log, prep, P, H, G, d, q_scale, unit_eps, back)
    if (dtype == PICO_F32) { if (per_head) DP_LAUNCH(float, true); else DP_LAUNCH(float, false); }
    else if (dtype == PICO_BF16) { if (per_head) DP_LAUNCH(bf16, true); else DP_LAUNCH(bf16, false); }
    else
#undef DP_LAUNCH
        return PICO_ERR_DTYPE;
    return pico_launch_status();
}

__device__ __forceinline__ void dr_cp4(float* dst, const float* src) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(src) : "memory");
}
__device__ __forceinline__ void dr_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
__device__ __forceinline__ void dr_wait_all() { asm volatile("cp.async.wait_group 0;\n" ::: "memory"); }

// prep: the rows delta_prepare_kernel wrote (q at 0, k at G d, a at 2 G d, beta and k . q after them); v float32 rows with
// head h's values at h * dv; state float32 [slots, H, dv, d]; out float32 [T, H * dv].  Grid (column tiles, H, segments).
// A column is held by LPC lanes of a warp; lane l of a column holds the rows 4 l .. 4 l + 3, 4 LPC + 4 l .., ... (RPL of
// them), so a sum over rows is RPL multiply-adds in a lane (four chains side by side) and log2(LPC) exchanges among the lanes: the
// token-to-token chain - decay, two sums, write - is what sets this kernel's time, since tokens cannot run side by side.
// PER_HEAD: the decay is one number a token; it rides behind k . q instead of d numbers of their own.
template <int RPL, int LPC, bool PER_HEAD>      // rows a lane, lanes a column (8 or 16): a block holds 16 columns in 16 * LPC threads
__global__ void __launch_bounds__(16 * LPC)
gated_delta_rule_kernel(const float* __restrict__ prep, int P, const float* __restrict__ v, int v_stride,
                        float* __restrict__ state, const int* __restrict__ seg_slots, const int* __restrict__ cu_q,
                        const int* __restrict__ positions, float* __restrict__ out, int out_stride, int H, int G, int d,
                        int dv) {
    // The kernel that follows is released at the end, not here: its blocks, resident and waiting beside this kernel's
    // few warps, made the token loop 2.7 times slower (2.0 instead of 0.76 ms for 2,048 tokens).
    pdl_wait();
    extern __shared__ __align__(16) float dsm[];
    constexpr int dp = RPL * LPC;
    constexpr int NC = 16, CPW = 32 / LPC, NTH = 16 * LPC;
    // two buffers of DR_TOK tokens: q [dp], k [dp], a [dp] (not PER_HEAD), v [NC], beta, kq, a (PER_HEAD), and what keeps a
    // token 16-byte aligned
    constexpr int VAT = (PER_HEAD ? 2 : 3) * dp, tok_floats = VAT + NC + 4, NSC = PER_HEAD ? 3 : 2;
    const int seg = blockIdx.z, h = blockIdx.y, col_base = blockIdx.x * NC;
    const int t_begin = cu_q[seg], t_end = cu_q[seg + 1];
    if (t_end <= t_begin || positions[t_begin] < 0) return;      // an empty or a padding segment
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane % LPC, cw = lane / LPC;                  // row lane and column of the warp
    const int col = col_base + warp * CPW + cw;
    const int hq = h / (H / G);
    float* st = state + ((size_t)seg_slots[seg] * H + h) * (size_t)dv * d;
    float S[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int i = 4 * sub + 4 * LPC * (r >> 2) + (r & 3);  // four neighbouring rows at a time: one 16-byte load a token
        S[r] = (i < d && col < dv) ? st[(size_t)col * d + i] : 0.f;
    }
    const int q_at = hq * d, k_at = G * d + hq * d, a_at = 2 * G * d + (PER_HEAD ? 4 * h : h * d),
              b_at = PER_HEAD ? a_at + 1 : 2 * G * d + H * d + h, kq_at = 2 * G * d + (PER_HEAD ? 4 * H + 8 * hq : H * d + H + hq);
    auto fetch = [&](int t0, int nt, float* buf) {
        for (int idx = threadIdx.x; idx < nt * dp; idx += NTH) {
            const int tt = idx / dp, i = idx - tt * dp;
            float* dst = buf + tt * tok_floats;
            if (i < d) {
                const float* src = prep + (size_t)(t0 + tt) * P;
                dr_cp4(dst + i, src + q_at + i);
                dr_cp4(dst + dp + i, src + k_at + i);
                if (!PER_HEAD) dr_cp4(dst + 2 * dp + i, src + a_at + i);
            } else {
                dst[i] = 0.f;
                dst[dp + i] = 0.f;
                if (!PER_HEAD) dst[2 * dp + i] = 1.f;
            }
        }
        for (int idx = threadIdx.x; idx < nt * (NC + NSC); idx += NTH) {
            const int tt = idx / (NC + NSC), c = idx - tt * (NC + NSC);
            float* dst = buf + tt * tok_floats + VAT;
            const float* src = prep + (size_t)(t0 + tt) * P;
            if (c < NC) {
                if (col_base + c < dv) dr_cp4(dst + c, v + (size_t)(t0 + tt) * v_stride + (size_t)h * dv + col_base + c);
                else dst[c] = 0.f;
            } else if (c == NC) dr_cp4(dst + c, src + b_at);
            else dr_cp4(dst + c, src + (PER_HEAD && c == NC + 2 ? a_at : kq_at));
        }
        dr_commit();
    };
    float* buf0 = dsm;
    float* buf1 = dsm + DR_TOK * tok_floats;
    fetch(t_begin, min(DR_TOK, t_end - t_begin), buf0);
    int turn = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += DR_TOK, turn ^= 1) {
        const int nt = min(DR_TOK, t_end - t0);
        dr_wait_all();
        __syncthreads();                    // these tokens are in; everyone is done with the other buffer
        if (t0 + DR_TOK < t_end) fetch(t0 + DR_TOK, min(DR_TOK, t_end - t0 - DR_TOK), turn ? buf0 : buf1);
        const float* buf = turn ? buf1 : buf0;
        float4 nq[RPL / 4], nk[RPL / 4], na[PER_HEAD ? 1 : RPL / 4];      // the next token's rows, asked for a token ahead
        auto rows_of = [&](int tt) {
            const float* tk = buf + tt * tok_floats + 4 * sub;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                nq[j] = *reinterpret_cast<const float4*>(tk + 4 * LPC * j);
                nk[j] = *reinterpret_cast<const float4*>(tk + dp + 4 * LPC * j);
                if (!PER_HEAD) na[j] = *reinterpret_cast<const float4*>(tk + 2 * dp + 4 * LPC * j);
            }
        };
        rows_of(0);
        for (int tt = 0; tt < nt; ++tt) {
            const float* tk = buf + tt * tok_floats;
            float p1[4] = {0.f, 0.f, 0.f, 0.f}, p2[4] = {0.f, 0.f, 0.f, 0.f};
            float kr[RPL];
            const float ah = PER_HEAD ? tk[VAT + NC + 2] : 1.0f;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                const float4 a4 = PER_HEAD ? make_float4(ah, ah, ah, ah) : na[PER_HEAD ? 0 : j];
                const float qv[4] = {nq[j].x, nq[j].y, nq[j].z, nq[j].w}, kv[4] = {nk[j].x, nk[j].y, nk[j].z, nk[j].w},
                            av[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = 4 * j + e;
                    const float s = S[r] * av[e];
                    kr[r] = kv[e];
                    S[r] = s;
                    p1[e] = fmaf(s, kv[e], p1[e]);
                    p2[e] = fmaf(s, qv[e], p2[e]);
                }
            }
            if (tt + 1 < nt) rows_of(tt + 1);
            float r1 = (p1[0] + p1[1]) + (p1[2] + p1[3]), r2 = (p2[0] + p2[1]) + (p2[2] + p2[3]);
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) {
                r1 += __shfl_xor_sync(0xffffffffu, r1, o);
                r2 += __shfl_xor_sync(0xffffffffu, r2, o);
            }
            const float u = tk[VAT + NC] * (tk[VAT + warp * CPW + cw] - r1);
#pragma unroll
            for (int r = 0; r < RPL; ++r) S[r] = fmaf(kr[r], u, S[r]);
            if (sub == 0 && col < dv)
                out[(size_t)(t0 + tt) * out_stride + (size_t)h * dv + col] = fmaf(u, tk[VAT + NC + 1], r2);
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int i = 4 * sub + 4 * LPC * (r >> 2) + (r & 3);
        if (i < d && col < dv) st[(size_t)col * d + i] = S[r];
    }
}

// ------------------------------------------------------------------------------------------ four tokens at a time
// With one decay a head (g_t) the memory needs to be touched only once for four tokens.  For a block of tokens 1 .. 4 that
// starts from the memory S, with r_i = S^T k_i, p_i = S^T q_i (eight sums over rows in one pass and one reduction),
// D_ij = g_(j+1) ... g_i and G_i = g_1 ... g_i:
//
//   u_i = beta_i (v_i - G_i r_i - sum_(j < i) D_ij (k_i . k_j) u_j)         o_i = G_i p_i + sum_(j <= i) D_ij (q_i . k_j) u_j
//   S  <- G_4 S + sum_j D_4j k_j u_j
//
// the same recurrence with the sums in another order; the products of decays are taken as products (none is above one, nothing is
// divided).  The dot products come from delta_prepare_kernel, the coefficients of a block from sixteen threads of this one.
// Tokens beyond the segment's end are blanks (k = q = v = 0, beta = 0, g = 1).  A block holds 16 columns as above; a lane holds the
// same rows of CPL columns (what it reads of q and k serves both) and multiplies two rows at a time (fma.rn.f32x2).
#define DB_TOK 32          // tokens fetched at a time
#define DB_COEF 48         // floats of coefficients a block of four tokens: B [4][4], E [4][4], beta G [4], beta [4], G [4], W [4]

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 db_fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 db_mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 db_pair(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};\n" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 db_split(f32x2 a) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;\n" : "=f"(r.x), "=f"(r.y) : "l"(a));
    return r;
}

__device__ __forceinline__ void dr_cp16(float* dst, const float* src) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(src) : "memory");
}

// RPL rows and CPL columns a lane, LPC lanes a column (at least 8 * CPL).  vec: d, dv, both row strides and all addresses are
// multiples of 16 bytes.  (Measured for 2,048 tokens of twelve heads with d = dv = 128: 285 us with two columns a lane, 303 us with
// one, 357 us when the next block's rows are asked for while the sums are exchanged; 692 us with a pass for every token.)
template <int RPL, int LPC, int CPL>
__global__ void __launch_bounds__(16 * LPC / CPL)
gated_delta_block_kernel(const float* __restrict__ prep, int P, const float* __restrict__ v, int v_stride,
                         float* __restrict__ state, const int* __restrict__ seg_slots, const int* __restrict__ cu_q,
                         const int* __restrict__ positions, float* __restrict__ out, int out_stride, int H, int G, int d,
                         int dv, int vec) {
    pdl_wait();                         // the kernel that follows is released at the end (see above)
    extern __shared__ __align__(16) float dsm[];
    constexpr int dp = RPL * LPC, NC = 16, NTH = NC / CPL * LPC, NV = 8 * CPL, VL = LPC / NV;      // VL: lanes that share a sum
    static_assert(VL >= 1, "a lane ends with one sum");
    constexpr int VAT = 2 * dp, SAT = VAT + NC, tok_floats = SAT + 12;      // q [dp], k [dp], v [NC], a, beta, -, -, eight dot products
    const int seg = blockIdx.z, h = blockIdx.y, col_base = blockIdx.x * NC;
    const int t_begin = cu_q[seg], t_end = cu_q[seg + 1];
    if (t_end <= t_begin || positions[t_begin] < 0) return;      // an empty or a padding segment
    const int sub = threadIdx.x % LPC, lcol = threadIdx.x / LPC * CPL, lane0 = (threadIdx.x & 31) - sub;
    const int hq = h / (H / G);
    float* st = state + ((size_t)seg_slots[seg] * H + h) * (size_t)dv * d;
    f32x2 S[CPL][RPL / 2];
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
        const int col = col_base + lcol + c;
#pragma unroll
        for (int r = 0; r < RPL; r += 2) {
            const int i = 4 * sub + 4 * LPC * (r >> 2) + (r & 3);
            S[c][r / 2] = db_pair(col < dv && i < d ? st[(size_t)col * d + i] : 0.f, col < dv && i + 1 < d ? st[(size_t)col * d + i + 1] : 0.f);
        }
    }
    const int q_at = hq * d, k_at = G * d + hq * d, a_at = 2 * G * d + 4 * h, dot_at = 2 * G * d + 4 * H + 8 * hq;
    auto fetch = [&](int t0, float* buf) {
        const int nt = min(DB_TOK, t_end - t0), nt4 = (nt + 3) & ~3;         // whole blocks of four, blanks at the end
        if (vec) {
            constexpr int DQ = dp / 4;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int idx = threadIdx.x; idx < nt4 * DQ; idx += NTH) {
                const int tt = idx / DQ, i = (idx - tt * DQ) * 4;
                float* dst = buf + tt * tok_floats + i;
                if (i < d && tt < nt) {
                    const float* src = prep + (size_t)(t0 + tt) * P + i;
                    dr_cp16(dst, src + q_at);
                    dr_cp16(dst + dp, src + k_at);
                } else {
                    *reinterpret_cast<float4*>(dst) = zero;
                    *reinterpret_cast<float4*>(dst + dp) = zero;
                }
            }
            for (int idx = threadIdx.x; idx < nt4 * 8; idx += NTH) {         // four vectors of v, one of a and beta, two of dot products
                const int tt = idx >> 3, c = idx & 7;
                float* dst = buf + tt * tok_floats + VAT + 4 * c;
                const float* src = prep + (size_t)(t0 + tt) * P;
                if (c < 4) {
                    if (tt < nt && col_base + 4 * c < dv) dr_cp16(dst, v + (size_t)(t0 + tt) * v_stride + (size_t)h * dv + col_base + 4 * c);
                    else *reinterpret_cast<float4*>(dst) = zero;
                } else if (c < 7) {
                    if (tt < nt) dr_cp16(dst, c == 4 ? src + a_at : src + dot_at + 4 * (c - 5));
                    else *reinterpret_cast<float4*>(dst) = make_float4(c == 4 ? 1.f : 0.f, 0.f, 0.f, 0.f);
                }
            }
        } else {
            for (int idx = threadIdx.x; idx < nt4 * dp; idx += NTH) {
                const int tt = idx / dp, i = idx - tt * dp;
                float* dst = buf + tt * tok_floats + i;
                if (i < d && tt < nt) {
                    const float* src = prep + (size_t)(t0 + tt) * P + i;
                    dr_cp4(dst, src + q_at);
                    dr_cp4(dst + dp, src + k_at);
                } else {
                    dst[0] = 0.f;
                    dst[dp] = 0.f;
                }
            }
            for (int idx = threadIdx.x; idx < nt4 * (NC + 12); idx += NTH) {
                const int tt = idx / (NC + 12), c = idx - tt * (NC + 12);
                float* dst = buf + tt * tok_floats + VAT + c;
                const float* src = prep + (size_t)(t0 + tt) * P;
                if (c < NC) {
                    if (tt < nt && col_base + c < dv) dr_cp4(dst, v + (size_t)(t0 + tt) * v_stride + (size_t)h * dv + col_base + c);
                    else *dst = 0.f;
                } else if (tt < nt) dr_cp4(dst, c < NC + 4 ? src + a_at + c - NC : src + dot_at + c - NC - 4);
                else *dst = c == NC ? 1.f : 0.f;
            }
        }
        dr_commit();
    };
    float* buf0 = dsm;
    float* buf1 = dsm + DB_TOK * tok_floats;
    float* coef = dsm + 2 * DB_TOK * tok_floats;
    fetch(t_begin, buf0);
    // which of the block's outputs this lane writes, if any: sum number sub / VL is p_(oi + 1) of column lcol + oc
    const int val = sub / VL, oc = val >> 3, oi = val & 3, ocol = col_base + lcol + oc;
    const bool writes = (val & 4) != 0 && sub % VL == 0 && ocol < dv;
    float* op = out + (size_t)(t_begin + oi) * out_stride + (size_t)h * dv + ocol;
    int turn = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += DB_TOK, turn ^= 1) {
        const int nt = min(DB_TOK, t_end - t0), nb = (nt + 3) >> 2;
        dr_wait_all();
        __syncthreads();                    // these tokens are in; everyone is done with the other buffer and the coefficients
        if (t0 + DB_TOK < t_end) fetch(t0 + DB_TOK, turn ? buf0 : buf1);
        const float* buf = turn ? buf1 : buf0;
        for (int idx = threadIdx.x; idx < 16 * nb; idx += NTH) {             // a thread per pair (i, j) of a block's tokens
            const int b = idx >> 4, i = (idx >> 2) & 3, j = idx & 3;
            const float* tk = buf + 4 * b * tok_floats + SAT;
            const float* ti = tk + i * tok_floats;
            float* c = coef + b * DB_COEF;
            float D = 1.f, W = 1.f, Gi = 1.f;
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                const float g = tk[m * tok_floats];
                if (m > j && m <= i) D *= g;
                if (m > j) W *= g;
                if (m <= i) Gi *= g;
            }
            c[4 * i + j] = j < i ? ti[1] * D * ti[7 + i - j] : 0.f;          // ti[8 ..]: k_i . k_(i-1), ...
            c[16 + 4 * i + j] = j <= i ? D * ti[4 + i - j] : 0.f;            // ti[4 ..]: q_i . k_i, q_i . k_(i-1), ...
            if (i == 0) c[44 + j] = W;
            if (j == 0) {
                c[32 + i] = ti[1] * Gi;
                c[36 + i] = ti[1];
                c[40 + i] = Gi;
            }
        }
        __syncthreads();
#pragma unroll 2
        for (int b = 0; b < nb; ++b, op += (size_t)4 * out_stride) {
            const float* tk = buf + 4 * b * tok_floats;
            const float* c = coef + b * DB_COEF;
            ulonglong2 kr[4][RPL / 4], qr[4][RPL / 4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int r = 0; r < RPL / 4; ++r) {
                    const float* at = tk + i * tok_floats + 4 * sub + 4 * LPC * r;
                    qr[i][r] = *reinterpret_cast<const ulonglong2*>(at);
                    kr[i][r] = *reinterpret_cast<const ulonglong2*>(at + dp);
                }
            float s[NV];
#pragma unroll
            for (int cc = 0; cc < CPL; ++cc)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    f32x2 ar = db_mul2(S[cc][0], kr[i][0].x), ap = db_mul2(S[cc][0], qr[i][0].x);
                    ar = db_fma2(S[cc][1], kr[i][0].y, ar);
                    ap = db_fma2(S[cc][1], qr[i][0].y, ap);
#pragma unroll
                    for (int r = 1; r < RPL / 4; ++r) {
                        ar = db_fma2(S[cc][2 * r], kr[i][r].x, ar);
                        ap = db_fma2(S[cc][2 * r], qr[i][r].x, ap);
                        ar = db_fma2(S[cc][2 * r + 1], kr[i][r].y, ar);
                        ap = db_fma2(S[cc][2 * r + 1], qr[i][r].y, ap);
                    }
                    const float2 fr = db_split(ar), fp = db_split(ap);
                    s[8 * cc + i] = fr.x + fr.y;
                    s[8 * cc + 4 + i] = fp.x + fp.y;
                }
            // on their way while the sums are exchanged: the block's values and coefficients
            float vv[4][CPL];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int cc = 0; cc < CPL; ++cc) vv[i][cc] = tk[i * tok_floats + VAT + lcol + cc];
            const float4 bG = *reinterpret_cast<const float4*>(c + 32), be = *reinterpret_cast<const float4*>(c + 36),
                         W = *reinterpret_cast<const float4*>(c + 44), B1 = *reinterpret_cast<const float4*>(c + 4),
                         B2 = *reinterpret_cast<const float4*>(c + 8), B3 = *reinterpret_cast<const float4*>(c + 12),
                         E = *reinterpret_cast<const float4*>(c + 16 + 4 * oi);
            const float Gn = c[43], Go = c[40 + oi];
            // the sums over the column's lanes: each exchange halves the number of sums a lane still carries
#pragma unroll
            for (int w = NV / 2; w > 0; w >>= 1) {
                const bool up = (sub & (w * VL)) != 0;
#pragma unroll
                for (int i = 0; i < w; ++i) {
                    const float send = up ? s[i] : s[i + w], keep = up ? s[i + w] : s[i];
                    s[i] = keep + __shfl_xor_sync(0xffffffffu, send, w * VL);
                }
            }
#pragma unroll
            for (int o = VL / 2; o > 0; o >>= 1) s[0] += __shfl_xor_sync(0xffffffffu, s[0], o);
            const float bg[4] = {bG.x, bG.y, bG.z, bG.w}, bb[4] = {be.x, be.y, be.z, be.w};
            float u[CPL][4];
#pragma unroll
            for (int cc = 0; cc < CPL; ++cc) {
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    u[cc][i] = fmaf(-bg[i], __shfl_sync(0xffffffffu, s[0], lane0 + (8 * cc + i) * VL), bb[i] * vv[i][cc]);
                u[cc][1] = fmaf(-B1.x, u[cc][0], u[cc][1]);
                u[cc][2] = fmaf(-B2.y, u[cc][1], fmaf(-B2.x, u[cc][0], u[cc][2]));
                u[cc][3] = fmaf(-B3.z, u[cc][2], fmaf(-B3.y, u[cc][1], fmaf(-B3.x, u[cc][0], u[cc][3])));
            }
            const float wt[4] = {W.x, W.y, W.z, W.w};
            const f32x2 G2 = db_pair(Gn, Gn);
#pragma unroll
            for (int cc = 0; cc < CPL; ++cc) {
#pragma unroll
                for (int r = 0; r < RPL / 2; ++r) S[cc][r] = db_mul2(S[cc][r], G2);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float w1 = wt[i] * u[cc][i];
                    const f32x2 w2 = db_pair(w1, w1);
#pragma unroll
                    for (int r = 0; r < RPL / 4; ++r) {
                        S[cc][2 * r] = db_fma2(kr[i][r].x, w2, S[cc][2 * r]);
                        S[cc][2 * r + 1] = db_fma2(kr[i][r].y, w2, S[cc][2 * r + 1]);
                    }
                }
            }
            if (writes && t0 + 4 * b + oi < t_end) {
                float uo[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) uo[i] = CPL == 2 && oc ? u[CPL - 1][i] : u[0][i];
                *op = fmaf(E.w, uo[3], fmaf(E.z, uo[2], fmaf(E.y, uo[1], fmaf(E.x, uo[0], Go * s[0]))));
            }
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
        const int col = col_base + lcol + c;
#pragma unroll
        for (int r = 0; r < RPL; r += 2) {
            const int i = 4 * sub + 4 * LPC * (r >> 2) + (r & 3);
            const float2 f = db_split(S[c][r / 2]);
            if (col < dv && i < d) st[(size_t)col * d + i] = f.x;
            if (col < dv && i + 1 < d) st[(size_t)col * d + i + 1] = f.y;
        }
    }
}

PICO_API int pico_gated_delta_rule(const float* prep, const float* v, int v_stride, float* state, const int* seg_slots,
                                   const int* cu_q, const int* positions, float* out, int out_stride, int S, int H, int G,
                                   int d, int dv, int per_head, int blocked, cudaStream_t stream) {
    if (S <= 0) return 0;
    if (H < 1 || G < 1 || H % G || d < 1 || d > 256 || dv < 1) return PICO_ERR_SIZE;
    const int P = 2 * G * d + (per_head ? 4 * H + 8 * G : H * d + H + G);
    const dim3 grid((dv + 15) / 16, H, S);
    if (grid.z > 65535 || grid.y > 65535) return PICO_ERR_SIZE;
    // A grid that fits on the device one block to a multiprocessor asks for more shared memory than half of one, so that
    // no two blocks share a multiprocessor: released early behind a kernel that is still draining, the blocks of a
    // 2,048-token prompt landed four to a multiprocessor on the first ones that had room and took 1.5 ms instead of 0.8.
    const bool alone = (long long)grid.x * grid.y * grid.z <= pico_num_sms();
#define DR_LAUNCH_AS(N, L, PH)                                                                                              \
    do {                                                                                                                    \
        size_t smem = (size_t)2 * DR_TOK * ((PH ? 2 : 3) * N * L + 16 + 4) * sizeof(float);                                 \
        if (alone && smem < 116 * 1024) smem = 116 * 1024;                                                                  \
        if (smem > 48 * 1024)                                                                                               \
            cudaFuncSetAttribute(gated_delta_rule_kernel<N, L, PH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
        pico_launch((gated_delta_rule_kernel<N, L, PH>), grid, dim3(16 * L), smem, stream, prep, P, v, v_stride, state,     \
                    seg_slots, cu_q, positions, out, out_stride, H, G, d, dv);                                              \
    } while (0)
#define DR_LAUNCH(N, L)                                                                                                     \
    do {                                                                                                                    \
        if (per_head) DR_LAUNCH_AS(N, L, true);                                                                             \
        else DR_LAUNCH_AS(N, L, false);                                                                                     \
    } while (0)
#define DB_LAUNCH(N, L, C)                                                                                             \
    do {                                                                                                                    \
        size_t smem = (size_t)(2 * DB_TOK * (2 * N * L + 16 + 12) + DB_TOK / 4 * DB_COEF) * sizeof(float);                  \
        if (alone && smem < 116 * 1024) smem = 116 * 1024;                                                                  \
        if (smem > 48 * 1024)                                                                                               \
            cudaFuncSetAttribute(gated_delta_block_kernel<N, L, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        pico_launch((gated_delta_block_kernel<N, L, C>), grid, dim3(16 * L / C), smem, stream, prep, P, v, v_stride, state, \
                    seg_slots, cu_q, positions, out, out_stride, H, G, d, dv, vec);                                         \
    } while (0)
    if (per_head && blocked) {
        const int vec = d % 4 == 0 && dv % 4 == 0 && v_stride % 4 == 0 && (((uintptr_t)prep | (uintptr_t)v) & 15) == 0;
        if (d <= 32) DB_LAUNCH(4, 8, 1);
        else if (d <= 64) DB_LAUNCH(4, 16, 2);
        else if (d <= 128) DB_LAUNCH(8, 16, 2);
        else DB_LAUNCH(16, 16, 2);
        return pico_launch_status();
    }
#undef DB_LAUNCH
    // keys of up to 32: eight lanes a column (four warps a block); longer keys: sixteen (eight warps), so that a
    // multiprocessor's four schedulers each have two warps to choose from
    if (d <= 32) DR_LAUNCH(4, 8);
    else if (d <= 64) DR_LAUNCH(4, 16);
    else if (d <= 128) DR_LAUNCH(8, 16);
    else DR_LAUNCH(16, 16);
#undef DR_LAUNCH
#undef DR_LAUNCH_AS
    return pico_launch_status();
}
