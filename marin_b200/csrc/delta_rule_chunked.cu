// The gated delta rule over prompt portions, 64 tokens at a time on the tensor cores (mma.sync), compiled for one head layout:
// -DQK_DIM (key channels, a multiple of 16 up to 128), -DV_SLICE (value channels a CTA takes: 16 or 32).
//
// The recurrence (delta_rule.cu) per head:  S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q.  With S0 the state before
// a chunk of 64 tokens, G_i the sum of the log-decays of its tokens 0 .. i (per key channel), and the weighted products
//     A_ij = sum_c k_i[c] k_j[c] exp(G_i[c] - G_j[c])  (j < i),      P_ij = sum_c q_i[c] k_j[c] exp(G_i[c] - G_j[c])  (j <= i),
// unrolling it gives (Yang, Wang, Zhang, Shen, Kim, "Parallelizing Linear Transformers with the Delta Rule over Sequence Length")
//     (I + diag(beta) A) U = diag(beta) (V - K+ S0),   K+_i = exp(G_i) k_i,
//     O = Q+ S0 + P U,   Q+_i = exp(G_i) q_i,          S = exp(G_63) S0 + sum_j (exp(G_63 - G_j) k_j) u_j^T.
// prepare_kernel (a CTA per chunk and head, all of them side by side) makes what does not need the state: P, and by forward
// substitution W = (I + diag(beta) A)^-1 diag(beta) K+ and U0 = (I + diag(beta) A)^-1 diag(beta) V.  walk_kernel (a CTA per request, head
// and slice of value channels) then walks the chunks in order: U = U0 - W S0, O, S.
//
// Exactness.  Every exponent that is taken is of a non-positive number: with one decay per channel a block of 16 rows is worked out
// against a reference between it and the earlier rows (exp(G_i - R) exp(R - G_j), both at most 1), the lower half of a block's diagonal
// square against one in its middle, and the 8 x 8 squares left on the diagonal pair by pair.  Decays, sums, unit vectors, A, the substitution and the state are float32; where a float32 number has to be an
// operand of a product it is split into two bf16 numbers (value = hi + lo) and the three larger products are taken, so that about 16
// bits of it enter.
#define MB_LIB "delta_rule_chunked"
#define MB_LIB_ID 21
#include "common.cuh"
#include "launch.cuh"
#include "mma_helpers.cuh"

#ifndef QK_DIM
#define QK_DIM 128
#endif
#ifndef V_SLICE
#define V_SLICE 32
#endif
static_assert(QK_DIM % 16 == 0 && QK_DIM >= 16 && QK_DIM <= 128, "key channels: a multiple of 16 up to 128");
static_assert(V_SLICE == 16 || V_SLICE == 32, "a CTA takes 16 or 32 value channels");

#define DQ QK_DIM
#define VS V_SLICE
#define CH 64
#define LOG2E 1.4426950408889634f
#define UNIT_EPS 1e-6f

__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float2 bf2(uint32_t w) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w)); }

__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 back = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = pack_bf16(x - back.x, y - back.y);
}
__device__ __forceinline__ void mma3(float* c, const uint32_t* ah, const uint32_t* al, uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    mma_bf16_16816(c, ah, bh0, bh1);
    mma_bf16_16816(c, al, bh0, bh1);
    mma_bf16_16816(c, ah, bl0, bl1);
}

// The same into three sums (added up at the end): three chains of products instead of one three times as long.
struct Sums3 {
    float hh[2][4], lh[2][4], hl[2][4];
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) hh[n][e] = lh[n][e] = hl[n][e] = 0.0f;
    }
    __device__ __forceinline__ void add(const uint32_t* ah, const uint32_t* al, const uint32_t* bh, const uint32_t* bl) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            mma_bf16_16816(hh[n], ah, bh[2 * n], bh[2 * n + 1]);
            mma_bf16_16816(lh[n], al, bh[2 * n], bh[2 * n + 1]);
            mma_bf16_16816(hl[n], ah, bl[2 * n], bl[2 * n + 1]);
        }
    }
    __device__ __forceinline__ float at(int n, int e) const { return hh[n][e] + (lh[n][e] + hl[n][e]); }
};

// What a chunk and head leaves for the walk, in bf16 planes of [64][DQ] (W, Q+, K exp(G_63 - G), each hi then lo), [64][64] (P hi, lo),
// then float32 U0 [64][dv] and exp(G_63) [DQ].
#define PLANE (CH * DQ)
#define PPLANE (CH * CH)
#define CHUNK_BF16 (6 * PLANE + 2 * PPLANE)
#define CHUNK_F32(dv) (CH * (dv) + DQ)

// Where request r's chunks start among all chunks of the step (room is left for a partial chunk per request).
__device__ __forceinline__ int first_chunk(const int* cu_tokens, int first_req, int r) { return (cu_tokens[r] - cu_tokens[first_req]) / CH + (r - first_req); }

#define LDR (DQ + 8)                  // raw q and k rows in shared memory (bf16) and sums (float32): eight rows of four lanes meet all banks
#define LDG (DQ + 8)
#define LDL (CH + 4)
#define PREP_SMEM(CHANNEL, dv) (2 * CH * LDR * 2 + ((CHANNEL) ? CH * LDG : CH) * 4 + CH * LDL * 4 + 4 * CH * 4 + CH * ((dv) + 8) * 2 + 16)
#define PREP_THREADS 256

template <bool CHANNEL>
__global__ void __launch_bounds__(PREP_THREADS, 2) prepare_kernel(
    const bf16* __restrict__ qkv, const bf16* __restrict__ b_rows, int b_stride, const bf16* __restrict__ a_rows, int a_stride,
    const float* __restrict__ rate_log, const float* __restrict__ dt_bias, const int* __restrict__ cu_tokens, int first_req,
    bf16* __restrict__ planes, float* __restrict__ floats, int H, int G, int dv, int a_vec) {
    PDL_ENTER();
    qkv = pdl_fresh(qkv); b_rows = pdl_fresh(b_rows); a_rows = pdl_fresh(a_rows);
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* sq = reinterpret_cast<bf16*>(smem_raw);              // [CH][LDR]
    bf16* sk = sq + CH * LDR;
    float* sL = reinterpret_cast<float*>(sk + CH * LDR);       // [CH][LDL] beta_i A_ij
    float* sG = sL + CH * LDL;                                 // [CH][LDG], or [CH] with one decay per head (log2 units)
    float* s_beta = sG + (CHANNEL ? CH * LDG : CH);
    float* s_fq = s_beta + CH;
    float* s_fk = s_fq + CH;
    float* s_qk = s_fk + CH;                                   // q_i . k_i as they are
    const int req = first_req + blockIdx.z, head = blockIdx.y;
    const int tok0 = cu_tokens[req] + blockIdx.x * CH;
    const int rows = min(CH, cu_tokens[req + 1] - tok0);
    if (rows <= 0) return;
    const int kh = head / (H / G), channels = 2 * G * DQ + H * dv;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const size_t slot = (size_t)(first_chunk(cu_tokens, first_req, req) + blockIdx.x) * H + head;
    bf16* out = planes + slot * CHUNK_BF16;
    float* fout = floats + slot * CHUNK_F32(dv);
    // ---- q, k and v as the convolution left them; rows past the request's tokens are zero
    bf16* sv = reinterpret_cast<bf16*>(s_qk + CH);             // [CH][dv + 8]
    {
        const bf16* base = qkv + (size_t)tok0 * channels;
        for (int idx = tid; idx < 2 * CH * (DQ / 8); idx += PREP_THREADS) {
            const int which = idx / (CH * (DQ / 8)), rest = idx % (CH * (DQ / 8));
            const int row = rest / (DQ / 8), c = rest % (DQ / 8);
            bf16* dst = (which ? sk : sq) + row * LDR + c * 8;
            if (row < rows) cp_async16(dst, base + (size_t)row * channels + (size_t)which * G * DQ + (size_t)kh * DQ + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        const int per = dv / 8;
        for (int idx = tid; idx < CH * per; idx += PREP_THREADS) {
            const int row = idx / per, c = idx - row * per;
            bf16* dst = sv + row * (dv + 8) + c * 8;
            if (row < rows) cp_async16(dst, base + (size_t)row * channels + (size_t)2 * G * DQ + (size_t)head * dv + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    }
    const float rate = expf(rate_log[head]) * LOG2E;
    if (CHANNEL && a_vec) {
        constexpr int ITERS = (CH * (DQ / 8) + PREP_THREADS - 1) / PREP_THREADS;
        uint4 raw[ITERS];
#pragma unroll
        for (int u = 0; u < ITERS; ++u) {
            const int idx = tid + u * PREP_THREADS, row = idx / (DQ / 8), c = idx % (DQ / 8) * 8;
            raw[u] = make_uint4(0, 0, 0, 0);
            if (row < rows) raw[u] = *reinterpret_cast<const uint4*>(a_rows + (size_t)(tok0 + row) * a_stride + (size_t)head * DQ + c);
        }
#pragma unroll
        for (int u = 0; u < ITERS; ++u) {
            const int idx = tid + u * PREP_THREADS, row = idx / (DQ / 8), c = idx % (DQ / 8) * 8;
            if (row >= CH) continue;
            const float4 d0 = *reinterpret_cast<const float4*>(dt_bias + head * DQ + c), d1 = *reinterpret_cast<const float4*>(dt_bias + head * DQ + c + 4);
            const float bias[8] = {d0.x, d0.y, d0.z, d0.w, d1.x, d1.y, d1.z, d1.w};
            const uint32_t w[4] = {raw[u].x, raw[u].y, raw[u].z, raw[u].w};
            float* dst = sG + row * LDG + c;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 a2 = bf2(w[e]);
                dst[2 * e] = row < rows ? -rate * softplus_f(a2.x + bias[2 * e]) : 0.0f;
                dst[2 * e + 1] = row < rows ? -rate * softplus_f(a2.y + bias[2 * e + 1]) : 0.0f;
            }
        }
    } else if (CHANNEL) {
        for (int idx = tid; idx < CH * DQ; idx += PREP_THREADS) {
            const int row = idx / DQ, c = idx % DQ;
            float lg = 0.0f;
            if (row < rows) lg = -rate * softplus_f(__bfloat162float(a_rows[(size_t)(tok0 + row) * a_stride + (size_t)head * DQ + c]) + dt_bias[head * DQ + c]);
            sG[row * LDG + c] = lg;
        }
    } else if (tid < CH) {
        sG[tid] = tid < rows ? -rate * softplus_f(__bfloat162float(a_rows[(size_t)(tok0 + tid) * a_stride + head]) + dt_bias[head]) : 0.0f;
    }
    if (tid < CH) s_beta[tid] = tid < rows ? 1.0f / (1.0f + expf(-__bfloat162float(b_rows[(size_t)(tok0 + tid) * b_stride + head]))) : 0.0f;
    cp_async_wait<0>();
    __syncthreads();
    // ---- running sums of the log-decays; unit lengths
    if (CHANNEL) {
        for (int c = tid; c < DQ; c += PREP_THREADS) {
            float run = 0.0f;
            for (int i = 0; i < CH; ++i) { run += sG[i * LDG + c]; sG[i * LDG + c] = run; }
        }
    } else if (tid == 0) {
        float run = 0.0f;
        for (int i = 0; i < CH; ++i) { run += sG[i]; sG[i] = run; }
    }
    for (int row = warp; row < CH; row += PREP_THREADS / 32) {
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
        for (int c = lane; c < DQ; c += 32) {
            const float x = __bfloat162float(sq[row * LDR + c]), y = __bfloat162float(sk[row * LDR + c]);
            qq = fmaf(x, x, qq);
            kk = fmaf(y, y, kk);
            qk = fmaf(x, y, qk);
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        qk = warp_sum(qk);
        if (lane == 0) {
            s_fq[row] = 1.0f / (sqrtf((float)DQ) * sqrtf(qq + UNIT_EPS));
            s_fk[row] = 1.0f / sqrtf(kk + UNIT_EPS);
            s_qk[row] = qk;
        }
    }
    // (the upper triangles stay zero; of P's only what lies in a diagonal block is ever read)
    for (int idx = tid; idx < CH * LDL; idx += PREP_THREADS) sL[idx] = 0.0f;
    bf16* ph = out + 6 * PLANE;
    for (int idx = tid; idx < 4 * 16 * 8; idx += PREP_THREADS) {
        const int row = (idx >> 3), at = row * CH + (row & ~15) + (idx & 7) * 2;
        *reinterpret_cast<uint32_t*>(ph + at) = 0u;
        *reinterpret_cast<uint32_t*>(ph + PPLANE + at) = 0u;
    }
    __syncthreads();
    // ---- A and P: two warps make the rows 16 I .. 16 I + 15, each eight columns of every block of sixteen
    {
        const int I = warp >> 1, half = warp & 1;
        const int i0 = I * 16 + g, i1 = i0 + 8;
        float accA[4][4], accP[4][4];                          // [block of columns]; the fourth: this block's own
#pragma unroll
        for (int J = 0; J < 4; ++J)
#pragma unroll
            for (int e = 0; e < 4; ++e) { accA[J][e] = 0.0f; accP[J][e] = 0.0f; }
        // a reference for the rows of this block against earlier ones: the sum at the last row before it; for its rows 8 .. 15 against
        // its rows 0 .. 7 (worked out by the first of the two warps): the sum at its row 7
        const float* ref = sG + (I > 0 ? I * 16 - 1 : 0) * LDG;
        const float* mid = sG + (I * 16 + 7) * LDG;
#pragma unroll 1
        for (int kk = 0; kk < DQ / 16; ++kk) {
            uint32_t rk[4], rq[4];                             // raw bf16 pairs: rows i0, i1 at channels c, c + 8
            const int c = kk * 16 + t2;
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int row = (u & 1) ? i1 : i0;
                rk[u] = *reinterpret_cast<const uint32_t*>(sk + row * LDR + c + (u >> 1) * 8);
                rq[u] = *reinterpret_cast<const uint32_t*>(sq + row * LDR + c + (u >> 1) * 8);
            }
            if (!CHANNEL) {
#pragma unroll
                for (int J = 0; J < 4; ++J) {
                    const int jb = J < 3 ? J : I;
                    if (J < 3 && J >= I) continue;
                    const bf16* row = sk + (jb * 16 + half * 8 + g) * LDR + c;
                    const uint32_t b0 = *reinterpret_cast<const uint32_t*>(row), b1 = *reinterpret_cast<const uint32_t*>(row + 8);
                    mma_bf16_16816(accA[J], rk, b0, b1);
                    mma_bf16_16816(accP[J], rq, b0, b1);
                }
            } else {
                uint32_t kh_[4], kl_[4], qh_[4], ql_[4];
                if (I > 0) {
                    const float2 ra = *reinterpret_cast<const float2*>(ref + c), rb = *reinterpret_cast<const float2*>(ref + c + 8);
                    const float r[4] = {ra.x, ra.y, rb.x, rb.y};
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const float2 gi = *reinterpret_cast<const float2*>(sG + ((u & 1) ? i1 : i0) * LDG + c + (u >> 1) * 8);
                        const float e0 = ex2_approx(gi.x - r[(u >> 1) * 2]), e1 = ex2_approx(gi.y - r[(u >> 1) * 2 + 1]);
                        const float2 k2 = bf2(rk[u]), q2 = bf2(rq[u]);
                        split_bf16(k2.x * e0, k2.y * e1, kh_[u], kl_[u]);
                        split_bf16(q2.x * e0, q2.y * e1, qh_[u], ql_[u]);
                    }
#pragma unroll
                    for (int J = 0; J < 3; ++J) {
                        if (J >= I) continue;
                        const int j = J * 16 + half * 8 + g;
                        const float2 ga = *reinterpret_cast<const float2*>(sG + j * LDG + c), gb = *reinterpret_cast<const float2*>(sG + j * LDG + c + 8);
                        const float2 x = bf2(*reinterpret_cast<const uint32_t*>(sk + j * LDR + c)), y = bf2(*reinterpret_cast<const uint32_t*>(sk + j * LDR + c + 8));
                        uint32_t bh0, bl0, bh1, bl1;
                        split_bf16(x.x * ex2_approx(r[0] - ga.x), x.y * ex2_approx(r[1] - ga.y), bh0, bl0);
                        split_bf16(y.x * ex2_approx(r[2] - gb.x), y.y * ex2_approx(r[3] - gb.y), bh1, bl1);
                        mma3(accA[J], kh_, kl_, bh0, bh1, bl0, bl1);
                        mma3(accP[J], qh_, ql_, bh0, bh1, bl0, bl1);
                    }
                }
                if (half == 0) {                               // rows 8 .. 15 of the block (the operands of rows 0 .. 7 are zero)
                    const float2 ra = *reinterpret_cast<const float2*>(mid + c), rb = *reinterpret_cast<const float2*>(mid + c + 8);
                    const float r[4] = {ra.x, ra.y, rb.x, rb.y};
                    kh_[0] = kh_[2] = kl_[0] = kl_[2] = qh_[0] = qh_[2] = ql_[0] = ql_[2] = 0u;
#pragma unroll
                    for (int u = 1; u < 4; u += 2) {
                        const float2 gi = *reinterpret_cast<const float2*>(sG + i1 * LDG + c + (u >> 1) * 8);
                        const float e0 = ex2_approx(gi.x - r[(u >> 1) * 2]), e1 = ex2_approx(gi.y - r[(u >> 1) * 2 + 1]);
                        const float2 k2 = bf2(rk[u]), q2 = bf2(rq[u]);
                        split_bf16(k2.x * e0, k2.y * e1, kh_[u], kl_[u]);
                        split_bf16(q2.x * e0, q2.y * e1, qh_[u], ql_[u]);
                    }
                    const float2 ga = *reinterpret_cast<const float2*>(sG + i0 * LDG + c), gb = *reinterpret_cast<const float2*>(sG + i0 * LDG + c + 8);   // token g of the block: the same index as row i0
                    const float2 x = bf2(rk[0]), y = bf2(rk[2]);
                    uint32_t bh0, bl0, bh1, bl1;
                    split_bf16(x.x * ex2_approx(r[0] - ga.x), x.y * ex2_approx(r[1] - ga.y), bh0, bl0);
                    split_bf16(y.x * ex2_approx(r[2] - gb.x), y.y * ex2_approx(r[3] - gb.y), bh1, bl1);
                    mma3(accA[3], kh_, kl_, bh0, bh1, bl0, bl1);
                    mma3(accP[3], qh_, ql_, bh0, bh1, bl0, bl1);
                }
            }
        }
#pragma unroll
        for (int J = 0; J < 4; ++J) {
            const int jb = J < 3 ? J : I;
            if ((J < 3 && J >= I) || (CHANNEL && J == 3 && half == 1)) continue;
            const int j = jb * 16 + half * 8 + t2;
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                if (CHANNEL && J == 3 && rr == 0) continue;    // rows 0 .. 7 of the block's own square: pair by pair below
                const int i = rr ? i1 : i0;
                float a[2], b[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float w = CHANNEL ? 1.0f : j + e <= i ? ex2_approx(sG[i] - sG[j + e]) : 0.0f;
                    a[e] = s_beta[i] * s_fk[i] * s_fk[j + e] * accA[J][rr * 2 + e] * w;
                    b[e] = s_fq[i] * s_fk[j + e] * accP[J][rr * 2 + e] * w;
                    if (j + e < i) sL[i * LDL + j + e] = a[e];
                }
                uint32_t hi, lo;                               // (a weight of zero where j > i)
                split_bf16(b[0], b[1], hi, lo);
                *reinterpret_cast<uint32_t*>(ph + i * CH + j) = hi;
                *reinterpret_cast<uint32_t*>(ph + PPLANE + i * CH + j) = lo;
            }
        }
        if (CHANNEL && lane < 28) {                            // the 8 x 8 square on the diagonal that is this warp's, a pair of rows per lane
            int ii = 1;
            while ((ii + 1) * ii / 2 <= lane) ++ii;
            const int i = warp * 8 + ii, j = warp * 8 + lane - ii * (ii - 1) / 2;
            float a = 0.0f, b = 0.0f;
#pragma unroll 4
            for (int c = 0; c < DQ; c += 2) {
                const float2 ki = bf2(*reinterpret_cast<const uint32_t*>(sk + i * LDR + c)), kj = bf2(*reinterpret_cast<const uint32_t*>(sk + j * LDR + c));
                const float2 qi = bf2(*reinterpret_cast<const uint32_t*>(sq + i * LDR + c));
                const float2 gi = *reinterpret_cast<const float2*>(sG + i * LDG + c), gj = *reinterpret_cast<const float2*>(sG + j * LDG + c);
                const float x = kj.x * ex2_approx(gi.x - gj.x), y = kj.y * ex2_approx(gi.y - gj.y);
                a = fmaf(ki.x, x, a); a = fmaf(ki.y, y, a);
                b = fmaf(qi.x, x, b); b = fmaf(qi.y, y, b);
            }
            sL[i * LDL + j] = s_beta[i] * s_fk[i] * s_fk[j] * a;
            b *= s_fq[i] * s_fk[j];
            const bf16 hi = __float2bfloat16_rn(b);
            ph[i * CH + j] = hi;
            ph[PPLANE + i * CH + j] = __float2bfloat16_rn(b - __bfloat162float(hi));
        }
        if (CHANNEL && tid < CH) {                             // P_ii = q_i . k_i
            const float b = s_qk[tid] * s_fq[tid] * s_fk[tid];
            const bf16 hi = __float2bfloat16_rn(b);
            ph[tid * CH + tid] = hi;
            ph[PPLANE + tid * CH + tid] = __float2bfloat16_rn(b - __bfloat162float(hi));
        }
    }
    __syncthreads();
    // ---- Q+, K exp(G_63 - G), exp(G_63)
    {
        for (int idx = tid; idx < CH * DQ / 2; idx += PREP_THREADS) {
            const int i = idx / (DQ / 2), c = (idx % (DQ / 2)) * 2;
            const float g0 = CHANNEL ? sG[i * LDG + c] : sG[i], g1 = CHANNEL ? sG[i * LDG + c + 1] : g0;
            const float e0 = CHANNEL ? sG[(CH - 1) * LDG + c] : sG[CH - 1], e1 = CHANNEL ? sG[(CH - 1) * LDG + c + 1] : e0;
            const float2 k2 = bf2(*reinterpret_cast<const uint32_t*>(sk + i * LDR + c)), q2 = bf2(*reinterpret_cast<const uint32_t*>(sq + i * LDR + c));
            uint32_t hi, lo;
            split_bf16(q2.x * s_fq[i] * ex2_approx(g0), q2.y * s_fq[i] * ex2_approx(g1), hi, lo);
            *reinterpret_cast<uint32_t*>(out + 2 * PLANE + i * DQ + c) = hi;
            *reinterpret_cast<uint32_t*>(out + 3 * PLANE + i * DQ + c) = lo;
            split_bf16(k2.x * s_fk[i] * ex2_approx(e0 - g0), k2.y * s_fk[i] * ex2_approx(e1 - g1), hi, lo);
            *reinterpret_cast<uint32_t*>(out + 4 * PLANE + i * DQ + c) = hi;
            *reinterpret_cast<uint32_t*>(out + 5 * PLANE + i * DQ + c) = lo;
        }
        for (int c = tid; c < DQ; c += PREP_THREADS) fout[CH * dv + c] = ex2_approx(CHANNEL ? sG[(CH - 1) * LDG + c] : sG[CH - 1]);
    }
    // ---- forward substitution, a column per thread: x_i = rhs_i - sum_(j < i) L_ij x_j
    for (int col = tid; col < DQ + dv; col += PREP_THREADS) {
        const bool is_w = col < DQ;
        const bf16* v = sv + (col - DQ);
        float x[CH];
#pragma unroll
        for (int i = 0; i < CH; ++i) {
            if (is_w) x[i] = s_beta[i] * s_fk[i] * __bfloat162float(sk[i * LDR + col]) * ex2_approx(CHANNEL ? sG[i * LDG + col] : sG[i]);
            else x[i] = s_beta[i] * __bfloat162float(v[i * (dv + 8)]);
        }
#pragma unroll
        for (int i = 1; i < CH; ++i) {
            float acc0 = x[i], acc1 = 0.0f;
#pragma unroll
            for (int j = 0; j < i; j += 4) {
                const float4 l = *reinterpret_cast<const float4*>(sL + i * LDL + j);        // (zero from the diagonal on)
                acc0 = fmaf(-l.x, x[j], acc0);
                if (j + 1 < i) acc1 = fmaf(-l.y, x[j + 1], acc1);
                if (j + 2 < i) acc0 = fmaf(-l.z, x[j + 2], acc0);
                if (j + 3 < i) acc1 = fmaf(-l.w, x[j + 3], acc1);
            }
            x[i] = acc0 + acc1;
        }
        if (is_w) {
#pragma unroll
            for (int i = 0; i < CH; ++i) {
                const bf16 hi = __float2bfloat16_rn(x[i]);
                out[i * DQ + col] = hi;
                out[PLANE + i * DQ + col] = __float2bfloat16_rn(x[i] - __bfloat162float(hi));
            }
        } else {
#pragma unroll
            for (int i = 0; i < CH; ++i) fout[(size_t)i * dv + col - DQ] = x[i];
        }
    }
}

// ---- the walk -------------------------------------------------------------------------------------------------------------------------
#define LDQ (DQ + 8)
#define LDS (VS + 8)
#define LDP (CH + 8)
#define WC (VS / 16)                  // column groups of 16
#define WARPS (4 * WC)
#define WALK_THREADS (32 * WARPS)
#define MT (DQ / 16)                  // 16-row tiles of the state, tiles warp, warp + WARPS, ... belong to a warp
#define MT_W ((MT + WARPS - 1) / WARPS)
#define NT (VS / 8)
#define WALK_SMEM ((6 * CH * LDQ + 2 * CH * LDP + 2 * DQ * LDS + 2 * CH * LDS) * 2)

__device__ __forceinline__ void copy_plane(bf16* dst, int ld, const bf16* src, int width) {     // [64][width] into rows of ld
    const int per = width / 8;
    for (int idx = threadIdx.x; idx < CH * per; idx += WALK_THREADS) {
        const int row = idx / per, c = idx - row * per;
        cp_async16(dst + row * ld + c * 8, src + row * width + c * 8);
    }
}

__global__ void __launch_bounds__(WALK_THREADS) walk_kernel(const bf16* __restrict__ planes, const float* __restrict__ floats, float* __restrict__ state,
                                                            const int* __restrict__ cu_tokens, const int* __restrict__ slots, float* __restrict__ o,
                                                            int first_req, int H, int dv) {
    PDL_ENTER_WALK();
    planes = pdl_fresh(planes); floats = pdl_fresh(floats);
    extern __shared__ __align__(16) uint8_t smem_raw[];
    bf16* sW = reinterpret_cast<bf16*>(smem_raw);      // [2][CH][LDQ] hi, lo
    bf16* sQ = sW + 2 * CH * LDQ;
    bf16* sK = sQ + 2 * CH * LDQ;
    bf16* sP = sK + 2 * CH * LDQ;                      // [2][CH][LDP]
    bf16* sS = sP + 2 * CH * LDP;                      // [2][DQ][LDS]
    bf16* sU = sS + 2 * DQ * LDS;                      // [2][CH][LDS]
    const int req = first_req + blockIdx.x, head = blockIdx.y, vs0 = blockIdx.z * VS;
    const int first = cu_tokens[req], count = cu_tokens[req + 1] - first;
    if (count <= 0) return;
    const int chunks = (count + CH - 1) / CH;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const int wr = warp & 3, wc = warp >> 2;           // this warp's 16 tokens and 16 columns in the products over tokens
    const size_t slot0 = (size_t)first_chunk(cu_tokens, first_req, req) * H + head;
    float* st = state + (((size_t)slots[req] * H + head) * DQ) * dv + vs0;
    float S[MT_W][NT][4];
#pragma unroll
    for (int mi = 0; mi < MT_W; ++mi) {
        const int m0 = (warp + WARPS * mi) * 16;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            S[mi][nt][0] = S[mi][nt][1] = S[mi][nt][2] = S[mi][nt][3] = 0.0f;
            if (m0 < DQ) {
                const float2 a = *reinterpret_cast<const float2*>(st + (size_t)(m0 + g) * dv + nt * 8 + t2);
                const float2 b = *reinterpret_cast<const float2*>(st + (size_t)(m0 + g + 8) * dv + nt * 8 + t2);
                S[mi][nt][0] = a.x; S[mi][nt][1] = a.y; S[mi][nt][2] = b.x; S[mi][nt][3] = b.y;
            }
        }
    }
    auto load_w = [&](int c) {
        if (c < chunks) {
            const bf16* p = planes + (slot0 + (size_t)c * H) * CHUNK_BF16;
            copy_plane(sW, LDQ, p, DQ);
            copy_plane(sW + CH * LDQ, LDQ, p + PLANE, DQ);
        }
        cp_async_commit();
    };
    auto load_qp = [&](int c) {
        if (c < chunks) {
            const bf16* p = planes + (slot0 + (size_t)c * H) * CHUNK_BF16;
            copy_plane(sQ, LDQ, p + 2 * PLANE, DQ);
            copy_plane(sQ + CH * LDQ, LDQ, p + 3 * PLANE, DQ);
            copy_plane(sP, LDP, p + 6 * PLANE, CH);
            copy_plane(sP + CH * LDP, LDP, p + 6 * PLANE + PPLANE, CH);
        }
        cp_async_commit();
    };
    auto load_k = [&](int c) {
        const bf16* p = planes + (slot0 + (size_t)c * H) * CHUNK_BF16;
        copy_plane(sK, LDQ, p + 4 * PLANE, DQ);
        copy_plane(sK + CH * LDQ, LDQ, p + 5 * PLANE, DQ);
        cp_async_commit();
    };
    load_w(0);
    load_qp(0);
    const size_t o_stride = (size_t)H * dv;
    const int a_row = wr * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;          // ldmatrix addresses: row operands ...
    const int b_row = (lane & 7) + ((lane >> 3) & 1) * 8, b_col = (lane >> 4) * 8;                    // ... and column operands read transposed
    const uint32_t w_addr = (uint32_t)__cvta_generic_to_shared(sW + a_row * LDQ + a_col), q_addr = (uint32_t)__cvta_generic_to_shared(sQ + a_row * LDQ + a_col);
    const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(sP + a_row * LDP + a_col);
    const uint32_t s_addr = (uint32_t)__cvta_generic_to_shared(sS + b_row * LDS + b_col + wc * 16), u_addr = (uint32_t)__cvta_generic_to_shared(sU + b_row * LDS + b_col);
    const uint32_t PL_Q = CH * LDQ * 2, PL_P = CH * LDP * 2, PL_S = DQ * LDS * 2, PL_U = CH * LDS * 2;     // bytes from a hi plane to its lo plane
    const int i0 = wr * 16 + g, i1 = i0 + 8, col = wc * 16 + t2;
    for (int c = 0; c < chunks; ++c) {
        const int rows = min(CH, count - c * CH);
        const float* f = floats + (slot0 + (size_t)c * H) * CHUNK_F32(dv);
        float u[2][4], last[MT_W][2];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            const float2 a = *reinterpret_cast<const float2*>(f + (size_t)i0 * dv + vs0 + col + nt * 8), b = *reinterpret_cast<const float2*>(f + (size_t)i1 * dv + vs0 + col + nt * 8);
            u[nt][0] = a.x; u[nt][1] = a.y; u[nt][2] = b.x; u[nt][3] = b.y;
        }
#pragma unroll
        for (int mi = 0; mi < MT_W; ++mi) {
            const int m0 = (warp + WARPS * mi) * 16;
            last[mi][0] = m0 < DQ ? f[CH * dv + m0 + g] : 0.0f;
            last[mi][1] = m0 < DQ ? f[CH * dv + m0 + g + 8] : 0.0f;
        }
        // the state as two bf16 operands (the products of the chunk before have read the old ones)
#pragma unroll
        for (int mi = 0; mi < MT_W; ++mi) {
            const int m0 = (warp + WARPS * mi) * 16;
            if (m0 < DQ) {
#pragma unroll
                for (int nt = 0; nt < NT; ++nt) {
                    uint32_t hi, lo;
                    split_bf16(S[mi][nt][0], S[mi][nt][1], hi, lo);
                    *reinterpret_cast<uint32_t*>(sS + (m0 + g) * LDS + nt * 8 + t2) = hi;
                    *reinterpret_cast<uint32_t*>(sS + DQ * LDS + (m0 + g) * LDS + nt * 8 + t2) = lo;
                    split_bf16(S[mi][nt][2], S[mi][nt][3], hi, lo);
                    *reinterpret_cast<uint32_t*>(sS + (m0 + g + 8) * LDS + nt * 8 + t2) = hi;
                    *reinterpret_cast<uint32_t*>(sS + DQ * LDS + (m0 + g + 8) * LDS + nt * 8 + t2) = lo;
                }
            }
        }
        cp_async_wait<1>();                            // W of this chunk (Q and P may still be on their way)
        __syncthreads();
        load_k(c);                                     // everyone has left the chunk before
        // U = U0 - W S
        {
            Sums3 acc;
            acc.clear();
#pragma unroll
            for (int kk = 0; kk < DQ / 16; ++kk) {
                uint32_t ah[4], al[4], bh[4], bl[4];
                ldsm_x4(w_addr + kk * 32, ah[0], ah[1], ah[2], ah[3]);
                ldsm_x4(w_addr + PL_Q + kk * 32, al[0], al[1], al[2], al[3]);
                ldsm_x4_trans(s_addr + kk * 16 * LDS * 2, bh[0], bh[1], bh[2], bh[3]);
                ldsm_x4_trans(s_addr + PL_S + kk * 16 * LDS * 2, bl[0], bl[1], bl[2], bl[3]);
                acc.add(ah, al, bh, bl);
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                uint32_t hi, lo;
                split_bf16(u[nt][0] - acc.at(nt, 0), u[nt][1] - acc.at(nt, 1), hi, lo);
                *reinterpret_cast<uint32_t*>(sU + i0 * LDS + col + nt * 8) = hi;
                *reinterpret_cast<uint32_t*>(sU + CH * LDS + i0 * LDS + col + nt * 8) = lo;
                split_bf16(u[nt][2] - acc.at(nt, 2), u[nt][3] - acc.at(nt, 3), hi, lo);
                *reinterpret_cast<uint32_t*>(sU + i1 * LDS + col + nt * 8) = hi;
                *reinterpret_cast<uint32_t*>(sU + CH * LDS + i1 * LDS + col + nt * 8) = lo;
            }
        }
        cp_async_wait<1>();                            // Q and P (K may still be on its way)
        __syncthreads();
        load_w(c + 1);                                 // everyone is done with W
        // O = Q+ S + P U
        {
            Sums3 acc;
            acc.clear();
#pragma unroll
            for (int kk = 0; kk < DQ / 16; ++kk) {
                uint32_t ah[4], al[4], bh[4], bl[4];
                ldsm_x4(q_addr + kk * 32, ah[0], ah[1], ah[2], ah[3]);
                ldsm_x4(q_addr + PL_Q + kk * 32, al[0], al[1], al[2], al[3]);
                ldsm_x4_trans(s_addr + kk * 16 * LDS * 2, bh[0], bh[1], bh[2], bh[3]);
                ldsm_x4_trans(s_addr + PL_S + kk * 16 * LDS * 2, bl[0], bl[1], bl[2], bl[3]);
                acc.add(ah, al, bh, bl);
            }
#pragma unroll
            for (int kk = 0; kk < CH / 16; ++kk) {
                if (kk > wr) continue;                 // later tokens have no weight
                uint32_t ah[4], al[4], bh[4], bl[4];
                ldsm_x4(p_addr + kk * 32, ah[0], ah[1], ah[2], ah[3]);
                ldsm_x4(p_addr + PL_P + kk * 32, al[0], al[1], al[2], al[3]);
                ldsm_x4_trans(u_addr + (kk * 16 * LDS + wc * 16) * 2, bh[0], bh[1], bh[2], bh[3]);
                ldsm_x4_trans(u_addr + PL_U + (kk * 16 * LDS + wc * 16) * 2, bl[0], bl[1], bl[2], bl[3]);
                acc.add(ah, al, bh, bl);
            }
            float* dst = o + (size_t)(first + c * CH) * o_stride + (size_t)head * dv + vs0 + col;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                if (i0 < rows) *reinterpret_cast<float2*>(dst + (size_t)i0 * o_stride + nt * 8) = make_float2(acc.at(nt, 0), acc.at(nt, 1));
                if (i1 < rows) *reinterpret_cast<float2*>(dst + (size_t)i1 * o_stride + nt * 8) = make_float2(acc.at(nt, 2), acc.at(nt, 3));
            }
        }
        cp_async_wait<1>();                            // K
        __syncthreads();
        load_qp(c + 1);                                // everyone is done with Q and P
        // S = exp(G_63) S + (K exp(G_63 - G))^T U
#pragma unroll
        for (int mi = 0; mi < MT_W; ++mi) {
            const int m0 = (warp + WARPS * mi) * 16;
            if (m0 < DQ) {
                // K^T as the row operand: tokens are its columns, read transposed from the [token][channel] tile
                const uint32_t k_addr = (uint32_t)__cvta_generic_to_shared(sK + ((lane & 7) + (lane >> 4) * 8) * LDQ + m0 + ((lane >> 3) & 1) * 8);
                Sums3 acc[NT / 2];
#pragma unroll
                for (int dt = 0; dt < NT / 2; ++dt) acc[dt].clear();
#pragma unroll
                for (int kk = 0; kk < CH / 16; ++kk) {
                    uint32_t ah[4], al[4];
                    ldsm_x4_trans(k_addr + kk * 16 * LDQ * 2, ah[0], ah[1], ah[2], ah[3]);
                    ldsm_x4_trans(k_addr + PL_Q + kk * 16 * LDQ * 2, al[0], al[1], al[2], al[3]);
#pragma unroll
                    for (int dt = 0; dt < NT / 2; ++dt) {
                        uint32_t bh[4], bl[4];
                        ldsm_x4_trans(u_addr + (kk * 16 * LDS + dt * 16) * 2, bh[0], bh[1], bh[2], bh[3]);
                        ldsm_x4_trans(u_addr + PL_U + (kk * 16 * LDS + dt * 16) * 2, bl[0], bl[1], bl[2], bl[3]);
                        acc[dt].add(ah, al, bh, bl);
                    }
                }
#pragma unroll
                for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[mi][nt][e] = fmaf(S[mi][nt][e], last[mi][e >> 1], acc[nt >> 1].at(nt & 1, e));
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int mi = 0; mi < MT_W; ++mi) {
        const int m0 = (warp + WARPS * mi) * 16;
        if (m0 < DQ) {
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                *reinterpret_cast<float2*>(st + (size_t)(m0 + g) * dv + nt * 8 + t2) = make_float2(S[mi][nt][0], S[mi][nt][1]);
                *reinterpret_cast<float2*>(st + (size_t)(m0 + g + 8) * dv + nt * 8 + t2) = make_float2(S[mi][nt][2], S[mi][nt][3]);
            }
        }
    }
}

// How many bf16 and float32 numbers a chunk and head needs between the two kernels.
MB_API int mb_delta_chunked_scratch(int dv, int* bf16s, int* floats) { *bf16s = CHUNK_BF16; *floats = CHUNK_F32(dv); return 0; }

// Requests first_req .. requests - 1.  qkv: bf16 [tokens][2 G QK_DIM + H dv] after the convolution (rows 16-byte aligned); b, a, their
// strides, per_channel, rate_log, dt_bias, state, o as mb_delta_scan takes them; dv a multiple of V_SLICE.  planes and floats hold
// (tokens / 64 + requests) * H pieces of mb_delta_chunked_scratch each.
MB_API int mb_delta_chunked(const void* qkv, const void* b_rows, int b_stride, const void* a_rows, int a_stride, int per_channel, const float* rate_log,
                            const float* dt_bias, float* state, const int* cu_tokens, const int* slots, float* o, void* planes, float* floats, int first_req,
                            int requests, int max_query_len, int H, int G, int dv, int which, cudaStream_t s) {
    if (requests <= first_req || max_query_len <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G != 0 || dv <= 0 || dv % VS != 0 || first_req < 0 || ((2 * G * DQ + H * dv) % 8) != 0) return MB_ERR_BAD_SIZE;
    if ((((uintptr_t)qkv | (uintptr_t)planes) & 15) != 0 || ((uintptr_t)floats & 7) != 0) return MB_ERR_BAD_SIZE;
    if (which == 0) {
        const int a_vec = a_stride % 8 == 0 && (((uintptr_t)a_rows | (uintptr_t)dt_bias) & 15) == 0;      // decays per channel by 16-byte loads
        dim3 grid((max_query_len + CH - 1) / CH, H, requests - first_req);
        if (per_channel) {
            cudaFuncSetAttribute(prepare_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, PREP_SMEM(1, dv));
            return launch_kernel(prepare_kernel<true>, grid, PREP_THREADS, PREP_SMEM(1, dv), s, 0, (const bf16*)qkv, (const bf16*)b_rows, b_stride,
                                 (const bf16*)a_rows, a_stride, rate_log, dt_bias, cu_tokens, first_req, (bf16*)planes, floats, H, G, dv, a_vec);
        }
        cudaFuncSetAttribute(prepare_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, PREP_SMEM(0, dv));
        return launch_kernel(prepare_kernel<false>, grid, PREP_THREADS, PREP_SMEM(0, dv), s, 0, (const bf16*)qkv, (const bf16*)b_rows, b_stride,
                             (const bf16*)a_rows, a_stride, rate_log, dt_bias, cu_tokens, first_req, (bf16*)planes, floats, H, G, dv, a_vec);
    }
    cudaFuncSetAttribute(walk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, WALK_SMEM);
    return launch_kernel(walk_kernel, dim3(requests - first_req, H, dv / VS), WALK_THREADS, WALK_SMEM, s, 0, (const bf16*)planes, (const float*)floats,
                         state, cu_tokens, slots, o, first_req, H, dv);
}
