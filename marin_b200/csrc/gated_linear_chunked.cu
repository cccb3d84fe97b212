// Gated linear attention (gated_linear.cu) over prompt portions, 64 tokens at a time on the tensor cores (mma.sync), compiled for one head
// layout: -DQK_DIM (key channels, a multiple of 16 up to 128), -DV_SLICE (value channels a CTA takes: a multiple of 16 up to 128).
//
// With S0 the state before a chunk and G_i[c] the sum of the log-decays of its tokens 0 .. i in key channel c,
//     o_i = (q_i exp(G_i)) S0 + sum_(j <= i) P_ij v_j,   P_ij = sum_c q_i[c] k_j[c] exp(G_i[c] - G_j[c]),
//     S   = exp(G_63) S0 + sum_j (k_j exp(G_63 - G_j)) v_j^T.
// Nothing but exp(G_63) S0 ties a chunk to the one before, so three kernels do it, only the second of them in order:
//   add_kernel    (a CTA per chunk, head and slice): the log-decays and their sums G, and what the chunk adds to the state;
//   carry_kernel  (a thread per four numbers of a state): walks the chunks, leaves in each chunk's place the state before it;
//   read_kernel   (a CTA per chunk, head and slice): P, then the outputs; where a CTA has a whole head, also its norm, weight and gate.
//
// Exactness.  Every exponent that is taken is of a non-positive number: a block of 16 rows of P is worked out against a reference between it
// and the earlier rows (exp(G_i - R) exp(R - G_j), both at most 1), the lower half of a block's diagonal square against one in its
// middle, and the 8 x 8 squares left on the diagonal pair by pair.  Decays, sums and the state are float32; where a float32 number has to be
// an operand of a product it is split into two bf16 numbers (value = hi + lo) and the larger products are taken, so that about 16
// bits of it enter.  k and v are bf16 as the projection left them.
#define MB_LIB "gated_linear_chunked"
#define MB_LIB_ID 23
#include "common.cuh"
#include "launch.cuh"
#include "mma_helpers.cuh"

#ifndef QK_DIM
#define QK_DIM 128
#endif
#ifndef V_SLICE
#define V_SLICE 128
#endif
static_assert(QK_DIM % 16 == 0 && QK_DIM >= 16 && QK_DIM <= 128, "key channels: a multiple of 16 up to 128");
static_assert(V_SLICE % 16 == 0 && V_SLICE >= 16 && V_SLICE <= 128, "value channels of a CTA: a multiple of 16 up to 128");

#define DQ QK_DIM
#define VS V_SLICE
#define VP ((VS + 31) / 32 * 32)      // the slice in whole pairs of 16 columns (what lies beyond it is zero)
#define CH 64
#define THREADS 256
#define LOG2E 1.4426950408889634f
#define LDR (DQ + 8)                  // q and k rows in shared memory (bf16)
#define LDG (DQ + 8)                  // sums (float32)
#define LDV (VP + 8)
#define LDP (CH + 8)
#define ST 32                         // rows of the state in shared memory at a time, twice

__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float2 bf2(uint32_t w) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w)); }
__device__ __forceinline__ uint32_t word(const bf16* p) { return *reinterpret_cast<const uint32_t*>(p); }

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

// What a chunk and head keeps between the kernels, float32: G in log2 units [64][DQ], then what it adds to the state, replaced by the state before it, [DQ][dv].
#define CHUNK_F32(dv) (CH * DQ + DQ * (dv))

// Where request r's chunks start among all chunks of the step (room is left for a partial chunk per request).
__device__ __forceinline__ int first_chunk(const int* cu_tokens, int first_req, int r) { return (cu_tokens[r] - cu_tokens[first_req]) / CH + (r - first_req); }

// `rows` rows of `width` bf16 (a multiple of 8) into shared rows of `ld`, rows past them up to CH zero, columns up to `padded` zero.
__device__ __forceinline__ void take_rows(bf16* dst, int ld, const bf16* src, size_t stride, int rows, int width, int padded) {
    const int per = padded / 8;
    for (int idx = threadIdx.x; idx < CH * per; idx += THREADS) {
        const int row = idx / per, c = (idx - row * per) * 8;
        if (row < rows && c < width) cp_async16(dst + row * ld + c, src + (size_t)row * stride + c);
        else *reinterpret_cast<uint4*>(dst + row * ld + c) = make_uint4(0, 0, 0, 0);
    }
}

#define ADD_SMEM(rank) (CH * LDR * 2 + CH * LDV * 2 + CH * LDG * 4 + (CH + DQ) * ((rank) + 8) * 2)

__global__ void __launch_bounds__(THREADS, 2) add_kernel(
    const bf16* __restrict__ k, const bf16* __restrict__ v, const bf16* __restrict__ l, int in_stride, const bf16* __restrict__ w2,
    const float* __restrict__ bias, int rank, float inv_tau, const int* __restrict__ cu_tokens, int first_req, float* __restrict__ floats, int H, int dv,
    int slices) {
    PDL_ENTER();
    k = pdl_fresh(k); v = pdl_fresh(v); l = pdl_fresh(l);
    extern __shared__ __align__(16) uint8_t smem_raw[];
    float* sG = reinterpret_cast<float*>(smem_raw);            // [CH][LDG], log2 units
    bf16* sk = reinterpret_cast<bf16*>(sG + CH * LDG);         // [CH][LDR]
    bf16* sv = sk + CH * LDR;                                  // [CH][LDV]
    bf16* sl = sv + CH * LDV;                                  // [CH][rank + 8]
    const int LDL = rank + 8;
    bf16* sw = sl + CH * LDL;                                  // [DQ][rank + 8]
    const int req = first_req + blockIdx.z / slices, slice = blockIdx.z % slices, head = blockIdx.y, vs0 = slice * VS;
    const int tok0 = cu_tokens[req] + blockIdx.x * CH;
    const int rows = min(CH, cu_tokens[req + 1] - tok0);
    if (rows <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    float* out = floats + ((size_t)(first_chunk(cu_tokens, first_req, req) + blockIdx.x) * H + head) * CHUNK_F32(dv);
    take_rows(sl, LDL, l + (size_t)tok0 * in_stride, in_stride, rows, rank, rank);
    {
        const int per = rank / 8;
        for (int idx = tid; idx < DQ * per; idx += THREADS) {
            const int row = idx / per, c = (idx - row * per) * 8;
            cp_async16(sw + row * LDL + c, w2 + ((size_t)head * DQ + row) * rank + c);
        }
    }
    cp_async_commit();
    take_rows(sk, LDR, k + (size_t)tok0 * in_stride + (size_t)head * DQ, in_stride, rows, DQ, DQ);
    take_rows(sv, LDV, v + (size_t)tok0 * in_stride + (size_t)head * dv + vs0, in_stride, rows, VS, VP);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    // ---- log-decays: z = l W_2^T, 16 tokens and half of the channels per warp
    {
        const int i0 = (warp & 3) * 16 + g, i1 = i0 + 8, n_first = (warp >> 2) * (DQ / 16);
        const float rate = -inv_tau * LOG2E;
#pragma unroll 2
        for (int n = 0; n < DQ / 16; ++n) {
            const int c = (n_first + n) * 8;
            float z[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            for (int kk = 0; kk < rank; kk += 16) {
                uint32_t a[4];
                a[0] = word(sl + i0 * LDL + kk + t2); a[1] = word(sl + i1 * LDL + kk + t2);
                a[2] = word(sl + i0 * LDL + kk + 8 + t2); a[3] = word(sl + i1 * LDL + kk + 8 + t2);
                mma_bf16_16816(z, a, word(sw + (c + g) * LDL + kk + t2), word(sw + (c + g) * LDL + kk + 8 + t2));
            }
            const float2 b = *reinterpret_cast<const float2*>(bias + head * DQ + c + t2);
            float2 x, y;
            x.x = i0 < rows ? rate * softplus_f(-(z[0] + b.x)) : 0.0f;
            x.y = i0 < rows ? rate * softplus_f(-(z[1] + b.y)) : 0.0f;
            y.x = i1 < rows ? rate * softplus_f(-(z[2] + b.x)) : 0.0f;
            y.y = i1 < rows ? rate * softplus_f(-(z[3] + b.y)) : 0.0f;
            *reinterpret_cast<float2*>(sG + i0 * LDG + c + t2) = x;
            *reinterpret_cast<float2*>(sG + i1 * LDG + c + t2) = y;
        }
    }
    __syncthreads();
    // ---- running sums: SEG threads a channel, each a run of rows, then the runs before
    {
        constexpr int SEG = THREADS / DQ >= 8 ? 8 : THREADS / DQ >= 4 ? 4 : 2, RUN = CH / SEG;
        const int c = tid % DQ, seg = tid / DQ;
        float run = 0.0f, before = 0.0f;
        if (seg < SEG)
#pragma unroll 8
            for (int i = seg * RUN; i < seg * RUN + RUN; ++i) { run += sG[i * LDG + c]; sG[i * LDG + c] = run; }
        __syncthreads();
        if (seg < SEG)
            for (int s = 0; s < seg; ++s) before += sG[(s * RUN + RUN - 1) * LDG + c];
        __syncthreads();
        if (seg > 0 && seg < SEG)
#pragma unroll 8
            for (int i = seg * RUN; i < seg * RUN + RUN; ++i) sG[i * LDG + c] += before;
    }
    cp_async_wait<0>();
    __syncthreads();
    if (slice == 0)
        for (int idx = tid; idx < CH * DQ / 4; idx += THREADS) {
            const int row = idx / (DQ / 4), c = idx % (DQ / 4) * 4;
            *reinterpret_cast<float4*>(out + row * DQ + c) = *reinterpret_cast<const float4*>(sG + row * LDG + c);
        }
    // ---- (k exp(G_63 - G))^T v: a warp has 16 key channels (and a part of the columns where there are more warps than that)
    constexpr int MT = DQ / 16, SHARE = MT >= 8 ? 1 : MT >= 4 ? 2 : MT >= 2 ? 4 : 8, NPAIR = VP / 16;
    for (int job = warp; job < MT * SHARE; job += THREADS / 32) {
        const int m0 = job % MT * 16, part = job / MT;
        const float e0 = sG[(CH - 1) * LDG + m0 + g], e1 = sG[(CH - 1) * LDG + m0 + g + 8];
        constexpr int NP_W = (NPAIR + SHARE - 1) / SHARE;      // pairs of 8 columns a warp has
        float acc[NP_W][2][4];
#pragma unroll
        for (int n = 0; n < NP_W; ++n)
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[n][h][e] = 0.0f;
        const uint32_t v_addr = (uint32_t)__cvta_generic_to_shared(sv + ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (lane >> 4) * 8 + part * NP_W * 16);
#pragma unroll
        for (int kk = 0; kk < CH / 16; ++kk) {
            uint32_t ah[4], al[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int c = m0 + g + (u & 1) * 8, t = kk * 16 + t2 + (u >> 1) * 8;
                const float last = (u & 1) ? e1 : e0;
                split_bf16(__bfloat162float(sk[t * LDR + c]) * ex2_approx(last - sG[t * LDG + c]),
                           __bfloat162float(sk[(t + 1) * LDR + c]) * ex2_approx(last - sG[(t + 1) * LDG + c]), ah[u], al[u]);
            }
#pragma unroll
            for (int n = 0; n < NP_W; ++n) {
                if (part * NP_W + n >= NPAIR) continue;
                uint32_t b0, b1, b2, b3;
                ldsm_x4_trans(v_addr + (kk * 16 * LDV + n * 16) * 2, b0, b1, b2, b3);
                mma_bf16_16816(acc[n][0], ah, b0, b1);
                mma_bf16_16816(acc[n][1], ah, b2, b3);
                mma_bf16_16816(acc[n][0], al, b0, b1);
                mma_bf16_16816(acc[n][1], al, b2, b3);
            }
        }
        float* dst = out + CH * DQ + (size_t)(m0 + g) * dv + vs0 + t2;
#pragma unroll
        for (int n = 0; n < NP_W; ++n)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int col = (part * NP_W + n) * 16 + h * 8;
                if (col >= VS) continue;
                *reinterpret_cast<float2*>(dst + col) = make_float2(acc[n][h][0], acc[n][h][1]);
                *reinterpret_cast<float2*>(dst + (size_t)8 * dv + col) = make_float2(acc[n][h][2], acc[n][h][3]);
            }
    }
}

// ---- the states before every chunk, and the one behind the last -----------------------------------------------------------------
#define CARRY_AHEAD 4
__global__ void __launch_bounds__(256) carry_kernel(float* floats, float* __restrict__ state, const int* __restrict__ cu_tokens, const int* __restrict__ slots,
                                                    int first_req, int H, int dv) {
    PDL_ENTER();
    floats = pdl_fresh(floats);
    const int req = first_req + blockIdx.z, head = blockIdx.y;
    const int count = cu_tokens[req + 1] - cu_tokens[req];
    const int at = (blockIdx.x * 256 + threadIdx.x) * 4;       // four numbers of one row (dv is a multiple of 4)
    if (count <= 0 || at >= DQ * dv) return;
    const int chunks = (count + CH - 1) / CH, n = at / dv;
    const size_t step = (size_t)H * CHUNK_F32(dv);
    float* base = floats + ((size_t)first_chunk(cu_tokens, first_req, req) * H + head) * CHUNK_F32(dv);
    float4* kept = reinterpret_cast<float4*>(state + ((size_t)slots[req] * H + head) * DQ * dv + at);
    float4 s = *kept;
    float4 add[CARRY_AHEAD];
    float decay[CARRY_AHEAD];
    for (int c0 = 0; c0 < chunks; c0 += CARRY_AHEAD) {
#pragma unroll
        for (int u = 0; u < CARRY_AHEAD; ++u)
            if (c0 + u < chunks) {
                const float* p = base + (c0 + u) * step;
                add[u] = *reinterpret_cast<const float4*>(p + CH * DQ + at);
                decay[u] = p[(CH - 1) * DQ + n];
            }
#pragma unroll
        for (int u = 0; u < CARRY_AHEAD; ++u)
            if (c0 + u < chunks) {
                *reinterpret_cast<float4*>(base + (c0 + u) * step + CH * DQ + at) = s;
                const float e = ex2_approx(decay[u]);
                s.x = fmaf(s.x, e, add[u].x); s.y = fmaf(s.y, e, add[u].y); s.z = fmaf(s.z, e, add[u].z); s.w = fmaf(s.w, e, add[u].w);
            }
    }
    *kept = s;
}

// ---- the outputs -------------------------------------------------------------------------------------------------------------------
#define QK_BYTES (2 * CH * LDR * 2)
#define S_BYTES (2 * 2 * ST * LDV * 2)
#define READ_SMEM (CH * LDG * 4 + (QK_BYTES > S_BYTES ? QK_BYTES : S_BYTES) + CH * LDV * 2 + 2 * CH * LDP * 2)
static_assert(CH * LDG * 4 == 2 * CH * LDR * 2, "the weighted queries take the sums' place");

template <bool WHOLE>
__global__ void __launch_bounds__(THREADS, 2) read_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, int in_stride, const float* __restrict__ floats,
    const int* __restrict__ cu_tokens, int first_req, int H, int dv, int slices, float* __restrict__ o, const bf16* __restrict__ gate_rows, int gate_stride,
    int gate, const float* __restrict__ norm_w, float eps, float factor, bf16* __restrict__ out, int out_stride) {
    PDL_ENTER();
    q = pdl_fresh(q); k = pdl_fresh(k); v = pdl_fresh(v); floats = pdl_fresh(floats); gate_rows = pdl_fresh(gate_rows);
    extern __shared__ __align__(16) uint8_t smem_raw[];
    __shared__ float s_qk[CH], s_ss[2][CH];
    float* sG = reinterpret_cast<float*>(smem_raw);            // [CH][LDG]; later q exp(G), hi and lo: [2][CH][LDR] bf16
    bf16* sQ = reinterpret_cast<bf16*>(sG);
    bf16* sq = reinterpret_cast<bf16*>(sG + CH * LDG);         // [CH][LDR] q, then k; later two tiles of the state, hi and lo: [2][2][ST][LDV]
    bf16* sk = sq + CH * LDR;
    bf16* sS = sq;
    bf16* sv = reinterpret_cast<bf16*>(smem_raw + CH * LDG * 4 + (QK_BYTES > S_BYTES ? QK_BYTES : S_BYTES));
    bf16* sP = sv + CH * LDV;                                  // [2][CH][LDP] hi, lo
    const int req = first_req + blockIdx.z / slices, head = blockIdx.y, vs0 = (blockIdx.z % slices) * VS;
    const int tok0 = cu_tokens[req] + blockIdx.x * CH;
    const int rows = min(CH, cu_tokens[req + 1] - tok0);
    if (rows <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = 2 * (lane & 3);
    const float* kept = floats + ((size_t)(first_chunk(cu_tokens, first_req, req) + blockIdx.x) * H + head) * CHUNK_F32(dv);
    const float* S = kept + CH * DQ + vs0;
    for (int idx = tid; idx < CH * DQ / 4; idx += THREADS) {
        const int row = idx / (DQ / 4), c = idx % (DQ / 4) * 4;
        cp_async16(sG + row * LDG + c, kept + row * DQ + c);
    }
    take_rows(sq, LDR, q + (size_t)tok0 * in_stride + (size_t)head * DQ, in_stride, rows, DQ, DQ);
    take_rows(sk, LDR, k + (size_t)tok0 * in_stride + (size_t)head * DQ, in_stride, rows, DQ, DQ);
    take_rows(sv, LDV, v + (size_t)tok0 * in_stride + (size_t)head * dv + vs0, in_stride, rows, VS, VP);
    cp_async_commit();
    // the state's first tile, asked for now and stored once q and k are done with
    constexpr int S_ITEMS = (ST * VP / 4 + THREADS - 1) / THREADS;
    float4 tile[S_ITEMS];
    auto ask = [&](int kt) {
#pragma unroll
        for (int u = 0; u < S_ITEMS; ++u) {
            const int idx = tid + u * THREADS, row = idx / (VP / 4), c = idx % (VP / 4) * 4;
            tile[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (row < ST && kt * ST + row < DQ && c < VS) tile[u] = *reinterpret_cast<const float4*>(S + (size_t)(kt * ST + row) * dv + c);
        }
    };
    auto lay = [&](int kt) {
        bf16* hi = sS + (kt & 1) * 2 * ST * LDV;
#pragma unroll
        for (int u = 0; u < S_ITEMS; ++u) {
            const int idx = tid + u * THREADS, row = idx / (VP / 4), c = idx % (VP / 4) * 4;
            if (row >= ST) continue;
            uint2 h, w;
            split_bf16(tile[u].x, tile[u].y, h.x, w.x);
            split_bf16(tile[u].z, tile[u].w, h.y, w.y);
            *reinterpret_cast<uint2*>(hi + row * LDV + c) = h;
            *reinterpret_cast<uint2*>(hi + ST * LDV + row * LDV + c) = w;
        }
    };
    ask(0);
    const float scale = 1.0f / sqrtf((float)DQ);
    cp_async_wait<0>();
    __syncthreads();
    for (int row = warp; row < CH; row += THREADS / 32) {
        float qk = 0.0f;
        for (int c = lane; c < DQ; c += 32) qk = fmaf(__bfloat162float(sq[row * LDR + c]), __bfloat162float(sk[row * LDR + c]), qk);
        qk = warp_sum(qk);
        if (lane == 0) s_qk[row] = qk;
    }
    for (int idx = tid; idx < 4 * 16 * 8; idx += THREADS) {    // (of the upper triangle only what lies in a diagonal block is ever read)
        const int row = (idx >> 3), at = row * LDP + (row & ~15) + (idx & 7) * 2;
        *reinterpret_cast<uint32_t*>(sP + at) = 0u;
        *reinterpret_cast<uint32_t*>(sP + CH * LDP + at) = 0u;
    }
    __syncthreads();
    // ---- P: two warps make the rows 16 I .. 16 I + 15, each eight columns of every block of sixteen
    {
        const int I = warp >> 1, half = warp & 1;
        const int i0 = I * 16 + g, i1 = i0 + 8;
        float acc[4][4];                                       // [block of columns]; the fourth: this block's own
#pragma unroll
        for (int J = 0; J < 4; ++J)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[J][e] = 0.0f;
        // a reference for the rows of this block against earlier ones: the sum at the last row before it; for its rows 8 .. 15 against
        // its rows 0 .. 7 (worked out by the first of the two warps): the sum at its row 7
        const float* ref = sG + (I > 0 ? I * 16 - 1 : 0) * LDG;
        const float* mid = sG + (I * 16 + 7) * LDG;
#pragma unroll 1
        for (int kk = 0; kk < DQ / 16; ++kk) {
            const int c = kk * 16 + t2;
            uint32_t rq[4], qh[4], ql[4];                      // raw bf16 pairs: rows i0, i1 at channels c, c + 8
#pragma unroll
            for (int u = 0; u < 4; ++u) rq[u] = word(sq + ((u & 1) ? i1 : i0) * LDR + c + (u >> 1) * 8);
            if (I > 0) {
                const float2 ra = *reinterpret_cast<const float2*>(ref + c), rb = *reinterpret_cast<const float2*>(ref + c + 8);
                const float r[4] = {ra.x, ra.y, rb.x, rb.y};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const float2 gi = *reinterpret_cast<const float2*>(sG + ((u & 1) ? i1 : i0) * LDG + c + (u >> 1) * 8), q2 = bf2(rq[u]);
                    split_bf16(q2.x * ex2_approx(gi.x - r[(u >> 1) * 2]), q2.y * ex2_approx(gi.y - r[(u >> 1) * 2 + 1]), qh[u], ql[u]);
                }
#pragma unroll
                for (int J = 0; J < 3; ++J) {
                    if (J >= I) continue;
                    const int j = J * 16 + half * 8 + g;
                    const float2 ga = *reinterpret_cast<const float2*>(sG + j * LDG + c), gb = *reinterpret_cast<const float2*>(sG + j * LDG + c + 8);
                    const float2 x = bf2(word(sk + j * LDR + c)), y = bf2(word(sk + j * LDR + c + 8));
                    uint32_t bh0, bl0, bh1, bl1;
                    split_bf16(x.x * ex2_approx(r[0] - ga.x), x.y * ex2_approx(r[1] - ga.y), bh0, bl0);
                    split_bf16(y.x * ex2_approx(r[2] - gb.x), y.y * ex2_approx(r[3] - gb.y), bh1, bl1);
                    mma3(acc[J], qh, ql, bh0, bh1, bl0, bl1);
                }
            }
            if (half == 0) {                                   // rows 8 .. 15 of the block (the operands of rows 0 .. 7 are zero)
                const float2 ra = *reinterpret_cast<const float2*>(mid + c), rb = *reinterpret_cast<const float2*>(mid + c + 8);
                const float r[4] = {ra.x, ra.y, rb.x, rb.y};
                qh[0] = qh[2] = ql[0] = ql[2] = 0u;
#pragma unroll
                for (int u = 1; u < 4; u += 2) {
                    const float2 gi = *reinterpret_cast<const float2*>(sG + i1 * LDG + c + (u >> 1) * 8), q2 = bf2(rq[u]);
                    split_bf16(q2.x * ex2_approx(gi.x - r[(u >> 1) * 2]), q2.y * ex2_approx(gi.y - r[(u >> 1) * 2 + 1]), qh[u], ql[u]);
                }
                // (token g of the block: the same index as row i0)
                const float2 ga = *reinterpret_cast<const float2*>(sG + i0 * LDG + c), gb = *reinterpret_cast<const float2*>(sG + i0 * LDG + c + 8);
                const float2 x = bf2(word(sk + i0 * LDR + c)), y = bf2(word(sk + i0 * LDR + c + 8));
                uint32_t bh0, bl0, bh1, bl1;
                split_bf16(x.x * ex2_approx(r[0] - ga.x), x.y * ex2_approx(r[1] - ga.y), bh0, bl0);
                split_bf16(y.x * ex2_approx(r[2] - gb.x), y.y * ex2_approx(r[3] - gb.y), bh1, bl1);
                mma3(acc[3], qh, ql, bh0, bh1, bl0, bl1);
            }
        }
#pragma unroll
        for (int J = 0; J < 4; ++J) {
            if ((J < 3 && J >= I) || (J == 3 && half == 1)) continue;
            const int j = (J < 3 ? J : I) * 16 + half * 8 + t2;
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                if (J == 3 && rr == 0) continue;               // rows 0 .. 7 of the block's own square: pair by pair below
                const int i = rr ? i1 : i0;
                uint32_t hi, lo;
                split_bf16(acc[J][rr * 2] * scale, acc[J][rr * 2 + 1] * scale, hi, lo);
                *reinterpret_cast<uint32_t*>(sP + i * LDP + j) = hi;
                *reinterpret_cast<uint32_t*>(sP + CH * LDP + i * LDP + j) = lo;
            }
        }
        if (lane < 28) {                                       // the 8 x 8 square on the diagonal that is this warp's, a pair of rows per lane
            int ii = 1;
            while ((ii + 1) * ii / 2 <= lane) ++ii;
            const int i = warp * 8 + ii, j = warp * 8 + lane - ii * (ii - 1) / 2;
            float b = 0.0f, b2 = 0.0f;
#pragma unroll 4
            for (int c = 0; c < DQ; c += 2) {
                const float2 qi = bf2(word(sq + i * LDR + c)), kj = bf2(word(sk + j * LDR + c));
                const float2 gi = *reinterpret_cast<const float2*>(sG + i * LDG + c), gj = *reinterpret_cast<const float2*>(sG + j * LDG + c);
                b = fmaf(qi.x * kj.x, ex2_approx(gi.x - gj.x), b);
                b2 = fmaf(qi.y * kj.y, ex2_approx(gi.y - gj.y), b2);
            }
            b = (b + b2) * scale;
            const bf16 hi = __float2bfloat16_rn(b);
            sP[i * LDP + j] = hi;
            sP[CH * LDP + i * LDP + j] = __float2bfloat16_rn(b - __bfloat162float(hi));
        }
        if (tid < CH) {                                        // P_ii = q_i . k_i
            const float b = s_qk[tid] * scale;
            const bf16 hi = __float2bfloat16_rn(b);
            sP[tid * LDP + tid] = hi;
            sP[CH * LDP + tid * LDP + tid] = __float2bfloat16_rn(b - __bfloat162float(hi));
        }
    }
    // ---- q exp(G) takes G's place
    {
        constexpr int ITEMS = CH * DQ / 2 / THREADS;
        uint32_t hi[ITEMS], lo[ITEMS];
#pragma unroll
        for (int u = 0; u < ITEMS; ++u) {
            const int idx = tid + u * THREADS, row = idx / (DQ / 2), c = idx % (DQ / 2) * 2;
            const float2 g2 = *reinterpret_cast<const float2*>(sG + row * LDG + c), q2 = bf2(word(sq + row * LDR + c));
            split_bf16(q2.x * scale * ex2_approx(g2.x), q2.y * scale * ex2_approx(g2.y), hi[u], lo[u]);
        }
        __syncthreads();                                       // everyone has left G, q and k
#pragma unroll
        for (int u = 0; u < ITEMS; ++u) {
            const int idx = tid + u * THREADS, row = idx / (DQ / 2), c = idx % (DQ / 2) * 2;
            *reinterpret_cast<uint32_t*>(sQ + row * LDR + c) = hi[u];
            *reinterpret_cast<uint32_t*>(sQ + CH * LDR + row * LDR + c) = lo[u];
        }
    }
    lay(0);
    // ---- O = P V + (q exp(G)) S: a warp has 16 tokens and half of the columns
    const int wr = warp & 3, wc = warp >> 2, i0 = wr * 16 + g, i1 = i0 + 8;
    constexpr int NP = VP / 32;                                // pairs of 8 columns a warp has
    float acc[NP][2][4];
#pragma unroll
    for (int n = 0; n < NP; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[n][h][e] = 0.0f;
    const int a_row = wr * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;          // ldmatrix addresses: row operands ...
    const int b_row = (lane & 7) + ((lane >> 3) & 1) * 8, b_col = (lane >> 4) * 8 + wc * (VP / 2);    // ... and column operands read transposed
    const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(sP + a_row * LDP + a_col), q_addr = (uint32_t)__cvta_generic_to_shared(sQ + a_row * LDR + a_col);
    const uint32_t v_addr = (uint32_t)__cvta_generic_to_shared(sv + b_row * LDV + b_col), s_addr = (uint32_t)__cvta_generic_to_shared(sS + b_row * LDV + b_col);
    constexpr int TILES = (DQ + ST - 1) / ST;
#pragma unroll 1
    for (int kt = 0; kt < TILES; ++kt) {
        if (kt + 1 < TILES) ask(kt + 1);
        __syncthreads();                                       // this tile (and, at first, P and q exp(G)) is there
        if (kt == 0) {
#pragma unroll
            for (int kk = 0; kk < CH / 16; ++kk) {
                if (kk > wr) continue;                         // later tokens have no weight
                uint32_t ah[4], al[4];
                ldsm_x4(p_addr + kk * 32, ah[0], ah[1], ah[2], ah[3]);
                ldsm_x4(p_addr + CH * LDP * 2 + kk * 32, al[0], al[1], al[2], al[3]);
#pragma unroll
                for (int n = 0; n < NP; ++n) {
                    uint32_t b[4];
                    ldsm_x4_trans(v_addr + (kk * 16 * LDV + n * 16) * 2, b[0], b[1], b[2], b[3]);
                    mma_bf16_16816(acc[n][0], ah, b[0], b[1]);
                    mma_bf16_16816(acc[n][1], ah, b[2], b[3]);
                    mma_bf16_16816(acc[n][0], al, b[0], b[1]);
                    mma_bf16_16816(acc[n][1], al, b[2], b[3]);
                }
            }
        }
        const uint32_t hi = s_addr + (kt & 1) * 2 * ST * LDV * 2;
#pragma unroll
        for (int kk = 0; kk < ST / 16; ++kk) {
            if (kt * ST + kk * 16 >= DQ) break;
            uint32_t ah[4], al[4];
            ldsm_x4(q_addr + (kt * ST + kk * 16) * 2, ah[0], ah[1], ah[2], ah[3]);
            ldsm_x4(q_addr + (CH * LDR + kt * ST + kk * 16) * 2, al[0], al[1], al[2], al[3]);
#pragma unroll
            for (int n = 0; n < NP; ++n) {
                uint32_t b[4], c[4];
                ldsm_x4_trans(hi + (kk * 16 * LDV + n * 16) * 2, b[0], b[1], b[2], b[3]);
                ldsm_x4_trans(hi + (ST * LDV + kk * 16 * LDV + n * 16) * 2, c[0], c[1], c[2], c[3]);
                mma3(acc[n][0], ah, al, b[0], b[1], c[0], c[1]);
                mma3(acc[n][1], ah, al, b[2], b[3], c[2], c[3]);
            }
        }
        if (kt + 1 < TILES) lay(kt + 1);                       // (its buffer was read a tile ago: the barrier above lies between)
    }
    if (!WHOLE) {
        float* dst = o + (size_t)tok0 * H * dv + (size_t)head * dv + vs0 + t2;
#pragma unroll
        for (int n = 0; n < NP; ++n)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int col = wc * (VP / 2) + n * 16 + h * 8;
                if (col >= VS) continue;
                if (i0 < rows) *reinterpret_cast<float2*>(dst + (size_t)i0 * H * dv + col) = make_float2(acc[n][h][0], acc[n][h][1]);
                if (i1 < rows) *reinterpret_cast<float2*>(dst + (size_t)i1 * H * dv + col) = make_float2(acc[n][h][2], acc[n][h][3]);
            }
        return;
    }
    // ---- the norm over the head's channels (columns beyond it are zero), weight and gate
    float ss0 = 0.0f, ss1 = 0.0f;
#pragma unroll
    for (int n = 0; n < NP; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            ss0 += acc[n][h][0] * acc[n][h][0] + acc[n][h][1] * acc[n][h][1];
            ss1 += acc[n][h][2] * acc[n][h][2] + acc[n][h][3] * acc[n][h][3];
        }
    ss0 += __shfl_xor_sync(0xffffffffu, ss0, 1); ss0 += __shfl_xor_sync(0xffffffffu, ss0, 2);
    ss1 += __shfl_xor_sync(0xffffffffu, ss1, 1); ss1 += __shfl_xor_sync(0xffffffffu, ss1, 2);
    if ((lane & 3) == 0) { s_ss[wc][i0] = ss0; s_ss[wc][i1] = ss1; }
    __syncthreads();
    const float f0 = factor / sqrtf((s_ss[0][i0] + s_ss[1][i0]) / (float)VS + eps), f1 = factor / sqrtf((s_ss[0][i1] + s_ss[1][i1]) / (float)VS + eps);
#pragma unroll
    for (int n = 0; n < NP; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int col = wc * (VP / 2) + n * 16 + h * 8 + t2;
            if (col >= VS) continue;
            const float2 w = *reinterpret_cast<const float2*>(norm_w + col);
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                const int i = rr ? i1 : i0;
                if (i >= rows) continue;
                const float f = rr ? f1 : f0;
                const float2 z = bf2(word(gate_rows + (size_t)(tok0 + i) * gate_stride + (size_t)head * dv + col));
                float2 y = make_float2(__fdividef(1.0f, 1.0f + __expf(-z.x)), __fdividef(1.0f, 1.0f + __expf(-z.y)));
                if (gate == 1) { y.x *= z.x; y.y *= z.y; }
                *reinterpret_cast<uint32_t*>(out + (size_t)(tok0 + i) * out_stride + (size_t)head * dv + col) =
                    pack_bf16(acc[n][h][rr * 2] * f * w.x * y.x, acc[n][h][rr * 2 + 1] * f * w.y * y.y);
            }
        }
}

// How many float32 numbers a chunk and head needs between the kernels.
MB_API int mb_gla_chunked_scratch(int dv) { return CHUNK_F32(dv); }

// Requests first_req .. requests - 1; which: 0 adds, 1 carries, 2 reads (in this order).  q, k, v, l, w2, bias, state as mb_gla_scan takes them (bf16, 16-byte
// aligned, in_stride a multiple of 8, rank a multiple of 16 up to 128); dv a multiple of V_SLICE.  floats holds (tokens / 64 + requests) * H
// pieces of mb_gla_chunked_scratch.  A whole head in one slice (dv == V_SLICE): normed and gated rows go to `out`; else the sums to `o`.
MB_API int mb_gla_chunked(int which, const void* q, const void* k, const void* v, const void* l, int in_stride, const void* w2, const float* bias, int rank,
                          float inv_tau, float* state, const int* cu_tokens, const int* slots, float* floats, float* o, const void* gate_rows, int gate_stride,
                          int gate, const float* norm_w, float eps, float factor, void* out, int out_stride, int first_req, int requests, int max_query_len,
                          int H, int dv, cudaStream_t s) {
    if (requests <= first_req || max_query_len <= 0) return 0;
    if (H <= 0 || dv <= 0 || dv % VS != 0 || first_req < 0 || rank <= 0 || rank % 16 != 0 || rank > 128 || in_stride % 8 != 0 || gate < 0 || gate > 1) return MB_ERR_BAD_SIZE;
    if ((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)l | (uintptr_t)w2 | (uintptr_t)floats | (uintptr_t)state) & 15) != 0 || ((uintptr_t)bias & 7) != 0)
        return MB_ERR_BAD_SIZE;
    const int slices = dv / VS, count = requests - first_req;
    dim3 grid((max_query_len + CH - 1) / CH, H, count * slices);
    if (which == 0) {
        cudaFuncSetAttribute(add_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, ADD_SMEM(rank));
        return launch_kernel(add_kernel, grid, THREADS, ADD_SMEM(rank), s, 0, (const bf16*)k, (const bf16*)v, (const bf16*)l, in_stride, (const bf16*)w2, bias, rank,
                             inv_tau, cu_tokens, first_req, floats, H, dv, slices);
    }
    if (which == 1)
        return launch_kernel(carry_kernel, dim3((DQ * dv / 4 + 255) / 256, H, count), 256, 0, s, 0, floats, state, cu_tokens, slots, first_req, H, dv);
    if (slices == 1) {
        if ((((uintptr_t)gate_rows | (uintptr_t)out) & 3) != 0 || gate_stride % 2 != 0 || out_stride % 2 != 0 || out_stride < H * dv || ((uintptr_t)norm_w & 7) != 0) return MB_ERR_BAD_SIZE;
        cudaFuncSetAttribute(read_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, READ_SMEM);
        return launch_kernel(read_kernel<true>, grid, THREADS, READ_SMEM, s, 0, (const bf16*)q, (const bf16*)k, (const bf16*)v, in_stride, (const float*)floats, cu_tokens,
                             first_req, H, dv, slices, o, (const bf16*)gate_rows, gate_stride, gate, norm_w, eps, factor, (bf16*)out, out_stride);
    }
    cudaFuncSetAttribute(read_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, READ_SMEM);
    return launch_kernel(read_kernel<false>, grid, THREADS, READ_SMEM, s, 0, (const bf16*)q, (const bf16*)k, (const bf16*)v, in_stride, (const float*)floats, cu_tokens,
                         first_req, H, dv, slices, o, (const bf16*)gate_rows, gate_stride, gate, norm_w, eps, factor, (bf16*)out, out_stride);
}
