// Gated linear attention (Yang, Wang, Shen, Panda, Kim, "Gated Linear Attention Transformers with Hardware-Efficient Training"): a matrix
// per head whose rows, one per key channel, every token decays by a factor of its own and adds to,
//     S <- diag(alpha) S + k v^T,   o = S^T q,   alpha = sigmoid(z)^(1 / tau),   z = W_2 l + bias,
// S a dim x vdim matrix in float32 ([slot][head][dim][vdim], zero at a sequence's start), q times dim^(-1/2).  l (`rank` numbers a token) is
// what a first small matrix made of the layer's input; the second one, W_2, is applied here, so that z and the decays are never
// rounded: log alpha = -softplus(-z) / tau.  o per head is divided by its root mean square over vdim, times a weight [vdim], times silu or
// sigmoid of a gate, times a factor.
// q, k, v, l and the gate come as the projections left them (column blocks of one product's rows, `in_stride` elements apart); everything
// else is float32 in both dtypes.
// This file: the recurrence token by token (any size, both dtypes; the norm with its gate is delta_rule.cu's), and all of it for single
// tokens in one kernel.
#define MB_LIB "gated_linear"
#define MB_LIB_ID 22
#include "common.cuh"
#include "launch.cuh"

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// z of one channel: its row of W_2 (`rank` numbers, 16-byte aligned rows where vec) times l (shared memory).
template <typename T>
__device__ __forceinline__ float decay_input(const T* __restrict__ w, const float* l, int rank) {
    float a = 0.0f, b = 0.0f;
    for (int r = 0; r + 1 < rank; r += 2) { a = fmaf(to_f32(w[r]), l[r], a); b = fmaf(to_f32(w[r + 1]), l[r + 1], b); }
    if (rank & 1) a = fmaf(to_f32(w[rank - 1]), l[rank - 1], a);
    return a + b;
}

// ---- the recurrence token by token: a block per (request, head, slice of GS_COLS value channels) ------------------------------
// Four threads share a column of the state: thread (column, part) keeps the rows part, part + 4, ... in registers, ROWS of them.
// Tokens are taken in runs of GS_RUN: their q, k, v and decays go to shared memory, then the run is walked without a barrier (the
// four partial sums of a column meet by shuffles).
#define GS_COLS 32
#define GS_THREADS (GS_COLS * 4)
#define GS_RUN 8

template <typename T, int ROWS>
__global__ void __launch_bounds__(GS_THREADS) gla_scan_kernel(
    const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ l, int in_stride, const T* __restrict__ w2,
    const float* __restrict__ bias, int rank, float inv_tau, float* __restrict__ state, const int* __restrict__ cu_tokens,
    const int* __restrict__ slots, float* __restrict__ o, int first_req, int H, int d, int dv) {
    PDL_ENTER_WALK();
    q = pdl_fresh(q); k = pdl_fresh(k); v = pdl_fresh(v); l = pdl_fresh(l);
    extern __shared__ float smem[];
    float* ks = smem;                          // [GS_RUN][d]
    float* qs = ks + GS_RUN * d;               // [GS_RUN][d]
    float* gs = qs + GS_RUN * d;               // [GS_RUN][d] decays
    float* vs = gs + GS_RUN * d;               // [GS_RUN][GS_COLS]
    float* ls = vs + GS_RUN * GS_COLS;         // [GS_RUN][rank]
    const int req = first_req + blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * GS_COLS;
    const int first = cu_tokens[req], count = cu_tokens[req + 1] - first;
    if (count <= 0) return;
    const int col = threadIdx.x >> 2, part = threadIdx.x & 3, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = col0 + col;
    const bool in_range = c < dv;
    float* S = state + ((size_t)slots[req] * H + head) * d * dv;
    float s[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = part + 4 * j;
        s[j] = (in_range && n < d) ? S[(size_t)n * dv + c] : 0.0f;
    }
    const float q_scale = 1.0f / sqrtf((float)d);
    for (int base = 0; base < count; base += GS_RUN) {
        const int run = min(GS_RUN, count - base);
        __syncthreads();
        for (int tt = warp; tt < run; tt += GS_THREADS / 32) {     // a warp per token
            const size_t t = (size_t)(first + base + tt) * in_stride;
            for (int r = lane; r < rank; r += 32) ls[tt * rank + r] = to_f32(l[t + r]);
            __syncwarp();
            for (int n = lane; n < d; n += 32) {
                qs[tt * d + n] = to_f32(q[t + head * d + n]) * q_scale;
                ks[tt * d + n] = to_f32(k[t + head * d + n]);
                const float z = decay_input(w2 + (size_t)(head * d + n) * rank, ls + tt * rank, rank) + bias[head * d + n];
                gs[tt * d + n] = expf(-softplus_f(-z) * inv_tau);
            }
            vs[tt * GS_COLS + lane] = col0 + lane < dv ? to_f32(v[t + (size_t)head * dv + col0 + lane]) : 0.0f;
        }
        __syncthreads();
        for (int tt = 0; tt < run; ++tt) {
            float sums[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const float vv = vs[tt * GS_COLS + col];
#pragma unroll
            for (int j = 0; j < ROWS; ++j) {
                const int n = part + 4 * j;
                if (n < d) {
                    s[j] = fmaf(ks[tt * d + n], vv, s[j] * gs[tt * d + n]);
                    sums[j & 3] = fmaf(s[j], qs[tt * d + n], sums[j & 3]);
                }
            }
            float out = (sums[0] + sums[1]) + (sums[2] + sums[3]);
            out += __shfl_xor_sync(0xffffffffu, out, 1);
            out += __shfl_xor_sync(0xffffffffu, out, 2);
            if (part == 0 && in_range) o[(size_t)(first + base + tt) * H * dv + (size_t)head * dv + c] = out;
        }
    }
    if (in_range) {
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
            const int n = part + 4 * j;
            if (n < d) S[(size_t)n * dv + c] = s[j];
        }
    }
}

template <typename T>
static int gla_scan_rows(int rows, dim3 grid, size_t smem, cudaStream_t s, const T* q, const T* k, const T* v, const T* l, int in_stride, const T* w2,
                         const float* bias, int rank, float inv_tau, float* state, const int* cu_tokens, const int* slots, float* o, int first_req, int H,
                         int d, int dv) {
#define GS_CASE(R)                                                                                                                        \
    if (rows <= R)                                                                                                                        \
        return launch_kernel(gla_scan_kernel<T, R>, grid, GS_THREADS, smem, s, 0, q, k, v, l, in_stride, w2, bias, rank, inv_tau, state, cu_tokens, \
                             slots, o, first_req, H, d, dv);
    GS_CASE(4) GS_CASE(8) GS_CASE(16) GS_CASE(32) GS_CASE(64)
#undef GS_CASE
    return MB_ERR_BAD_SIZE;
}

// Requests first_req .. requests - 1.  q, k: the first of H heads of d in token 0's row, v of H heads of dv, l of `rank` numbers; w2: [H d][rank];
// o: float32 [tokens][H dv].
MB_API int mb_gla_scan(const void* q, const void* k, const void* v, const void* l, int in_stride, int dtype, const void* w2, const float* bias, int rank,
                       float inv_tau, float* state, const int* cu_tokens, const int* slots, float* o, int first_req, int requests, int H, int d, int dv,
                       cudaStream_t s) {
    if (requests <= first_req) return 0;
    if (H <= 0 || d <= 0 || d > 256 || dv <= 0 || rank <= 0 || rank > 512 || first_req < 0) return MB_ERR_BAD_SIZE;
    dim3 grid(requests - first_req, H, (dv + GS_COLS - 1) / GS_COLS);
    const size_t smem = (size_t)(3 * GS_RUN * d + GS_RUN * GS_COLS + GS_RUN * rank) * sizeof(float);
    if (smem > 48 * 1024) return MB_ERR_BAD_SIZE;
    const int rows = (d + 3) / 4;
    if (dtype == MB_F32)
        return gla_scan_rows<float>(rows, grid, smem, s, (const float*)q, (const float*)k, (const float*)v, (const float*)l, in_stride, (const float*)w2, bias,
                                    rank, inv_tau, state, cu_tokens, slots, o, first_req, H, d, dv);
    if (dtype == MB_BF16)
        return gla_scan_rows<bf16>(rows, grid, smem, s, (const bf16*)q, (const bf16*)k, (const bf16*)v, (const bf16*)l, in_stride, (const bf16*)w2, bias, rank,
                                   inv_tau, state, cu_tokens, slots, o, first_req, H, d, dv);
    return MB_ERR_BAD_DTYPE;
}

// ---- single tokens, all of it in one kernel: a block per (head, request) --------------------------------------------------------
// The state of a head is read once, all loads in flight while the decays are worked out, and written once.  Thread (group, part): the
// four columns 4 group .. 4 group + 3 of the rows part, part + PARTS, ..., ROWS of them, in registers; the PARTS partial sums of a
// column meet in shared memory in a fixed order.
template <typename T, int ROWS, int PARTS>
__global__ void __launch_bounds__(512) gla_single_kernel(
    const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ l, int in_stride, const T* __restrict__ w2,
    const float* __restrict__ bias, int rank, float inv_tau, float* __restrict__ state, const int* __restrict__ seq_lens, const int* __restrict__ slots,
    const T* __restrict__ g, int gate, const float* __restrict__ norm_w, float eps, float factor, T* __restrict__ out, int out_stride, int H, int d, int dv) {
    // The state is asked for before the wait for the kernel ahead: only this kernel (and the prompt kernels) of an earlier step wrote it,
    // and every step has kernels in between that let nothing start before all work ahead of them is done (its embedding, the norms);
    // slots and lengths are the step's inputs, copied before its first kernel.  All else waits.
#ifdef PDL_LAUNCH_FIRST
    PDL_ENTER();
#endif
    extern __shared__ float smem[];
    const int d4 = (d + 3) / 4 * 4;
    float* qs = smem;                          // [d]
    float* ks = qs + d4;                       // [d]
    float* gs = ks + d4;                       // [d]
    float* vs = gs + d4;                       // [dv]
    float* sums = vs + dv;                     // [PARTS][dv]
    float* ls = sums + PARTS * dv;             // [rank]
    __shared__ float scratch[32];
    const int head = blockIdx.x, r = blockIdx.y;
    if (seq_lens[r] <= 0) return;              // a row that pads a captured batch
    const int groups = dv >> 2, threads = blockDim.x;
    const int slot = slots[r];
    const int grp = threadIdx.x % groups, part = threadIdx.x / groups;
    const bool owner = part < PARTS;
    float4* S = reinterpret_cast<float4*>(state + ((size_t)slot * H + head) * d * dv) + grp;
    float4 s[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = part + PARTS * j;
        s[j] = (owner && n < d) ? S[(size_t)n * groups] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#ifndef PDL_LAUNCH_FIRST
    PDL_ENTER();
#endif
    q = pdl_fresh(q); k = pdl_fresh(k); v = pdl_fresh(v); l = pdl_fresh(l); g = pdl_fresh(g);
    const size_t row = (size_t)r * in_stride;
    float gate_raw = 0.0f, norm_raw = 0.0f;    // asked for early, used late
    if (threadIdx.x < dv) {
        gate_raw = to_f32(g[row + (size_t)head * dv + threadIdx.x]);
        norm_raw = norm_w[threadIdx.x];
    }
    for (int i = threadIdx.x; i < rank; i += threads) ls[i] = to_f32(l[row + i]);
    for (int i = threadIdx.x; i < dv; i += threads) vs[i] = to_f32(v[row + (size_t)head * dv + i]);
    const float q_scale = 1.0f / sqrtf((float)d);
    for (int i = threadIdx.x; i < d; i += threads) {
        qs[i] = to_f32(q[row + (size_t)head * d + i]) * q_scale;
        ks[i] = to_f32(k[row + (size_t)head * d + i]);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < d; i += threads) {
        const float z = decay_input(w2 + (size_t)(head * d + i) * rank, ls, rank) + bias[head * d + i];
        gs[i] = expf(-softplus_f(-z) * inv_tau);
    }
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner) {
        const float4 vv = *reinterpret_cast<const float4*>(vs + 4 * grp);
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
            const int n = part + PARTS * j;
            if (n < d) {
                const float gn = gs[n], kn = ks[n], qn = qs[n];
                s[j].x = fmaf(kn, vv.x, s[j].x * gn); s[j].y = fmaf(kn, vv.y, s[j].y * gn); s[j].z = fmaf(kn, vv.z, s[j].z * gn); s[j].w = fmaf(kn, vv.w, s[j].w * gn);
                acc.x = fmaf(s[j].x, qn, acc.x); acc.y = fmaf(s[j].y, qn, acc.y); acc.z = fmaf(s[j].z, qn, acc.z); acc.w = fmaf(s[j].w, qn, acc.w);
                S[(size_t)n * groups] = s[j];
            }
        }
        *reinterpret_cast<float4*>(sums + part * dv + 4 * grp) = acc;
    }
    __syncthreads();
    // the norm over the head's channels and the gate
    float ss = 0.0f;
    for (int i = threadIdx.x; i < dv; i += threads) {
        float a = 0.0f;
#pragma unroll
        for (int p = 0; p < PARTS; ++p) a += sums[p * dv + i];
        vs[i] = a;                             // (v itself is not needed any more; a thread reads back only what it wrote)
        ss = fmaf(a, a, ss);
    }
    ss = block_sum(ss, scratch);
    const float f = factor / sqrtf(ss / (float)dv + eps);
    for (int i = threadIdx.x; i < dv; i += threads) {
        const float z = i < threads ? gate_raw : to_f32(g[row + (size_t)head * dv + i]);
        const float wn = i < threads ? norm_raw : norm_w[i];
        out[(size_t)r * out_stride + (size_t)head * dv + i] = from_f32<T>(vs[i] * f * wn * (gate == 0 ? sigmoid_f(z) : silu_f(z)));
    }
}

// Whether the one kernel takes these sizes: a head's state in the registers of one block.
MB_API int mb_gla_single_supported(int d, int dv) {
    return d >= 1 && d <= 256 && dv >= 4 && dv <= 256 && dv % 4 == 0 && (dv / 4) * (d > 128 ? 16 : 8) <= 512;
}

template <typename T>
static int gla_single_launch(dim3 grid, cudaStream_t s, const T* q, const T* k, const T* v, const T* l, int in_stride, const T* w2, const float* bias, int rank,
                             float inv_tau, float* state, const int* seq_lens, const int* slots, const T* g, int gate, const float* norm_w, float eps,
                             float factor, T* out, int out_stride, int H, int d, int dv) {
    const int parts = d > 128 ? 16 : 8, rows = (d + parts - 1) / parts;
    const int threads = ((dv / 4) * parts + 31) / 32 * 32;
    const size_t smem = (size_t)(3 * ((d + 3) / 4 * 4) + dv + parts * dv + rank) * sizeof(float);
#define G1_CASE(R, P)                                                                                                                          \
    if (parts == P && rows <= R)                                                                                                               \
        return launch_kernel(gla_single_kernel<T, R, P>, grid, threads, smem, s, 0, q, k, v, l, in_stride, w2, bias, rank, inv_tau, state, seq_lens, slots, \
                             g, gate, norm_w, eps, factor, out, out_stride, H, d, dv);
    G1_CASE(2, 8) G1_CASE(4, 8) G1_CASE(8, 8) G1_CASE(16, 8) G1_CASE(16, 16)
#undef G1_CASE
    return MB_ERR_BAD_SIZE;
}

// Requests 0 .. requests - 1 bring one token each (token r is request r's); gate 0: sigmoid, 1: silu, of g (H heads of dv in the same rows).
MB_API int mb_gla_single(const void* q, const void* k, const void* v, const void* l, int in_stride, int dtype, const void* w2, const float* bias, int rank,
                         float inv_tau, float* state, const int* seq_lens, const int* slots, const void* g, int gate, const float* norm_w, float eps,
                         float factor, void* out, int out_stride, int requests, int H, int d, int dv, cudaStream_t s) {
    if (requests <= 0) return 0;
    if (H <= 0 || rank <= 0 || rank > 512 || gate < 0 || gate > 1 || !mb_gla_single_supported(d, dv) || out_stride < H * dv) return MB_ERR_BAD_SIZE;
    dim3 grid(H, requests);
    if (dtype == MB_F32)
        return gla_single_launch<float>(grid, s, (const float*)q, (const float*)k, (const float*)v, (const float*)l, in_stride, (const float*)w2, bias, rank,
                                        inv_tau, state, seq_lens, slots, (const float*)g, gate, norm_w, eps, factor, (float*)out, out_stride, H, d, dv);
    if (dtype == MB_BF16)
        return gla_single_launch<bf16>(grid, s, (const bf16*)q, (const bf16*)k, (const bf16*)v, (const bf16*)l, in_stride, (const bf16*)w2, bias, rank, inv_tau,
                                       state, seq_lens, slots, (const bf16*)g, gate, norm_w, eps, factor, (bf16*)out, out_stride, H, d, dv);
    return MB_ERR_BAD_DTYPE;
}
