// The gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"): a matrix per head
// that every token decays, corrects and reads,
//     S <- g S (row by row),   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q,
// S a dim x vdim matrix in float32 ([slot][head][dim][vdim], zero at a sequence's start).  Around it:
//   * q | k | v (G heads of dim, G heads of dim, H heads of vdim; head h uses q and k head h / (H / G)) through a short causal
//     convolution per channel and silu.  A request keeps its latest inputs as a ring of `taps` rows (float32 [slot][taps]
//     [channels]): the input at position p lies in row p mod taps, so a single token reads rows p - 1 .. p - taps + 1 and
//     writes row p with nothing to shift, and a sequence's first tokens are told by their positions (zeros before the start);
//   * q and k divided by sqrt(sum of squares + 1e-6) per head, q also times dim^(-1/2);
//   * beta = sigmoid(b);  g = exp(-exp(A_log_h) softplus(a + dt_bias)): one per head, or one per head and key channel;
//   * o per head divided by its root mean square over vdim, times a weight [vdim], times sigmoid or silu of a gate, times a factor.
// Convolution inputs, b, a and the gate come as the projections left them; everything else is float32 in both dtypes.
// This file: the convolution, the recurrence token by token (any size, both dtypes), the norm with its gate, and all of it for
// single tokens in one kernel.
#define MB_LIB "delta_rule"
#define MB_LIB_ID 20
#include "common.cuh"
#include "launch.cuh"

#define UNIT_EPS 1e-6f

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// ---- the convolution over the step's tokens from `first_token` on: a thread per (token, channel) -----------------------------
template <typename T>
__global__ void delta_conv_kernel(const T* __restrict__ in, int in_stride, const float* __restrict__ w, const float* __restrict__ ring,
                                  const int* __restrict__ positions, const int* __restrict__ req_index, const int* __restrict__ cu_tokens,
                                  const int* __restrict__ slots, T* __restrict__ out, int first_token, int channels, int taps) {
    PDL_ENTER();
    in = pdl_fresh(in); ring = pdl_fresh(ring);
    const int c = blockIdx.y * blockDim.x + threadIdx.x, t = first_token + blockIdx.x;
    if (c >= channels) return;
    const int req = req_index[t], pos = positions[t];
    const int first = cu_tokens[req];
    const float* kept = ring + (size_t)slots[req] * taps * channels;
    float sum = 0.0f;
    for (int back = min(taps - 1, pos); back >= 0; --back) {
        const float v = t - back >= first ? to_f32(in[(size_t)(t - back) * in_stride + c]) : kept[(size_t)((pos - back) % taps) * channels + c];
        sum = fmaf(w[(size_t)(taps - 1 - back) * channels + c], v, sum);
    }
    out[(size_t)t * channels + c] = from_f32<T>(silu_f(sum));
}

// The same for bf16 channels in multiples of 8: a thread owns 8 channels of CONV_RUN consecutive tokens, keeps the last TAPS - 1
// inputs in registers and reads every row once (16-byte loads).  At a request's first token the window is filled from its ring.
#define CONV_RUN 8

__device__ __forceinline__ void unpack8(const uint4& raw, float* x) {
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h2[i]); x[2 * i] = f.x; x[2 * i + 1] = f.y; }
}

template <int TAPS>
__global__ void __launch_bounds__(128) delta_conv_run_kernel(
    const bf16* __restrict__ in, int in_stride, const float* __restrict__ w, const float* __restrict__ ring, const int* __restrict__ positions,
    const int* __restrict__ req_index, const int* __restrict__ cu_tokens, const int* __restrict__ slots, bf16* __restrict__ out, int first_token,
    int tokens, int channels) {
    PDL_ENTER();
    in = pdl_fresh(in); ring = pdl_fresh(ring);
    const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (c0 >= channels) return;
    const int t0 = first_token + blockIdx.x * CONV_RUN, t1 = min(tokens, t0 + CONV_RUN);
    float wt[8][TAPS], past[TAPS > 1 ? TAPS - 1 : 1][8];       // past[b]: the input b + 1 tokens back
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        const float4 a = *reinterpret_cast<const float4*>(w + (size_t)j * channels + c0), b = *reinterpret_cast<const float4*>(w + (size_t)j * channels + c0 + 4);
        wt[0][j] = a.x; wt[1][j] = a.y; wt[2][j] = a.z; wt[3][j] = a.w; wt[4][j] = b.x; wt[5][j] = b.y; wt[6][j] = b.z; wt[7][j] = b.w;
    }
    uint4 raw[CONV_RUN];                                       // every row of the run in flight at once
#pragma unroll
    for (int u = 0; u < CONV_RUN; ++u)
        if (t0 + u < t1) raw[u] = *reinterpret_cast<const uint4*>(in + (size_t)(t0 + u) * in_stride + c0);
    int req = req_index[t0], first = cu_tokens[req], end = cu_tokens[req + 1];
#pragma unroll
    for (int u = 0; u < CONV_RUN; ++u) {
        const int t = t0 + u;
        if (t >= t1) break;
        if (t == end) { req = req_index[t]; first = t; end = cu_tokens[req + 1]; }
        if (TAPS > 1 && (u == 0 || t == first)) {              // fill the window: from this step's rows, the ring, or nothing
            const int pos = positions[t];
            const float* kept = ring + (size_t)slots[req] * TAPS * channels + c0;
#pragma unroll
            for (int b = 0; b < TAPS - 1; ++b) {
                if (t - b - 1 >= first) unpack8(*reinterpret_cast<const uint4*>(in + (size_t)(t - b - 1) * in_stride + c0), past[b]);
                else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) past[b][e] = pos - b - 1 >= 0 ? kept[(size_t)((pos - b - 1) % TAPS) * channels + e] : 0.0f;
                }
            }
        }
        float now[8];
        unpack8(raw[u], now);
        uint4 packed;
        __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(&packed);
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            float sum = 0.0f;                                  // (the oldest first, as the plain kernel adds)
#pragma unroll
            for (int b = TAPS - 2; b >= 0; --b) sum = fmaf(wt[e][TAPS - 2 - b], past[b][e], sum);
            sum = fmaf(wt[e][TAPS - 1], now[e], sum);
            y[e] = __fdividef(sum, 1.0f + __expf(-sum));       // (a few float32 ulps, far inside the rounding to bf16)
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) p2[i] = __floats2bfloat162_rn(y[2 * i], y[2 * i + 1]);
        *reinterpret_cast<uint4*>(out + (size_t)t * channels + c0) = packed;
#pragma unroll
        for (int b = TAPS - 2; b > 0; --b)
#pragma unroll
            for (int e = 0; e < 8; ++e) past[b][e] = past[b - 1][e];
        if (TAPS > 1) {
#pragma unroll
            for (int e = 0; e < 8; ++e) past[0][e] = now[e];
        }
    }
}

// The ring after the step: the inputs of a request's last taps - 1 tokens (or as many as it brought).
template <typename T>
__global__ void delta_ring_kernel(const T* __restrict__ in, int in_stride, float* __restrict__ ring, const int* __restrict__ positions,
                                  const int* __restrict__ cu_tokens, const int* __restrict__ slots, int first_req, int channels, int taps) {
    PDL_ENTER();
    in = pdl_fresh(in);
    const int c = blockIdx.x * blockDim.x + threadIdx.x, req = first_req + blockIdx.y;
    if (c >= channels) return;
    const int end = cu_tokens[req + 1], first = max(cu_tokens[req], end - (taps - 1));
    float* kept = ring + (size_t)slots[req] * taps * channels;
    for (int t = first; t < end; ++t) kept[(size_t)(positions[t] % taps) * channels + c] = to_f32(in[(size_t)t * in_stride + c]);
}

// w: float32 [taps][channels], the last row meets the current token.  Tokens first_token .. tokens - 1, requests first_req .. requests - 1; out: [tokens][channels].
MB_API int mb_delta_conv(const void* in, int in_stride, int dtype, const float* w, const float* ring, const int* positions, const int* req_index,
                         const int* cu_tokens, const int* slots, void* out, int first_token, int tokens, int channels, int taps, cudaStream_t s) {
    if (tokens <= first_token) return 0;
    if (channels <= 0 || taps <= 0 || taps > 64 || first_token < 0) return MB_ERR_BAD_SIZE;
    dim3 grid(tokens - first_token, (channels + 127) / 128);
    if (dtype == MB_F32)
        return launch_kernel(delta_conv_kernel<float>, grid, 128, 0, s, 0, (const float*)in, in_stride, w, ring, positions, req_index, cu_tokens,
                             slots, (float*)out, first_token, channels, taps);
    if (dtype == MB_BF16 && taps <= 4 && channels % 8 == 0 && in_stride % 8 == 0 && (((uintptr_t)in | (uintptr_t)out | (uintptr_t)w) & 15) == 0) {
        dim3 runs((tokens - first_token + CONV_RUN - 1) / CONV_RUN, (channels / 8 + 127) / 128);
#define CONV_CASE(N)                                                                                                                              \
    if (taps == N)                                                                                                                                \
        return launch_kernel(delta_conv_run_kernel<N>, runs, 128, 0, s, 0, (const bf16*)in, in_stride, w, ring, positions, req_index, cu_tokens, slots, \
                             (bf16*)out, first_token, tokens, channels);
        CONV_CASE(1) CONV_CASE(2) CONV_CASE(3) CONV_CASE(4)
#undef CONV_CASE
    }
    if (dtype == MB_BF16)
        return launch_kernel(delta_conv_kernel<bf16>, grid, 128, 0, s, 0, (const bf16*)in, in_stride, w, ring, positions, req_index, cu_tokens,
                             slots, (bf16*)out, first_token, channels, taps);
    return MB_ERR_BAD_DTYPE;
}

MB_API int mb_delta_ring(const void* in, int in_stride, int dtype, float* ring, const int* positions, const int* cu_tokens, const int* slots,
                         int first_req, int requests, int channels, int taps, cudaStream_t s) {
    if (requests <= first_req || taps <= 1) return 0;
    if (channels <= 0 || taps > 64 || first_req < 0) return MB_ERR_BAD_SIZE;
    dim3 grid((channels + 127) / 128, requests - first_req);
    if (dtype == MB_F32)
        return launch_kernel(delta_ring_kernel<float>, grid, 128, 0, s, 0, (const float*)in, in_stride, ring, positions, cu_tokens, slots, first_req,
                             channels, taps);
    if (dtype == MB_BF16)
        return launch_kernel(delta_ring_kernel<bf16>, grid, 128, 0, s, 0, (const bf16*)in, in_stride, ring, positions, cu_tokens, slots, first_req,
                             channels, taps);
    return MB_ERR_BAD_DTYPE;
}

// ---- the recurrence token by token: a block per (request, head, slice of DS_COLS value channels) --------------------------------
// Four threads share a column of the state: thread (column, part) keeps the rows part, part + 4, ... in registers, ROWS of
// them.  Tokens are taken in runs of DS_RUN: their k, q (made unit vectors here), v, decays and betas go to shared memory, then
// the run is walked without a barrier (the four partial sums of a column meet by shuffles).
#define DS_COLS 32
#define DS_THREADS (DS_COLS * 4)
#define DS_RUN 8

template <typename T, int ROWS>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(
    const T* __restrict__ qkv, const T* __restrict__ b_rows, int b_stride, const T* __restrict__ a_rows, int a_stride, int per_channel,
    const float* __restrict__ rate_log, const float* __restrict__ dt_bias, float* __restrict__ state, const int* __restrict__ cu_tokens,
    const int* __restrict__ slots, float* __restrict__ o, int first_req, int H, int G, int d, int dv) {
    PDL_ENTER_WALK();
    qkv = pdl_fresh(qkv); b_rows = pdl_fresh(b_rows); a_rows = pdl_fresh(a_rows);
    extern __shared__ float smem[];
    float* ks = smem;                          // [DS_RUN][d]
    float* qs = ks + DS_RUN * d;               // [DS_RUN][d]
    float* gs = qs + DS_RUN * d;               // [DS_RUN][d] decays
    float* vs = gs + DS_RUN * d;               // [DS_RUN][DS_COLS]
    float* betas = vs + DS_RUN * DS_COLS;      // [DS_RUN]
    const int req = first_req + blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * DS_COLS;
    const int first = cu_tokens[req], count = cu_tokens[req + 1] - first;
    if (count <= 0) return;
    const int kh = head / (H / G), channels = 2 * G * d + H * dv;
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
    const float rate = expf(rate_log[head]), q_scale = 1.0f / sqrtf((float)d);
    for (int base = 0; base < count; base += DS_RUN) {
        const int run = min(DS_RUN, count - base);
        __syncthreads();
        for (int tt = warp; tt < run; tt += DS_THREADS / 32) {     // a warp per token: unit vectors and decays
            const size_t t = (size_t)(first + base + tt);
            const T* qrow = qkv + t * channels + (size_t)kh * d;
            const T* krow = qrow + (size_t)G * d;
            float qq = 0.0f, kk = 0.0f;
            for (int n = lane; n < d; n += 32) {
                const float x = to_f32(qrow[n]), y = to_f32(krow[n]);
                qq = fmaf(x, x, qq);
                kk = fmaf(y, y, kk);
            }
            const float fq = q_scale / sqrtf(warp_sum(qq) + UNIT_EPS), fk = 1.0f / sqrtf(warp_sum(kk) + UNIT_EPS);
            float one = 0.0f;
            if (!per_channel) one = expf(-rate * softplus_f(to_f32(a_rows[t * a_stride + head]) + dt_bias[head]));
            for (int n = lane; n < d; n += 32) {
                qs[tt * d + n] = to_f32(qrow[n]) * fq;
                ks[tt * d + n] = to_f32(krow[n]) * fk;
                gs[tt * d + n] = per_channel ? expf(-rate * softplus_f(to_f32(a_rows[t * a_stride + (size_t)head * d + n]) + dt_bias[head * d + n])) : one;
            }
            const T* vrow = qkv + t * channels + (size_t)2 * G * d + (size_t)head * dv;
            vs[tt * DS_COLS + lane] = col0 + lane < dv ? to_f32(vrow[col0 + lane]) : 0.0f;
            if (lane == 0) betas[tt] = sigmoid_f(to_f32(b_rows[t * b_stride + head]));
        }
        __syncthreads();
        for (int tt = 0; tt < run; ++tt) {
            float sums[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int j = 0; j < ROWS; ++j) {
                const int n = part + 4 * j;
                if (n < d) {
                    s[j] *= gs[tt * d + n];
                    sums[j & 3] = fmaf(s[j], ks[tt * d + n], sums[j & 3]);
                }
            }
            float kv = (sums[0] + sums[1]) + (sums[2] + sums[3]);
            kv += __shfl_xor_sync(0xffffffffu, kv, 1);
            kv += __shfl_xor_sync(0xffffffffu, kv, 2);
            const float u = betas[tt] * (vs[tt * DS_COLS + col] - kv);
            sums[0] = sums[1] = sums[2] = sums[3] = 0.0f;
#pragma unroll
            for (int j = 0; j < ROWS; ++j) {
                const int n = part + 4 * j;
                if (n < d) {
                    s[j] = fmaf(ks[tt * d + n], u, s[j]);
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
static int delta_scan_rows(int rows, dim3 grid, size_t smem, cudaStream_t s, const T* qkv, const T* b_rows, int b_stride, const T* a_rows, int a_stride,
                           int per_channel, const float* rate_log, const float* dt_bias, float* state, const int* cu_tokens, const int* slots, float* o,
                           int first_req, int H, int G, int d, int dv) {
#define DS_CASE(R)                                                                                                                     \
    if (rows <= R)                                                                                                                     \
        return launch_kernel(delta_scan_kernel<T, R>, grid, DS_THREADS, smem, s, 0, qkv, b_rows, b_stride, a_rows, a_stride, per_channel, \
                             rate_log, dt_bias, state, cu_tokens, slots, o, first_req, H, G, d, dv);
    DS_CASE(4) DS_CASE(8) DS_CASE(16) DS_CASE(32) DS_CASE(64)
#undef DS_CASE
    return MB_ERR_BAD_SIZE;
}

// qkv: [tokens][2 G d + H dv] after the convolution.  b_rows / a_rows: the projections' numbers of token 0 (rows b_stride / a_stride
// apart); per_channel: a has H d of them and dt_bias [H d], else H and [H].  o: float32 [tokens][H dv].
MB_API int mb_delta_scan(const void* qkv, int dtype, const void* b_rows, int b_stride, const void* a_rows, int a_stride, int per_channel,
                         const float* rate_log, const float* dt_bias, float* state, const int* cu_tokens, const int* slots, float* o, int first_req,
                         int requests, int H, int G, int d, int dv, cudaStream_t s) {
    if (requests <= first_req) return 0;
    if (H <= 0 || G <= 0 || H % G != 0 || d <= 0 || d > 256 || dv <= 0 || first_req < 0) return MB_ERR_BAD_SIZE;
    dim3 grid(requests - first_req, H, (dv + DS_COLS - 1) / DS_COLS);
    const size_t smem = (size_t)(3 * DS_RUN * d + DS_RUN * DS_COLS + DS_RUN) * sizeof(float);
    const int rows = (d + 3) / 4;
    if (dtype == MB_F32)
        return delta_scan_rows<float>(rows, grid, smem, s, (const float*)qkv, (const float*)b_rows, b_stride, (const float*)a_rows, a_stride, per_channel,
                                      rate_log, dt_bias, state, cu_tokens, slots, o, first_req, H, G, d, dv);
    if (dtype == MB_BF16)
        return delta_scan_rows<bf16>(rows, grid, smem, s, (const bf16*)qkv, (const bf16*)b_rows, b_stride, (const bf16*)a_rows, a_stride, per_channel,
                                     rate_log, dt_bias, state, cu_tokens, slots, o, first_req, H, G, d, dv);
    return MB_ERR_BAD_DTYPE;
}

// ---- norm per head and gate: a warp per (token, head) --------------------------------------------------------------------------
// out = o / rms_head(o) * weight[vdim] * gate(g) * factor; gate 0: sigmoid, 1: silu.  g: [tokens][g_stride].
template <typename T>
__global__ void delta_norm_kernel(const float* __restrict__ o, const T* __restrict__ g, int g_stride, int gate, const float* __restrict__ w, float eps,
                                  float factor, T* __restrict__ out, int out_stride, int first_token, int pairs, int H, int dv, int vec) {
    PDL_ENTER();
    o = pdl_fresh(o); g = pdl_fresh(g);
    const int p = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (p >= pairs) return;
    const int t = first_token + p / H, head = p % H;
    const float* row = o + ((size_t)t * H + head) * dv;
    float ss = 0.0f;
    const T* gr = g + (size_t)t * g_stride + (size_t)head * dv;
    T* dst = out + (size_t)t * out_stride + (size_t)head * dv;
    if (sizeof(T) == 2 && vec) {                               // four elements a lane and turn, at most 256 of a head
        float4 v[2], z[2];
        const int turns = (dv + 127) / 128;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int i = u * 128 + lane * 4;
            v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            z[u] = v[u];
            if (u < turns && i < dv) {
                v[u] = *reinterpret_cast<const float4*>(row + i);
                const uint2 raw = *reinterpret_cast<const uint2*>(gr + i);
                const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                z[u] = make_float4(a.x, a.y, b.x, b.y);
            }
            ss += (v[u].x * v[u].x + v[u].y * v[u].y) + (v[u].z * v[u].z + v[u].w * v[u].w);
        }
        const float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int i = u * 128 + lane * 4;
            if (u >= turns || i >= dv) continue;
            const float4 ww = *reinterpret_cast<const float4*>(w + i);
            float4 s4 = make_float4(__fdividef(1.0f, 1.0f + __expf(-z[u].x)), __fdividef(1.0f, 1.0f + __expf(-z[u].y)), __fdividef(1.0f, 1.0f + __expf(-z[u].z)),
                                    __fdividef(1.0f, 1.0f + __expf(-z[u].w)));
            if (gate == 1) { s4.x *= z[u].x; s4.y *= z[u].y; s4.z *= z[u].z; s4.w *= z[u].w; }
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v[u].x * f * ww.x * s4.x, v[u].y * f * ww.y * s4.y), hi = __floats2bfloat162_rn(v[u].z * f * ww.z * s4.z, v[u].w * f * ww.w * s4.w);
            uint2 packed;
            packed.x = *reinterpret_cast<const uint32_t*>(&lo);
            packed.y = *reinterpret_cast<const uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(dst + i) = packed;
        }
        return;
    }
    for (int i = lane; i < dv; i += 32) { const float v = row[i]; ss = fmaf(v, v, ss); }
    const float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
    for (int i = lane; i < dv; i += 32) {
        const float z = to_f32(gr[i]);
        dst[i] = from_f32<T>(row[i] * f * w[i] * (gate == 0 ? sigmoid_f(z) : silu_f(z)));
    }
}

MB_API int mb_delta_norm(const float* o, const void* g, int g_stride, int gate, int dtype, const float* w, float eps, float factor, void* out,
                         int out_stride, int first_token, int tokens, int H, int dv, cudaStream_t s) {
    if (tokens <= first_token) return 0;
    if (H <= 0 || dv <= 0 || gate < 0 || gate > 1 || first_token < 0 || out_stride < H * dv) return MB_ERR_BAD_SIZE;
    const int pairs = (tokens - first_token) * H, blocks = (pairs + 7) / 8;
    const int vec = dv % 4 == 0 && dv <= 256 && g_stride % 4 == 0 && out_stride % 4 == 0 && (((uintptr_t)o | (uintptr_t)w) & 15) == 0 && (((uintptr_t)g | (uintptr_t)out) & 7) == 0;
    if (dtype == MB_F32)
        return launch_kernel(delta_norm_kernel<float>, blocks, 256, 0, s, 0, o, (const float*)g, g_stride, gate, w, eps, factor, (float*)out, out_stride,
                             first_token, pairs, H, dv, vec);
    if (dtype == MB_BF16)
        return launch_kernel(delta_norm_kernel<bf16>, blocks, 256, 0, s, 0, o, (const bf16*)g, g_stride, gate, w, eps, factor, (bf16*)out, out_stride,
                             first_token, pairs, H, dv, vec);
    return MB_ERR_BAD_DTYPE;
}

// ---- single tokens, all of it in one kernel: a block per (head, request) --------------------------------------------------------
// The state of a head is read once, all loads in flight while the convolution is worked out, and written once.  Thread (group,
// part): the four columns 4 group .. 4 group + 3 of the rows part, part + PARTS, ..., ROWS of them, in registers; the PARTS
// partial sums of a column meet in shared memory in a fixed order.  Heads that share a q and k head each work out its
// convolution; the first of them keeps the new input in the ring (its row is read by nobody in this step).
template <typename T, int ROWS, int PARTS>
__global__ void __launch_bounds__(512) delta_single_kernel(
    const T* __restrict__ in, int in_stride, const float* __restrict__ conv_w, float* ring, int taps, const T* __restrict__ b_rows, int b_stride,
    const T* __restrict__ a_rows, int a_stride, int per_channel, const float* __restrict__ rate_log, const float* __restrict__ dt_bias,
    float* __restrict__ state, const int* __restrict__ positions, const int* __restrict__ seq_lens, const int* __restrict__ slots,
    const T* __restrict__ g, int g_stride, int gate, const float* __restrict__ norm_w, float eps, float factor, T* __restrict__ out, int out_stride, int H,
    int G, int d, int dv) {
    // The state is asked for before the wait for the kernel ahead: only this kernel (and the prompt kernels) of an earlier step wrote it,
    // and every step has kernels in between that let nothing start before all work ahead of them is done (its embedding, the norms);
    // slots, positions and lengths are the step's inputs, copied before its first kernel.  All else waits.
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
    __shared__ float scratch[32], scratch2[32];
    const int head = blockIdx.x, r = blockIdx.y;
    if (seq_lens[r] <= 0) return;              // a row that pads a captured batch
    const int groups = dv >> 2, threads = blockDim.x;
    const int slot = slots[r], pos = positions[r];
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
    in = pdl_fresh(in); b_rows = pdl_fresh(b_rows); a_rows = pdl_fresh(a_rows); g = pdl_fresh(g); ring = pdl_fresh(ring);
    const float rate_raw = rate_log[head], beta_raw = to_f32(b_rows[(size_t)r * b_stride + head]);
    float decay_raw = 0.0f, decay_bias = 0.0f, gate_raw = 0.0f, norm_raw = 0.0f;         // asked for early, used late
    if (threadIdx.x < d) {
        const int at = per_channel ? head * d + threadIdx.x : head;
        decay_raw = to_f32(a_rows[(size_t)r * a_stride + at]);
        decay_bias = dt_bias[at];
    }
    if (threadIdx.x < dv) {
        gate_raw = to_f32(g[(size_t)r * g_stride + (size_t)head * dv + threadIdx.x]);
        norm_raw = norm_w[threadIdx.x];
    }
    // the convolution of this head's q, k and v channels
    const int share = H / G, kh = head / share, channels = 2 * G * d + H * dv;
    float* kept = ring + (size_t)slot * taps * channels;
    const T* row = in + (size_t)r * in_stride;
    const int pos_row = pos % taps;
    float qq = 0.0f, kk = 0.0f;
    for (int i = threadIdx.x; i < 2 * d + dv; i += threads) {
        const int c = i < d ? kh * d + i : i < 2 * d ? G * d + kh * d + (i - d) : 2 * G * d + head * dv + (i - 2 * d);
        const float now = to_f32(row[c]);
        float sum = 0.0f;
        const int most = min(taps - 1, pos);
        if (taps <= 4) {                       // all loads in flight at once
            float x[3], y[3];
#pragma unroll
            for (int back = 3; back > 0; --back) {
                x[back - 1] = y[back - 1] = 0.0f;
                if (back <= most) {
                    int at = pos_row - back;
                    at = at < 0 ? at + taps : at;
                    x[back - 1] = kept[(size_t)at * channels + c];
                    y[back - 1] = conv_w[(size_t)(taps - 1 - back) * channels + c];
                }
            }
#pragma unroll
            for (int back = 3; back > 0; --back) sum = fmaf(y[back - 1], x[back - 1], sum);
        } else {
            for (int back = most; back > 0; --back)
                sum = fmaf(conv_w[(size_t)(taps - 1 - back) * channels + c], kept[(size_t)((pos - back) % taps) * channels + c], sum);
        }
        sum = silu_f(fmaf(conv_w[(size_t)(taps - 1) * channels + c], now, sum));
        if (taps > 1 && (i >= 2 * d || head == kh * share)) kept[(size_t)pos_row * channels + c] = now;
        sum = to_f32(from_f32<T>(sum));        // as the convolution of many tokens leaves it
        if (i < d) { qs[i] = sum; qq = fmaf(sum, sum, qq); }
        else if (i < 2 * d) { ks[i - d] = sum; kk = fmaf(sum, sum, kk); }
        else vs[i - 2 * d] = sum;
    }
    const float rate = expf(rate_raw);
    for (int i = threadIdx.x; i < d; i += threads) {
        if (i >= threads) {
            const int at = per_channel ? head * d + i : head;
            decay_raw = to_f32(a_rows[(size_t)r * a_stride + at]);
            decay_bias = dt_bias[at];
        }
        gs[i] = expf(-rate * softplus_f(decay_raw + decay_bias));
    }
    const float beta = sigmoid_f(beta_raw);
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    if ((threadIdx.x & 31) == 0) { scratch[threadIdx.x >> 5] = qq; scratch2[threadIdx.x >> 5] = kk; }
    __syncthreads();                           // (publishes qs, ks, gs and vs too)
    {
        const int lane = threadIdx.x & 31, warps = (threads + 31) >> 5;
        qq = warp_sum(lane < warps ? scratch[lane] : 0.0f);
        kk = warp_sum(lane < warps ? scratch2[lane] : 0.0f);
    }
    const float fq = 1.0f / (sqrtf((float)d) * sqrtf(qq + UNIT_EPS)), fk = 1.0f / sqrtf(kk + UNIT_EPS);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = part + PARTS * j;
        if (owner && n < d) {
            const float gn = gs[n], kn = ks[n] * fk;
            s[j].x *= gn; s[j].y *= gn; s[j].z *= gn; s[j].w *= gn;
            acc.x = fmaf(s[j].x, kn, acc.x); acc.y = fmaf(s[j].y, kn, acc.y); acc.z = fmaf(s[j].z, kn, acc.z); acc.w = fmaf(s[j].w, kn, acc.w);
        }
    }
    if (owner) *reinterpret_cast<float4*>(sums + part * dv + 4 * grp) = acc;
    __syncthreads();
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (owner) {
#pragma unroll
        for (int p = 0; p < PARTS; ++p) {
            const float4 a = *reinterpret_cast<const float4*>(sums + p * dv + 4 * grp);
            u.x += a.x; u.y += a.y; u.z += a.z; u.w += a.w;
        }
        const float4 v = *reinterpret_cast<const float4*>(vs + 4 * grp);
        u.x = beta * (v.x - u.x); u.y = beta * (v.y - u.y); u.z = beta * (v.z - u.z); u.w = beta * (v.w - u.w);
    }
    __syncthreads();                           // everyone has read the sums
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = part + PARTS * j;
        if (owner && n < d) {
            const float kn = ks[n] * fk, qn = qs[n] * fq;
            s[j].x = fmaf(kn, u.x, s[j].x); s[j].y = fmaf(kn, u.y, s[j].y); s[j].z = fmaf(kn, u.z, s[j].z); s[j].w = fmaf(kn, u.w, s[j].w);
            acc.x = fmaf(s[j].x, qn, acc.x); acc.y = fmaf(s[j].y, qn, acc.y); acc.z = fmaf(s[j].z, qn, acc.z); acc.w = fmaf(s[j].w, qn, acc.w);
            S[(size_t)n * groups] = s[j];
        }
    }
    if (owner) *reinterpret_cast<float4*>(sums + part * dv + 4 * grp) = acc;
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
        const float z = i < threads ? gate_raw : to_f32(g[(size_t)r * g_stride + (size_t)head * dv + i]);
        const float wn = i < threads ? norm_raw : norm_w[i];
        out[(size_t)r * out_stride + (size_t)head * dv + i] = from_f32<T>(vs[i] * f * wn * (gate == 0 ? sigmoid_f(z) : silu_f(z)));
    }
}

// Whether the one kernel takes these sizes: a head's state in the registers of one block.
MB_API int mb_delta_single_supported(int d, int dv) {
    return d >= 1 && d <= 256 && dv >= 4 && dv <= 256 && dv % 4 == 0 && (dv / 4) * (d > 128 ? 16 : 8) <= 512;
}

template <typename T>
static int delta_single_launch(dim3 grid, cudaStream_t s, const T* in, int in_stride, const float* conv_w, float* ring, int taps, const T* b_rows,
                               int b_stride, const T* a_rows, int a_stride, int per_channel, const float* rate_log, const float* dt_bias, float* state,
                               const int* positions, const int* seq_lens, const int* slots, const T* g, int g_stride, int gate, const float* norm_w,
                               float eps, float factor, T* out, int out_stride, int H, int G, int d, int dv) {
    const int parts = d > 128 ? 16 : 8, rows = (d + parts - 1) / parts;
    const int threads = ((dv / 4) * parts + 31) / 32 * 32;
    const size_t smem = (size_t)(3 * ((d + 3) / 4 * 4) + dv + parts * dv) * sizeof(float);
#define D1_CASE(R, P)                                                                                                                       \
    if (parts == P && rows <= R)                                                                                                            \
        return launch_kernel(delta_single_kernel<T, R, P>, grid, threads, smem, s, 0, in, in_stride, conv_w, ring, taps, b_rows, b_stride, a_rows, \
                             a_stride, per_channel, rate_log, dt_bias, state, positions, seq_lens, slots, g, g_stride, gate, norm_w, eps, factor, out, \
                             out_stride, H, G, d, dv);
    D1_CASE(2, 8) D1_CASE(4, 8) D1_CASE(8, 8) D1_CASE(16, 8) D1_CASE(16, 16)
#undef D1_CASE
    return MB_ERR_BAD_SIZE;
}

// Requests 0 .. requests - 1 bring one token each (token r is request r's).  in: the projections' q | k | v before the convolution.
MB_API int mb_delta_single(const void* in, int in_stride, int dtype, const float* conv_w, float* ring, int taps, const void* b_rows, int b_stride,
                           const void* a_rows, int a_stride, int per_channel, const float* rate_log, const float* dt_bias, float* state,
                           const int* positions, const int* seq_lens, const int* slots, const void* g, int g_stride, int gate, const float* norm_w,
                           float eps, float factor, void* out, int out_stride, int requests, int H, int G, int d, int dv, cudaStream_t s) {
    if (requests <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G != 0 || taps <= 0 || taps > 64 || gate < 0 || gate > 1 || !mb_delta_single_supported(d, dv) || out_stride < H * dv)
        return MB_ERR_BAD_SIZE;
    dim3 grid(H, requests);
    if (dtype == MB_F32)
        return delta_single_launch<float>(grid, s, (const float*)in, in_stride, conv_w, ring, taps, (const float*)b_rows, b_stride, (const float*)a_rows,
                                          a_stride, per_channel, rate_log, dt_bias, state, positions, seq_lens, slots, (const float*)g, g_stride, gate, norm_w,
                                          eps, factor, (float*)out, out_stride, H, G, d, dv);
    if (dtype == MB_BF16)
        return delta_single_launch<bf16>(grid, s, (const bf16*)in, in_stride, conv_w, ring, taps, (const bf16*)b_rows, b_stride, (const bf16*)a_rows, a_stride,
                                         per_channel, rate_log, dt_bias, state, positions, seq_lens, slots, (const bf16*)g, g_stride, gate, norm_w, eps,
                                         factor, (bf16*)out, out_stride, H, G, d, dv);
    return MB_ERR_BAD_DTYPE;
}
