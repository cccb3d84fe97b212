// Causal grouped-query softmax attention over the paged cache with the options several designs combine:
//   * keys of `d` elements, values of `dv` (they may differ): K pages [page][kv_head][offset][d], V pages [..][dv];
//   * which keys a position sees: all before it, the last `window`, or those of its own chunk of `chunk` positions
//     (chunks counted from position 0 of the sequence, wherever a prompt was cut);
//   * the sequence's first `keep` positions, visible however far behind the window or chunk they lie;
//   * scores capped: s <- cap tanh(s / cap), the sink's score is not;
//   * a sink: one more term in the softmax's denominator, a key without a value whose score is 0 or a learned number per
//     query head (not scaled),  p_j = exp(s_j) / (exp(sink_h) + sum_j exp(s_j));
//   * values that are the leading `dv` elements of the key rows (a latent shared by keys and values): the value pointer is
//     the key pointer and `v_stride`, the distance between two positions' values, is the key rows' width;
//   * an output gate: the result is multiplied element by element with sigmoid(g), g a column block of the fused
//     projection; and a plain factor `out_scale`;
//   * several maps per head over the same values (differential attention: Ye, Dong, Xia, Sun, Zhu, Huang, Wei, "Differential
//     Transformer"): the keys of a kv head's maps lie side by side in one key row, a map's query is zero outside its own part of that
//     row, so that to the attention kernels the maps are query heads like any others that share a kv head; their results are
//     combined, o = a_1 - lambda a_2, o / rms(o) * factor (pair_combine_kernel, or the ends of the tensor-core kernels).
// This file holds the head preparation (biases, a short causal convolution per channel over the projection's rows, RMS norm of q
// and k per head or over the whole projection, partial rotation with scaled sines and cosines, value mixing with the values an
// earlier layer left for the same tokens, cache write) and the plain attention kernel that serves any size in both dtypes.  Sums,
// norms, angles, scores and weights are float32.
#define MB_LIB "attention_sink"
#define MB_LIB_ID 13
#include "common.cuh"
#include "launch.cuh"

#define QF_THREADS 256            // at least; 1024 where a token's q and k have 4,096 elements and more

// A causal convolution over the rows of the projection, one per channel (q, k and v columns), before norm and rotation: with
// u = projection + bias, y_t = sum_j w[j] u_(t - taps + 1 + j), zeros before the sequence's start.  A request keeps its latest u as a
// ring of `taps` rows (float32 [slot][taps][channels], position p in row p mod taps).  The step's tokens below `singles` are the only ones
// of their requests: they replace their ring row here (nobody in the step reads it); the rows of longer portions are kept by
// conv_ring_kernel behind this one.
struct ConvRows {
    const float* w;               // [taps][channels], the last row on the current token; nullptr: no convolution
    float* ring;
    const int* slots;
    const int* req_index;
    const int* cu_tokens;
    int taps, channels, singles;
};

// Channel c of token t (its projection's row `row`, position pos): bias and convolution.  first: the request's first token of the step.
template <typename T>
__device__ __forceinline__ float conv_channel(const ConvRows& cv, const T* row, int row_stride, int t, int c, float bias, int first, int pos, float* kept) {
    const float now = to_f32(row[c]) + bias;
    if (cv.w == nullptr) return now;
    float sum = 0.0f;
    for (int back = min(cv.taps - 1, pos); back > 0; --back) {
        const float u = t - back >= first ? to_f32(row[c - (ptrdiff_t)back * row_stride]) + bias : kept[(size_t)((pos - back) % cv.taps) * cv.channels + c];
        sum = fmaf(cv.w[(size_t)(cv.taps - 1 - back) * cv.channels + c], u, sum);
    }
    if (t < cv.singles && cv.taps > 1) kept[(size_t)(pos % cv.taps) * cv.channels + c] = now;
    return fmaf(cv.w[(size_t)(cv.taps - 1) * cv.channels + c], now, sum);
}

// The rings after the step, requests first_req .. : what their last taps - 1 tokens (or as many as they brought) left in front of the convolution.
template <typename T>
__global__ void conv_ring_kernel(const T* __restrict__ row, int row_stride, const float* __restrict__ q_b, const float* __restrict__ k_b,
                                 const float* __restrict__ v_b, ConvRows cv, const int* __restrict__ positions, int first_req, int q_cols, int k_cols) {
    PDL_ENTER();
    row = pdl_fresh(row);
    const int c = blockIdx.x * blockDim.x + threadIdx.x, req = first_req + blockIdx.y;
    if (c >= cv.channels) return;
    const float* b = c < q_cols ? q_b : c < q_cols + k_cols ? k_b : v_b;
    const float bias = b != nullptr ? b[c < q_cols ? c : c < q_cols + k_cols ? c - q_cols : c - q_cols - k_cols] : 0.0f;
    const int end = cv.cu_tokens[req + 1], first = max(cv.cu_tokens[req], end - (cv.taps - 1));
    float* kept = cv.ring + (size_t)cv.slots[req] * cv.taps * cv.channels;
    for (int t = first; t < end; ++t) kept[(size_t)(positions[t] % cv.taps) * cv.channels + c] = to_f32(row[(size_t)t * row_stride + c]) + bias;
}

// ---- heads of the fused q|k|v(|g) projection, a token per block ---------------------------------------------------------
// A row of `row` holds q (H heads of d), k (K heads of d), v (K heads of dv), then whatever follows (the gate's columns).
// norm_mode 0: none; 1: per head over d, weight [d] shared by the heads; 2: over all of q (and all of k) at once, before
// the split into heads, weight [H d] (and [K d]).  The first rot_dim elements of a head are rotated in pairs
// (i, i + rot_dim/2), or (2i, 2i + 1) if `interleaved`, by the angle pos * inv_freq[i]; sines and cosines are multiplied by
// rot_mag.
// v_mode 0: values as they are; 1: they are also left in v_shared (activation dtype [tokens][K dv]) for later layers;
// 2: v <- (1 - lam) v + lam v_shared, lam = *v_lambda, and the mixed values go to the cache.
// maps > 1: H and K count maps (heads times maps, a head's maps side by side), there are K / maps value heads; key map m of a kv
// head goes to elements m d .. of its row of maps * d, a query map likewise, with zeros around it.
template <typename T>
__global__ void __launch_bounds__(1024) qkv_finish_kernel(
    const T* __restrict__ row, int row_stride, T* __restrict__ q_out, const float* __restrict__ q_b, const float* __restrict__ k_b,
    const float* __restrict__ v_b, int norm_mode, const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
    const int* __restrict__ positions, const float* __restrict__ inv_freq, int rot_dim, float rot_mag,
    const int* __restrict__ slot_mapping, T* __restrict__ k_cache, T* __restrict__ v_cache, int v_mode, T* __restrict__ v_shared,
    const float* __restrict__ v_lambda, int H, int K, int d, int dv, int page_size, int write_kv, int interleaved, int maps, ConvRows cv) {
    PDL_ENTER();
    row = pdl_fresh(row); v_shared = pdl_fresh(v_shared); cv.ring = pdl_fresh(cv.ring);
    extern __shared__ float smem[];
    const int heads = write_kv ? H + K : H;
    const int half = rot_dim >> 1;
    float* vals = smem;                        // [heads * d]: q then k, float32
    float* cs_tab = vals + (size_t)heads * d;  // [half] cosines, [half] sines
    float* head_ss = cs_tab + 2 * half;        // [heads]
    __shared__ float s_factor[2];
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x / 32, threads = blockDim.x;
    const T* src = row + (size_t)t * row_stride;
    if (inv_freq != nullptr) {
        const float pos = (float)positions[t];
        for (int i = threadIdx.x; i < half; i += threads) {
            float sn, cs;
            sincosf(pos * inv_freq[i], &sn, &cs);
            cs_tab[i] = cs * rot_mag;
            cs_tab[half + i] = sn * rot_mag;
        }
    }
    int first = 0, pos = 0;
    float* kept = nullptr;
    if (cv.w != nullptr) {
        const int req = cv.req_index[t];
        first = cv.cu_tokens[req];
        pos = positions[t];
        kept = cv.ring + (size_t)cv.slots[req] * cv.taps * cv.channels;
    }
    // every element of q and k (+ bias, through the convolution) into shared memory as float32, all threads side by side
    const int qk = heads * d, q_len = H * d;
    for (int idx = threadIdx.x; idx < qk; idx += threads) {
        float bias = 0.0f;
        if (idx < q_len) { if (q_b != nullptr) bias = q_b[idx]; }
        else if (k_b != nullptr) bias = k_b[idx - q_len];
        vals[idx] = conv_channel(cv, src, row_stride, t, idx, bias, first, pos, kept);
    }
    __syncthreads();
    // sums of squares per head: a warp per head, lanes in a fixed order
    for (int head = warp; head < heads; head += warps) {
        float ss = 0.0f;
        for (int i = lane; i < d; i += 32) { const float v = vals[head * d + i]; ss += v * v; }
        ss = warp_sum(ss);
        if (lane == 0) head_ss[head] = ss;
    }
    __syncthreads();
    if (norm_mode == 2 && threadIdx.x < 2) {
        const int first = threadIdx.x == 0 ? 0 : H, count = threadIdx.x == 0 ? H : heads - H;
        float total = 0.0f;
        for (int j = 0; j < count; ++j) total += head_ss[first + j];
        s_factor[threadIdx.x] = count > 0 ? 1.0f / sqrtf(total / (float)(count * d) + eps) : 0.0f;
    }
    __syncthreads();
    const int slot = write_kv ? slot_mapping[t] : -1;
    const int KG = K / maps, wide = d * maps;                  // kv heads, and the width of a key row
    T* k_dst = slot >= 0 ? k_cache + (((size_t)(slot / page_size)) * KG * page_size + (size_t)(slot % page_size)) * wide : nullptr;
    // a warp per head, lanes along the head: no division per element, 64-byte runs per store
    for (int head = warp; head < heads; head += warps) {
        const bool is_q = head < H;
        const int kh = head - H;
        if (!is_q && k_dst == nullptr) continue;
        float factor = 1.0f;
        const float* w = nullptr;
        if (norm_mode == 1) {
            factor = 1.0f / sqrtf(head_ss[head] / (float)d + eps);
            w = is_q ? q_w : k_w;
        } else if (norm_mode == 2) {
            factor = s_factor[is_q ? 0 : 1];
            w = is_q ? q_w + (size_t)head * d : k_w + (size_t)kh * d;
        }
        const float* hv = vals + (size_t)head * d;
        T* dst = is_q ? q_out + ((size_t)t * H + head) * wide + (head % maps) * d : k_dst + (size_t)(kh / maps) * page_size * wide + (kh % maps) * d;
        if (is_q && maps > 1) {
            T* whole = dst - (head % maps) * d;
            for (int i = lane; i < wide; i += 32)
                if (i / d != head % maps) whole[i] = from_f32<T>(0.0f);
        }
        for (int i = lane; i < d; i += 32) {
            float a = hv[i] * factor * (w != nullptr ? w[i] : 1.0f);
            if (i < rot_dim) {                                 // (rot_dim is 0 without a rotation)
                const bool low = interleaved ? (i & 1) == 0 : i < half;
                const int j = interleaved ? i >> 1 : low ? i : i - half;
                const int other = interleaved ? i ^ 1 : low ? i + half : i - half;
                const float b = hv[other] * factor * (w != nullptr ? w[other] : 1.0f);
                const float cs = cs_tab[j], sn = cs_tab[half + j];
                a = low ? a * cs - b * sn : a * cs + b * sn;
            }
            dst[i] = from_f32<T>(a);
        }
    }
    if (!write_kv) return;
    const float lam = v_mode == 2 ? *v_lambda : 0.0f;
    const int vcol0 = (H + K) * d;
    for (int kh = warp; kh < KG; kh += warps) {
        T* dst = slot >= 0 ? v_cache + ((((size_t)(slot / page_size)) * KG + kh) * page_size + (size_t)(slot % page_size)) * dv : nullptr;
        for (int e = lane; e < dv; e += 32) {
            const int i = kh * dv + e;
            float v = conv_channel(cv, src, row_stride, t, vcol0 + i, v_b != nullptr ? v_b[i] : 0.0f, first, pos, kept);
            if (v_mode == 1) v_shared[(size_t)t * KG * dv + i] = from_f32<T>(v);
            else if (v_mode == 2) v = (1.0f - lam) * v + lam * to_f32(v_shared[(size_t)t * KG * dv + i]);
            if (dst != nullptr) dst[e] = from_f32<T>(v);
        }
    }
}

// The same for bf16 rows whose sizes are multiples of 8 (heads, value heads, half the rotated width, the row's stride):
// a thread owns runs of 8 elements (one 16-byte load, one 16-byte store), keeps them in registers between the two phases
// and fetches only its rotation partners from shared memory.  Sums of squares: a thread's 8 elements in order, then the
// block's (norm over the whole projection) or a warp per head over shared memory (per-head norm): fixed orders.
// RUNS runs per thread: one or two with few tokens (every load of a token in flight at once), four with many (smaller
// blocks, several of them on an SM at different stages: a block's life is a chain of waits on memory and barriers).
__device__ __forceinline__ void unpack8(const uint4& raw, float* x) {
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h2[i]); x[2 * i] = f.x; x[2 * i + 1] = f.y; }
}
__device__ __forceinline__ uint4 pack8(const float* x) {
    uint4 out;
    __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int i = 0; i < 4; ++i) h2[i] = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
    return out;
}
__device__ __forceinline__ void load8(const float* p, float* x) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}

// conv_channel for eight neighbouring channels from c on; x comes in as projection + bias of the current token.
__device__ __forceinline__ void conv_run8(const ConvRows& cv, const bf16* row, int row_stride, int t, int c, const float* bias, int first, int pos, float* kept,
                                          float* x) {
    if (cv.w == nullptr) return;
    float sum[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) sum[e] = 0.0f;
    auto add = [&](int back) {
        float u[8], w[8];
        if (t - back >= first) {
            unpack8(*reinterpret_cast<const uint4*>(row + c - (ptrdiff_t)back * row_stride), u);
#pragma unroll
            for (int e = 0; e < 8; ++e) u[e] += bias[e];
        } else {
            load8(kept + (size_t)((pos - back) % cv.taps) * cv.channels + c, u);
        }
        load8(cv.w + (size_t)(cv.taps - 1 - back) * cv.channels + c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] = fmaf(w[e], u[e], sum[e]);
    };
    const int most = min(cv.taps - 1, pos);
    if (cv.taps <= 4) {                        // (unrolled: the loads of all rows in flight at once)
#pragma unroll
        for (int back = 3; back > 0; --back)
            if (back <= most) add(back);
    } else {
        for (int back = most; back > 0; --back) add(back);
    }
    if (t < cv.singles && cv.taps > 1) {
        float* dst = kept + (size_t)(pos % cv.taps) * cv.channels + c;
        *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
        *reinterpret_cast<float4*>(dst + 4) = make_float4(x[4], x[5], x[6], x[7]);
    }
    float w[8];
    load8(cv.w + (size_t)(cv.taps - 1) * cv.channels + c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = fmaf(w[e], x[e], sum[e]);
}

template <int RUNS>
__global__ void __launch_bounds__(RUNS <= 2 ? 1024 : 256) qkv_finish_vec_kernel(
    const bf16* __restrict__ row, int row_stride, bf16* __restrict__ q_out, const float* __restrict__ q_b, const float* __restrict__ k_b,
    const float* __restrict__ v_b, int norm_mode, const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
    const int* __restrict__ positions, const float* __restrict__ inv_freq, int rot_dim, float rot_mag,
    const int* __restrict__ slot_mapping, bf16* __restrict__ k_cache, bf16* __restrict__ v_cache, int v_mode, bf16* __restrict__ v_shared,
    const float* __restrict__ v_lambda, int H, int K, int d, int dv, int page_size, int write_kv, int interleaved, int maps, ConvRows cv) {
    PDL_ENTER();
    row = pdl_fresh(row); v_shared = pdl_fresh(v_shared); cv.ring = pdl_fresh(cv.ring);
    extern __shared__ __align__(16) float smem[];
    __shared__ float scratch[32];
    const int heads = write_kv ? H + K : H;
    const int half = rot_dim >> 1;
    float* vals = smem;                        // [heads * d]
    float* cs_tab = vals + (size_t)heads * d;  // [half] cosines, [half] sines
    float* head_ss = cs_tab + 2 * half;        // [heads]
    const int t = blockIdx.x, threads = blockDim.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = threads >> 5;
    const bf16* src = row + (size_t)t * row_stride;
    if (inv_freq != nullptr) {
        const float pos = (float)positions[t];
        for (int i = threadIdx.x; i < half; i += threads) {
            float sn, cs;
            sincosf(pos * inv_freq[i], &sn, &cs);
            cs_tab[i] = cs * rot_mag;
            cs_tab[half + i] = sn * rot_mag;
        }
    }
    int first = 0, pos = 0;
    float* kept = nullptr;
    if (cv.w != nullptr) {
        const int req = cv.req_index[t];
        first = cv.cu_tokens[req];
        pos = positions[t];
        kept = cv.ring + (size_t)cv.slots[req] * cv.taps * cv.channels;
    }
    const int runs = heads * d / 8, q_runs = H * d / 8;
    float x[RUNS][8];
    float ss_q = 0.0f, ss_k = 0.0f;
#pragma unroll
    for (int u = 0; u < RUNS; ++u) {
        const int v = threadIdx.x + u * threads;
        if (v < runs) {
            unpack8(*reinterpret_cast<const uint4*>(src + v * 8), x[u]);
            const float* bias = v < q_runs ? q_b : k_b;
            float b[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
            if (bias != nullptr) {
                load8(bias + (v < q_runs ? v : v - q_runs) * 8, b);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[u][e] += b[e];
            }
            conv_run8(cv, src, row_stride, t, v * 8, b, first, pos, kept, x[u]);
            float ss = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += x[u][e] * x[u][e];
            if (v < q_runs) ss_q += ss; else ss_k += ss;
            *reinterpret_cast<float4*>(vals + v * 8) = make_float4(x[u][0], x[u][1], x[u][2], x[u][3]);
            *reinterpret_cast<float4*>(vals + v * 8 + 4) = make_float4(x[u][4], x[u][5], x[u][6], x[u][7]);
        }
    }
    float f_q = 1.0f, f_k = 1.0f;
    if (norm_mode == 2) {
        ss_q = block_sum(ss_q, scratch);
        ss_k = block_sum(ss_k, scratch);
        f_q = 1.0f / sqrtf(ss_q / (float)(H * d) + eps);
        f_k = heads > H ? 1.0f / sqrtf(ss_k / (float)((heads - H) * d) + eps) : 0.0f;
        __syncthreads();
    } else {
        __syncthreads();
        if (norm_mode == 1) {
            for (int head = warp; head < heads; head += warps) {
                float ss = 0.0f;
                for (int i = lane; i < d; i += 32) { const float v = vals[head * d + i]; ss += v * v; }
                ss = warp_sum(ss);
                if (lane == 0) head_ss[head] = ss;
            }
            __syncthreads();
        }
    }
    const int slot = write_kv ? slot_mapping[t] : -1;
    const int KG = K / maps, wide = d * maps;                  // kv heads, and the width of a key row
    bf16* k_dst = slot >= 0 ? k_cache + (((size_t)(slot / page_size)) * KG * page_size + (size_t)(slot % page_size)) * wide : nullptr;
#pragma unroll
    for (int u = 0; u < RUNS; ++u) {
        const int v = threadIdx.x + u * threads;
        if (v >= runs) continue;
        const int head = (v * 8) / d, i0 = v * 8 - head * d;
        const bool is_q = head < H;
        const int kh = head - H;
        if (!is_q && k_dst == nullptr) continue;
        float factor = 1.0f;
        const float* w = nullptr;
        if (norm_mode == 1) {
            factor = 1.0f / sqrtf(head_ss[head] / (float)d + eps);
            w = is_q ? q_w : k_w;
        } else if (norm_mode == 2) {
            factor = is_q ? f_q : f_k;
            w = is_q ? q_w + (size_t)head * d : k_w + (size_t)kh * d;
        }
        float a[8];
        if (w != nullptr) {
            float ww[8];
            load8(w + i0, ww);
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] = x[u][e] * factor * ww[e];
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] = x[u][e] * factor;
        }
        if (i0 < rot_dim && interleaved) {                     // partners are neighbours inside the run
            const float4 c4 = *reinterpret_cast<const float4*>(cs_tab + (i0 >> 1)), s4 = *reinterpret_cast<const float4*>(cs_tab + half + (i0 >> 1));
            const float cs[4] = {c4.x, c4.y, c4.z, c4.w}, sn[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float u = a[2 * e], v = a[2 * e + 1];
                a[2 * e] = u * cs[e] - v * sn[e];
                a[2 * e + 1] = v * cs[e] + u * sn[e];
            }
        } else if (i0 < rot_dim) {
            const bool low = i0 < half;
            const int j0 = low ? i0 : i0 - half, other = low ? i0 + half : i0 - half;
            float b[8], cs[8], sn[8];
            load8(vals + head * d + other, b);
            if (w != nullptr) {
                float ww[8];
                load8(w + other, ww);
#pragma unroll
                for (int e = 0; e < 8; ++e) b[e] *= factor * ww[e];
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) b[e] *= factor;
            }
            load8(cs_tab + j0, cs);
            load8(cs_tab + half + j0, sn);
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] = low ? a[e] * cs[e] - b[e] * sn[e] : a[e] * cs[e] + b[e] * sn[e];
        }
        if (maps == 1) {
            bf16* dst = is_q ? q_out + (size_t)t * H * d + (size_t)v * 8 : k_dst + (size_t)kh * page_size * d + i0;
            *reinterpret_cast<uint4*>(dst) = pack8(a);
        } else if (is_q) {
            const int m = head % maps;
            bf16* dst = q_out + ((size_t)t * H + head) * wide + i0;
            for (int o = 0; o < maps; ++o) *reinterpret_cast<uint4*>(dst + o * d) = o == m ? pack8(a) : make_uint4(0, 0, 0, 0);
        } else {
            *reinterpret_cast<uint4*>(k_dst + (size_t)(kh / maps) * page_size * wide + (kh % maps) * d + i0) = pack8(a);
        }
    }
    if (!write_kv) return;
    const float lam = v_mode == 2 ? *v_lambda : 0.0f;
    const int vcol0 = (H + K) * d;
    for (int v = threadIdx.x; v < KG * dv / 8; v += threads) {
        float val[8];
        unpack8(*reinterpret_cast<const uint4*>(src + vcol0 + v * 8), val);
        float b[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
        if (v_b != nullptr) {
            load8(v_b + v * 8, b);
#pragma unroll
            for (int e = 0; e < 8; ++e) val[e] += b[e];
        }
        conv_run8(cv, src, row_stride, t, vcol0 + v * 8, b, first, pos, kept, val);
        bf16* shared_at = v_shared + (size_t)t * KG * dv + v * 8;
        if (v_mode == 1) {
            *reinterpret_cast<uint4*>(shared_at) = pack8(val);
        } else if (v_mode == 2) {
            float first[8];
            unpack8(*reinterpret_cast<const uint4*>(shared_at), first);
#pragma unroll
            for (int e = 0; e < 8; ++e) val[e] = (1.0f - lam) * val[e] + lam * first[e];
        }
        if (slot >= 0) {
            const int kh = (v * 8) / dv, e0 = v * 8 - kh * dv;
            *reinterpret_cast<uint4*>(v_cache + ((((size_t)(slot / page_size)) * KG + kh) * page_size + (size_t)(slot % page_size)) * dv + e0) = pack8(val);
        }
    }
}

// The same without a barrier, for bf16 heads whose runs of 8 are a power of two and lie in one warp (values of any multiple of 8; no norm over the
// whole projection, no mixed values): a thread owns one run of 8 neighbouring channels of q, k or v over a run of consecutive tokens, a
// head's sum of squares and its rotation partners come by shuffles, cosines and sines from a table made once a step (rope: [tokens][rot_dim],
// cosines then sines).  With a convolution the thread's weights and last TAPS - 1 inputs stay in registers, so that every row is read once a run.
// TAPS 0: no convolution.
#define FR_THREADS 128
#define FR_RUN 8

template <int TAPS>
__global__ void __launch_bounds__(FR_THREADS, 3) qkv_finish_runs_kernel(
    const bf16* __restrict__ row, int row_stride, bf16* __restrict__ q_out, const float* __restrict__ q_b, const float* __restrict__ k_b,
    const float* __restrict__ v_b, int norm, const float* __restrict__ q_w, const float* __restrict__ k_w, float eps, const int* __restrict__ positions,
    const float* __restrict__ rope, int rot_dim, const int* __restrict__ slot_mapping, bf16* __restrict__ k_cache, bf16* __restrict__ v_cache, int H, int K,
    int d, int dv, int page_size, int write_kv, int interleaved, int maps, ConvRows cv, int tokens, int run) {
    PDL_ENTER();
    row = pdl_fresh(row); rope = pdl_fresh(rope); cv.ring = pdl_fresh(cv.ring);
    constexpr int RING = TAPS > 0 ? TAPS : 1;
    const int KG = K / maps, wide = d * maps, half = rot_dim >> 1;
    const int q_cols = H * d, k_end = q_cols + (write_kv ? K * d : 0), cols = k_end + (write_kv ? KG * dv : 0);
    const int c = (blockIdx.y * FR_THREADS + threadIdx.x) * 8, lane = threadIdx.x & 31;
    const bool active = c < cols;
    const bool is_q = c < q_cols, is_v = c >= k_end;
    const int rel = is_q ? c : is_v ? c - k_end : c - q_cols;
    const int width = is_v ? dv : d, head = rel / width, i0 = rel - head * width;
    const int t0 = blockIdx.x * run, t1 = min(tokens, t0 + run);
    const bool rotated = !is_v && i0 < rot_dim, low = i0 < half;
    const int partner = rotated && !interleaved ? lane + (low ? half / 8 : -half / 8) : lane;
    const int j0 = interleaved ? i0 >> 1 : low ? i0 : i0 - half;      // the first of this run's angles
    float bias[8], w[8];
    {
        const float* b = is_q ? q_b : is_v ? v_b : k_b;
        const float* ww = is_q ? q_w : k_w;
#pragma unroll
        for (int e = 0; e < 8; ++e) { bias[e] = 0.0f; w[e] = 1.0f; }
        if (active && b != nullptr) load8(b + rel, bias);
        if (active && norm && !is_v) load8(ww + i0, w);
    }
    float wt[TAPS > 0 ? TAPS : 1][8], past[TAPS > 1 ? TAPS - 1 : 1][8];      // past[b]: the input b + 1 tokens back
    if (TAPS > 0 && active)
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load8(cv.w + (size_t)j * cv.channels + c, wt[j]);
    uint4 raw[FR_RUN];                                         // every row of the run in flight at once
#pragma unroll
    for (int u = 0; u < FR_RUN; ++u) {
        raw[u] = make_uint4(0, 0, 0, 0);
        if (active && t0 + u < t1) raw[u] = *reinterpret_cast<const uint4*>(row + (size_t)(t0 + u) * row_stride + c);
    }
    int first = 0, end = 0;
    float* kept = nullptr;
#pragma unroll
    for (int u = 0; u < FR_RUN; ++u) {
        const int t = t0 + u;
        if (t >= t1) break;                                    // (the same for the whole block)
        float x[8];
        unpack8(raw[u], x);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] += bias[e];
        if (TAPS > 0) {
            if (u == 0 || t == end) {                          // another request: its window, from this step's rows, the ring, or nothing
                const int req = cv.req_index[t], pos = positions[t];
                first = cv.cu_tokens[req];
                end = cv.cu_tokens[req + 1];
                kept = cv.ring + (size_t)cv.slots[req] * TAPS * cv.channels + c;
                if (TAPS > 1 && active)
#pragma unroll
                    for (int b = 0; b < TAPS - 1; ++b) {
                        if (t - b - 1 >= first) {
                            unpack8(*reinterpret_cast<const uint4*>(row + (size_t)(t - b - 1) * row_stride + c), past[b]);
#pragma unroll
                            for (int e = 0; e < 8; ++e) past[b][e] += bias[e];
                        } else if (pos - b - 1 >= 0) {
                            load8(kept + (size_t)((pos - b - 1) % RING) * cv.channels, past[b]);
                        } else {
#pragma unroll
                            for (int e = 0; e < 8; ++e) past[b][e] = 0.0f;
                        }
                    }
            }
            if (TAPS > 1 && active && t < cv.singles) {
                float* dst = kept + (size_t)(positions[t] % RING) * cv.channels;
                *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
                *reinterpret_cast<float4*>(dst + 4) = make_float4(x[4], x[5], x[6], x[7]);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                float sum = 0.0f;                              // (the oldest first, as the other kernels add)
#pragma unroll
                for (int b = TAPS - 2; b >= 0; --b) sum = fmaf(wt[TAPS - 2 - b][e], past[b][e], sum);
                const float now = x[e];
                x[e] = fmaf(wt[TAPS > 0 ? TAPS - 1 : 0][e], now, sum);
#pragma unroll
                for (int b = TAPS - 2; b > 0; --b) past[b][e] = past[b - 1][e];
                if (TAPS > 1) past[0][e] = now;
            }
        }
        if (norm) {
            float ss = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
            for (int o = 1; o < d / 8; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);       // (a head's lanes; values do not use theirs)
            if (!is_v) {
                const float factor = 1.0f / sqrtf(ss / (float)d + eps);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = x[e] * factor * w[e];
            }
        }
        if (rot_dim > 0) {
            const float* cs_row = rope + (size_t)t * rot_dim + j0;
            if (interleaved) {
                if (rotated) {
                    const float4 c4 = *reinterpret_cast<const float4*>(cs_row), s4 = *reinterpret_cast<const float4*>(cs_row + half);
                    const float cs[4] = {c4.x, c4.y, c4.z, c4.w}, sn[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float a = x[2 * e], b = x[2 * e + 1];
                        x[2 * e] = a * cs[e] - b * sn[e];
                        x[2 * e + 1] = b * cs[e] + a * sn[e];
                    }
                }
            } else {
                float b[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) b[e] = __shfl_sync(0xffffffffu, x[e], partner);
                if (rotated) {
                    float cs[8], sn[8];
                    load8(cs_row, cs);
                    load8(cs_row + half, sn);
#pragma unroll
                    for (int e = 0; e < 8; ++e) x[e] = low ? x[e] * cs[e] - b[e] * sn[e] : x[e] * cs[e] + b[e] * sn[e];
                }
            }
        }
        if (!active) continue;
        if (is_q) {
            const int m = head % maps;
            bf16* dst = q_out + ((size_t)t * H + head) * wide + i0;
            for (int o = 0; o < maps; ++o) *reinterpret_cast<uint4*>(dst + o * d) = o == m ? pack8(x) : make_uint4(0, 0, 0, 0);
        } else {
            const int slot = slot_mapping[t];
            if (slot < 0) continue;
            const size_t page = (size_t)(slot / page_size), at = (size_t)(slot % page_size);
            if (is_v) *reinterpret_cast<uint4*>(v_cache + ((page * KG + head) * page_size + at) * dv + i0) = pack8(x);
            else *reinterpret_cast<uint4*>(k_cache + ((page * KG + head / maps) * page_size + at) * wide + (head % maps) * d + i0) = pack8(x);
        }
    }
}

static bool aligned16(const void* p) { return (((uintptr_t)p) & 15) == 0; }

// rope: null, or what qkv_finish_runs_kernel takes (rot_mag is then 1).
MB_API int mb_qkv_finish(const void* row, int row_stride, int dtype, void* q_out, const float* q_b, const float* k_b, const float* v_b,
                         int norm_mode, const float* q_w, const float* k_w, float eps, const int* positions, const float* inv_freq,
                         int rot_dim, float rot_mag, const int* slot_mapping, void* k_cache, void* v_cache, int v_mode, void* v_shared,
                         const float* v_lambda, int tokens, int H, int K, int d, int dv, int page_size, int write_kv, int interleaved,
                         int maps, const float* conv_w, float* ring, const int* slots, const int* req_index, const int* cu_tokens, int taps, int singles,
                         const float* rope, cudaStream_t s) {
    if (tokens <= 0) return 0;
    if (maps < 1 || H % maps != 0 || K % maps != 0) return MB_ERR_BAD_SIZE;
    if (conv_w != nullptr && (taps < 1 || taps > 64 || !write_kv)) return MB_ERR_BAD_SIZE;
    const ConvRows cv = {conv_w, ring, slots, req_index, cu_tokens, taps, (H + K) * d + K / maps * dv, singles};
    if (d <= 0 || dv <= 0 || H <= 0 || K <= 0 || rot_dim > d || (rot_dim & 1) || norm_mode < 0 || norm_mode > 2) return MB_ERR_BAD_SIZE;
    if ((v_mode == 1 || v_mode == 2) && v_shared == nullptr) return MB_ERR_BAD_SIZE;
    if (v_mode == 2 && v_lambda == nullptr) return MB_ERR_BAD_SIZE;
    if (inv_freq == nullptr) rot_dim = 0;
    const int lanes = d / 8;                                   // of a head: a power of two within a warp
    if (dtype == MB_BF16 && (rope != nullptr || rot_dim == 0) && norm_mode != 2 && v_mode == 0 && d % 8 == 0 && dv % 8 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 &&
        (interleaved ? rot_dim % 8 == 0 : rot_dim % 16 == 0) && row_stride % 8 == 0 && (conv_w == nullptr || taps <= 4) && aligned16(row) && aligned16(q_out) &&
        aligned16(q_b) && aligned16(k_b) && aligned16(v_b) && aligned16(q_w) && aligned16(k_w) && aligned16(k_cache) && aligned16(v_cache) && aligned16(conv_w) &&
        aligned16(ring) && aligned16(rope)) {
        const int cols = H * d + (write_kv ? K * d + K / maps * dv : 0);
        const int run = tokens >= 256 ? FR_RUN : tokens >= 64 ? 2 : 1;
        dim3 grid((tokens + run - 1) / run, (cols / 8 + FR_THREADS - 1) / FR_THREADS);
#define FR_CASE(TAPS)                                                                                                                                \
    if ((conv_w == nullptr ? 0 : taps) == TAPS)                                                                                                      \
        return launch_kernel(qkv_finish_runs_kernel<TAPS>, grid, FR_THREADS, 0, s, 0, (const bf16*)row, row_stride, (bf16*)q_out, q_b, k_b, v_b, norm_mode, q_w, \
                             k_w, eps, positions, rope, rot_dim, slot_mapping, (bf16*)k_cache, (bf16*)v_cache, H, K, d, dv, page_size, write_kv,      \
                             interleaved, maps, cv, tokens, run);
        FR_CASE(0) FR_CASE(1) FR_CASE(2) FR_CASE(3) FR_CASE(4)
#undef FR_CASE
    }
    const size_t smem = ((size_t)(H + K) * d + rot_dim + H + K) * sizeof(float);
    if (smem > 160 * 1024) return MB_ERR_BAD_SIZE;
    const int runs8 = (H + K) * d / 8;
    if (dtype == MB_BF16 && d % 8 == 0 && dv % 8 == 0 && (interleaved ? rot_dim % 8 == 0 : (rot_dim / 2) % 8 == 0) && row_stride % 8 == 0 && runs8 <= 1024 * 2 &&
        aligned16(row) && aligned16(q_out) && aligned16(q_b) && aligned16(k_b) && aligned16(v_b) && aligned16(q_w) && aligned16(k_w) &&
        aligned16(k_cache) && aligned16(v_cache) && aligned16(v_shared) && aligned16(conv_w) && aligned16(ring)) {
#define QV_LAUNCH(RUNS, threads)                                                                                                        \
    do {                                                                                                                                \
        if (smem > 48 * 1024) {                                                                                                         \
            const int rc = (int)cudaFuncSetAttribute(qkv_finish_vec_kernel<RUNS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (rc != 0) return rc;                                                                                                     \
        }                                                                                                                               \
        return launch_kernel(qkv_finish_vec_kernel<RUNS>, tokens, threads, smem, s, 0, (const bf16*)row, row_stride, (bf16*)q_out, q_b, k_b, \
                             v_b, norm_mode, q_w, k_w, eps, positions, inv_freq, rot_dim, rot_mag, slot_mapping, (bf16*)k_cache,         \
                             (bf16*)v_cache, v_mode, (bf16*)v_shared, v_lambda, H, K, d, dv, page_size, write_kv, interleaved, maps, cv);          \
    } while (0)
        const int quarter = (((runs8 + 3) / 4 + 31) / 32) * 32;
        if (tokens >= 512 && quarter <= 256) QV_LAUNCH(4, quarter < 64 ? 64 : quarter);
        const int whole = ((runs8 + 31) / 32) * 32;
        if (whole <= 1024) QV_LAUNCH(1, whole < 128 ? 128 : whole);
        QV_LAUNCH(2, (((runs8 + 1) / 2 + 31) / 32) * 32);
#undef QV_LAUNCH
    }
#define QF_LAUNCH(TT)                                                                                                                \
    do {                                                                                                                             \
        if (smem > 48 * 1024) {                                                                                                      \
            const int rc = (int)cudaFuncSetAttribute(qkv_finish_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (rc != 0) return rc;                                                                                                  \
        }                                                                                                                            \
        return launch_kernel(qkv_finish_kernel<TT>, tokens, (H + K) * d < 4096 ? QF_THREADS : tokens <= 64 ? 1024 : 512, smem, s, 0, (const TT*)row, row_stride, (TT*)q_out, q_b, k_b, \
                             v_b, norm_mode, q_w, k_w, eps, positions, inv_freq, rot_dim, rot_mag, slot_mapping, (TT*)k_cache,      \
                             (TT*)v_cache, v_mode, (TT*)v_shared, v_lambda, H, K, d, dv, page_size, write_kv, interleaved, maps, cv);          \
    } while (0)
    if (dtype == MB_F32) QF_LAUNCH(float);
    if (dtype == MB_BF16) QF_LAUNCH(bf16);
#undef QF_LAUNCH
    return MB_ERR_BAD_DTYPE;
}

MB_API int mb_conv_ring(const void* row, int row_stride, int dtype, const float* q_b, const float* k_b, const float* v_b, float* ring, const int* slots,
                        const int* cu_tokens, const int* positions, int taps, int first_req, int requests, int q_cols, int k_cols, int v_cols, cudaStream_t s) {
    if (requests <= first_req || taps <= 1) return 0;
    if (taps > 64 || first_req < 0) return MB_ERR_BAD_SIZE;
    const int channels = q_cols + k_cols + v_cols;
    const ConvRows cv = {nullptr, ring, slots, nullptr, cu_tokens, taps, channels, 0};
    dim3 grid((channels + 127) / 128, requests - first_req);
    if (dtype == MB_F32)
        return launch_kernel(conv_ring_kernel<float>, grid, 128, 0, s, 0, (const float*)row, row_stride, q_b, k_b, v_b, cv, positions, first_req, q_cols, k_cols);
    if (dtype == MB_BF16)
        return launch_kernel(conv_ring_kernel<bf16>, grid, 128, 0, s, 0, (const bf16*)row, row_stride, q_b, k_b, v_b, cv, positions, first_req, q_cols, k_cols);
    return MB_ERR_BAD_DTYPE;
}

// ---- two maps of a head combined: out = n / rms(n) * factor, n = a_1 - lam a_2, a warp per (token, head) -----------------
// a: float32 [tokens][2 H][dv], a head's maps side by side.
template <typename T>
__global__ void pair_combine_kernel(const float* __restrict__ a, T* __restrict__ out, int out_stride, float lam, float eps, float factor, int first_token,
                                    int pairs, int H, int dv) {
    PDL_ENTER();
    a = pdl_fresh(a);
    const int p = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (p >= pairs) return;
    const int t = first_token + p / H, head = p % H;
    const float* a1 = a + ((size_t)t * H + head) * 2 * dv;
    const float* a2 = a1 + dv;
    float ss = 0.0f;
    for (int i = lane; i < dv; i += 32) { const float v = a1[i] - lam * a2[i]; ss = fmaf(v, v, ss); }
    const float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
    T* dst = out + (size_t)t * out_stride + (size_t)head * dv;
    for (int i = lane; i < dv; i += 32) dst[i] = from_f32<T>((a1[i] - lam * a2[i]) * f);
}

MB_API int mb_pair_combine(const float* a, void* out, int out_stride, int dtype, float lam, float eps, float factor, int first_token, int tokens, int H, int dv,
                           cudaStream_t s) {
    if (tokens <= first_token) return 0;
    if (H <= 0 || dv <= 0 || first_token < 0 || out_stride < H * dv) return MB_ERR_BAD_SIZE;
    const int pairs = (tokens - first_token) * H, blocks = (pairs + 7) / 8;
    if (dtype == MB_F32) return launch_kernel(pair_combine_kernel<float>, blocks, 256, 0, s, 0, a, (float*)out, out_stride, lam, eps, factor, first_token, pairs, H, dv);
    if (dtype == MB_BF16) return launch_kernel(pair_combine_kernel<bf16>, blocks, 256, 0, s, 0, a, (bf16*)out, out_stride, lam, eps, factor, first_token, pairs, H, dv);
    return MB_ERR_BAD_DTYPE;
}

// ---- the plain kernel: one block per (token, query head), keys in blocks of 128 in increasing order ----------------------
#define SK_THREADS 128
#define SK_MAX_PER_THREAD 4

template <typename T>
__global__ void __launch_bounds__(SK_THREADS) attention_sink_kernel(
    const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ out,
    const int* __restrict__ block_table, int max_pages, const int* __restrict__ req_index, const int* __restrict__ positions,
    int H, int K, int d, int dv, int page_size, float scale, int window, int chunk, int sink, const float* __restrict__ sink_logit,
    int v_stride, const T* __restrict__ gate, int gate_stride, int keep, float softcap, float out_scale, int out_stride, float* __restrict__ wide_out) {
    PDL_ENTER();
    q = pdl_fresh(q); k_cache = pdl_fresh(k_cache); v_cache = pdl_fresh(v_cache); gate = pdl_fresh(gate);
    extern __shared__ float smem[];
    float* qs = smem;                 // [d]
    float* ps = smem + d;             // [SK_THREADS]
    float* scratch = ps + SK_THREADS; // [32]
    const int t = blockIdx.x, head = blockIdx.y;
    const int kh = head / (H / K);
    const int req = req_index[t];
    const int pos = positions[t];
    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, (pos / chunk) * chunk);
    // the keys in order: the kept ones before lo, then lo .. pos; key number j is j or lo + j - kept
    const int kept = min(keep, lo), keys = kept + pos - lo + 1;
    const int* table = block_table + (size_t)req * max_pages;
    const T* qrow = q + ((size_t)t * H + head) * d;
    for (int i = threadIdx.x; i < d; i += SK_THREADS) qs[i] = to_f32(qrow[i]);
    __syncthreads();

    // the sink is a key whose value is zero: the running maximum starts at its score (0 or the head's learned number) and
    // the sum at 1
    float m = sink ? (sink_logit != nullptr ? sink_logit[head] : 0.0f) : -INFINITY, l = sink ? 1.0f : 0.0f;
    float acc[SK_MAX_PER_THREAD];
#pragma unroll
    for (int r = 0; r < SK_MAX_PER_THREAD; ++r) acc[r] = 0.0f;

    for (int base = 0; base < keys; base += SK_THREADS) {
        const int at = base + threadIdx.x;
        float s = -INFINITY;
        if (at < keys) {
            const int key = at < kept ? at : lo + at - kept;
            const size_t page = (size_t)table[key / page_size];
            const T* krow = k_cache + ((page * K + kh) * page_size + (size_t)(key % page_size)) * d;
            float dot = 0.0f;
            for (int i = 0; i < d; ++i) dot = fmaf(qs[i], to_f32(krow[i]), dot);
            s = dot * scale;
            if (softcap > 0.0f) s = softcap * tanhf(s / softcap);
        }
        const float block_top = block_max(s, scratch);
        const float m_new = fmaxf(m, block_top);
        const float corr = expf(m - m_new);   // exp(-inf) = 0 on the first block without a sink
        const float p = at < keys ? expf(s - m_new) : 0.0f;
        __syncthreads();
        ps[threadIdx.x] = p;
        const float block_total = block_sum(p, scratch);  // has the barriers that publish ps
        l = l * corr + block_total;
        m = m_new;
        const int count = min(SK_THREADS, keys - base);
#pragma unroll
        for (int r = 0; r < SK_MAX_PER_THREAD; ++r) {
            const int dd = threadIdx.x + r * SK_THREADS;
            if (dd < dv) {
                float a = acc[r] * corr;
                for (int j = 0; j < count; ++j) {
                    const int kj = base + j < kept ? base + j : lo + base + j - kept;
                    const size_t page = (size_t)table[kj / page_size];
                    const T* vrow = v_cache + ((page * K + kh) * page_size + (size_t)(kj % page_size)) * v_stride;
                    a = fmaf(ps[j], to_f32(vrow[dd]), a);
                }
                acc[r] = a;
            }
        }
        __syncthreads();
    }
    T* orow = out + (size_t)t * out_stride + (size_t)head * dv;
    const T* grow = gate != nullptr ? gate + (size_t)t * gate_stride + (size_t)head * dv : nullptr;
#pragma unroll
    for (int r = 0; r < SK_MAX_PER_THREAD; ++r) {
        const int dd = threadIdx.x + r * SK_THREADS;
        if (dd < dv) {
            float o = acc[r] / l * out_scale;
            if (grow != nullptr) o *= 1.0f / (1.0f + expf(-to_f32(grow[dd])));
            if (wide_out != nullptr) wide_out[((size_t)t * H + head) * dv + dd] = o;
            else orow[dd] = from_f32<T>(o);
        }
    }
}

// gate: null, or the first gate column of token 0 (rows `gate_stride` elements apart, H heads of dv side by side).
// sink_logit: null (a sink of score 0, if `sink`) or a float32 score per query head.  v_stride: elements between the values of
// two positions of a page (dv for value pages of their own; the key rows' width where values are the start of the key rows).
// keep: first positions that are always seen; softcap 0: scores are not capped; out rows are out_stride elements apart.
// wide_out: null, or float32 [tokens][H][dv] that takes the result instead of `out`.
MB_API int mb_attention_sink(const void* q, const void* k_cache, const void* v_cache, void* out, int dtype, const int* block_table,
                             int max_pages, const int* req_index, const int* positions, int tokens, int H, int K, int d, int dv,
                             int page_size, float scale, int window, int chunk, int sink, const float* sink_logit, int v_stride,
                             const void* gate, int gate_stride, int keep, float softcap, float out_scale, int out_stride, float* wide_out, cudaStream_t s) {
    if (tokens <= 0) return 0;
    if (v_stride < dv || keep < 0 || softcap < 0.0f || (wide_out == nullptr && out_stride < H * dv)) return MB_ERR_BAD_SIZE;
    if (d <= 0 || dv <= 0 || dv > SK_THREADS * SK_MAX_PER_THREAD || K <= 0 || H % K != 0 || window < 0 || chunk < 0) return MB_ERR_BAD_SIZE;
    dim3 grid(tokens, H);
    const size_t smem = (size_t)(d + SK_THREADS + 32) * sizeof(float);
    if (smem > 48 * 1024) return MB_ERR_BAD_SIZE;
    if (dtype == MB_F32)
        return launch_kernel(attention_sink_kernel<float>, grid, SK_THREADS, smem, s, 0, (const float*)q, (const float*)k_cache,
                             (const float*)v_cache, (float*)out, block_table, max_pages, req_index, positions, H, K, d, dv, page_size,
                             scale, window, chunk, sink, sink_logit, v_stride, (const float*)gate, gate_stride, keep, softcap, out_scale, out_stride, wide_out);
    if (dtype == MB_BF16)
        return launch_kernel(attention_sink_kernel<bf16>, grid, SK_THREADS, smem, s, 0, (const bf16*)q, (const bf16*)k_cache,
                             (const bf16*)v_cache, (bf16*)out, block_table, max_pages, req_index, positions, H, K, d, dv, page_size,
                             scale, window, chunk, sink, sink_logit, v_stride, (const bf16*)gate, gate_stride, keep, softcap, out_scale, out_stride, wide_out);
    return MB_ERR_BAD_DTYPE;
}
