// Layer norm of float32 rows, alone or as the end of a sublayer whose output is normed before it joins the residual stream:
//   v = (y - mean(y)) / sqrt(mean((y - mean)^2) + eps) * w + b        (mode 0, layer norm; b may be absent)
//   v = y / sqrt(mean(y^2) + eps) * w                                 (mode 1, root mean square)
// plain:     out = v;
// sublayer:  hidden <- hidden + v * scale (scale: a vector, or absent), y <- 0 (the next sublayer adds into it) and, where
//            asked for, the new row of the stream in the activation dtype for the next sublayer to read.
// A row per block, held in registers: one pass over memory, the deviations squared around the mean that was found first.
#define MB_LIB "layer_norm"
#define MB_LIB_ID 19
#include "common.cuh"
#include "launch.cuh"

template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 packed;
    packed.x = *reinterpret_cast<const uint32_t*>(&lo);
    packed.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = packed;
}

// n a multiple of 4, at most 4 R blockDim.x
template <typename T, int R>
__global__ void __launch_bounds__(1024) layer_norm_vec_kernel(float* y, const float* __restrict__ w, const float* __restrict__ b,
                                                              const float* __restrict__ scale, float* hidden, T* __restrict__ out, int n, float eps,
                                                              int mode) {
    PDL_ENTER();
    y = pdl_fresh(y); hidden = pdl_fresh(hidden);
    __shared__ float scratch[32];
    const int n4 = n >> 2, threads = blockDim.x;
    float4* row = reinterpret_cast<float4*>(y + (size_t)blockIdx.x * n);
    float4 v[R];
    float sum = 0.0f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = threadIdx.x + r * threads;
        v[r] = i < n4 ? row[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        sum += (v[r].x + v[r].y) + (v[r].z + v[r].w);
    }
    float mean = 0.0f;
    if (mode == 0) mean = block_sum(sum, scratch) / (float)n;
    float ss = 0.0f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (threadIdx.x + r * threads < n4) {
            v[r].x -= mean; v[r].y -= mean; v[r].z -= mean; v[r].w -= mean;
            ss += (v[r].x * v[r].x + v[r].y * v[r].y) + (v[r].z * v[r].z + v[r].w * v[r].w);
        }
    }
    ss = block_sum(ss, scratch);
    const float f = 1.0f / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = threadIdx.x + r * threads;
        if (i >= n4) continue;
        const float4 g = reinterpret_cast<const float4*>(w)[i];
        float4 o = make_float4(v[r].x * f * g.x, v[r].y * f * g.y, v[r].z * f * g.z, v[r].w * f * g.w);
        if (b != nullptr) {
            const float4 c = reinterpret_cast<const float4*>(b)[i];
            o.x += c.x; o.y += c.y; o.z += c.z; o.w += c.w;
        }
        if (hidden != nullptr) {
            float4* h = reinterpret_cast<float4*>(hidden + (size_t)blockIdx.x * n) + i;
            float4 old = *h;
            if (scale != nullptr) {
                const float4 s = reinterpret_cast<const float4*>(scale)[i];
                o.x *= s.x; o.y *= s.y; o.z *= s.z; o.w *= s.w;
            }
            o.x += old.x; o.y += old.y; o.z += old.z; o.w += old.w;
            *h = o;
            row[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (out != nullptr) store4(out + (size_t)blockIdx.x * n + 4 * i, o);
    }
}

// any n: the row stays in shared memory
template <typename T>
__global__ void __launch_bounds__(256) layer_norm_kernel(float* y, const float* __restrict__ w, const float* __restrict__ b, const float* __restrict__ scale,
                                                         float* hidden, T* __restrict__ out, int n, float eps, int mode) {
    PDL_ENTER();
    y = pdl_fresh(y); hidden = pdl_fresh(hidden);
    extern __shared__ float vals[];
    __shared__ float scratch[32];
    float* row = y + (size_t)blockIdx.x * n;
    float sum = 0.0f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) { vals[i] = row[i]; sum += vals[i]; }     // (a thread reads back only what it wrote)
    float mean = 0.0f;
    if (mode == 0) mean = block_sum(sum, scratch) / (float)n;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) { const float d = vals[i] - mean; ss += d * d; }
    ss = block_sum(ss, scratch);
    const float f = 1.0f / sqrtf(ss / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        float o = (vals[i] - mean) * f * w[i];
        if (b != nullptr) o += b[i];
        if (hidden != nullptr) {
            float* h = hidden + (size_t)blockIdx.x * n + i;
            if (scale != nullptr) o *= scale[i];
            o += *h;
            *h = o;
            row[i] = 0.0f;
        }
        if (out != nullptr) out[(size_t)blockIdx.x * n + i] = from_f32<T>(o);
    }
}

// hidden null: out = norm(y) and y stays as it is.  mode 0: layer norm, 1: root mean square (no mean taken off).
MB_API int mb_layer_norm(float* y, const float* w, const float* b, const float* scale, float* hidden, void* out, int out_dtype, int rows, int n,
                         float eps, int mode, cudaStream_t s) {
    if (rows <= 0) return 0;
    if (n <= 0 || mode < 0 || mode > 1 || (hidden == nullptr && out == nullptr)) return MB_ERR_BAD_SIZE;
    if (out_dtype != MB_F32 && out_dtype != MB_BF16) return MB_ERR_BAD_DTYPE;
    const uintptr_t all = (uintptr_t)y | (uintptr_t)w | (uintptr_t)b | (uintptr_t)scale | (uintptr_t)hidden | (uintptr_t)out;
    const int n4 = n / 4;
    int threads = rows <= 148 ? (n4 + 31) / 32 * 32 : 256;      // few rows: every load of a row in flight at once
    if (threads > 1024) threads = 1024;
    if (threads < 64) threads = 64;
    const int runs = (n4 + threads - 1) / threads;
    if (n % 4 == 0 && (all & 15) == 0 && runs <= 8) {
#define LN_CASE(R)                                                                                                                          \
    if (runs <= R) {                                                                                                                        \
        if (out_dtype == MB_F32) return launch_kernel(layer_norm_vec_kernel<float, R>, rows, threads, 0, s, 0, y, w, b, scale, hidden, (float*)out, n, eps, mode); \
        return launch_kernel(layer_norm_vec_kernel<bf16, R>, rows, threads, 0, s, 0, y, w, b, scale, hidden, (bf16*)out, n, eps, mode);      \
    }
        LN_CASE(1) LN_CASE(2) LN_CASE(4) LN_CASE(8)
#undef LN_CASE
    }
    const size_t smem = (size_t)n * sizeof(float);
    if (smem > 48 * 1024) return MB_ERR_BAD_SIZE;
    if (out_dtype == MB_F32) return launch_kernel(layer_norm_kernel<float>, rows, 256, smem, s, 0, y, w, b, scale, hidden, (float*)out, n, eps, mode);
    return launch_kernel(layer_norm_kernel<bf16>, rows, 256, smem, s, 0, y, w, b, scale, hidden, (bf16*)out, n, eps, mode);
}

// ---- float32 rows in the activation dtype (the first sublayer's input), and a zeroed buffer for it to add into -----------
__global__ void stream_rows_kernel(const float* __restrict__ x, bf16* __restrict__ out, float* __restrict__ y, size_t total) {
    PDL_ENTER();
    x = pdl_fresh(x);
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < total; idx += stride) {
        if (out != nullptr) out[idx] = __float2bfloat16_rn(x[idx]);
        y[idx] = 0.0f;
    }
}

__global__ void stream_rows_vec_kernel(const float* __restrict__ x, bf16* __restrict__ out, float* __restrict__ y, size_t quads) {
    PDL_ENTER();
    x = pdl_fresh(x);
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < quads; idx += stride) {
        if (out != nullptr) store4(out + 4 * idx, reinterpret_cast<const float4*>(x)[idx]);
        reinterpret_cast<float4*>(y)[idx] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
}

// out null: only y is written.
MB_API int mb_stream_rows(const float* x, void* out, float* y, size_t total, cudaStream_t s) {
    if (total == 0) return 0;
    if (total % 4 == 0 && (((uintptr_t)x | (uintptr_t)out | (uintptr_t)y) & 15) == 0) {
        const size_t quads = (total / 4 + 255) / 256;
        return launch_kernel(stream_rows_vec_kernel, (unsigned)(quads < 148 * 8 ? quads : 148 * 8), 256, 0, s, 0, x, (bf16*)out, y, total / 4);
    }
    const size_t blocks = (total + 255) / 256;
    return launch_kernel(stream_rows_kernel, (unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, s, 0, x, (bf16*)out, y, total);
}
