// Residual add fused with RMSNorm.
//
//   all rows:       x[t] += delta[t];  y[t] = x[t] / sqrt(mean(x[t]^2) + eps) * w
//   selected rows:  v = x[rows[r]] + delta[rows[r]];  y[r] = v / sqrt(mean(v^2) + eps) * w
//   groups > 1:     the mean is taken over each of `groups` equal consecutive parts of the row by itself
//   two addends:    x[t] += delta[t] + delta2[t] (a layer whose two sublayers read the same norm's output)
//   normed addend:  d = delta[t] / sqrt(mean(delta[t]^2) + eps_d) * w_d takes the place of delta[t] (a sublayer with a
//                   norm behind it as well as before it: its norm, the sum and the next sublayer's norm are one kernel)
//
// The residual stream x is 32-bit in every mode; sum and norm are 32-bit
// (crates/cellm-kernels/src/cpu_kernels.rs:17-34 is the formula: the weight is
// used as it is, with no +1). delta may be absent (a plain norm). One block
// per row; the order of the sum depends only on the row length, so a row's
// result does not depend on what else is in the batch.
#include "common.cuh"

template <typename TA, typename TW>
__global__ void add_rmsnorm_kernel(float* __restrict__ x, const TA* __restrict__ delta, const TA* __restrict__ delta2,
                                   const TW* __restrict__ w, TA* __restrict__ y,
                                   const int* __restrict__ rows, int H, int groups, float eps) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const int t = rows ? rows[r] : r;
    float* xr = x + (size_t)t * H;
    const TA* dr = delta ? delta + (size_t)t * H : nullptr;
    const TA* dr2 = (delta && delta2) ? delta2 + (size_t)t * H : nullptr;
    const bool write_back = (rows == nullptr) && (delta != nullptr);
    TA* yr = y + (size_t)r * H;
    // groups > 1: the row in equal consecutive parts, each divided by its own root mean square
    const int Hg = H / groups;
    for (int g = 0; g < groups; ++g) {
        const int lo = g * Hg, hi = lo + Hg;
        float ss = 0.f;
        for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) {
            float v = xr[i];
            if (dr) v += dr2 ? to_float(dr[i]) + to_float(dr2[i]) : to_float(dr[i]);
            if (write_back) xr[i] = v;
            ss += v * v;
        }
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)Hg + eps);
        for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) {
            float v = xr[i];
            if (dr && !write_back) v += dr2 ? to_float(dr[i]) + to_float(dr2[i]) : to_float(dr[i]);
            yr[i] = from_float<TA>(v * inv * to_float(w[i]));
        }
    }
}

// The same for rows of bfloat16 activations whose length is a multiple of 8 and at
// most 8 * 1024: every thread keeps its 8 values in registers, so each element is
// read once and written once, in 16-byte pieces. The sum over a row is taken in
// the same order whatever the batch (thread partials of 8, then the block tree).
template <typename TW>
__global__ void add_rmsnorm_vec8_kernel(float* __restrict__ x, const __nv_bfloat16* __restrict__ delta,
                                        const __nv_bfloat16* __restrict__ delta2, const TW* __restrict__ w, __nv_bfloat16* __restrict__ y,
                                        const int* __restrict__ rows, int H, float eps) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const int t = rows ? rows[r] : r;
    const int i0 = threadIdx.x * 8;
    const bool on = i0 < H;
    const bool write_back = (rows == nullptr) && (delta != nullptr);
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
    if (on) {
        const float4 a = *reinterpret_cast<const float4*>(x + (size_t)t * H + i0);
        const float4 b = *reinterpret_cast<const float4*>(x + (size_t)t * H + i0 + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
        if (delta && delta2) {
            const uint4 d = *reinterpret_cast<const uint4*>(delta + (size_t)t * H + i0);
            const uint4 e = *reinterpret_cast<const uint4*>(delta2 + (size_t)t * H + i0);
            const __nv_bfloat162* dp = reinterpret_cast<const __nv_bfloat162*>(&d);
            const __nv_bfloat162* ep = reinterpret_cast<const __nv_bfloat162*>(&e);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(dp[j]), g = __bfloat1622float2(ep[j]);
                v[2 * j] += f.x + g.x;
                v[2 * j + 1] += f.y + g.y;
            }
        } else if (delta) {
            const uint4 d = *reinterpret_cast<const uint4*>(delta + (size_t)t * H + i0);
            const __nv_bfloat162* dp = reinterpret_cast<const __nv_bfloat162*>(&d);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(dp[j]);
                v[2 * j] += f.x;
                v[2 * j + 1] += f.y;
            }
        }
        if (write_back) {
            *reinterpret_cast<float4*>(x + (size_t)t * H + i0) = make_float4(v[0], v[1], v[2], v[3]);
            *reinterpret_cast<float4*>(x + (size_t)t * H + i0 + 4) = make_float4(v[4], v[5], v[6], v[7]);
        }
    }
    float wv[8];                 // the weights travel while the row's sum is taken
#pragma unroll
    for (int j = 0; j < 8; ++j) wv[j] = on ? to_float(w[i0 + j]) : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    if (on) {
        uint32_t o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            __nv_bfloat162 pk = __floats2bfloat162_rn(v[2 * j] * inv * wv[2 * j], v[2 * j + 1] * inv * wv[2 * j + 1]);
            o[j] = *reinterpret_cast<uint32_t*>(&pk);
        }
        *reinterpret_cast<uint4*>(y + (size_t)r * H + i0) = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

// x: [*, H] float; delta, delta2: [*, H] act dtype or null (delta2 only beside delta); w: [H]; y: [n_rows, H] act dtype;
// rows: null (all n_rows rows, x updated in place) or n_rows row indices (x left as is).
static int add_rmsnorm_impl(float* x, const void* delta, const void* delta2, const void* w, int w_dtype, void* y,
                            const int* rows, int n_rows, int H, int groups, float eps, int act_dtype,
                            cudaStream_t stream) {
    if (n_rows <= 0) return CELLM_OK;
    if (delta2 && !delta) return CELLM_ERR_ARG;
    if (groups < 1 || H % groups) return CELLM_ERR_SIZE;
    if (groups == 1 && act_dtype == CELLM_BF16 && (H & 7) == 0 && H <= 8192 && (((uintptr_t)x | (uintptr_t)delta | (uintptr_t)delta2 | (uintptr_t)y) & 15) == 0) {
        const int vthreads = ((H / 8 + 31) / 32) * 32;
        if (w_dtype == CELLM_BF16)
            CELLM_RUN(add_rmsnorm_vec8_kernel<__nv_bfloat16>, n_rows, vthreads, 0, stream, x, (const __nv_bfloat16*)delta,
                      (const __nv_bfloat16*)delta2, (const __nv_bfloat16*)w, (__nv_bfloat16*)y, rows, H, eps);
        else if (w_dtype == CELLM_F32)
            CELLM_RUN(add_rmsnorm_vec8_kernel<float>, n_rows, vthreads, 0, stream, x, (const __nv_bfloat16*)delta,
                      (const __nv_bfloat16*)delta2, (const float*)w, (__nv_bfloat16*)y, rows, H, eps);
        else return CELLM_ERR_DTYPE;
        return CELLM_OK;
    }
    const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
#define LAUNCH(TA, TW) \
    CELLM_RUN((add_rmsnorm_kernel<TA, TW>), n_rows, threads, 0, stream, x, (const TA*)delta, (const TA*)delta2, (const TW*)w, (TA*)y, rows, H, groups, eps)
    if (act_dtype == CELLM_F32 && w_dtype == CELLM_F32) LAUNCH(float, float);
    else if (act_dtype == CELLM_F32 && w_dtype == CELLM_BF16) LAUNCH(float, __nv_bfloat16);
    else if (act_dtype == CELLM_BF16 && w_dtype == CELLM_F32) LAUNCH(__nv_bfloat16, float);
    else if (act_dtype == CELLM_BF16 && w_dtype == CELLM_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else return CELLM_ERR_DTYPE;
#undef LAUNCH
    return CELLM_OK;
}

CELLM_API int cellm_add_rmsnorm(float* x, const void* delta, const void* w, int w_dtype, void* y,
                                const int* rows, int n_rows, int H, int groups, float eps, int act_dtype,
                                cudaStream_t stream) {
    return add_rmsnorm_impl(x, delta, nullptr, w, w_dtype, y, rows, n_rows, H, groups, eps, act_dtype, stream);
}

// Two addends that wait at once (either may be null; the sum delta + delta2 is formed first, then added to x).
CELLM_API int cellm_add2_rmsnorm(float* x, const void* delta, const void* delta2, const void* w, int w_dtype, void* y,
                                 const int* rows, int n_rows, int H, int groups, float eps, int act_dtype,
                                 cudaStream_t stream) {
    if (!delta) { delta = delta2; delta2 = nullptr; }
    return add_rmsnorm_impl(x, delta, delta2, w, w_dtype, y, rows, n_rows, H, groups, eps, act_dtype, stream);
}

// ---- an addend that is normed before it joins the stream -------------------------------------------------------------
template <typename TA, typename TW>
__global__ void norm_add_norm_kernel(float* x, const TA* delta, const TW* __restrict__ w_d, float eps_d,
                                     const TW* __restrict__ w, TA* __restrict__ y, const int* __restrict__ rows, int H, float eps) {
    extern __shared__ float vals[];      // [H]
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const int t = rows ? rows[r] : r;
    float* xr = x + (size_t)t * H;
    const TA* dr = delta + (size_t)t * H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = to_float(dr[i]);
        vals[i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv_d = 1.0f / sqrtf(ss / (float)H + eps_d);
    ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = xr[i] + vals[i] * inv_d * to_float(w_d[i]);
        vals[i] = v;
        if (!rows) xr[i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) y[(size_t)r * H + i] = from_float<TA>(vals[i] * inv * to_float(w[i]));
}

__device__ __forceinline__ void load8(float (&v)[8], const __nv_bfloat16* p) {
    const uint4 q = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
__device__ __forceinline__ void load8(float (&v)[8], const float* p) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

// The same for bfloat16 activations and rows whose length is a multiple of 8 and at most 8 * 1024: a thread keeps its 8
// values in registers, every element is read once and written once in 16-byte pieces; the weights' loads go out before the
// wait on the kernel before this one. (x and delta are not declared __restrict__: their loads, which look like the weights'
// to the compiler and have the same condition, must stay behind that wait.)
template <typename TW>
__global__ void norm_add_norm_vec8_kernel(float* x, const __nv_bfloat16* delta, const TW* __restrict__ w_d, float eps_d,
                                          const TW* __restrict__ w, __nv_bfloat16* y, const int* rows, int H, float eps) {
    __shared__ float scratch[32];
    pdl_trigger();
    const int i0 = threadIdx.x * 8;
    const bool on = i0 < H;
    float wd[8], wv[8], v[8], d[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) wd[j] = wv[j] = v[j] = d[j] = 0.f;
    if (on) { load8(wd, w_d + i0); load8(wv, w + i0); }         // the weights are not the work of the kernel before this one
    pdl_wait();
    const int r = blockIdx.x;
    const int t = rows ? rows[r] : r;
    const size_t at = (size_t)t * H + i0;
    if (on) { load8(d, delta + at); load8(v, x + at); }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += d[j] * d[j];
    ss = block_sum(ss, scratch);
    const float inv_d = 1.0f / sqrtf(ss / (float)H + eps_d);
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        v[j] += d[j] * inv_d * wd[j];
        ss += v[j] * v[j];
    }
    if (on && !rows) {
        *reinterpret_cast<float4*>(x + at) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(x + at + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    if (on) {
        uint32_t o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            __nv_bfloat162 pk = __floats2bfloat162_rn(v[2 * j] * inv * wv[2 * j], v[2 * j + 1] * inv * wv[2 * j + 1]);
            o[j] = *reinterpret_cast<uint32_t*>(&pk);
        }
        *reinterpret_cast<uint4*>(y + (size_t)r * H + i0) = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

// x[t] += d(delta[t]);  y[t] = x[t] / sqrt(mean(x[t]^2) + eps) * w, with d the norm of the addend (w_d, eps_d). x: [*, H]
// float; delta: [*, H] and y: [n_rows, H] of the activations' type; w_d, w: [H] of one type; rows as in cellm_add_rmsnorm.
CELLM_API int cellm_norm_add_norm(float* x, const void* delta, const void* w_d, float eps_d, const void* w, int w_dtype, void* y,
                                  const int* rows, int n_rows, int H, float eps, int act_dtype, cudaStream_t stream) {
    if (n_rows <= 0) return CELLM_OK;
    if (H <= 0) return CELLM_ERR_SIZE;
    if (!x || !delta || !w_d || !w || !y) return CELLM_ERR_ARG;
    if (act_dtype == CELLM_BF16 && (H & 7) == 0 && H <= 8192 && (((uintptr_t)x | (uintptr_t)delta | (uintptr_t)w_d | (uintptr_t)w | (uintptr_t)y) & 15) == 0) {
        const int vthreads = ((H / 8 + 31) / 32) * 32;
        if (w_dtype == CELLM_BF16)
            CELLM_RUN(norm_add_norm_vec8_kernel<__nv_bfloat16>, n_rows, vthreads, 0, stream, x, (const __nv_bfloat16*)delta, (const __nv_bfloat16*)w_d,
                      eps_d, (const __nv_bfloat16*)w, (__nv_bfloat16*)y, rows, H, eps);
        else if (w_dtype == CELLM_F32)
            CELLM_RUN(norm_add_norm_vec8_kernel<float>, n_rows, vthreads, 0, stream, x, (const __nv_bfloat16*)delta, (const float*)w_d, eps_d,
                      (const float*)w, (__nv_bfloat16*)y, rows, H, eps);
        else return CELLM_ERR_DTYPE;
        return CELLM_OK;
    }
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return CELLM_ERR_SIZE;
    const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
#define LAUNCH(TA, TW)                                                                                                  \
    do {                                                                                                                \
        if (smem > 48 * 1024) {                                                                                         \
            cudaError_t e = cudaFuncSetAttribute(norm_add_norm_kernel<TA, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                        \
        }                                                                                                               \
        CELLM_RUN((norm_add_norm_kernel<TA, TW>), n_rows, threads, smem, stream, x, (const TA*)delta, (const TW*)w_d, eps_d, (const TW*)w, (TA*)y, \
                  rows, H, eps);                                                                                        \
    } while (0)
    if (act_dtype == CELLM_F32 && w_dtype == CELLM_F32) LAUNCH(float, float);
    else if (act_dtype == CELLM_F32 && w_dtype == CELLM_BF16) LAUNCH(float, __nv_bfloat16);
    else if (act_dtype == CELLM_BF16 && w_dtype == CELLM_F32) LAUNCH(__nv_bfloat16, float);
    else if (act_dtype == CELLM_BF16 && w_dtype == CELLM_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else return CELLM_ERR_DTYPE;
#undef LAUNCH
    return CELLM_OK;
}

// z = cap * tanh(z / cap) in place over n 32-bit values (logits held between -cap and cap).
__global__ void soft_cap_kernel(float* __restrict__ z, size_t n, float cap) {
    pdl_trigger();
    pdl_wait();
    const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i + 4 <= n) {
        float4 v = *reinterpret_cast<const float4*>(z + i);
        v.x = cap * tanhf(v.x / cap);
        v.y = cap * tanhf(v.y / cap);
        v.z = cap * tanhf(v.z / cap);
        v.w = cap * tanhf(v.w / cap);
        *reinterpret_cast<float4*>(z + i) = v;
    } else {
        for (size_t j = i; j < n; ++j) z[j] = cap * tanhf(z[j] / cap);
    }
}

CELLM_API int cellm_soft_cap(float* z, long long n, float cap, cudaStream_t stream) {
    if (n <= 0) return CELLM_OK;
    if (!(cap > 0.f)) return CELLM_ERR_ARG;
    if ((uintptr_t)z & 15) return CELLM_ERR_ALIGN;
    const unsigned blocks = (unsigned)((n + 1023) / 1024);
    CELLM_RUN(soft_cap_kernel, blocks, 256, 0, stream, z, (size_t)n, cap);
    return CELLM_OK;
}

// Adds a pending delta into the residual stream without a norm (used when a
// block's output is not followed by a norm that could absorb it).
template <typename TA>
__global__ void residual_add_kernel(float* __restrict__ x, const TA* __restrict__ delta, size_t n) {
    pdl_trigger();
    pdl_wait();
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += to_float(delta[i]);
}

CELLM_API int cellm_residual_add(float* x, const void* delta, long long n, int act_dtype,
                                 cudaStream_t stream) {
    if (n <= 0) return CELLM_OK;
    const int threads = 256;
    const unsigned blocks = (unsigned)((n + threads - 1) / threads);
    if (act_dtype == CELLM_F32)
        CELLM_RUN(residual_add_kernel<float>, blocks, threads, 0, stream, x, (const float*)delta, (size_t)n);
    else if (act_dtype == CELLM_BF16)
        CELLM_RUN(residual_add_kernel<__nv_bfloat16>, blocks, threads, 0, stream, x, (const __nv_bfloat16*)delta, (size_t)n);
    else return CELLM_ERR_DTYPE;
    return CELLM_OK;
}
