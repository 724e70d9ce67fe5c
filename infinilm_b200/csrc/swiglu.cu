// Gated activation on a fused gate-up product: out[t,i] = act(gu[t,i]) * gu[t,I+i], computed in f32; act: SiLU (SwiGLU) or
// the tanh form of GELU, or the clamped gate (limit, alpha). `row_scale` (or null): a factor per row, multiplied into gate and
// up products alike before anything else (rows whose factor belongs to the product's input).
// Also a bias add for library matrix products that have no bias epilogue.
#include "common.cuh"

template <typename TA>
__device__ __forceinline__ float gated(float g, float u, int act, float limit, float alpha) {
    if (act == IL_ACT_CLAMPED) return sizeof(TA) == 2 ? il_clamped_glu_fast(g, u, limit, alpha) : il_clamped_glu(g, u, limit, alpha);
    if (act == IL_ACT_GELU_TANH) return sizeof(TA) == 2 ? il_gelu_tanh_mul_fast(g, u) : il_gelu_tanh_mul(g, u);
    return sizeof(TA) == 2 ? il_silu_mul_fast(g, u) : g / (1.f + expf(-g)) * u;
}

template <typename TA>
__global__ void swiglu_kernel(const TA* __restrict__ gu, TA* __restrict__ out, int I, size_t total, int act, float limit, float alpha,
                              const float* __restrict__ row_scale) {
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < total; idx += stride) {
        const size_t t = idx / I;
        const int i = (int)(idx - t * I);
        const float rs = row_scale ? row_scale[t] : 1.f;
        const float g = il_to_f(gu[t * 2 * I + i]) * rs;
        const float u = il_to_f(gu[t * 2 * I + I + i]) * rs;
        out[idx] = il_from_f<TA>(gated<TA>(g, u, act, limit, alpha));
    }
}

// 8 bfloat16 (or 4 float) per thread and access; I must be a multiple of the vector width.
template <typename TA, int VEC>
__global__ void swiglu_vec_kernel(const TA* __restrict__ gu, TA* __restrict__ out, int I, size_t total_vec, int act, float limit, float alpha,
                                  const float* __restrict__ row_scale) {
    const int ivec = I / VEC;
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < total_vec; idx += stride) {
        const size_t t = idx / ivec;
        const int i = (int)(idx - t * ivec) * VEC;
        const uint4 gq = *reinterpret_cast<const uint4*>(gu + t * 2 * I + i);
        const uint4 uq = *reinterpret_cast<const uint4*>(gu + t * 2 * I + I + i);
        const float rs = row_scale ? row_scale[t] : 1.f;
        uint4 oq;
        const TA* gp = reinterpret_cast<const TA*>(&gq);
        const TA* up = reinterpret_cast<const TA*>(&uq);
        TA* op = reinterpret_cast<TA*>(&oq);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float g = il_to_f(gp[k]) * rs, u = il_to_f(up[k]) * rs;
            op[k] = il_from_f<TA>(gated<TA>(g, u, act, limit, alpha));
        }
        *reinterpret_cast<uint4*>(out + t * I + i) = oq;
    }
}

template <typename TA>
__global__ void add_bias_kernel(TA* __restrict__ y, const void* __restrict__ b, int b_kind, int N, size_t total) {
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; idx < total; idx += stride) {
        const int n = (int)(idx % N);
        y[idx] = il_from_f<TA>(il_to_f(y[idx]) + il_load_any(b, b_kind, n));
    }
}

static inline int grid_for(size_t total, int threads) {
    size_t g = (total + threads - 1) / threads;
    const size_t cap = 148 * 16;
    return (int)(g > cap ? cap : g);
}

IL_EXPORT int il_swiglu(const void* gu, void* out, int act_kind, int T, int I, int act, float limit, float alpha, const float* row_scale,
                        cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (act != IL_ACT_SILU && act != IL_ACT_GELU_TANH && act != IL_ACT_CLAMPED) return IL_BAD_ARG;
    if (I <= 0) return IL_BAD_ARG;
    const size_t total = (size_t)T * I;
    if (act_kind == IL_BF16 && I % 8 == 0) {
        const size_t tv = total / 8;
        size_t g = (tv + 255) / 256;
        if (g > 148 * 32) g = 148 * 32;
        swiglu_vec_kernel<__nv_bfloat16, 8><<<(int)g, 256, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, I, tv, act, limit, alpha, row_scale);
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    if (act_kind == IL_F32 && I % 4 == 0) {
        const size_t tv = total / 4;
        size_t g = (tv + 255) / 256;
        if (g > 148 * 32) g = 148 * 32;
        swiglu_vec_kernel<float, 4><<<(int)g, 256, 0, stream>>>((const float*)gu, (float*)out, I, tv, act, limit, alpha, row_scale);
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    const int threads = 256, grid = grid_for(total, threads);
    if (act_kind == IL_F32)
        swiglu_kernel<float><<<grid, threads, 0, stream>>>((const float*)gu, (float*)out, I, total, act, limit, alpha, row_scale);
    else if (act_kind == IL_BF16)
        swiglu_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, I, total, act, limit, alpha, row_scale);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

IL_EXPORT int il_add_bias(void* y, int act_kind, const void* bias, int bias_kind, int T, int N, cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (N <= 0) return IL_BAD_ARG;
    const size_t total = (size_t)T * N;
    const int threads = 256, grid = grid_for(total, threads);
    if (act_kind == IL_F32)
        add_bias_kernel<float><<<grid, threads, 0, stream>>>((float*)y, bias, bias_kind, N, total);
    else if (act_kind == IL_BF16)
        add_bias_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>((__nv_bfloat16*)y, bias, bias_kind, N, total);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}
