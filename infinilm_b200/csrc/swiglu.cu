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

// ---- activations that stand on their own ---------------------------------------------------------------------------------
// y[i] = relu(z[i])^2, VEC neighbours a thread (out may be z).
template <typename TA, int VEC>
__global__ void relu2_kernel(const TA* z, TA* out, size_t total_vec) {
    il_pdl_wait();
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total_vec; idx += stride) {
        if (VEC == 1) {
            out[idx] = il_from_f<TA>(il_relu2(il_to_f(z[idx])));
        } else {
            uint4 q = reinterpret_cast<const uint4*>(z)[idx];
            TA* p = reinterpret_cast<TA*>(&q);
#pragma unroll
            for (int k = 0; k < VEC; ++k) p[k] = il_from_f<TA>(il_relu2(il_to_f(p[k])));
            reinterpret_cast<uint4*>(out)[idx] = q;
        }
    }
}

// out[t, n] = gelu_tanh(z[t, n]) * table[ids[t], off + n] for n < dim, 0 for dim <= n < ldo: a token's own row of a table, gated (z f32).
template <typename TA>
__global__ void gelu_row_kernel(const float* z, int ldz, const int* __restrict__ ids, const TA* __restrict__ table, int ldt, int off, int dim, int vocab,
                                TA* __restrict__ out, int ldo, unsigned total) {
    il_pdl_wait();
    const unsigned stride = gridDim.x * blockDim.x;
    for (unsigned i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
        const unsigned t = i / (unsigned)ldo;
        const int n = (int)(i - t * (unsigned)ldo), id = ids[t];
        float y = 0.f;
        if (n < dim && id >= 0 && id < vocab) {   // (the host rejects other ids before launch; never read out of range)
            const float g = z[(size_t)t * ldz + n], e = il_to_f(table[(size_t)id * ldt + off + n]);
            y = sizeof(TA) == 2 ? il_gelu_tanh_mul_fast(g, e) : il_gelu_tanh_mul(g, e);
        }
        out[i] = il_from_f<TA>(y);
    }
}

// The same, four neighbouring columns a thread.
__device__ __forceinline__ float4 gr_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 gr_ld4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void gr_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void gr_st4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
template <typename TA>
__global__ void gelu_row4_kernel(const float* z, int ldz, const int* __restrict__ ids, const TA* __restrict__ table, int ldt, int off, int dim, int vocab,
                                 TA* __restrict__ out, int ldo, unsigned total4) {
    il_pdl_wait();
    const unsigned stride = gridDim.x * blockDim.x, ld4 = (unsigned)ldo >> 2;
    for (unsigned i = blockIdx.x * blockDim.x + threadIdx.x; i < total4; i += stride) {
        const unsigned t = i / ld4;
        const int n = (int)(i - t * ld4) << 2, id = ids[t];
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (n < dim && id >= 0 && id < vocab) {   // (dim is a multiple of 4 here)
            const float4 g = gr_ld4(z + (size_t)t * ldz + n), e = gr_ld4(table + (size_t)id * ldt + off + n);
            if (sizeof(TA) == 2)
                y = make_float4(il_gelu_tanh_mul_fast(g.x, e.x), il_gelu_tanh_mul_fast(g.y, e.y), il_gelu_tanh_mul_fast(g.z, e.z), il_gelu_tanh_mul_fast(g.w, e.w));
            else
                y = make_float4(il_gelu_tanh_mul(g.x, e.x), il_gelu_tanh_mul(g.y, e.y), il_gelu_tanh_mul(g.z, e.z), il_gelu_tanh_mul(g.w, e.w));
        }
        gr_st4(out + (size_t)t * ldo + n, y);
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

IL_EXPORT int il_relu2(const void* z, void* out, int act_kind, long long total, cudaStream_t stream) {
    if (total <= 0) return IL_OK;
    if (act_kind != IL_F32 && act_kind != IL_BF16) return IL_BAD_ARG;
    const int vec = act_kind == IL_F32 ? 4 : 8;
    const bool v = total % vec == 0 && (((uintptr_t)z | (uintptr_t)out) & 15) == 0;
    const long long n = v ? total / vec : total, g = (n + 255) / 256;
    const int blocks = (int)(g > 148 * 32 ? 148 * 32 : g);
    if (act_kind == IL_F32) {
        if (v) IL_LAUNCH((relu2_kernel<float, 4>), blocks, 256, 0, stream, (const float*)z, (float*)out, (size_t)n);
        else IL_LAUNCH((relu2_kernel<float, 1>), blocks, 256, 0, stream, (const float*)z, (float*)out, (size_t)n);
    } else {
        if (v) IL_LAUNCH((relu2_kernel<__nv_bfloat16, 8>), blocks, 256, 0, stream, (const __nv_bfloat16*)z, (__nv_bfloat16*)out, (size_t)n);
        else IL_LAUNCH((relu2_kernel<__nv_bfloat16, 1>), blocks, 256, 0, stream, (const __nv_bfloat16*)z, (__nv_bfloat16*)out, (size_t)n);
    }
    IL_LAUNCH_CHECK();
    return IL_OK;
}

IL_EXPORT int il_gelu_row(const float* z, int act_kind, int ldz, const int* ids, const void* table, int ldt, int off, int dim, int vocab, void* out,
                          int ldo, int T, cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (dim <= 0 || ldz < dim || ldo < dim || off < 0 || off + dim > ldt || vocab <= 0) return IL_BAD_ARG;
    if (act_kind != IL_F32 && act_kind != IL_BF16) return IL_BAD_ARG;
    const int eb = act_kind == IL_F32 ? 4 : 2;    // four columns at a time where every row's pieces start on whole borders
    const bool vec = ((ldz | ldo | ldt | off | dim) & 3) == 0 && ((uintptr_t)z & 15) == 0 && (((uintptr_t)table | (uintptr_t)out) & (4 * eb - 1)) == 0;
    const long long all = (long long)T * ldo, g = (all + 255) / 256;
    if (all > 0x7fffffffLL) return IL_UNSUPPORTED;
    const unsigned total = (unsigned)all;
    const int blocks = (int)(g > 148 * 16 ? 148 * 16 : g);
    if (vec) {
        const long long g4 = (all / 4 + 255) / 256;
        const int blocks4 = (int)(g4 > 148 * 16 ? 148 * 16 : g4);
        if (act_kind == IL_F32)
            IL_LAUNCH(gelu_row4_kernel<float>, blocks4, 256, 0, stream, z, ldz, ids, (const float*)table, ldt, off, dim, vocab, (float*)out, ldo, total / 4);
        else
            IL_LAUNCH(gelu_row4_kernel<__nv_bfloat16>, blocks4, 256, 0, stream, z, ldz, ids, (const __nv_bfloat16*)table, ldt, off, dim, vocab,
                      (__nv_bfloat16*)out, ldo, total / 4);
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    if (act_kind == IL_F32)
        IL_LAUNCH(gelu_row_kernel<float>, blocks, 256, 0, stream, z, ldz, ids, (const float*)table, ldt, off, dim, vocab, (float*)out, ldo, total);
    else
        IL_LAUNCH(gelu_row_kernel<__nv_bfloat16>, blocks, 256, 0, stream, z, ldz, ids, (const __nv_bfloat16*)table, ldt, off, dim, vocab,
                  (__nv_bfloat16*)out, ldo, total);
    IL_LAUNCH_CHECK();
    return IL_OK;
}
