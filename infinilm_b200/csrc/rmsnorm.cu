// Residual add fused with RMSNorm.
//   x = resid[r] + branch_scale * branch[r] + vec   (branch may be absent; vec too: f32, one vector added to every row, or -
//                                                    vec_stride = H - a row of its own for every row of resid)
//   resid[r] = x                              (kept in f32; skipped when a row list is given)
//   out[i]  = x / sqrt(mean(x^2) + eps) * w
// Sum of squares, rsqrt and the scaling are f32; one block per row with a fixed thread count,
// so a row's result does not depend on what else is in the batch.
#include "common.cuh"

template <typename TA>
__global__ void add_rmsnorm_kernel(float* __restrict__ resid, const TA* __restrict__ branch, float bscale,
                                   const void* __restrict__ w, int w_kind, float eps, TA* __restrict__ out,
                                   const int* __restrict__ rows, int H, const float* __restrict__ vec, int vec_stride) {
    extern __shared__ float xs[];
    __shared__ float red[32];
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    float* rr = resid + (size_t)r * H;
    const TA* br = branch ? branch + (size_t)r * H : nullptr;
    if (vec) vec += (size_t)r * vec_stride;
    float ss = 0.f;
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        float x = rr[h];
        if (br) x += bscale * il_to_f(br[h]);
        if (vec) x += vec[h];
        xs[h] = x;
        ss += x * x;
        if (!rows && (br || vec)) rr[h] = x;
    }
    ss = il_block_sum(ss, red);
    const float rstd = rsqrtf(ss / (float)H + eps);
    TA* o = out + (size_t)i * H;
    for (int h = threadIdx.x; h < H; h += blockDim.x)
        o[h] = il_from_f<TA>(xs[h] * rstd * il_load_any(w, w_kind, h));
}

// The same with 4 elements per thread and access: 16-byte loads of the residual, 8- or 16-byte loads of
// the branch and the weight, all of a thread's loads issued before the first use.
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

template <typename TA, int MAXV>
__global__ void __launch_bounds__(256) add_rmsnorm_vec_kernel(float* resid, const TA* branch, float bscale,
                                                              const void* __restrict__ w, int w_kind, float eps, TA* __restrict__ out,
                                                              const int* __restrict__ rows, int H, const float* __restrict__ vec, int vec_stride) {
    __shared__ float red[32];
    const int i = blockIdx.x;
    const int nv = H >> 2;                        // float4 groups in a row
    // the norm's weights and the row index do not come from the kernel before this one: read while it still runs
    float4 wv[MAXV];
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        wv[k] = v < nv ? (w_kind == IL_F32 ? ld4((const float*)w + 4 * v) : ld4((const __nv_bfloat16*)w + 4 * v)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int r = rows ? rows[i] : i;
    il_pdl_wait();
    float* rr = resid + (size_t)r * H;
    const TA* br = branch ? branch + (size_t)r * H : nullptr;
    float4 x[MAXV];
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        x[k] = v < nv ? ld4(rr + 4 * v) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (br) {
        float4 b[MAXV];
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            const int v = threadIdx.x + k * 256;
            b[k] = v < nv ? ld4(br + 4 * v) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            x[k].x += bscale * b[k].x;
            x[k].y += bscale * b[k].y;
            x[k].z += bscale * b[k].z;
            x[k].w += bscale * b[k].w;
        }
    }
    if (vec) {
        vec += (size_t)r * vec_stride;
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            const int v = threadIdx.x + k * 256;
            const float4 a = v < nv ? ld4(vec + 4 * v) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[k].x += a.x, x[k].y += a.y, x[k].z += a.z, x[k].w += a.w;
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < MAXV; ++k) ss += x[k].x * x[k].x + x[k].y * x[k].y + x[k].z * x[k].z + x[k].w * x[k].w;
    if (!rows && (br || vec)) {
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            const int v = threadIdx.x + k * 256;
            if (v < nv) st4(rr + 4 * v, x[k]);
        }
    }
    ss = il_block_sum(ss, red);
    const float rstd = rsqrtf(ss / (float)H + eps);
    TA* o = out + (size_t)i * H;
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        if (v < nv) st4(o + 4 * v, make_float4(x[k].x * rstd * wv[k].x, x[k].y * rstd * wv[k].y, x[k].z * rstd * wv[k].z, x[k].w * rstd * wv[k].w));
    }
}

template <typename TA>
static int launch_vec(float* resid, const void* branch, float bscale, const void* w, int w_kind, float eps, void* out,
                      const int* rows, int n_rows, int H, const float* vec, int vec_stride, cudaStream_t stream) {
    const int nv = H >> 2;
    if (nv <= 256 * 2)
        IL_LAUNCH((add_rmsnorm_vec_kernel<TA, 2>), n_rows, 256, 0, stream, resid, (const TA*)branch, bscale, w, w_kind, eps, (TA*)out, rows, H, vec, vec_stride);
    else if (nv <= 256 * 4)
        IL_LAUNCH((add_rmsnorm_vec_kernel<TA, 4>), n_rows, 256, 0, stream, resid, (const TA*)branch, bscale, w, w_kind, eps, (TA*)out, rows, H, vec, vec_stride);
    else
        IL_LAUNCH((add_rmsnorm_vec_kernel<TA, 8>), n_rows, 256, 0, stream, resid, (const TA*)branch, bscale, w, w_kind, eps, (TA*)out, rows, H, vec, vec_stride);
    return 0;
}

IL_EXPORT int il_add_rmsnorm(float* resid, const void* branch, float bscale, const void* w, int w_kind,
                             float eps, void* out, int act_kind, const int* rows, int n_rows, int H,
                             const float* vec, int vec_stride, cudaStream_t stream) {
    if (n_rows <= 0) return IL_OK;
    if (H <= 0) return IL_BAD_ARG;
    if (H % 4 == 0 && H <= 256 * 8 * 4 && (act_kind == IL_F32 || act_kind == IL_BF16)) {
        if (act_kind == IL_F32) launch_vec<float>(resid, branch, bscale, w, w_kind, eps, out, rows, n_rows, H, vec, vec_stride, stream);
        else launch_vec<__nv_bfloat16>(resid, branch, bscale, w, w_kind, eps, out, rows, n_rows, H, vec, vec_stride, stream);
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return IL_UNSUPPORTED;
    const int threads = 256;
    if (act_kind == IL_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(add_rmsnorm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        add_rmsnorm_kernel<float><<<n_rows, threads, smem, stream>>>(resid, (const float*)branch, bscale, w, w_kind, eps, (float*)out, rows, H, vec, vec_stride);
    } else if (act_kind == IL_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(add_rmsnorm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        add_rmsnorm_kernel<__nv_bfloat16><<<n_rows, threads, smem, stream>>>(resid, (const __nv_bfloat16*)branch, bscale, w, w_kind, eps, (__nv_bfloat16*)out, rows, H, vec, vec_stride);
    } else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// ---- the norm on the branch, then the residual add -------------------------------------------------------------------
//   resid[r] += scale * branch[r] / sqrt(mean(branch[r]^2) + eps) * w        (f32)
//   copy[r]   = resid[r] in the activations' type (optional: what the next sublayer reads)
// The block layout of a model whose sublayers read the residual stream itself and whose norms sit on the sublayers'
// outputs. One block per row with a fixed thread count; the branch row waits in shared memory as f32 between the two passes.
template <typename TA>
__global__ void __launch_bounds__(256) norm_add_kernel(float* resid, const TA* branch, float scale, const void* __restrict__ w, int w_kind,
                                                       float eps, TA* copy, int H) {
    extern __shared__ float bs[];
    __shared__ float red[32];
    const int r = blockIdx.x;
    il_pdl_wait();
    const TA* br = branch + (size_t)r * H;
    float* rr = resid + (size_t)r * H;
    float ss = 0.f;
    if ((H & 3) == 0) {
        for (int v = threadIdx.x; v < (H >> 2); v += blockDim.x) {
            const float4 b = ld4(br + 4 * v);
            st4(bs + 4 * v, b);
            ss += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
        }
    } else {
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            const float b = il_to_f(br[h]);
            bs[h] = b;
            ss += b * b;
        }
    }
    ss = il_block_sum(ss, red);
    const float k = scale * (1.f / sqrtf(ss / (float)H + eps));
    if ((H & 3) == 0) {
        for (int v = threadIdx.x; v < (H >> 2); v += blockDim.x) {
            const float4 b = ld4(bs + 4 * v);
            const float4 wv = w_kind == IL_F32 ? ld4((const float*)w + 4 * v) : ld4((const __nv_bfloat16*)w + 4 * v);
            float4 x = ld4(rr + 4 * v);
            x.x = fmaf(k * b.x, wv.x, x.x), x.y = fmaf(k * b.y, wv.y, x.y), x.z = fmaf(k * b.z, wv.z, x.z), x.w = fmaf(k * b.w, wv.w, x.w);
            st4(rr + 4 * v, x);
            if (copy) st4(copy + (size_t)r * H + 4 * v, x);
        }
    } else {
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            const float x = fmaf(k * bs[h], il_load_any(w, w_kind, h), rr[h]);
            rr[h] = x;
            if (copy) copy[(size_t)r * H + h] = il_from_f<TA>(x);
        }
    }
}

// ---- the norm on the branch, the residual add and the next norm in one pass --------------------------------------------
//   b         = branch[r], or the sum over a token's routed rows: sum_k wt[r, k] * y[pos[r, k]]  (wt null: plain sum)
//   resid[r] += b / sqrt(mean(b^2) + eps_b) * w_b                                   (f32)
//   out[r]    = resid[r] / sqrt(mean(resid[r]^2) + eps_n) * w_n                     (out null: only the add)
// What lies between two sublayers of a model with a norm before and one after each. One block per row with a fixed thread
// count; a thread's columns (v = thread, thread + 256, ... groups of VW) stay in registers between the passes.
template <typename TA, int VW> struct NanVec;
template <typename TA> struct NanVec<TA, 4> {
    static __device__ __forceinline__ float4 ld(const TA* p) { return ld4(p); }
    static __device__ __forceinline__ void st(TA* p, float4 v) { st4(p, v); }
};
template <typename TA> struct NanVec<TA, 1> {
    static __device__ __forceinline__ float4 ld(const TA* p) { return make_float4(il_to_f(*p), 0.f, 0.f, 0.f); }
    static __device__ __forceinline__ void st(TA* p, float4 v) { *p = il_from_f<TA>(v.x); }
};
template <int VW> __device__ __forceinline__ float4 nan_w(const void* w, int kind, int h) {
    if (VW == 4) return kind == IL_F32 ? ld4((const float*)w + h) : ld4((const __nv_bfloat16*)w + h);
    return make_float4(il_load_any(w, kind, h), 0.f, 0.f, 0.f);
}
#define NAN_MAX_TOP 32
template <typename TA, int VW, int MAXV>
__global__ void __launch_bounds__(256) norm_add_norm_kernel(float* resid, const TA* branch, const int* pos, const float* wt, int top,
                                                            const void* __restrict__ wb, int wb_kind, float eps_b, const void* __restrict__ wn,
                                                            int wn_kind, float eps_n, TA* __restrict__ out, int H) {
    __shared__ float red[32];
    __shared__ int sp[NAN_MAX_TOP];
    __shared__ float sw[NAN_MAX_TOP];
    const int r = blockIdx.x, nv = (H + VW - 1) / VW;
    // the norms' weights do not come from the kernel before this one: read while it still runs
    float4 a[MAXV], b[MAXV];
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        a[k] = v < nv ? nan_w<VW>(wb, wb_kind, v * VW) : make_float4(0.f, 0.f, 0.f, 0.f);
        b[k] = (out && v < nv) ? nan_w<VW>(wn, wn_kind, v * VW) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    il_pdl_wait();
    if (pos) {
        if (threadIdx.x < top) {
            sp[threadIdx.x] = pos[(size_t)r * top + threadIdx.x];
            sw[threadIdx.x] = wt ? wt[(size_t)r * top + threadIdx.x] : 1.f;
        }
        __syncthreads();
    }
    float* rr = resid + (size_t)r * H;
    float4 x[MAXV], c[MAXV];
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        x[k] = v < nv ? NanVec<float, VW>::ld(rr + v * VW) : make_float4(0.f, 0.f, 0.f, 0.f);
        c[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (v < nv && !pos) c[k] = NanVec<TA, VW>::ld(branch + (size_t)r * H + v * VW);
    }
    if (pos) {                                    // the rows of a token's choices, added in the order of the choices, NR of them asked for at a time
        constexpr int NR = MAXV <= 2 ? 4 : MAXV <= 4 ? 2 : 1;
        for (int i0 = 0; i0 < top; i0 += NR) {
            float4 t[NR][MAXV];
#pragma unroll
            for (int i = 0; i < NR; ++i)
#pragma unroll
                for (int k = 0; k < MAXV; ++k) {
                    const int v = threadIdx.x + k * 256;
                    t[i][k] = (i0 + i < top && v < nv) ? NanVec<TA, VW>::ld(branch + (size_t)sp[i0 + i] * H + v * VW) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const float w = i0 + i < top ? sw[i0 + i] : 0.f;
#pragma unroll
                for (int k = 0; k < MAXV; ++k)
                    c[k].x = fmaf(w, t[i][k].x, c[k].x), c[k].y = fmaf(w, t[i][k].y, c[k].y), c[k].z = fmaf(w, t[i][k].z, c[k].z), c[k].w = fmaf(w, t[i][k].w, c[k].w);
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < MAXV; ++k) ss += c[k].x * c[k].x + c[k].y * c[k].y + c[k].z * c[k].z + c[k].w * c[k].w;
    ss = il_block_sum(ss, red);
    const float kb = 1.f / sqrtf(ss / (float)H + eps_b);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        x[k].x = fmaf(kb * c[k].x, a[k].x, x[k].x), x[k].y = fmaf(kb * c[k].y, a[k].y, x[k].y);
        x[k].z = fmaf(kb * c[k].z, a[k].z, x[k].z), x[k].w = fmaf(kb * c[k].w, a[k].w, x[k].w);
        if (v < nv) NanVec<float, VW>::st(rr + v * VW, x[k]);
        ss += x[k].x * x[k].x + x[k].y * x[k].y + x[k].z * x[k].z + x[k].w * x[k].w;
    }
    if (!out) return;
    ss = il_block_sum(ss, red);
    const float kn = 1.f / sqrtf(ss / (float)H + eps_n);
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        if (v < nv)
            NanVec<TA, VW>::st(out + (size_t)r * H + v * VW, make_float4(x[k].x * kn * b[k].x, x[k].y * kn * b[k].y, x[k].z * kn * b[k].z, x[k].w * kn * b[k].w));
    }
}

template <typename TA>
static int nan_launch(float* resid, const void* branch, const int* pos, const float* wt, int top, const void* wb, int wb_kind, float eps_b,
                      const void* wn, int wn_kind, float eps_n, void* out, int n_rows, int H, cudaStream_t stream) {
    const bool vec = (H & 3) == 0 && (((uintptr_t)resid | (uintptr_t)branch | (uintptr_t)wb | (uintptr_t)wn | (uintptr_t)out) & 15) == 0;
#define NAN_GO(VW, MAXV)                                                                                                                     \
    IL_LAUNCH((norm_add_norm_kernel<TA, VW, MAXV>), n_rows, 256, 0, stream, resid, (const TA*)branch, pos, wt, top, wb, wb_kind, eps_b, wn, \
              wn_kind, eps_n, (TA*)out, H)
    if (vec && H <= 256 * 4) NAN_GO(4, 1);
    else if (vec && H <= 256 * 4 * 2) NAN_GO(4, 2);
    else if (vec && H <= 256 * 4 * 4) NAN_GO(4, 4);
    else if (vec && H <= 256 * 4 * 8) NAN_GO(4, 8);
    else if (H <= 256 * 4) NAN_GO(1, 4);
    else if (H <= 256 * 16) NAN_GO(1, 16);
    else return IL_UNSUPPORTED;
#undef NAN_GO
    return IL_OK;
}

// branch: [n_rows, H], or - with `pos` [n_rows, top] - the rows y that the places in `pos` name.
IL_EXPORT int il_norm_add_norm(float* resid, const void* branch, const int* pos, const float* wt, int top, const void* wb, int wb_kind, float eps_b,
                               const void* wn, int wn_kind, float eps_n, void* out, int act_kind, int n_rows, int H, cudaStream_t stream) {
    if (n_rows <= 0) return IL_OK;
    if (H <= 0 || !branch || !wb || (out && !wn) || (pos && (top <= 0 || top > NAN_MAX_TOP))) return IL_BAD_ARG;
    int rc;
    if (act_kind == IL_F32) rc = nan_launch<float>(resid, branch, pos, wt, top, wb, wb_kind, eps_b, wn, wn_kind, eps_n, out, n_rows, H, stream);
    else if (act_kind == IL_BF16) rc = nan_launch<__nv_bfloat16>(resid, branch, pos, wt, top, wb, wb_kind, eps_b, wn, wn_kind, eps_n, out, n_rows, H, stream);
    else return IL_BAD_ARG;
    if (rc != IL_OK) return rc;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// ---- several branches joined in one pass ----------------------------------------------------------------------------------
//   total    = sum_i scale_i * cs_i * (y_i, or y_i / sqrt(mean(y_i^2) + eps_i) * nw_i)       up to BS_MAX_TERMS branches y_i [rows, H]
//   resid[r] += total (resid null: not)                                                       f32
//   copy[r]   = resid[r], or total where resid is null, in the activations' type (null: not)
//   out[r]    = resid[r] / sqrt(mean(resid[r]^2) + eps_n) * wn (null: not)
// nw_i (the branch's own norm) and cs_i (a factor per column) are each optional. What stands behind the sublayers of a block that
// run side by side on one input. One block per row with a fixed thread count; a thread's columns stay in registers, the
// branches are added in their order.
#define BS_MAX_TERMS 4
struct BsTerm {
    const void* y;
    const void* nw;
    const void* cs;
    int nw_kind, cs_kind;
    float scale, eps;
};
struct BsTerms { BsTerm t[BS_MAX_TERMS]; };

template <typename TA, int VW, int MAXV, int NT>
__global__ void __launch_bounds__(256) branch_sum_kernel(float* resid, const BsTerms ts, TA* copy, const void* __restrict__ wn, int wn_kind,
                                                         float eps_n, TA* __restrict__ out, int H) {
    __shared__ float red[NT + 1][8];
    const int r = blockIdx.x, nv = (H + VW - 1) / VW, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    il_pdl_wait();
    float4 c[NT][MAXV], x[MAXV];
    float* rr = resid ? resid + (size_t)r * H : nullptr;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            const int v = threadIdx.x + k * 256;
            c[i][k] = v < nv ? NanVec<TA, VW>::ld((const TA*)ts.t[i].y + (size_t)r * H + v * VW) : zero;
        }
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        x[k] = (rr && v < nv) ? NanVec<float, VW>::ld(rr + v * VW) : zero;
    }
    bool any = false;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        if (!ts.t[i].nw) continue;                // (the same for the whole grid)
        any = true;
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < MAXV; ++k) ss += c[i][k].x * c[i][k].x + c[i][k].y * c[i][k].y + c[i][k].z * c[i][k].z + c[i][k].w * c[i][k].w;
        ss = il_warp_sum(ss);
        if (lane == 0) red[i][warp] = ss;
    }
    if (any) __syncthreads();
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const BsTerm& t = ts.t[i];
        float f = t.scale;
        if (t.nw) {
            float ss = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) ss += red[i][w];
            f *= 1.f / sqrtf(ss / (float)H + t.eps);
        }
#pragma unroll
        for (int k = 0; k < MAXV; ++k) {
            const int v = threadIdx.x + k * 256;
            if (v >= nv) continue;
            float4 w = make_float4(f, f, f, f);
            if (t.nw) {
                const float4 a = nan_w<VW>(t.nw, t.nw_kind, v * VW);
                w.x *= a.x, w.y *= a.y, w.z *= a.z, w.w *= a.w;
            }
            if (t.cs) {
                const float4 a = nan_w<VW>(t.cs, t.cs_kind, v * VW);
                w.x *= a.x, w.y *= a.y, w.z *= a.z, w.w *= a.w;
            }
            x[k].x = fmaf(w.x, c[i][k].x, x[k].x), x[k].y = fmaf(w.y, c[i][k].y, x[k].y);
            x[k].z = fmaf(w.z, c[i][k].z, x[k].z), x[k].w = fmaf(w.w, c[i][k].w, x[k].w);
        }
    }
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        if (v >= nv) continue;
        if (rr) NanVec<float, VW>::st(rr + v * VW, x[k]);
        if (copy) NanVec<TA, VW>::st(copy + (size_t)r * H + v * VW, x[k]);
    }
    if (!out) return;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < MAXV; ++k) ss += x[k].x * x[k].x + x[k].y * x[k].y + x[k].z * x[k].z + x[k].w * x[k].w;
    ss = il_warp_sum(ss);
    if (lane == 0) red[NT][warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += red[NT][w];
    const float kn = 1.f / sqrtf(ss / (float)H + eps_n);
#pragma unroll
    for (int k = 0; k < MAXV; ++k) {
        const int v = threadIdx.x + k * 256;
        if (v >= nv) continue;
        const float4 b = nan_w<VW>(wn, wn_kind, v * VW);
        NanVec<TA, VW>::st(out + (size_t)r * H + v * VW, make_float4(x[k].x * kn * b.x, x[k].y * kn * b.y, x[k].z * kn * b.z, x[k].w * kn * b.w));
    }
}

template <typename TA, int NT>
static int bs_launch(float* resid, const BsTerms& ts, void* copy, const void* wn, int wn_kind, float eps_n, void* out, int n_rows, int H,
                     cudaStream_t stream) {
    uintptr_t all = (uintptr_t)resid | (uintptr_t)copy | (uintptr_t)wn | (uintptr_t)out;
    for (int i = 0; i < NT; ++i) all |= (uintptr_t)ts.t[i].y | (uintptr_t)ts.t[i].nw | (uintptr_t)ts.t[i].cs;
    const bool vec = (H & 3) == 0 && (all & 15) == 0;
#define BS_GO(VW, MAXV) \
    IL_LAUNCH((branch_sum_kernel<TA, VW, MAXV, NT>), n_rows, 256, 0, stream, resid, ts, (TA*)copy, wn, wn_kind, eps_n, (TA*)out, H)
    if (vec && H <= 256 * 4) BS_GO(4, 1);
    else if (vec && H <= 256 * 4 * 2) BS_GO(4, 2);
    else if (vec && H <= 256 * 4 * 4) BS_GO(4, 4);
    else if (vec && H <= 256 * 4 * 8) BS_GO(4, 8);
    else if (H <= 256 * 4) BS_GO(1, 4);
    else if (H <= 256 * 16) BS_GO(1, 16);
    else return IL_UNSUPPORTED;
#undef BS_GO
    return IL_OK;
}

// Branches behind the n_terms-th are not looked at. kinds: bit i: nw_i is bfloat16 (else f32), bit 8 + i: cs_i is.
IL_EXPORT int il_branch_sum(float* resid, int n_terms, const void* y0, const void* y1, const void* y2, const void* y3, const void* nw0, const void* nw1,
                            const void* nw2, const void* nw3, const void* cs0, const void* cs1, const void* cs2, const void* cs3, int kinds, float s0, float s1,
                            float s2, float s3, float e0, float e1, float e2, float e3, void* copy, const void* wn, int wn_kind, float eps_n, void* out,
                            int act_kind, int n_rows, int H, cudaStream_t stream) {
    if (n_rows <= 0) return IL_OK;
    if (n_terms <= 0 || n_terms > BS_MAX_TERMS || H <= 0 || (!resid && !copy) || (out && (!wn || !resid))) return IL_BAD_ARG;
    if (act_kind != IL_F32 && act_kind != IL_BF16) return IL_BAD_ARG;
    const void *y[] = {y0, y1, y2, y3}, *nw[] = {nw0, nw1, nw2, nw3}, *cs[] = {cs0, cs1, cs2, cs3};
    const float scale[] = {s0, s1, s2, s3}, eps[] = {e0, e1, e2, e3};
    BsTerms ts = {};
    for (int i = 0; i < n_terms; ++i) {
        if (!y[i]) return IL_BAD_ARG;
        ts.t[i] = BsTerm{y[i], nw[i], cs[i], (kinds >> i) & 1 ? IL_BF16 : IL_F32, (kinds >> (8 + i)) & 1 ? IL_BF16 : IL_F32, scale[i], eps[i]};
    }
    int rc = IL_OK;
#define BS_PICK(TA)                                                                                           \
    do {                                                                                                      \
        if (n_terms == 1) rc = bs_launch<TA, 1>(resid, ts, copy, wn, wn_kind, eps_n, out, n_rows, H, stream); \
        else if (n_terms == 2) rc = bs_launch<TA, 2>(resid, ts, copy, wn, wn_kind, eps_n, out, n_rows, H, stream); \
        else if (n_terms == 3) rc = bs_launch<TA, 3>(resid, ts, copy, wn, wn_kind, eps_n, out, n_rows, H, stream); \
        else rc = bs_launch<TA, 4>(resid, ts, copy, wn, wn_kind, eps_n, out, n_rows, H, stream);              \
    } while (0)
    if (act_kind == IL_F32) BS_PICK(float);
    else BS_PICK(__nv_bfloat16);
#undef BS_PICK
    if (rc != IL_OK) return rc;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// rows of f32 copied into the activations' type (the first sublayer's input, where no norm_add ran before it)
template <typename TA>
__global__ void cast_rows_kernel(const float* x, TA* out, size_t total) {
    il_pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) out[i] = il_from_f<TA>(x[i]);
}

IL_EXPORT int il_norm_add(float* resid, const void* branch, float scale, const void* w, int w_kind, float eps, void* copy, int act_kind,
                          int n_rows, int H, cudaStream_t stream) {
    if (n_rows <= 0) return IL_OK;
    if (H <= 0 || !branch) return IL_BAD_ARG;
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return IL_UNSUPPORTED;
    if (act_kind == IL_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(norm_add_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        IL_LAUNCH(norm_add_kernel<float>, n_rows, 256, smem, stream, resid, (const float*)branch, scale, w, w_kind, eps, (float*)copy, H);
    } else if (act_kind == IL_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(norm_add_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        IL_LAUNCH(norm_add_kernel<__nv_bfloat16>, n_rows, 256, smem, stream, resid, (const __nv_bfloat16*)branch, scale, w, w_kind, eps,
                  (__nv_bfloat16*)copy, H);
    } else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

IL_EXPORT int il_cast_rows(const float* x, void* out, int out_kind, long long total, cudaStream_t stream) {
    if (total <= 0) return IL_OK;
    if (out_kind != IL_BF16) return IL_BAD_ARG;
    const long long g = (total + 255) / 256;
    IL_LAUNCH(cast_rows_kernel<__nv_bfloat16>, (int)(g > 148 * 16 ? 148 * 16 : g), 256, 0, stream, x, (__nv_bfloat16*)out, (size_t)total);
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// ---- several copies of the residual stream ("hyper-connections") ---------------------------------------------------------------
// A model may keep S copies x_1 .. x_S of the residual stream (streams [T, S, H], f32). A sublayer reads u = sum_s in[s] x_s
// through a norm, and its output y goes back as x_t <- sum_s mix[s, t] x_s + out[t] y, every new copy from the old ones.
// One kernel does what lies between two sublayers, for one row a block:
//   init (or null):   x_s = init[r] for every s           (the copies start as the embedding's output)
//   y (or null):      the write-back of the sublayer before, with mix [S, S] (from, to) and out [S]
//   in_next (or null): u = sum_t in_next[t] x_t, normed = u / sqrt(mean(u^2) + eps) * w   -> normed[r] (the next sublayer's input)
//   sum_out (or null): sum_out[r] = sum_t x_t              (the stream as one row: what the model's last norm reads)
// Everything is f32 but y (read) and normed (written), which have the compute dtype. S <= HC_MAX_STREAMS.
// Dynamic shared memory: H floats (u between its two passes).
#define HC_MAX_STREAMS 16
// (MAXS: the copies a thread holds in registers, 4, 8 or 16 - the smallest that takes S)
template <typename TA, int MAXS>
__global__ void hyper_step_kernel(float* streams, const float* init, const TA* y, const float* __restrict__ mix,
                                  const float* __restrict__ out_w, const float* __restrict__ in_next, const void* __restrict__ w, int w_kind,
                                  float eps, TA* __restrict__ normed, float* __restrict__ sum_out, int S, int H) {
    extern __shared__ float us[];
    __shared__ float red[32];
    __shared__ float s_mix[HC_MAX_STREAMS * HC_MAX_STREAMS], s_out[HC_MAX_STREAMS], s_in[HC_MAX_STREAMS];
    const int r = blockIdx.x;
    for (int i = threadIdx.x; i < S * S && y; i += blockDim.x) s_mix[i] = mix[i];
    if (threadIdx.x < S) {
        if (y) s_out[threadIdx.x] = out_w[threadIdx.x];
        if (in_next) s_in[threadIdx.x] = in_next[threadIdx.x];
    }
    il_pdl_wait();
    __syncthreads();
    float* xr = streams + (size_t)r * S * H;
    float ss = 0.f;
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        float x[MAXS], xn[MAXS];
#pragma unroll
        for (int s = 0; s < MAXS; ++s)
            if (s < S) x[s] = init ? init[(size_t)r * H + h] : xr[(size_t)s * H + h];
        if (y) {
            const float yv = il_to_f(y[(size_t)r * H + h]);
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) {
                    float a = 0.f;
#pragma unroll
                    for (int s = 0; s < MAXS; ++s)
                        if (s < S) a = fmaf(s_mix[s * S + t], x[s], a);
                    xn[t] = fmaf(s_out[t], yv, a);
                }
        } else {
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) xn[t] = x[t];
        }
        if (y || init) {
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) xr[(size_t)t * H + h] = xn[t];
        }
        if (sum_out) {
            float a = 0.f;
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) a += xn[t];
            sum_out[(size_t)r * H + h] = a;
        }
        if (in_next) {
            float u = 0.f;
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) u = fmaf(s_in[t], xn[t], u);
            us[h] = u;
            ss += u * u;
        }
    }
    if (!in_next) return;
    ss = il_block_sum(ss, red);
    const float rstd = 1.f / sqrtf(ss / (float)H + eps);
    for (int h = threadIdx.x; h < H; h += blockDim.x)
        normed[(size_t)r * H + h] = il_from_f<TA>(us[h] * rstd * il_load_any(w, w_kind, h));
}

// The same with four neighbouring columns a thread (H a multiple of 4, rows on 16-byte borders): 16-byte loads of the copies,
// all of a thread's loads issued before the first use. Every column's sums run in the scalar kernel's order.
template <typename TA, int MAXS>
__global__ void __launch_bounds__(256) hyper_step_vec_kernel(float* streams, const float* init, const TA* y, const float* __restrict__ mix,
                                                             const float* __restrict__ out_w, const float* __restrict__ in_next,
                                                             const void* __restrict__ w, int w_kind, float eps, TA* __restrict__ normed,
                                                             float* __restrict__ sum_out, int S, int H) {
    extern __shared__ __align__(16) float us[];
    __shared__ float red[32];
    __shared__ float s_mix[MAXS * MAXS], s_out[MAXS], s_in[MAXS];
    const int r = blockIdx.x;
    for (int i = threadIdx.x; i < S * S && y; i += blockDim.x) s_mix[i] = mix[i];
    if (threadIdx.x < S) {
        if (y) s_out[threadIdx.x] = out_w[threadIdx.x];
        if (in_next) s_in[threadIdx.x] = in_next[threadIdx.x];
    }
    il_pdl_wait();
    __syncthreads();
    float* xr = streams + (size_t)r * S * H;
    const int nv = H >> 2;
    float ss = 0.f;
    for (int v = threadIdx.x; v < nv; v += blockDim.x) {
        const int h = 4 * v;
        float4 x[MAXS], xn[MAXS];
        if (init) {
            const float4 e = ld4(init + (size_t)r * H + h);
#pragma unroll
            for (int s = 0; s < MAXS; ++s) x[s] = e;
        } else {
#pragma unroll
            for (int s = 0; s < MAXS; ++s)
                if (s < S) x[s] = ld4(xr + (size_t)s * H + h);
        }
        if (y) {
            const float4 yv = ld4(y + (size_t)r * H + h);
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) {
                    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                    for (int s = 0; s < MAXS; ++s)
                        if (s < S) {
                            const float m = s_mix[s * S + t];
                            a.x = fmaf(m, x[s].x, a.x), a.y = fmaf(m, x[s].y, a.y), a.z = fmaf(m, x[s].z, a.z), a.w = fmaf(m, x[s].w, a.w);
                        }
                    const float o = s_out[t];
                    xn[t] = make_float4(fmaf(o, yv.x, a.x), fmaf(o, yv.y, a.y), fmaf(o, yv.z, a.z), fmaf(o, yv.w, a.w));
                }
        } else {
#pragma unroll
            for (int t = 0; t < MAXS; ++t) xn[t] = x[t];
        }
        if (y || init) {
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) st4(xr + (size_t)t * H + h, xn[t]);
        }
        if (sum_out) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) a.x += xn[t].x, a.y += xn[t].y, a.z += xn[t].z, a.w += xn[t].w;
            st4(sum_out + (size_t)r * H + h, a);
        }
        if (in_next) {
            float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int t = 0; t < MAXS; ++t)
                if (t < S) {
                    const float m = s_in[t];
                    u.x = fmaf(m, xn[t].x, u.x), u.y = fmaf(m, xn[t].y, u.y), u.z = fmaf(m, xn[t].z, u.z), u.w = fmaf(m, xn[t].w, u.w);
                }
            *reinterpret_cast<float4*>(us + h) = u;
            ss += (u.x * u.x + u.y * u.y) + (u.z * u.z + u.w * u.w);
        }
    }
    if (!in_next) return;
    ss = il_block_sum(ss, red);
    const float rstd = 1.f / sqrtf(ss / (float)H + eps);
    for (int v = threadIdx.x; v < nv; v += blockDim.x) {
        const int h = 4 * v;
        const float4 u = *reinterpret_cast<const float4*>(us + h);
        const float4 wv = w_kind == IL_F32 ? ld4((const float*)w + h) : ld4((const __nv_bfloat16*)w + h);
        st4(normed + (size_t)r * H + h, make_float4(u.x * rstd * wv.x, u.y * rstd * wv.y, u.z * rstd * wv.z, u.w * rstd * wv.w));
    }
}

IL_EXPORT int il_hyper_step(float* streams, const float* init, const void* y, int act_kind, const float* mix, const float* out_w,
                            const float* in_next, const void* w, int w_kind, float eps, void* normed, float* sum_out, int S, int H, int T,
                            cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (S <= 0 || S > HC_MAX_STREAMS || H <= 0 || (y && (!mix || !out_w)) || (in_next && (!w || !normed))) return IL_BAD_ARG;
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return IL_UNSUPPORTED;
    const int threads = H >= 4096 ? 512 : H >= 1024 ? 256 : 128;
    // four columns a thread where rows are whole 16-byte pieces (and the copies fit the registers)
    const bool vec = (H & 3) == 0 && S <= 8 &&
                     (((uintptr_t)streams | (uintptr_t)init | (uintptr_t)y | (uintptr_t)w | (uintptr_t)normed | (uintptr_t)sum_out) & 15) == 0;
    const int vthreads = H >= 1024 ? 256 : H >= 512 ? 128 : 64;
#define HC_GO(TA, MAXS)                                                                                                                  \
    do {                                                                                                                                 \
        if (smem > 48 * 1024) cudaFuncSetAttribute(hyper_step_kernel<TA, MAXS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        IL_LAUNCH((hyper_step_kernel<TA, MAXS>), T, threads, smem, stream, streams, init, (const TA*)y, mix, out_w, in_next, w, w_kind, eps, \
                  (TA*)normed, sum_out, S, H);                                                                                           \
    } while (0)
#define HC_GOV(TA, MAXS)                                                                                                                     \
    do {                                                                                                                                     \
        if (smem > 48 * 1024) cudaFuncSetAttribute(hyper_step_vec_kernel<TA, MAXS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        IL_LAUNCH((hyper_step_vec_kernel<TA, MAXS>), T, vthreads, smem, stream, streams, init, (const TA*)y, mix, out_w, in_next, w, w_kind, \
                  eps, (TA*)normed, sum_out, S, H);                                                                                          \
    } while (0)
#define HC_PICK(TA)                                          \
    do {                                                     \
        if (vec && S <= 2) HC_GOV(TA, 2);                    \
        else if (vec && S <= 4) HC_GOV(TA, 4);               \
        else if (vec) HC_GOV(TA, 8);                         \
        else if (S <= 4) HC_GO(TA, 4);                       \
        else if (S <= 8) HC_GO(TA, 8);                       \
        else HC_GO(TA, 16);                                  \
    } while (0)
    if (act_kind == IL_F32) HC_PICK(float);
    else if (act_kind == IL_BF16) HC_PICK(__nv_bfloat16);
    else return IL_BAD_ARG;
#undef HC_PICK
#undef HC_GOV
#undef HC_GO
    IL_LAUNCH_CHECK();
    return IL_OK;
}
