// Shared helpers of the sm_100a kernels: element conversion, reductions, launch checks.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define IL_EXPORT extern "C" __attribute__((visibility("default")))

// Element kinds passed from the host as integers.
enum { IL_F32 = 0, IL_BF16 = 1 };

// Error codes returned by the entry points (0 = launched).
enum { IL_OK = 0, IL_BAD_ARG = -1, IL_UNSUPPORTED = -2 };

#define IL_LAUNCH_CHECK()                                         \
    do {                                                          \
        cudaError_t e__ = cudaGetLastError();                     \
        if (e__ != cudaSuccess) return 1000 + (int)e__;           \
    } while (0)

__device__ __forceinline__ float il_to_f(float x) { return x; }
__device__ __forceinline__ float il_to_f(__nv_bfloat16 x) { return __bfloat162float(x); }

template <typename T> __device__ __forceinline__ T il_from_f(float x);
template <> __device__ __forceinline__ float il_from_f<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 il_from_f<__nv_bfloat16>(float x) {
    return __float2bfloat16_rn(x);
}

// Reads element i of a vector stored as f32 or bf16.
__device__ __forceinline__ float il_load_any(const void* p, int kind, size_t i) {
    return kind == IL_F32 ? ((const float*)p)[i] : __bfloat162float(((const __nv_bfloat16*)p)[i]);
}

__device__ __forceinline__ float il_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float il_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. `sh` holds 32 floats.
__device__ __forceinline__ float il_block_sum(float v, float* sh) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nw = (blockDim.x + 31) >> 5;
    v = il_warp_sum(v);
    __syncthreads();
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    float t = (lane < nw) ? sh[lane] : 0.f;
    t = il_warp_sum(t);
    return t;
}
__device__ __forceinline__ float il_block_max(float v, float* sh) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nw = (blockDim.x + 31) >> 5;
    v = il_warp_max(v);
    __syncthreads();
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    float t = (lane < nw) ? sh[lane] : -INFINITY;
    t = il_warp_max(t);
    return t;
}

// The lowest position a query at position `pos` sees, for the one integer by which the attention kernels take their mask:
// window > 0: a sliding window, positions pos - window + 1 .. pos; window < 0: runs ("chunks") of -window positions counted
// from position 0 of the sequence, a query seeing its own run only, from the run's first position to itself; 0: every
// position up to pos. It never decreases with pos, so the lowest bound of a tile of consecutive queries is its first query's.
__device__ __forceinline__ int il_mask_lo(int pos, int window) {
    if (window > 0) return pos - window + 1 > 0 ? pos - window + 1 : 0;
    if (window < 0 && pos > 0) return pos - pos % (-window);
    return 0;
}

// SiLU(g) * u for the bfloat16 path: exponential and division by the fast units (relative error near 2^-21, far below a
// bfloat16 step). The decode product's epilogue and the SwiGLU kernel both use it, so a token's activation does not
// depend on which of the two computed it. The float32 path keeps expf and a true division.
__device__ __forceinline__ float il_silu_mul_fast(float g, float u) { return __fmul_rn(__fdividef(g, __fadd_rn(1.f, __expf(-g))), u); }

// gelu_tanh(g) * u with gelu_tanh(z) = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))): the other gate of a gated feed-forward.
// 0.5 (1 + tanh(a)) = 1 / (1 + exp(-2a)); the bfloat16 path takes the fast exponential and division, as the SiLU form does.
__device__ __forceinline__ float il_gelu_tanh_mul_fast(float g, float u) {
    const float a = 0.7978845608028654f * __fmaf_rn(0.044715f * g * g, g, g);
    return __fmul_rn(__fdividef(g, __fadd_rn(1.f, __expf(-2.f * a))), u);
}
__device__ __forceinline__ float il_gelu_tanh_mul(float g, float u) {
    const float a = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return 0.5f * g * (1.f + tanhf(a)) * u;
}
// A clamped gate: g' = min(g, limit), u' = u kept within -limit .. limit, result g' * sigmoid(alpha g') * (u' + 1).
__device__ __forceinline__ float il_clamped_glu_fast(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fmul_rn(__fdividef(g, __fadd_rn(1.f, __expf(__fmul_rn(-alpha, g)))), __fadd_rn(u, 1.f));
}
__device__ __forceinline__ float il_clamped_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
// The gate of a gated feed-forward by number: 1 SiLU, 2 the tanh form of GELU, 3 the clamped gate (which has two numbers
// of its own, limit and alpha).
// Activations of a product that stand on their own: 4 the square of relu; 5 the tanh form of GELU times a row of a table that
// the row's token names.
enum { IL_ACT_SILU = 1, IL_ACT_GELU_TANH = 2, IL_ACT_CLAMPED = 3, IL_ACT_RELU2 = 4, IL_ACT_GELU_TANH_ROW = 5 };
__device__ __forceinline__ float il_relu2(float z) {
    z = fmaxf(z, 0.f);
    return __fmul_rn(z, z);
}

// 1 / (1 + 2^-v), the logistic function of v / log2(e): -inf gives 0. Exponential and reciprocal by the fast units (relative
// error near 2^-21).
__device__ __forceinline__ float il_sigmoid_log2_fast(float v) {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(-v));
    return __fdividef(1.f, 1.f + fminf(e, 1e38f));
}

// A capped score in the exponent's base: c * tanh(x) where 2^(k s) = e^(2x), so k = 2 log2(e) scale / cap and c = cap log2(e).
// tanh(x) = 1 - 2 / (1 + e^(2x)); exponential and reciprocal by the fast units (absolute error near 2^-21 c).
__device__ __forceinline__ float il_cap_log2_fast(float s, float k, float c) {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(s * k));
    return fmaf(-2.f * c, __fdividef(1.f, 1.f + fminf(e, 1e38f)), c);
}

// Two f32 at once (the packed forms of sm_100: one instruction for both, each rounded as the single form rounds).
typedef unsigned long long il_f2;
__device__ __forceinline__ il_f2 il_f2_make(float lo, float hi) {
    il_f2 v;
    asm("mov.b64 %0, {%1, %2};\n" : "=l"(v) : "f"(lo), "f"(hi));
    return v;
}
__device__ __forceinline__ void il_f2_get(il_f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;\n" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ il_f2 il_f2_fma(il_f2 a, il_f2 b, il_f2 c) {
    il_f2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ il_f2 il_f2_mul(il_f2 a, il_f2 b) {
    il_f2 d;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ il_f2 il_f2_add(il_f2 a, il_f2 b) {
    il_f2 d;
    asm("add.rn.f32x2 %0, %1, %2;\n" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ il_f2 il_f2_dup(float x) { return il_f2_make(x, x); }

// The same as il_cap_log2_fast, two scores at once, for arguments |y| <= IL_CAP_SMALL with y = s kx and 2^(k s) = e^(2y):
// tanh(y) = y P(y^2), P of degree 5 fitted to tanh(y) / y on [0, IL_CAP_SMALL^2] (weighted least squares, reweighted until the
// relative error levels out: 3e-8; with f32 arithmetic 1.6e-7). p[i]: the coefficients times c.
constexpr float IL_CAP_SMALL = 0.75f;
struct IlCapPoly { il_f2 kx, p[6]; };
__device__ __forceinline__ IlCapPoly il_cap_poly(float kx, float c) {
    IlCapPoly q;
    q.kx = il_f2_dup(kx);
    q.p[0] = il_f2_dup(c);
    q.p[1] = il_f2_dup(c * -0.33332958817481995f);
    q.p[2] = il_f2_dup(c * 0.1332540661096573f);
    q.p[3] = il_f2_dup(c * -0.05334443226456642f);
    q.p[4] = il_f2_dup(c * 0.01958290860056877f);
    q.p[5] = il_f2_dup(c * -0.004716257564723492f);
    return q;
}
__device__ __forceinline__ il_f2 il_cap_log2_small(il_f2 s, const IlCapPoly& q) {
    const il_f2 y = il_f2_mul(s, q.kx), z = il_f2_mul(y, y);
    il_f2 p = il_f2_fma(z, q.p[5], q.p[4]);
    p = il_f2_fma(z, p, q.p[3]);
    p = il_f2_fma(z, p, q.p[2]);
    p = il_f2_fma(z, p, q.p[1]);
    p = il_f2_fma(z, p, q.p[0]);
    return il_f2_mul(y, p);
}

// ---- programmatic dependent launch --------------------------------------------------------------
// Kernels of the decode path are launched so that the next kernel in the stream may become resident
// while this one drains (INFINILM_B200_PDL=0 turns it off). A kernel waits for its predecessor to have
// finished and flushed (il_pdl_begin) before it touches anything another kernel produces or reads, and
// lets its successor in once its main loop is over (il_pdl_tail; a kernel without one does so by ending).
// Both are no-ops in a kernel that was launched the ordinary way. A kernel may do, before its wait, whatever does not
// depend on its predecessor (read weights, step descriptors, cache pages of earlier tokens). What the predecessor
// writes must then NOT be read through a `const __restrict__` pointer: such loads count as read-only data for the
// whole kernel (ld.global.nc) and were seen scheduled above the wait, which replayed graphs then showed as wrong tokens. Measured on the 8B decode step at
// batch 8: 3.65 ms so, 3.70 ms without; with every kernel letting its successor in at its very start
// (IL_PDL_MODE 0) 6.7 ms, because waiting blocks of later kernels then crowd the SMs.
__device__ __forceinline__ void il_pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }
__device__ __forceinline__ void il_pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
// Where a kernel lets its successor in: IL_PDL_MODE 0 at its start, 1 after its main loop, 2 only by ending.
#ifndef IL_PDL_MODE
#define IL_PDL_MODE 1
#endif
__device__ __forceinline__ void il_pdl_begin() {
    if (IL_PDL_MODE == 0) il_pdl_launch_dependents();
    il_pdl_wait();
}
__device__ __forceinline__ void il_pdl_tail() {
    if (IL_PDL_MODE == 1) il_pdl_launch_dependents();
}

#include <cstdlib>
static inline bool il_pdl_enabled() {
    static int on = -1;
    if (on < 0) {
        const char* e = getenv("INFINILM_B200_PDL");
        on = (e && e[0] == '0') ? 0 : 1;
    }
    return on == 1;
}

template <typename... KArgs, typename... Args>
static inline cudaError_t il_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = il_pdl_enabled() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}
#define IL_LAUNCH(kernel, grid, block, smem, stream, ...)                                                \
    do {                                                                                                   \
        cudaError_t e__ = il_launch(kernel, dim3(grid), dim3(block), (size_t)(smem), stream, __VA_ARGS__); \
        if (e__ != cudaSuccess) return 1000 + (int)e__;                                                   \
    } while (0)
