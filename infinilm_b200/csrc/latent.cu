// The latent rows of a latent-attention mixer after their joint down-projection: per token, segment A of the projected
// row (the query latent) and segment B (the key/value latent) are each divided by their root mean square
// (x / sqrt(mean(x^2) + eps), f32) and multiplied by a weight vector. A goes to a row buffer for the query's
// up-projection; B - the only thing the mixer keeps of a token - is written to the token's slot of the paged cache,
// into the K plane and the V plane alike (the attention kernels read keys and values from the two planes; here they are
// the same vectors), and optionally to a row buffer.
// Cache layout of one layer: [page][0=K,1=V][kv head = 1][slot in page][width of B].
#include "common.cuh"

template <typename TA>
__global__ void latent_norm_store_kernel(const TA* proj, int row_stride, int off_a, int n_a, int off_b, int n_b,
                                         const void* __restrict__ w_a, const void* __restrict__ w_b, int w_kind, float eps,
                                         TA* __restrict__ out_a, TA* __restrict__ out_b, const int* __restrict__ tok_pos,
                                         const int* __restrict__ tok_entry, const int* __restrict__ block_table, int bt_stride,
                                         TA* __restrict__ cache, int page_size) {
    __shared__ float red[32];
    const int t = blockIdx.x;
    const int pos = tok_pos[t];
    TA* kdst = nullptr;
    size_t plane = 0;
    if (cache) {
        const int page = block_table[(size_t)tok_entry[t] * bt_stride + pos / page_size];
        if (page >= 0) {                          // the host reserves every page a step touches; never write elsewhere
            plane = (size_t)page_size * n_b;
            kdst = cache + (size_t)page * 2 * plane + (size_t)(pos % page_size) * n_b;
        }
    }
    il_pdl_begin();
    const TA* row = proj + (size_t)t * row_stride;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < n_a; i += blockDim.x) {
        const float x = il_to_f(row[off_a + i]);
        sa += x * x;
    }
    for (int i = threadIdx.x; i < n_b; i += blockDim.x) {
        const float x = il_to_f(row[off_b + i]);
        sb += x * x;
    }
    sa = il_block_sum(sa, red);
    sb = il_block_sum(sb, red);
    const float ra = n_a > 0 ? rsqrtf(sa / (float)n_a + eps) : 0.f, rb = rsqrtf(sb / (float)n_b + eps);
    for (int i = threadIdx.x; i < n_a; i += blockDim.x)
        out_a[(size_t)t * n_a + i] = il_from_f<TA>(il_to_f(row[off_a + i]) * ra * il_load_any(w_a, w_kind, i));
    for (int i = threadIdx.x; i < n_b; i += blockDim.x) {
        const TA v = il_from_f<TA>(il_to_f(row[off_b + i]) * rb * il_load_any(w_b, w_kind, i));
        if (out_b) out_b[(size_t)t * n_b + i] = v;
        if (kdst) {
            kdst[i] = v;
            kdst[plane + i] = v;
        }
    }
}

IL_EXPORT int il_latent_norm_store(const void* proj, int act_kind, int row_stride, int off_a, int n_a, int off_b, int n_b, const void* w_a,
                                   const void* w_b, int w_kind, float eps, void* out_a, void* out_b, const int* tok_pos,
                                   const int* tok_entry, const int* block_table, int bt_stride, void* cache, int page_size, int T,
                                   cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (n_b <= 0 || n_a < 0 || page_size <= 0 || (n_a > 0 && !out_a)) return IL_BAD_ARG;
    const int threads = (n_a + n_b) >= 1024 ? 256 : 128;
    if (act_kind == IL_F32)
        IL_LAUNCH(latent_norm_store_kernel<float>, T, threads, 0, stream, (const float*)proj, row_stride, off_a, n_a, off_b, n_b, w_a, w_b,
                  w_kind, eps, (float*)out_a, (float*)out_b, tok_pos, tok_entry, block_table, bt_stride, (float*)cache, page_size);
    else if (act_kind == IL_BF16)
        IL_LAUNCH(latent_norm_store_kernel<__nv_bfloat16>, T, threads, 0, stream, (const __nv_bfloat16*)proj, row_stride, off_a, n_a, off_b,
                  n_b, w_a, w_b, w_kind, eps, (__nv_bfloat16*)out_a, (__nv_bfloat16*)out_b, tok_pos, tok_entry, block_table, bt_stride,
                  (__nv_bfloat16*)cache, page_size);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// ---- a latent with a rotated key part beside it ---------------------------------------------------------------------------
// Per token: the latent (n_b columns at off_b) is divided by its root mean square and multiplied by w_b; the `rd` columns
// behind it are one key part for all heads, of which the first `rot` dimensions turn by pos * freq[i] (cosine and sine times
// mscale; pairs (2i, 2i + 1) or (i, i + rot / 2)) and the others pass. Latent, turned part and zeros up to hd columns go to the
// token's slot of the cache, K plane and V plane alike. Every head's query has its rotated part behind its other
// `qd` columns (head j at off_q + j * (qd + rd)): turned likewise, it goes to q_out[t, j * hd + n_b ..], zeros behind it; the
// columns in front of it are the business of the product that brings the query's other part to the latent's width.
// Angles are made in double precision and reduced to one turn before sine and cosine are taken in f32: an f32 product of
// position and frequency would be off by a rounding of the whole angle. Norm and rotation f32. One block per token.
#define LR_MAX_ROT 1024
__device__ __forceinline__ float2 lr_ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 lr_ld2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void lr_st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void lr_st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
template <typename TA, bool VEC>
__global__ void latent_rope_store_kernel(const TA* proj, int row_stride, int off_q, int nh, int qd, int off_b, int n_b, int rd, int hd,
                                         const void* __restrict__ w_b, int w_kind, float eps, int rot, const double* __restrict__ freq, float mscale,
                                         int interleaved, TA* __restrict__ q_out, const int* __restrict__ tok_pos, const int* __restrict__ tok_entry,
                                         const int* __restrict__ block_table, int bt_stride, TA* __restrict__ cache, int page_size) {
    __shared__ float red[32];
    __shared__ float s_cos[LR_MAX_ROT / 2], s_sin[LR_MAX_ROT / 2];
    const int t = blockIdx.x;
    const int pos = tok_pos[t];
    TA* kdst = nullptr;
    const size_t plane = (size_t)page_size * hd;
    if (cache) {
        const int page = block_table[(size_t)tok_entry[t] * bt_stride + pos / page_size];
        if (page >= 0) kdst = cache + (size_t)page * 2 * plane + (size_t)(pos % page_size) * hd;      // (the host reserves every page a step touches)
    }
    const int half = rot >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        double a = (double)pos * freq[i];
        a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
        float s, c;
        sincosf((float)a, &s, &c);
        s_sin[i] = s * mscale, s_cos[i] = c * mscale;
    }
    il_pdl_begin();
    const TA* row = proj + (size_t)t * row_stride;
    float sb = 0.f;
    for (int i = threadIdx.x; i < n_b; i += blockDim.x) {
        const float x = il_to_f(row[off_b + i]);
        sb += x * x;
    }
    sb = il_block_sum(sb, red);                   // (its barriers also stand between the writing and the reading of the angles)
    const float rb = 1.f / sqrtf(sb / (float)n_b + eps);
    auto turned = [&](const TA* x, int d) -> float {
        if (d >= rot) return il_to_f(x[d]);
        const bool low = interleaved ? !(d & 1) : d < half;
        const int i = interleaved ? d >> 1 : (low ? d : d - half), mate = interleaved ? d ^ 1 : (low ? d + half : d - half);
        const float a = il_to_f(x[d]), b = il_to_f(x[mate]), s = s_sin[i], c = s_cos[i];
        return low ? a * c - b * s : a * c + b * s;
    };
    const int tail = hd - n_b;
    if (VEC) {                                    // two neighbouring columns a thread: with interleaved pairs, a pair
        auto turned2 = [&](const TA* x, int d) -> float2 {
            if (d >= rd) return make_float2(0.f, 0.f);
            const float2 v = lr_ld2(x + d);
            if (d >= rot) return v;
            const float s = s_sin[d >> 1], c = s_cos[d >> 1];
            return make_float2(v.x * c - v.y * s, v.y * c + v.x * s);
        };
        if (kdst)
            for (int i = 2 * threadIdx.x; i < hd; i += 2 * blockDim.x) {
                float2 f;
                if (i < n_b) {
                    f = lr_ld2(row + off_b + i);
                    f.x *= rb * il_load_any(w_b, w_kind, i), f.y *= rb * il_load_any(w_b, w_kind, i + 1);
                } else {
                    f = turned2(row + off_b + n_b, i - n_b);
                }
                lr_st2(kdst + i, f);
                lr_st2(kdst + plane + i, f);
            }
        const int t2 = tail >> 1;
        for (int idx = threadIdx.x; idx < nh * t2; idx += blockDim.x) {
            const int j = idx / t2, d = 2 * (idx - j * t2);
            lr_st2(q_out + ((size_t)t * nh + j) * hd + n_b + d, turned2(row + off_q + (size_t)j * (qd + rd) + qd, d));
        }
        return;
    }
    if (kdst) {
        for (int i = threadIdx.x; i < hd; i += blockDim.x) {
            const float f = i < n_b ? il_to_f(row[off_b + i]) * rb * il_load_any(w_b, w_kind, i) : i < n_b + rd ? turned(row + off_b + n_b, i - n_b) : 0.f;
            const TA v = il_from_f<TA>(f);
            kdst[i] = v;
            kdst[plane + i] = v;
        }
    }
    for (int idx = threadIdx.x; idx < nh * tail; idx += blockDim.x) {
        const int j = idx / tail, d = idx - j * tail;
        q_out[((size_t)t * nh + j) * hd + n_b + d] = il_from_f<TA>(d < rd ? turned(row + off_q + (size_t)j * (qd + rd) + qd, d) : 0.f);
    }
}

IL_EXPORT int il_latent_rope_store(const void* proj, int act_kind, int row_stride, int off_q, int nh, int qd, int off_b, int n_b, int rd, int hd,
                                   const void* w_b, int w_kind, float eps, int rot, const double* freq, float mscale, int interleaved, void* q_out,
                                   const int* tok_pos, const int* tok_entry, const int* block_table, int bt_stride, void* cache, int page_size, int T,
                                   cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (nh <= 0 || qd < 0 || n_b <= 0 || rd < 0 || hd < n_b + rd || page_size <= 0 || !w_b || !q_out) return IL_BAD_ARG;
    if (rot < 0 || (rot & 1) || rot > rd || (rot > 0 && !freq)) return IL_BAD_ARG;
    if (rot > LR_MAX_ROT) return IL_UNSUPPORTED;
    const int work = hd + nh * (hd - n_b);
    const int threads = work >= 1024 ? 256 : 128;
    // two columns a thread: every segment starts on an even column of rows of even length, pairs are neighbours (or nothing turns)
    const bool vec = ((row_stride | off_q | qd | rd | off_b | n_b | hd) & 1) == 0 && (interleaved || rot == 0) &&
                     (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)cache) & 7) == 0;
#define LR_GO(TA, VEC)                                                                                                                      \
    IL_LAUNCH((latent_rope_store_kernel<TA, VEC>), T, threads, 0, stream, (const TA*)proj, row_stride, off_q, nh, qd, off_b, n_b, rd, hd, w_b, \
              w_kind, eps, rot, freq, mscale, interleaved, (TA*)q_out, tok_pos, tok_entry, block_table, bt_stride, (TA*)cache, page_size)
    if (act_kind == IL_F32) {
        if (vec) LR_GO(float, true); else LR_GO(float, false);
    } else if (act_kind == IL_BF16) {
        if (vec) LR_GO(__nv_bfloat16, true); else LR_GO(__nv_bfloat16, false);
    } else
        return IL_BAD_ARG;
#undef LR_GO
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// y[t, c] *= sigmoid(g[t, c]) for rows of `n` columns (y contiguous, g with a row stride): the heads' gate where the product
// before it was the library's and has no epilogue of ours.
template <typename TA>
__global__ void sigmoid_gate_kernel(TA* y, const TA* g, int ldg, int n, long long total) {
    il_pdl_begin();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n;
        const int c = (int)(i - t * n);
        const float gt = il_to_f(g[(size_t)t * ldg + c]);
        y[i] = il_from_f<TA>(il_to_f(y[i]) / (1.f + expf(-gt)));
    }
}

IL_EXPORT int il_sigmoid_gate(void* y, int act_kind, const void* g, int ldg, int T, int n, cudaStream_t stream) {
    if (T <= 0 || n <= 0) return IL_OK;
    const long long total = (long long)T * n;
    const int blocks = (int)((total + 255) / 256 > 148 * 16 ? 148 * 16 : (total + 255) / 256);
    if (act_kind == IL_F32)
        IL_LAUNCH(sigmoid_gate_kernel<float>, blocks, 256, 0, stream, (float*)y, (const float*)g, ldg, n, total);
    else if (act_kind == IL_BF16)
        IL_LAUNCH(sigmoid_gate_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)y, (const __nv_bfloat16*)g, ldg, n, total);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}
