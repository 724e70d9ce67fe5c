// What stands between an attention mixer's projection and its attention when queries and keys are normed per head and
// positions do not rotate anything: per token and head
//   q_h <- q_h / sqrt(mean(q_h^2) + eps) * w_q * temp(pos)        temp(p) = 1 + coef * ln(floor((p + 1) / every) + 1)  (or 1)
//   k_g <- k_g / sqrt(mean(k_g^2) + eps) * w_k                     -> the token's slot of the cache, K plane
//   v_g                                                            -> the V plane: the value columns, or the key columns as
//                                                                     projected, before the norm (a mixer whose values are its keys)
// all in f32 - with `bias` (f32, one per column of the projection, or null) added to q, k and v first; w_q and w_k are one vector each, shared by the heads. Heads are laid out at hd >= key size, value size: the
// surplus columns are written as zeros (a zero column adds nothing to a score). A mixer that reads another layer's cache
// gives no key columns (k_off < 0): only its queries are normed.
// `first` (VMIX): the values are blended with another row's, v_g <- (1 - mix) v_g + mix first[t, g * dv ..], in f32, before they
// are rounded into the cache.
// Cache layout of one layer: [page][0=K,1=V][kv head][slot in page][hd]. One warp per (token, head).
#include "common.cuh"

// four neighbouring values at a time (16 bytes of f32, 8 of bfloat16)
__device__ __forceinline__ float4 qn_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 qn_ld4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void qn_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void qn_st4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float4 qn_b4(float4 a, const float* b, int d) {      // a + the biases of its four columns
    a.x += b[d], a.y += b[d + 1], a.z += b[d + 2], a.w += b[d + 3];
    return a;
}
__device__ __forceinline__ float4 qn_w4(const void* w, int kind, int d) {
    return make_float4(il_load_any(w, kind, d), il_load_any(w, kind, d + 1), il_load_any(w, kind, d + 2), il_load_any(w, kind, d + 3));
}

// The form for sizes and offsets that are multiples of 4 (rows, segments and heads then start on 8- or 16-byte borders): the
// lanes hold 4 neighbouring columns instead of every 32nd (the sum of squares is gathered in another order). VEC 1 is the form for
// every size.
template <typename TA, int VEC, bool BIAS, bool VMIX>
__global__ void qk_norm_store_kernel(const TA* proj, int ld, int q_off, int k_off, int v_off, int nh, int nkv, int dk, int dv, int hd,
                                     const void* __restrict__ wq, const void* __restrict__ wk, int w_kind, float eps, float t_coef,
                                     int t_every, TA* __restrict__ q_out, const int* __restrict__ tok_pos,
                                     const int* __restrict__ tok_entry, const int* __restrict__ block_table, int bt_stride,
                                     TA* __restrict__ cache, int page_size, int T,
                                     const float* __restrict__ bias, const TA* first, int ld_first, float mix) {
    const int jobs = nh + (k_off >= 0 ? 2 * nkv : 0);
    const long long wid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (wid >= (long long)T * jobs) return;
    const int t = (int)(wid / jobs), j = (int)(wid - (long long)t * jobs);
    const int pos = tok_pos[t];
    il_pdl_wait();
    const TA* row = proj + (size_t)t * ld;
    if (j < nh) {                                 // a query head
        const TA* x = row + q_off + (size_t)j * dk;
        const float* bx = BIAS ? bias + q_off + (size_t)j * dk : nullptr;
        TA* o = q_out + ((size_t)t * nh + j) * hd;
        float ss = 0.f;
        if (VEC == 4) {
            for (int d = 4 * lane; d < dk; d += 128) {
                float4 a = qn_ld4(x + d);
                if (BIAS) a = qn_b4(a, bx, d);
                ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
            }
        } else {
            for (int d = lane; d < dk; d += 32) {
                float a = il_to_f(x[d]);
                if (BIAS) a += bx[d];
                ss += a * a;
            }
        }
        ss = il_warp_sum(ss);
        float r = 1.f / sqrtf(ss / (float)dk + eps);
        if (t_every > 0) r *= 1.f + t_coef * logf((float)((pos + 1) / t_every) + 1.f);
        if (VEC == 4) {
            for (int d = 4 * lane; d < hd; d += 128) {
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                if (d < dk) {
                    const float4 w = qn_w4(wq, w_kind, d);
                    a = qn_ld4(x + d);
                    if (BIAS) a = qn_b4(a, bx, d);
                    a.x *= r * w.x, a.y *= r * w.y, a.z *= r * w.z, a.w *= r * w.w;
                }
                qn_st4(o + d, a);
            }
        } else {
            for (int d = lane; d < hd; d += 32) o[d] = il_from_f<TA>(d < dk ? (BIAS ? il_to_f(x[d]) + bx[d] : il_to_f(x[d])) * r * il_load_any(wq, w_kind, d) : 0.f);
        }
        return;
    }
    if (!cache) return;
    const int page = block_table[(size_t)tok_entry[t] * bt_stride + pos / page_size];
    if (page < 0) return;                         // the host reserves every page a step touches; never write elsewhere
    const bool is_k = j < nh + nkv;
    const int g = is_k ? j - nh : j - nh - nkv;
    TA* dst = cache + (((size_t)page * 2 + (is_k ? 0 : 1)) * nkv + g) * (size_t)page_size * hd + (size_t)(pos % page_size) * hd;
    if (is_k) {
        const TA* x = row + k_off + (size_t)g * dk;
        const float* bx = BIAS ? bias + k_off + (size_t)g * dk : nullptr;
        float ss = 0.f;
        if (VEC == 4) {
            for (int d = 4 * lane; d < dk; d += 128) {
                float4 a = qn_ld4(x + d);
                if (BIAS) a = qn_b4(a, bx, d);
                ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
            }
        } else {
            for (int d = lane; d < dk; d += 32) {
                float a = il_to_f(x[d]);
                if (BIAS) a += bx[d];
                ss += a * a;
            }
        }
        ss = il_warp_sum(ss);
        const float r = 1.f / sqrtf(ss / (float)dk + eps);
        if (VEC == 4) {
            for (int d = 4 * lane; d < hd; d += 128) {
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                if (d < dk) {
                    const float4 w = qn_w4(wk, w_kind, d);
                    a = qn_ld4(x + d);
                    if (BIAS) a = qn_b4(a, bx, d);
                    a.x *= r * w.x, a.y *= r * w.y, a.z *= r * w.z, a.w *= r * w.w;
                }
                qn_st4(dst + d, a);
            }
        } else {
            for (int d = lane; d < hd; d += 32) dst[d] = il_from_f<TA>(d < dk ? (BIAS ? il_to_f(x[d]) + bx[d] : il_to_f(x[d])) * r * il_load_any(wk, w_kind, d) : 0.f);
        }
    } else {
        const TA* x = row + v_off + (size_t)g * dv;
        const float* bx = BIAS ? bias + v_off + (size_t)g * dv : nullptr;
        if (VMIX) {
            const TA* y = first + (size_t)t * ld_first + (size_t)g * dv;
            const float keep = 1.f - mix;
            if (VEC == 4) {
                for (int d = 4 * lane; d < hd; d += 128) {
                    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (d < dv) {
                        const float4 b = qn_ld4(y + d);
                        a = qn_ld4(x + d);
                        if (BIAS) a = qn_b4(a, bx, d);
                        a.x = fmaf(mix, b.x, keep * a.x), a.y = fmaf(mix, b.y, keep * a.y), a.z = fmaf(mix, b.z, keep * a.z), a.w = fmaf(mix, b.w, keep * a.w);
                    }
                    qn_st4(dst + d, a);
                }
            } else {
                for (int d = lane; d < hd; d += 32)
                    dst[d] = il_from_f<TA>(d < dv ? fmaf(mix, il_to_f(y[d]), keep * (BIAS ? il_to_f(x[d]) + bx[d] : il_to_f(x[d]))) : 0.f);
            }
        } else if (VEC == 4) {
            for (int d = 4 * lane; d < hd; d += 128) qn_st4(dst + d, d < dv ? (BIAS ? qn_b4(qn_ld4(x + d), bx, d) : qn_ld4(x + d)) : make_float4(0.f, 0.f, 0.f, 0.f));
        } else {
            for (int d = lane; d < hd; d += 32) dst[d] = d < dv ? (BIAS ? il_from_f<TA>(il_to_f(x[d]) + bx[d]) : x[d]) : il_from_f<TA>(0.f);
        }
    }
}

IL_EXPORT int il_qk_norm_store(const void* proj, int act_kind, int ld, int q_off, int k_off, int v_off, int nh, int nkv, int dk, int dv, int hd,
                               const void* wq, const void* wk, int w_kind, float eps, float t_coef, int t_every, void* q_out,
                               const int* tok_pos, const int* tok_entry, const int* block_table, int bt_stride, void* cache, int page_size,
                               int T, const float* bias, const void* first, int ld_first, float mix, cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (nh <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || hd < dk || hd < dv || page_size <= 0 || !wq || (k_off >= 0 && !wk)) return IL_BAD_ARG;
    const long long warps = (long long)T * (nh + (k_off >= 0 ? 2 * nkv : 0));
    const long long blocks = (warps + 3) / 4;
    if (blocks > 0x7fffffffLL) return IL_UNSUPPORTED;
    if (act_kind != IL_F32 && act_kind != IL_BF16) return IL_BAD_ARG;
    const bool vec = ((ld | q_off | v_off | dk | dv | hd) & 3) == 0 && (k_off < 0 || (k_off & 3) == 0) &&
                     (!first || ((ld_first & 3) == 0 && ((uintptr_t)first & (act_kind == IL_F32 ? 15 : 7)) == 0)) && (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)cache) & 15) == 0;
#define QN_GO1(TA, VEC, BIAS, VMIX)                                                                                                            \
    IL_LAUNCH((qk_norm_store_kernel<TA, VEC, BIAS, VMIX>), (int)blocks, 128, 0, stream, (const TA*)proj, ld, q_off, k_off, v_off, nh, nkv, dk, dv, hd, wq, wk, \
              w_kind, eps, t_coef, t_every, (TA*)q_out, tok_pos, tok_entry, block_table, bt_stride, (TA*)cache, page_size, T, bias, \
              (const TA*)first, ld_first, mix)
#define QN_GO(TA, VEC)                                                                 \
    do {                                                                               \
        if (bias && first) QN_GO1(TA, VEC, true, true);                                \
        else if (first) QN_GO1(TA, VEC, false, true);                                  \
        else if (bias) QN_GO1(TA, VEC, true, false);                                   \
        else QN_GO1(TA, VEC, false, false);                                            \
    } while (0)
    if (act_kind == IL_F32) {
        if (vec) QN_GO(float, 4); else QN_GO(float, 1);
    } else {
        if (vec) QN_GO(__nv_bfloat16, 4); else QN_GO(__nv_bfloat16, 1);
    }
#undef QN_GO
#undef QN_GO1
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// out[t, h * dv + c] = y[t, h * hd + c] * sigmoid(gate[t, g_off + h * dv + c]) for c < dv <= hd: a gate per output column,
// and heads that were laid out at hd columns come out packed. Without a gate only the packing is done.
template <typename TA>
__global__ void gate_pack_kernel(const TA* y, int hd, const TA* gate, int ldg, int g_off, TA* __restrict__ out, int nh, int dv, int T) {
    il_pdl_wait();
    const int n = nh * dv;
    const long long total = (long long)T * n;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n;
        const int jc = (int)(i - t * n), h = jc / dv, c = jc - h * dv;
        float v = il_to_f(y[((size_t)t * nh + h) * hd + c]);
        if (gate) v = v / (1.f + expf(-il_to_f(gate[(size_t)t * ldg + g_off + jc])));
        out[i] = il_from_f<TA>(v);
    }
}

template <typename TA>
__global__ void gate_pack4_kernel(const TA* y, int hd, const TA* gate, int ldg, int g_off, TA* __restrict__ out, int nh, int dv, int T) {
    il_pdl_wait();
    const int n4 = (nh * dv) >> 2;
    const long long total = (long long)T * n4;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n4;
        const int jc = (int)(i - t * n4) << 2, h = jc / dv, c = jc - h * dv;
        float4 v = qn_ld4(y + ((size_t)t * nh + h) * hd + c);
        if (gate) {
            const float4 z = qn_ld4(gate + (size_t)t * ldg + g_off + jc);
            v.x = v.x / (1.f + expf(-z.x)), v.y = v.y / (1.f + expf(-z.y)), v.z = v.z / (1.f + expf(-z.z)), v.w = v.w / (1.f + expf(-z.w));
        }
        qn_st4(out + (size_t)t * nh * dv + jc, v);
    }
}

IL_EXPORT int il_gate_pack(const void* y, int act_kind, int hd, const void* gate, int ldg, int g_off, void* out, int nh, int dv, int T,
                           cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (nh <= 0 || dv <= 0 || dv > hd) return IL_BAD_ARG;
    if (act_kind != IL_F32 && act_kind != IL_BF16) return IL_BAD_ARG;
    if (((hd | dv | ldg | g_off) & 3) == 0 && (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)out) & 15) == 0) {
        const long long g4 = ((long long)T * nh * dv / 4 + 255) / 256;
        const int blocks4 = (int)(g4 > 148 * 16 ? 148 * 16 : g4);
        if (act_kind == IL_F32)
            IL_LAUNCH(gate_pack4_kernel<float>, blocks4, 256, 0, stream, (const float*)y, hd, (const float*)gate, ldg, g_off, (float*)out, nh, dv, T);
        else
            IL_LAUNCH(gate_pack4_kernel<__nv_bfloat16>, blocks4, 256, 0, stream, (const __nv_bfloat16*)y, hd, (const __nv_bfloat16*)gate, ldg,
                      g_off, (__nv_bfloat16*)out, nh, dv, T);
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    const long long g = ((long long)T * nh * dv + 255) / 256;
    const int blocks = (int)(g > 148 * 16 ? 148 * 16 : g);
    if (act_kind == IL_F32)
        IL_LAUNCH(gate_pack_kernel<float>, blocks, 256, 0, stream, (const float*)y, hd, (const float*)gate, ldg, g_off, (float*)out, nh, dv, T);
    else if (act_kind == IL_BF16)
        IL_LAUNCH(gate_pack_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const __nv_bfloat16*)y, hd, (const __nv_bfloat16*)gate, ldg, g_off,
                  (__nv_bfloat16*)out, nh, dv, T);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}

// ---- queries and keys normed over the whole projection, then rotated ---------------------------------------------------
// Per token: the nh * dk query columns are divided by THEIR root mean square, all heads together, and multiplied by a
// weight of that many entries; the nkv * dk key columns likewise. Then, of every head, the first `rot` dimensions turn by
// angle = pos * inv_freq[i], dimension i paired with i + rot / 2 ((u, v) -> (u cos - v sin, v cos + u sin)); the others
// pass. Queries go to q_out [T, nh * hd], keys to the K plane of the token's cache slot, values to the V plane, heads laid
// out at hd columns with the surplus zero. k_off < 0: no keys or values (the mixer reads another layer's cache).
// Sums of squares, angles and the rotation are f32. One block per token.
#define QR_MAX_ROT 1024
template <typename TA>
__global__ void qk_rows_norm_rope_store_kernel(const TA* proj, int ld, int q_off, int k_off, int v_off, int nh, int nkv, int dk, int dv, int hd,
                                               const void* __restrict__ wq, const void* __restrict__ wk, int w_kind, float eps, int rot,
                                               const float* __restrict__ inv_freq, TA* __restrict__ q_out,
                                               const int* __restrict__ tok_pos, const int* __restrict__ tok_entry,
                                               const int* __restrict__ block_table, int bt_stride, TA* __restrict__ cache, int page_size) {
    __shared__ float red[32];
    __shared__ float s_cos[QR_MAX_ROT / 2], s_sin[QR_MAX_ROT / 2];      // the token's angles, once for all its heads
    const int t = blockIdx.x;
    const int pos = tok_pos[t];
    const bool has_k = k_off >= 0;
    int page = -1;
    if (has_k && cache) page = block_table[(size_t)tok_entry[t] * bt_stride + pos / page_size];
    for (int i = threadIdx.x; i < (rot >> 1); i += blockDim.x) sincosf((float)pos * inv_freq[i], &s_sin[i], &s_cos[i]);
    il_pdl_wait();
    const TA* row = proj + (size_t)t * ld;
    const int nq = nh * dk, nk = nkv * dk, half = rot >> 1;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
        const float x = il_to_f(row[q_off + i]);
        sq += x * x;
    }
    if (has_k)
        for (int i = threadIdx.x; i < nk; i += blockDim.x) {
            const float x = il_to_f(row[k_off + i]);
            sk += x * x;
        }
    sq = il_block_sum(sq, red);
    sk = il_block_sum(sk, red);
    const float rq = 1.f / sqrtf(sq / (float)nq + eps), rk = has_k ? 1.f / sqrtf(sk / (float)nk + eps) : 0.f;
    // element d of head j of a normed and weighted projection, rotated
    auto turned = [&](const TA* x, const void* w, float r, int j, int d) -> float {
        const int c = j * dk + d;
        const float a = il_to_f(x[c]) * r * il_load_any(w, w_kind, c);
        if (d >= rot) return a;
        const bool low = d < half;
        const int c2 = low ? c + half : c - half;
        const float b = il_to_f(x[c2]) * r * il_load_any(w, w_kind, c2);
        const float s = s_sin[low ? d : d - half], co = s_cos[low ? d : d - half];
        return low ? a * co - b * s : a * co + b * s;
    };
    for (int idx = threadIdx.x; idx < nh * hd; idx += blockDim.x) {
        const int j = idx / hd, d = idx - j * hd;
        q_out[(size_t)t * nh * hd + idx] = il_from_f<TA>(d < dk ? turned(row + q_off, wq, rq, j, d) : 0.f);
    }
    if (page < 0) return;                         // no keys of its own, or no slot (the host reserves every page a step touches)
    const size_t plane = (size_t)nkv * page_size * hd;
    TA* kdst = cache + (size_t)page * 2 * plane + (size_t)(pos % page_size) * hd;
    for (int idx = threadIdx.x; idx < nkv * hd; idx += blockDim.x) {
        const int g = idx / hd, d = idx - g * hd;
        const size_t at = (size_t)g * page_size * hd + d;
        kdst[at] = il_from_f<TA>(d < dk ? turned(row + k_off, wk, rk, g, d) : 0.f);
        kdst[plane + at] = d < dv ? row[v_off + g * dv + d] : il_from_f<TA>(0.f);
    }
}

// The same with neighbouring dimensions as pairs (2i turns with 2i + 1) and angles made in double precision, reduced to one turn
// before sine and cosine are taken in f32 (an f32 product of position and frequency would be off by a rounding of the whole
// angle). VEC 4: four neighbouring columns - two pairs - a thread, where sizes and offsets are multiples of 4. One block per
// token.
template <typename TA, int VEC>
__global__ void qk_rows_norm_pairs_store_kernel(const TA* proj, int ld, int q_off, int k_off, int v_off, int nh, int nkv, int dk, int dv, int hd,
                                                const void* __restrict__ wq, const void* __restrict__ wk, int w_kind, float eps, int rot,
                                                const double* __restrict__ freq, TA* __restrict__ q_out, const int* __restrict__ tok_pos,
                                                const int* __restrict__ tok_entry, const int* __restrict__ block_table, int bt_stride,
                                                TA* __restrict__ cache, int page_size) {
    __shared__ float red[2][32];
    __shared__ float s_cos[QR_MAX_ROT / 2], s_sin[QR_MAX_ROT / 2];
    const int t = blockIdx.x;
    const int pos = tok_pos[t];
    const bool has_k = k_off >= 0;
    int page = -1;
    if (has_k && cache) page = block_table[(size_t)tok_entry[t] * bt_stride + pos / page_size];
    for (int i = threadIdx.x; i < (rot >> 1); i += blockDim.x) {
        double a = (double)pos * freq[i];
        a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
        sincosf((float)a, &s_sin[i], &s_cos[i]);
    }
    il_pdl_wait();
    const TA* row = proj + (size_t)t * ld;
    const int nq = nh * dk, nk = has_k ? nkv * dk : 0;
    float sq = 0.f, sk = 0.f;
    if (VEC == 4) {
        for (int i = 4 * threadIdx.x; i < nq; i += 4 * blockDim.x) {
            const float4 x = qn_ld4(row + q_off + i);
            sq += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
        }
        for (int i = 4 * threadIdx.x; i < nk; i += 4 * blockDim.x) {
            const float4 x = qn_ld4(row + k_off + i);
            sk += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
        }
    } else {
        for (int i = threadIdx.x; i < nq; i += blockDim.x) {
            const float x = il_to_f(row[q_off + i]);
            sq += x * x;
        }
        for (int i = threadIdx.x; i < nk; i += blockDim.x) {
            const float x = il_to_f(row[k_off + i]);
            sk += x * x;
        }
    }
    sq = il_warp_sum(sq), sk = il_warp_sum(sk);
    if ((threadIdx.x & 31) == 0) red[0][threadIdx.x >> 5] = sq, red[1][threadIdx.x >> 5] = sk;
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) sq += red[0][w], sk += red[1][w];
    const float rq = 1.f / sqrtf(sq / (float)nq + eps), rk = has_k ? 1.f / sqrtf(sk / (float)nk + eps) : 0.f;
    // VEC columns from d of head j of a normed and weighted projection, turned
    auto turned = [&](const TA* x, const void* w, float r, int j, int d) -> float {
        const int c = j * dk + d;
        const float a = il_to_f(x[c]) * r * il_load_any(w, w_kind, c);
        if (d >= rot) return a;
        const int c2 = (d & 1) ? c - 1 : c + 1;
        const float b = il_to_f(x[c2]) * r * il_load_any(w, w_kind, c2);
        const float s = s_sin[d >> 1], co = s_cos[d >> 1];
        return (d & 1) ? a * co + b * s : a * co - b * s;
    };
    auto turned4 = [&](const TA* x, const void* w, float r, int j, int d) -> float4 {
        const int c = j * dk + d;
        float4 a = qn_ld4(x + c);
        const float4 b = qn_w4(w, w_kind, c);
        a.x *= r * b.x, a.y *= r * b.y, a.z *= r * b.z, a.w *= r * b.w;
        if (d < rot) {
            const float s = s_sin[d >> 1], co = s_cos[d >> 1], u = a.x, v = a.y;
            a.x = u * co - v * s, a.y = v * co + u * s;
        }
        if (d + 2 < rot) {
            const float s = s_sin[(d >> 1) + 1], co = s_cos[(d >> 1) + 1], u = a.z, v = a.w;
            a.z = u * co - v * s, a.w = v * co + u * s;
        }
        return a;
    };
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if (VEC == 4) {
        for (int idx = 4 * threadIdx.x; idx < nh * hd; idx += 4 * blockDim.x) {
            const int j = idx / hd, d = idx - j * hd;
            qn_st4(q_out + (size_t)t * nh * hd + idx, d < dk ? turned4(row + q_off, wq, rq, j, d) : zero);
        }
    } else {
        for (int idx = threadIdx.x; idx < nh * hd; idx += blockDim.x) {
            const int j = idx / hd, d = idx - j * hd;
            q_out[(size_t)t * nh * hd + idx] = il_from_f<TA>(d < dk ? turned(row + q_off, wq, rq, j, d) : 0.f);
        }
    }
    if (page < 0) return;                         // no keys of its own, or no slot (the host reserves every page a step touches)
    const size_t plane = (size_t)nkv * page_size * hd;
    TA* kdst = cache + (size_t)page * 2 * plane + (size_t)(pos % page_size) * hd;
    if (VEC == 4) {
        for (int idx = 4 * threadIdx.x; idx < nkv * hd; idx += 4 * blockDim.x) {
            const int g = idx / hd, d = idx - g * hd;
            const size_t at = (size_t)g * page_size * hd + d;
            qn_st4(kdst + at, d < dk ? turned4(row + k_off, wk, rk, g, d) : zero);
            qn_st4(kdst + plane + at, d < dv ? qn_ld4(row + v_off + g * dv + d) : zero);
        }
    } else {
        for (int idx = threadIdx.x; idx < nkv * hd; idx += blockDim.x) {
            const int g = idx / hd, d = idx - g * hd;
            const size_t at = (size_t)g * page_size * hd + d;
            kdst[at] = il_from_f<TA>(d < dk ? turned(row + k_off, wk, rk, g, d) : 0.f);
            kdst[plane + at] = d < dv ? row[v_off + g * dv + d] : il_from_f<TA>(0.f);
        }
    }
}

// freq: null, or float64 [rot / 2] - the pairs are then neighbours (2i, 2i + 1) and inv_freq is not read.
IL_EXPORT int il_qk_rows_norm_rope_store(const void* proj, int act_kind, int ld, int q_off, int k_off, int v_off, int nh, int nkv, int dk, int dv,
                                         int hd, const void* wq, const void* wk, int w_kind, float eps, int rot, const float* inv_freq,
                                         void* q_out, const int* tok_pos, const int* tok_entry, const int* block_table, int bt_stride,
                                         void* cache, int page_size, int T, const double* freq, cudaStream_t stream) {
    if (T <= 0) return IL_OK;
    if (nh <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || hd < dk || hd < dv || page_size <= 0 || !wq || (k_off >= 0 && !wk)) return IL_BAD_ARG;
    if (rot < 0 || (rot & 1) || rot > dk || (rot > 0 && !inv_freq && !freq)) return IL_BAD_ARG;
    if (rot > QR_MAX_ROT) return IL_UNSUPPORTED;
    const int work = nh * hd;
    const int threads = work >= 2048 ? 512 : work >= 512 ? 256 : 128;
    if (freq) {
        const bool vec = ((ld | q_off | v_off | dk | dv | hd) & 3) == 0 && (k_off < 0 || (k_off & 3) == 0) &&
                         (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)cache) & 15) == 0;
        const int vthreads = work >= 4096 ? 512 : work >= 1024 ? 256 : 128;
#define QP_GO(TA, VEC, TH)                                                                                                                      \
    IL_LAUNCH((qk_rows_norm_pairs_store_kernel<TA, VEC>), T, TH, 0, stream, (const TA*)proj, ld, q_off, k_off, v_off, nh, nkv, dk, dv, hd, wq, wk, \
              w_kind, eps, rot, freq, (TA*)q_out, tok_pos, tok_entry, block_table, bt_stride, (TA*)cache, page_size)
        if (act_kind == IL_F32) {
            if (vec) QP_GO(float, 4, vthreads); else QP_GO(float, 1, threads);
        } else if (act_kind == IL_BF16) {
            if (vec) QP_GO(__nv_bfloat16, 4, vthreads); else QP_GO(__nv_bfloat16, 1, threads);
        } else
            return IL_BAD_ARG;
#undef QP_GO
        IL_LAUNCH_CHECK();
        return IL_OK;
    }
    if (act_kind == IL_F32)
        IL_LAUNCH(qk_rows_norm_rope_store_kernel<float>, T, threads, 0, stream, (const float*)proj, ld, q_off, k_off, v_off, nh, nkv, dk, dv, hd, wq,
                  wk, w_kind, eps, rot, inv_freq, (float*)q_out, tok_pos, tok_entry, block_table, bt_stride, (float*)cache, page_size);
    else if (act_kind == IL_BF16)
        IL_LAUNCH(qk_rows_norm_rope_store_kernel<__nv_bfloat16>, T, threads, 0, stream, (const __nv_bfloat16*)proj, ld, q_off, k_off, v_off, nh, nkv,
                  dk, dv, hd, wq, wk, w_kind, eps, rot, inv_freq, (__nv_bfloat16*)q_out, tok_pos, tok_entry, block_table, bt_stride,
                  (__nv_bfloat16*)cache, page_size);
    else
        return IL_BAD_ARG;
    IL_LAUNCH_CHECK();
    return IL_OK;
}
