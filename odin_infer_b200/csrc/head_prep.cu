// Per-head preparation of the fused q|k|v projection, one warp per (token, head):
//   q heads: RMSNorm over the head (optional), rotation, written to q_out (which may be
//            the projection itself: in place);
//   k heads: RMSNorm (optional), rotation, written to the paged key cache;
//   v heads: copied to the paged value cache, or first mixed with the same token's values of
//            an earlier layer, v <- (1 - lambda) v + lambda v_first (struct VMix).
// Restates infer/forward.odin:58-85 (norm before rotation, one [hd] weight shared
// by all heads, half-split pairs (i, i + rot/2)) and the cache write of :47-49.
// The rotation reads cos/sin of 32-bit angles from a table built on the host.
// All arithmetic is 32-bit.
//
// Cache layout of one layer: [page][kv head][slot in page][hd]; a sequence's
// pages are named by its row of the block table.
#include "common.cuh"
#include "head_math.cuh"

#define HP_WARPS 4
#define HP_MAX_HD 512

// What happens to a value head on its way to the cache.  first: [rows][Hkv * vd] values of an earlier layer that are mixed
// in (null: none); keep: where this layer's own values go for later layers, in the same layout (null: nowhere).
template <typename T>
struct VMix {
    const T* first;
    T* keep;
    float lambda;
};

// TI: element type of the projection (bfloat16 or 32-bit; n_split 32-bit partial sums of a
// split product are added first, in order).  T: element type of q_out and of the cache.
// bias: one value per column of the projection, added first (null: none).  norm_mode 0: no norm;
// 1: RMSNorm with a weight before the rotation; 2: division by the root mean square after the
// rotation, no weight; 3: RMSNorm over the whole q projection (all query heads of the token at once; likewise k) with weights
// of that size, before the rotation.  vd: size of a value head (key and query heads have hd).
// pairs: the rotation pairs element 2i with 2i + 1 instead of i with i + rot/2.
// v_is_k: the projection holds no values; a key head's elements with their bias, before norm and rotation, are also its
// value head's (vd == hd), and its warp writes both.
template <typename TI, typename T>
__global__ void __launch_bounds__(HP_WARPS * 32)
head_prep_kernel(const TI* qkv, int n_split, size_t split_stride, T* q_out,  // may alias: no restrict
                 size_t q_out_stride, int Hq, int Hkv, int hd, int vd, size_t row_stride, VecRef bias, VecRef qw,
                 VecRef kw, int norm_mode, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                 int rot, int table_len, const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                 const int* __restrict__ block_table, int bt_stride, T* __restrict__ k_cache,
                 T* __restrict__ v_cache, int page_size, int write_kv, int pairs, int v_is_k, VMix<T> vmix) {
    __shared__ float buf[HP_WARPS][HP_MAX_HD];
    __shared__ float whole_ss[2][HP_WARPS];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * HP_WARPS + warp;
    const int n_heads = Hq + (v_is_k ? 1 : 2) * Hkv;
    const int seq = tok_seq[t];
    if (seq < 0) return;  // padding token (the whole CTA: it belongs to one token)
    if (norm_mode == 3) {
        // the sums of squares of the token's whole q and whole k projection, by the CTA's warps together and in an order
        // that the sizes alone fix (every CTA of the token forms the same two sums)
        // (only the sums that this CTA's four heads ask for: q heads come first, then k heads, then v heads)
        const int h0 = blockIdx.y * HP_WARPS, h1 = min(n_heads, h0 + HP_WARPS);
        for (int side = 0; side < 2; ++side) {
            if (side == 0 ? h0 >= Hq : (h1 <= Hq || h0 >= Hq + Hkv)) continue;
            const int whole = (side == 0 ? Hq : Hkv) * hd;
            const size_t wcol0 = side == 0 ? 0 : (size_t)Hq * hd;
            const TI* wsrc = qkv + (size_t)t * row_stride + wcol0;
            float sw = 0.f;
            for (int j = threadIdx.x; j < whole; j += HP_WARPS * 32) {
                float v = to_f32(wsrc[j]);
                for (int sp = 1; sp < n_split; ++sp) v += to_f32(wsrc[(size_t)sp * split_stride + j]);
                if (bias.p != nullptr) v += bias.at((int)wcol0 + j);
                sw += v * v;
            }
            sw = warp_sum(sw);
            if (lane == 0) whole_ss[side][warp] = sw;
        }
        __syncthreads();
    }
    if (head >= n_heads) return;
    const int pos = tok_pos[t];

    const bool is_q = head < Hq;
    const bool is_k = !is_q && head < Hq + Hkv;
    const int kvh = is_q ? 0 : (is_k ? head - Hq : head - Hq - Hkv);
    if (!is_q && !write_kv) return;
    const bool is_v = !is_q && !is_k;
    const int n = is_v ? vd : hd;  // this head's size
    const size_t col0 = is_v ? (size_t)(Hq + Hkv) * hd + (size_t)kvh * vd : (size_t)head * hd;
    const TI* src = qkv + (size_t)t * row_stride + col0;

    T* dst = q_out + (size_t)t * q_out_stride + (size_t)head * hd;
    if (!is_q) {
        const int page = block_table[(size_t)seq * bt_stride + pos / page_size];
        if (page < 0) return;
        T* base = is_k ? k_cache : v_cache;
        dst = base + (((size_t)page * Hkv + kvh) * page_size + (pos % page_size)) * n;
    }

    float* b = buf[warp];
    float ss = 0.f;
    for (int j = lane; j < n; j += 32) {
        float v = to_f32(src[j]);
        for (int sp = 1; sp < n_split; ++sp) v += to_f32(src[(size_t)sp * split_stride + j]);
        if (bias.p != nullptr) v += bias.at((int)col0 + j);
        b[j] = v;
        ss += v * v;
    }
    if (is_k && v_is_k) {   // the same place of the value cache (dst is its key's place)
        T* vdst = v_cache + (dst - k_cache);
        for (int j = lane; j < n; j += 32) vdst[j] = from_f32<T>(b[j]);
    }
    if (is_v) {  // value head: stored as it is, or mixed with an earlier layer's
        const size_t at = ((size_t)t * Hkv + kvh) * vd;
        for (int j = lane; j < n; j += 32) {
            float v = b[j];
            if (vmix.keep != nullptr) vmix.keep[at + j] = from_f32<T>(v);
            if (vmix.first != nullptr) v = (1.0f - vmix.lambda) * v + vmix.lambda * to_f32(vmix.first[at + j]);
            dst[j] = from_f32<T>(v);
        }
        return;
    }
    if (norm_mode == 1) {
        ss = warp_sum(ss);
        ss /= (float)hd;
        ss += eps;
        const float r = 1.0f / sqrtf(ss);
        const VecRef& w = is_q ? qw : kw;
        for (int j = lane; j < hd; j += 32) b[j] = w.at(j) * (r * b[j]);
    } else if (norm_mode == 3) {
        const int whole = (is_q ? Hq : Hkv) * hd;
        float sw = 0.f;
#pragma unroll
        for (int wi = 0; wi < HP_WARPS; ++wi) sw += whole_ss[is_q ? 0 : 1][wi];
        sw /= (float)whole;
        sw += eps;
        const float r = 1.0f / sqrtf(sw);
        const VecRef& w = is_q ? qw : kw;
        const int w0 = (is_q ? head : kvh) * hd;
        for (int j = lane; j < hd; j += 32) b[j] = w.at(w0 + j) * (r * b[j]);
    }
    __syncwarp();
    const int half = rot >> 1;
    const bool in_table = (pos >= 0 && pos < table_len);
    float o[HP_MAX_HD / 32];
    float s2 = 0.f;
#pragma unroll
    for (int e = 0; e < HP_MAX_HD / 32; ++e) {
        const int j = lane + 32 * e;
        if (j >= hd) break;
        if (j < rot && in_table && pairs) {
            const int i = j >> 1;
            const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
            const float x = b[2 * i], y = b[2 * i + 1];
            o[e] = (j & 1) ? (x * s + y * c) : (x * c - y * s);
        } else if (j < rot && in_table) {
            const int i = (j < half) ? j : j - half;
            const float c = cos_t[(size_t)pos * half + i], s = sin_t[(size_t)pos * half + i];
            const float x = b[i], y = b[i + half];
            o[e] = (j < half) ? (x * c - y * s) : (x * s + y * c);
        } else {
            o[e] = b[j];
        }
        s2 += o[e] * o[e];
    }
    float r2 = 1.0f;
    if (norm_mode == 2) {
        s2 = warp_sum(s2);
        s2 /= (float)hd;
        s2 += eps;
        r2 = 1.0f / sqrtf(s2);
    }
#pragma unroll
    for (int e = 0; e < HP_MAX_HD / 32; ++e) {
        const int j = lane + 32 * e;
        if (j >= hd) break;
        dst[j] = from_f32<T>(norm_mode == 2 ? o[e] * r2 : o[e]);
    }
}


// The common case with a bfloat16 cache (full rotary, head size 64 or 128): each lane holds
// VEC = hd/32 consecutive elements in registers, the rotation partner (i +- hd/2) lives in
// lane ^ 16, and rows move with vector loads and stores.  The input is bfloat16, or 32-bit
// partial sums of a split product that are added first, in order.  Same arithmetic as above.
using headmath::load_vec;
using headmath::store_vec_bf16;

// A value head's VEC elements of this lane on their way to the cache (see VMix); `at`: their place in its buffers.
template <int VEC>
__device__ __forceinline__ void value_to_cache(float (&v)[VEC], bf16* dst, const VMix<bf16>& vmix, size_t at) {
    if (vmix.keep != nullptr) store_vec_bf16<VEC>(vmix.keep + at, v);
    if (vmix.first != nullptr) {
        float f[VEC];
        load_vec<VEC>(vmix.first + at, f);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = (1.0f - vmix.lambda) * v[e] + vmix.lambda * f[e];
    }
    store_vec_bf16<VEC>(dst, v);
}

// A warp per (token, head), TOK tokens per warp (one: for few tokens the kernel is a chain of
// latencies, and everything that can be is fetched before the wait for the kernel before it).
template <int VEC, typename TI, int TOK>
__global__ void __launch_bounds__(HP_WARPS * 32)
head_prep_fast_kernel(const TI* qkv, int n_split, size_t split_stride, bf16* q_out, size_t q_out_stride, int T, int Hq,
                      int Hkv, size_t row_stride, VecRef qw, VecRef kw, int has_norm, float eps,
                      const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len,
                      const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                      const int* __restrict__ block_table, int bt_stride, bf16* __restrict__ k_cache,
                      bf16* __restrict__ v_cache, int page_size, int write_kv, VMix<bf16> vmix) {
    constexpr int HD = VEC * 32, HALF = HD / 2;
    pdl_trigger();
    // What no earlier kernel of the step writes is fetched before the wait for that kernel: the
    // step's tables, the page of the cache, the angles' cosines and sines, the norms' weights.
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * HP_WARPS + warp;
    const bool in_range = head < Hq + 2 * Hkv;
    const bool is_q = head < Hq;
    const bool is_k = !is_q && head < Hq + Hkv;
    const int kvh = is_q ? 0 : (is_k ? head - Hq : head - Hq - Hkv);
    bool active[TOK], in_table[TOK];
    bf16* dst[TOK];
    float c[TOK][VEC], sn[TOK][VEC], wn[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) wn[e] = 1.f;
    if (in_range && (is_q || is_k) && has_norm) {
        const VecRef& w = is_q ? qw : kw;
#pragma unroll
        for (int e = 0; e < VEC; ++e) wn[e] = w.at(lane * VEC + e);
    }
#pragma unroll
    for (int u = 0; u < TOK; ++u) {
        const int t = blockIdx.x * TOK + u;
        const int seq = (in_range && t < T) ? tok_seq[t] : -1;
        const int pos = (t < T) ? tok_pos[t] : 0;
        active[u] = seq >= 0 && (is_q || write_kv);
        dst[u] = q_out + (size_t)t * q_out_stride + (size_t)head * HD + lane * VEC;
        if (active[u] && !is_q) {
            const int page = block_table[(size_t)seq * bt_stride + pos / page_size];
            if (page < 0) active[u] = false;
            else dst[u] = (is_k ? k_cache : v_cache) + (((size_t)page * Hkv + kvh) * page_size + (pos % page_size)) * HD + lane * VEC;
        }
        in_table[u] = (pos >= 0 && pos < table_len);
#pragma unroll
        for (int e = 0; e < VEC; ++e) { c[u][e] = 1.f; sn[u][e] = 0.f; }
        if (active[u] && (is_q || is_k) && in_table[u]) {
            load_vec<VEC>(cos_t + (size_t)pos * HALF + (lane & 15) * VEC, c[u]);
            load_vec<VEC>(sin_t + (size_t)pos * HALF + (lane & 15) * VEC, sn[u]);
        }
    }
    pdl_wait();
    float v[TOK][VEC];
#pragma unroll
    for (int u = 0; u < TOK; ++u) {
        if (!active[u]) continue;
        const int t = blockIdx.x * TOK + u;
        headmath::load_parts<VEC, TI>(qkv + (size_t)t * row_stride + (size_t)head * HD + lane * VEC, n_split, split_stride, v[u]);
    }
#pragma unroll
    for (int u = 0; u < TOK; ++u) {
        if (!active[u]) continue;
        if (!is_q && !is_k) {  // value head: no norm, no rotation
            value_to_cache<VEC>(v[u], dst[u], vmix, ((size_t)(blockIdx.x * TOK + u) * Hkv + kvh) * HD + lane * VEC);
            continue;
        }
        float o[VEC];
        headmath::norm_rotate<VEC>(v[u], has_norm != 0, wn, eps, in_table[u], c[u], sn[u], lane, o);
        store_vec_bf16<VEC>(dst[u], o);
    }
}

// For prompts: a CTA per token, its four warps share the token's heads (warp w takes heads w, w + 4,
// ...), so the angles of the token's position are fetched once per warp and not once per head, and
// four heads' loads are in flight per warp.  Same arithmetic (head_math.cuh).
template <int VEC, typename TI>
__global__ void __launch_bounds__(HP_WARPS * 32)
head_prep_token_kernel(const TI* qkv, int n_split, size_t split_stride, bf16* q_out, size_t q_out_stride, int Hq,
                       int Hkv, size_t row_stride, VecRef qw, VecRef kw, int has_norm, float eps,
                       const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_len,
                       const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                       const int* __restrict__ block_table, int bt_stride, bf16* __restrict__ k_cache,
                       bf16* __restrict__ v_cache, int page_size, int write_kv, VMix<bf16> vmix) {
    constexpr int HD = VEC * 32, HALF = HD / 2, UNROLL = 4;
    pdl_trigger();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seq = tok_seq[t];
    const int pos = tok_pos[t];
    pdl_wait();
    if (seq < 0) return;
    // The first heads' loads go out before the loads that hang on the token's position (its page, its
    // angles): a CTA lives for a chain of three trips to memory otherwise, with data in flight during one.
    const int n_heads = Hq + 2 * Hkv;
    const TI* row = qkv + (size_t)t * row_stride + lane * VEC;
    float v[UNROLL][VEC];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
        const int head = warp + u * HP_WARPS;
        if (head < n_heads && (head < Hq || write_kv))
            headmath::load_parts<VEC, TI>(row + (size_t)head * HD, n_split, split_stride, v[u]);
    }
    const int page = write_kv ? block_table[(size_t)seq * bt_stride + pos / page_size] : -1;
    const bool in_table = (pos >= 0 && pos < table_len);
    float c[VEC], sn[VEC], wq[VEC], wk[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) { c[e] = 1.f; sn[e] = 0.f; wq[e] = 1.f; wk[e] = 1.f; }
    if (in_table) {
        load_vec<VEC>(cos_t + (size_t)pos * HALF + (lane & 15) * VEC, c);
        load_vec<VEC>(sin_t + (size_t)pos * HALF + (lane & 15) * VEC, sn);
    }
    if (has_norm) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { wq[e] = qw.at(lane * VEC + e); wk[e] = kw.at(lane * VEC + e); }
    }
    for (int h0 = warp; h0 < n_heads; h0 += HP_WARPS * UNROLL) {
        if (h0 != warp) {
#pragma unroll
            for (int u = 0; u < UNROLL; ++u) {
                const int head = h0 + u * HP_WARPS;
                if (head < n_heads && (head < Hq || page >= 0))
                    headmath::load_parts<VEC, TI>(row + (size_t)head * HD, n_split, split_stride, v[u]);
            }
        }
#pragma unroll
        for (int u = 0; u < UNROLL; ++u) {
            const int head = h0 + u * HP_WARPS;
            if (head >= n_heads) continue;
            const bool is_q = head < Hq, is_k = !is_q && head < Hq + Hkv;
            if (!is_q && page < 0) continue;
            bf16* dst;
            if (is_q) {
                dst = q_out + (size_t)t * q_out_stride + (size_t)head * HD + lane * VEC;
            } else {
                const int kvh = is_k ? head - Hq : head - Hq - Hkv;
                dst = (is_k ? k_cache : v_cache) + (((size_t)page * Hkv + kvh) * page_size + (pos % page_size)) * HD + lane * VEC;
            }
            if (!is_q && !is_k) {  // value head: no norm, no rotation
                value_to_cache<VEC>(v[u], dst, vmix, ((size_t)t * Hkv + (head - Hq - Hkv)) * HD + lane * VEC);
                continue;
            }
            float o[VEC];
            headmath::norm_rotate<VEC>(v[u], has_norm != 0, is_q ? wq : wk, eps, in_table, c, sn, lane, o);
            store_vec_bf16<VEC>(dst, o);
        }
    }
}

// qkv: [n_split][T, (Hq + 2 Hkv) hd] of in_dtype (row stride row_stride, parts split_stride
// elements apart).  q_out: [T, Hq hd] of dtype (row stride q_out_stride); it may be qkv
// itself when there is one part of the same type (q is then normalised and rotated in place).
// bias (null: none), norm_mode and vd as the general kernel describes them; the fast kernels take no
// bias, norm_mode 0 or 1 and vd == hd.  v_first, v_keep (each null: none; [T, Hkv vd] of dtype, contiguous), v_lambda: see VMix.
extern "C" int odin_head_prep(const void* qkv, int in_dtype, int n_split, long long split_stride, void* q_out,
                              long long q_out_stride, int dtype, int T, int Hq, int Hkv, int hd, int vd,
                              long long row_stride, const void* bias, int bias_dtype, const void* q_norm_w,
                              const void* k_norm_w, int w_dtype, int norm_mode, float eps,
                              const float* cos_t, const float* sin_t, int rot, int table_len,
                              const int* tok_pos, const int* tok_seq, const int* block_table, int bt_stride,
                              void* k_cache, void* v_cache, int page_size, int write_kv, int pairs, const void* v_first,
                              void* v_keep, float v_lambda, int v_is_k, void* stream) {
    if (T <= 0) return 0;
    if (v_is_k && (vd != hd || v_first != nullptr || v_keep != nullptr)) return ODIN_ERR_BAD_ARG;
    if (hd > HP_MAX_HD || hd <= 0 || vd > HP_MAX_HD || vd <= 0 || (rot & 1) || rot > hd || rot < 0 || n_split < 1 ||
        norm_mode < 0 || norm_mode > 3)
        return ODIN_ERR_UNSUPPORTED;
    const int has_norm = norm_mode == 1;
    const bool plain_heads = bias == nullptr && norm_mode < 2 && vd == hd && !pairs && !v_is_k;
    cudaStream_t s = (cudaStream_t)stream;
    const int n_heads = Hq + (v_is_k ? 1 : 2) * Hkv;
    dim3 grid(T, (n_heads + HP_WARPS - 1) / HP_WARPS);
    if (grid.y > 65535) return ODIN_ERR_UNSUPPORTED;
    VecRef qw{q_norm_w, w_dtype == ODIN_BF16}, kw{k_norm_w, w_dtype == ODIN_BF16};
    VecRef bv{bias, bias_dtype == ODIN_BF16};
    const bool fast_in = (in_dtype == ODIN_BF16 && n_split == 1) || in_dtype == ODIN_F32;
    if (plain_heads && fast_in && dtype == ODIN_BF16 && rot == hd && (hd == 64 || hd == 128) && (row_stride % 4) == 0 &&
        (split_stride % 4) == 0 && (q_out_stride % 4) == 0 &&
        ((((uintptr_t)qkv) | ((uintptr_t)q_out) | ((uintptr_t)cos_t) | ((uintptr_t)sin_t) | ((uintptr_t)v_first) |
          ((uintptr_t)v_keep)) & 15) == 0) {
        const VMix<bf16> vmix{(const bf16*)v_first, (bf16*)v_keep, v_lambda};
#define FAST(VEC, TI, TOK)                                                                                         \
    odin_launch(head_prep_fast_kernel<VEC, TI, TOK>, dim3((T + TOK - 1) / TOK, grid.y), dim3(HP_WARPS * 32), 0, s,     \
                (const TI*)qkv, n_split, (size_t)split_stride, (bf16*)q_out, (size_t)q_out_stride, T, Hq, Hkv,         \
                (size_t)row_stride, qw, kw, has_norm, eps, cos_t, sin_t, table_len, tok_pos, tok_seq, block_table,      \
                bt_stride, (bf16*)k_cache, (bf16*)v_cache, page_size, write_kv, vmix)
#define FAST_T(VEC, TI)                                                                                            \
    do {                                                                                                           \
        if (T >= 256)                                                                                              \
            odin_launch(head_prep_token_kernel<VEC, TI>, dim3(T), dim3(HP_WARPS * 32), 0, s, (const TI*)qkv, n_split,  \
                        (size_t)split_stride, (bf16*)q_out, (size_t)q_out_stride, Hq, Hkv, (size_t)row_stride, qw, kw, \
                        has_norm, eps, cos_t, sin_t, table_len, tok_pos, tok_seq, block_table, bt_stride,              \
                        (bf16*)k_cache, (bf16*)v_cache, page_size, write_kv, vmix);                                     \
        else FAST(VEC, TI, 1);                                                                                     \
    } while (0)
        if (hd == 128 && in_dtype == ODIN_BF16) FAST_T(4, bf16);
        else if (hd == 128) FAST_T(4, float);
        else if (in_dtype == ODIN_BF16) FAST_T(2, bf16);
        else FAST_T(2, float);
#undef FAST_T
#undef FAST
        ODIN_LAUNCH_CHECK();
        return 0;
    }
#define GO(TI, TT)                                                                                                  \
    odin_launch(head_prep_kernel<TI, TT>, grid, dim3(HP_WARPS * 32), 0, s,                                           \
        (const TI*)qkv, n_split, (size_t)split_stride, (TT*)q_out, (size_t)q_out_stride, Hq, Hkv, hd, vd,           \
        (size_t)row_stride, bv, qw, kw, norm_mode, eps, cos_t, sin_t, rot, table_len, tok_pos, tok_seq, block_table,     \
        (int)bt_stride, (TT*)k_cache, (TT*)v_cache, page_size, write_kv, pairs, v_is_k,                              \
        VMix<TT>{(const TT*)v_first, (TT*)v_keep, v_lambda})
    if (in_dtype == ODIN_BF16 && dtype == ODIN_BF16) GO(bf16, bf16);
    else if (in_dtype == ODIN_F32 && dtype == ODIN_F32) GO(float, float);
    else if (in_dtype == ODIN_F32 && dtype == ODIN_BF16) GO(float, bf16);
    else return ODIN_ERR_UNSUPPORTED;
#undef GO
    ODIN_LAUNCH_CHECK();
    return 0;
}
