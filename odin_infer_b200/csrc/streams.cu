// A residual of several streams X[0] .. X[s-1] ([s][rows][d], 32-bit): a sublayer's output joins all of them, and the next
// sublayer reads a norm of a weighted sum of them.
//
//   y      = the update: a sum of terms (combine_terms.cuh)
//   X'[j]  = sum_i mix[i][j] X[i] + add[j] y        (all streams at once from the old ones; without an update X' = X)
//   out    = w * u / sqrt(mean(u^2) + eps),  u = sum_j read[j] X'[j]
//
// One launch per sublayer, a CTA per row: a row of every stream is read and written once.  All arithmetic is 32-bit; a
// row's sums run in an order that the width and the block size fix, so a row does not depend on the other rows.
#include "combine_terms.cuh"

#define MAX_STREAMS 16
#define STREAM_THREADS 256

struct StreamArgs {
    float* x; size_t stream_stride; int s;
    CombineArgs terms; int update;                 // update 0: nothing joins, the streams are read only
    const float* mix; const float* add; const float* read;
    VecRef w; float eps;
    const int* rows;                               // gather these rows (the streams are then left as they are)
    int d;
};

// Any number of streams and terms, any width whose two rows fit in shared memory.
template <typename TO, bool VEC>
__global__ void __launch_bounds__(STREAM_THREADS)
mix_streams_kernel(StreamArgs a, TO* __restrict__ out) {
    __shared__ float red[32];
    __shared__ float cmix[MAX_STREAMS * MAX_STREAMS], cadd[MAX_STREAMS], cread[MAX_STREAMS];
    extern __shared__ __align__(16) float sbuf[];
    float* acc = sbuf;          // d: the update
    float* tmp = sbuf + a.d;    // d: a term before its norm, then the row that is read
    pdl_trigger();
    const int S = a.s, d = a.d;
    if (a.update) {
        for (int i = threadIdx.x; i < S * S; i += blockDim.x) cmix[i] = a.mix[i];
        for (int i = threadIdx.x; i < S; i += blockDim.x) cadd[i] = a.add[i];
    }
    for (int i = threadIdx.x; i < S; i += blockDim.x) cread[i] = a.read[i];
    const int r = a.rows != nullptr ? a.rows[blockIdx.x] : blockIdx.x;
    __syncthreads();
    pdl_wait();
    constexpr int W = VEC ? 4 : 1;   // four elements at a time where everything is that much aligned; the same sums either way
    const int j0 = threadIdx.x * W, dj = blockDim.x * W;
    auto weights = [&](const VecRef& w, int j, float* v) {
        if (VEC) { const float4 q = w.at4(j); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
        else v[0] = w.at(j);
    };
    for (int i = 0; i < (a.update ? a.terms.n : 0); ++i) {
        const CombineTerm& tm = a.terms.t[i];
        float ss = 0.f;
        for (int j = j0; j < d; j += dj) {
            float v[W], u[W];
#pragma unroll
            for (int e = 0; e < W; ++e) v[e] = 0.f;
            for (int sp = 0; sp < tm.n_split; ++sp) {
                const size_t at = (size_t)sp * tm.split_stride + (size_t)r * d + j;
                if (VEC) {
                    const float4 q = tm.is_bf16 ? ld4((const bf16*)tm.p + at) : ld4((const float*)tm.p + at);
                    u[0] = q.x; u[1] = q.y; u[2] = q.z; u[3] = q.w;
                } else {
                    u[0] = tm.is_bf16 ? __bfloat162float(((const bf16*)tm.p)[at]) : ((const float*)tm.p)[at];
                }
#pragma unroll
                for (int e = 0; e < W; ++e) v[e] += u[e];
            }
            if (tm.bias.p != nullptr) {
                weights(tm.bias, j, u);
#pragma unroll
                for (int e = 0; e < W; ++e) v[e] += u[e];
            }
#pragma unroll
            for (int e = 0; e < W; ++e) { tmp[j + e] = v[e]; ss += v[e] * v[e]; }
        }
        float f = tm.scale;
        if (tm.row_scale != nullptr) f *= tm.row_scale[r];
        float rs = 1.0f;
        if (tm.norm_w.p != nullptr) rs = 1.0f / sqrtf(block_sum(ss, red) / (float)d + tm.norm_eps);
        for (int j = j0; j < d; j += dj) {
            float w[W];
            if (tm.norm_w.p != nullptr) weights(tm.norm_w, j, w);
#pragma unroll
            for (int e = 0; e < W; ++e) {
                const float v = tm.norm_w.p != nullptr ? f * (w[e] * (rs * tmp[j + e])) : f * tmp[j + e];
                acc[j + e] = i == 0 ? v : acc[j + e] + v;
            }
        }
    }
    float ss = 0.f;
    for (int j = j0; j < d; j += dj) {
        float X[MAX_STREAMS][W], u[W];
        float* xr = a.x + (size_t)r * d + j;
#pragma unroll
        for (int i = 0; i < MAX_STREAMS; ++i) {
            if (i >= S) break;
            if (VEC) { const float4 q = ld4(xr + i * a.stream_stride); X[i][0] = q.x; X[i][1] = q.y; X[i][2] = q.z; X[i][3] = q.w; }
            else X[i][0] = xr[i * a.stream_stride];
        }
#pragma unroll
        for (int e = 0; e < W; ++e) u[e] = 0.f;
        for (int k = 0; k < S; ++k) {
            float n[W];
            if (a.update) {
#pragma unroll
                for (int e = 0; e < W; ++e) n[e] = 0.f;
#pragma unroll
                for (int i = 0; i < MAX_STREAMS; ++i) {
                    if (i >= S) break;
#pragma unroll
                    for (int e = 0; e < W; ++e) n[e] = fmaf(cmix[i * S + k], X[i][e], n[e]);
                }
#pragma unroll
                for (int e = 0; e < W; ++e) n[e] = fmaf(cadd[k], acc[j + e], n[e]);
                if (a.rows == nullptr) {
                    if (VEC) st4(xr + k * a.stream_stride, make_float4(n[0], n[VEC ? 1 : 0], n[VEC ? 2 : 0], n[VEC ? 3 : 0]));
                    else xr[k * a.stream_stride] = n[0];
                }
            } else {
#pragma unroll
                for (int i = 0; i < MAX_STREAMS; ++i)
                    if (i == k) {
#pragma unroll
                        for (int e = 0; e < W; ++e) n[e] = X[i][e];
                    }
            }
#pragma unroll
            for (int e = 0; e < W; ++e) u[e] = fmaf(cread[k], n[e], u[e]);
        }
#pragma unroll
        for (int e = 0; e < W; ++e) { tmp[j + e] = u[e]; ss += u[e] * u[e]; }
    }
    const float rs = 1.0f / sqrtf(block_sum(ss, red) / (float)d + a.eps);
    TO* o = out + (size_t)blockIdx.x * d;
    for (int j = j0; j < d; j += dj) {   // every thread reads back what it stored itself
        float w[W];
        weights(a.w, j, w);
        if (VEC) st4(o + j, make_float4(w[0] * (rs * tmp[j]), w[VEC ? 1 : 0] * (rs * tmp[j + (VEC ? 1 : 0)]),
                                        w[VEC ? 2 : 0] * (rs * tmp[j + (VEC ? 2 : 0)]), w[VEC ? 3 : 0] * (rs * tmp[j + (VEC ? 3 : 0)])));
        else o[j] = from_f32<TO>(w[0] * (rs * tmp[j]));
    }
}

// Up to four streams and two 32-bit terms without a number per row, a row of up to 4 NV blockDim.x elements (the width a
// multiple of four, everything 16-byte aligned): what is read stays in registers, loads go out together, and a sum over the
// row costs one barrier (every warp's share goes to a place of its own, every thread adds the shares in their order).
template <int S, int NT, int NV, typename TO>
__global__ void __launch_bounds__(512)
mix_streams_fast_kernel(StreamArgs a, TO* __restrict__ out) {
    __shared__ float shares[3][16];
    pdl_trigger();
    const int r = a.rows != nullptr ? a.rows[blockIdx.x] : blockIdx.x;
    const int d = a.d, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    float cmix[S][S], cadd[S], cread[S];
#pragma unroll
    for (int i = 0; i < S; ++i) {
        cread[i] = a.read[i];
        if (NT > 0) {
            cadd[i] = a.add[i];
#pragma unroll
            for (int k = 0; k < S; ++k) cmix[i][k] = a.mix[i * S + k];
        }
    }
    auto put_share = [&](int which, float v) {
        v = warp_sum(v);
        if (lane == 0) shares[which][warp] = v;
    };
    auto row_sum = [&](int which) {
        float v = 0.f;
        for (int i = 0; i < n_warps; ++i) v += shares[which][i];
        return v;
    };
    constexpr bool EARLY = S * NV <= 8;   // the streams' loads go out before the terms are summed, where registers allow
    float4 X[EARLY ? NV : 1][S];
    float4 t[NT > 0 ? NT : 1][NV], u[NV];
    pdl_wait();
    auto load_streams = [&](int i, float4 (&dst)[S]) {
        const int j = (threadIdx.x + i * blockDim.x) * 4;
#pragma unroll
        for (int k = 0; k < S; ++k) dst[k] = j < d ? ld4(a.x + k * a.stream_stride + (size_t)r * d + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    if (EARLY) {
#pragma unroll
        for (int i = 0; i < NV; ++i) load_streams(i, X[EARLY ? i : 0]);
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        const CombineTerm& tm = a.terms.t[n];
#pragma unroll
        for (int i = 0; i < NV; ++i) t[n][i] = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int sp = 0; sp < tm.n_split; ++sp) {
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int j = (threadIdx.x + i * blockDim.x) * 4;
                if (j < d) {
                    const float4 v = ld4((const float*)tm.p + (size_t)sp * tm.split_stride + (size_t)r * d + j);
                    t[n][i].x += v.x; t[n][i].y += v.y; t[n][i].z += v.z; t[n][i].w += v.w;
                }
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int j = (threadIdx.x + i * blockDim.x) * 4;
            if (j < d && tm.bias.p != nullptr) {
                const float4 b = tm.bias.at4(j);
                t[n][i].x += b.x; t[n][i].y += b.y; t[n][i].z += b.z; t[n][i].w += b.w;
            }
            ss += (t[n][i].x * t[n][i].x + t[n][i].y * t[n][i].y) + (t[n][i].z * t[n][i].z + t[n][i].w * t[n][i].w);
        }
        if (tm.norm_w.p != nullptr) put_share(n, ss);
    }
    if (NT > 0 && (a.terms.t[0].norm_w.p != nullptr || (NT > 1 && a.terms.t[NT - 1].norm_w.p != nullptr))) __syncthreads();
    float ss = 0.f;
    float rs[NT > 0 ? NT : 1];
#pragma unroll
    for (int n = 0; n < NT; ++n) rs[n] = a.terms.t[n].norm_w.p != nullptr ? 1.0f / sqrtf(row_sum(n) / (float)d + a.terms.t[n].norm_eps) : 1.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int j = (threadIdx.x + i * blockDim.x) * 4;
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j >= d) continue;
        float4 late[S];
        if (!EARLY) load_streams(i, late);
        const float4* Xi = EARLY ? X[EARLY ? i : 0] : late;
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const CombineTerm& tm = a.terms.t[n];
            const float f = tm.scale;
            float4 v = t[n][i];
            if (tm.norm_w.p != nullptr) {
                const float4 w = tm.norm_w.at4(j);
                v = make_float4(w.x * (rs[n] * v.x), w.y * (rs[n] * v.y), w.z * (rs[n] * v.z), w.w * (rs[n] * v.w));
            }
            y = make_float4(fmaf(f, v.x, y.x), fmaf(f, v.y, y.y), fmaf(f, v.z, y.z), fmaf(f, v.w, y.w));
        }
#pragma unroll
        for (int k = 0; k < S; ++k) {
            float4 n = Xi[k];
            if (NT > 0) {
                n = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int m = 0; m < S; ++m)
                    n = make_float4(fmaf(cmix[m][k], Xi[m].x, n.x), fmaf(cmix[m][k], Xi[m].y, n.y),
                                    fmaf(cmix[m][k], Xi[m].z, n.z), fmaf(cmix[m][k], Xi[m].w, n.w));
                n = make_float4(fmaf(cadd[k], y.x, n.x), fmaf(cadd[k], y.y, n.y), fmaf(cadd[k], y.z, n.z), fmaf(cadd[k], y.w, n.w));
                if (a.rows == nullptr) st4(a.x + k * a.stream_stride + (size_t)r * d + j, n);
            }
            u[i] = make_float4(fmaf(cread[k], n.x, u[i].x), fmaf(cread[k], n.y, u[i].y), fmaf(cread[k], n.z, u[i].z), fmaf(cread[k], n.w, u[i].w));
        }
        ss += (u[i].x * u[i].x + u[i].y * u[i].y) + (u[i].z * u[i].z + u[i].w * u[i].w);
    }
    put_share(2, ss);
    __syncthreads();
    const float ro = 1.0f / sqrtf(row_sum(2) / (float)d + a.eps);
    TO* o = out + (size_t)blockIdx.x * d;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int j = (threadIdx.x + i * blockDim.x) * 4;
        if (j >= d) continue;
        const float4 w = a.w.at4(j);
        st4(o + j, make_float4(w.x * (ro * u[i].x), w.y * (ro * u[i].y), w.z * (ro * u[i].z), w.w * (ro * u[i].w)));
    }
}

// mix, add: float32 [s][s] (from, to) and [s]; null with has_update = 0.  The terms as odin_combine_add takes them.
extern "C" int odin_mix_streams(float* x, long long stream_stride, int s, int has_update, int n_terms, const void* const* ptrs,
                                const int* dtypes, const int* n_splits, const long long* split_strides, const float* scales,
                                const float* const* row_scales, const void* const* norm_ws, const int* norm_w_dtypes,
                                const float* norm_eps, const void* const* biases, const int* bias_dtypes, const float* mix,
                                const float* add, const float* read, const void* w, int w_dtype, float eps, void* out,
                                int out_dtype, const int* rows, int n_rows, int d, void* stream) {
    if (n_rows <= 0) return 0;
    if (s < 1 || s > MAX_STREAMS || d <= 0 || x == nullptr || read == nullptr || w == nullptr || out == nullptr) return ODIN_ERR_BAD_ARG;
    if (has_update ? (n_terms < 1 || mix == nullptr || add == nullptr) : n_terms != 0) return ODIN_ERR_BAD_ARG;
    if (out_dtype != ODIN_BF16 && out_dtype != ODIN_F32) return ODIN_ERR_UNSUPPORTED;
    StreamArgs a;
    uintptr_t bits = (uintptr_t)x | (uintptr_t)w | (uintptr_t)out | (uintptr_t)(stream_stride * 4);
    if (const int rc = fill_combine_args(a.terms, bits, n_terms, ptrs, dtypes, n_splits, split_strides, scales, row_scales, norm_ws,
                                         norm_w_dtypes, norm_eps, biases, bias_dtypes)) return rc;
    a.x = x; a.stream_stride = (size_t)stream_stride; a.s = s; a.update = has_update; a.mix = mix; a.add = add; a.read = read;
    a.w = VecRef{w, w_dtype == ODIN_BF16}; a.eps = eps; a.rows = rows; a.d = d;
    const bool vec = (d % 4 == 0) && (bits % 16 == 0);
    cudaStream_t st = (cudaStream_t)stream;
    bool fast = vec && s <= 4 && n_terms <= 2 && d <= 4 * 4 * 512;
    for (int i = 0; i < n_terms; ++i) fast = fast && dtypes[i] == ODIN_F32 && row_scales[i] == nullptr;
    if (fast) {
        // few rows of 16-bit outputs: as many threads as the row keeps busy (a chain of latencies); else 256, or 512 for the
        // widest rows.  32-bit outputs take one block size per width, whatever the number of rows.
        int threads = d <= 4096 ? 256 : 512;
        if (out_dtype == ODIN_BF16 && n_rows <= 128) threads = d >= 2048 ? 512 : (d / 4 + 31) / 32 * 32;
        const int per = (d / 4 + threads - 1) / threads;
        const int nv = per <= 1 ? 1 : per <= 2 ? 2 : 4;
#define GO(S, NT, NV, TO) odin_launch(mix_streams_fast_kernel<S, NT, NV, TO>, dim3(n_rows), dim3(threads), 0, st, a, (TO*)out)
#define GO_NV(S, NT, TO)                     \
    do {                                     \
        if (nv == 1) GO(S, NT, 1, TO);       \
        else if (nv == 2) GO(S, NT, 2, TO);  \
        else GO(S, NT, 4, TO);               \
    } while (0)
#define GO_T(S, TO)                              \
    do {                                         \
        if (n_terms == 0) GO_NV(S, 0, TO);       \
        else if (n_terms == 1) GO_NV(S, 1, TO);  \
        else GO_NV(S, 2, TO);                    \
    } while (0)
#define GO_S(TO)                     \
    do {                             \
        if (s == 1) GO_T(1, TO);     \
        else if (s == 2) GO_T(2, TO); \
        else if (s == 3) GO_T(3, TO); \
        else GO_T(4, TO);            \
    } while (0)
        if (out_dtype == ODIN_BF16) GO_S(bf16);
        else GO_S(float);
#undef GO_S
#undef GO_T
#undef GO_NV
#undef GO
        ODIN_LAUNCH_CHECK();
        return 0;
    }
    const size_t smem = (size_t)2 * d * sizeof(float);
    if (smem > 200 * 1024) return ODIN_ERR_UNSUPPORTED;
#define GO(TO)                                                                                                       \
    do {                                                                                                             \
        auto kern = vec ? mix_streams_kernel<TO, true> : mix_streams_kernel<TO, false>;                              \
        if (smem > 48 * 1024) {                                                                                      \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);       \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        odin_launch(kern, dim3(n_rows), dim3(STREAM_THREADS), smem, st, a, (TO*)out);                                \
    } while (0)
    if (out_dtype == ODIN_BF16) GO(bf16);
    else GO(float);
#undef GO
    ODIN_LAUNCH_CHECK();
    return 0;
}
