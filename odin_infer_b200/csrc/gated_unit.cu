// A real-gated linear recurrent unit: one state number per channel.  Per token, with zr and zi the raw gates (products of
// the channel's block of u, without their biases) and ld = -sharpness * softplus(lam) of the channel:
//
//   r = sigmoid(zr + br);   i = sigmoid(zi + bi);   log a = ld * r;   S = a S + sqrt(1 - a^2) i u;   out = S * gelu_tanh(y + by)
//
//   step   one token per sequence: the block's gate products, the update and the output in one kernel;
//   scan   prompts and pieces of prompts: the raw gates come from a product per block; every sequence's rows are cut into
//          blocks of tokens, one kernel leaves each block's own state and decay (and the tokens' decays in place of their raw
//          gates), a second carries the states to the block's start and walks the block's tokens once more with their outputs.
//
// Gates, decays, exponentials and the state are 32-bit.  sqrt(1 - a^2) is taken of -expm1(2 log a), which keeps its digits
// where a is close to 1.  Raw gates and their biases lie block by block: [r of the block's m channels | i of them].
#include "common.cuh"

#define GU_CH 32       // channels of a CTA of the step kernel
#define GU_TOK 8       // tokens of a CTA of the step kernel
#define GU_SLICES 8    // parts into which it cuts the input channels
#define GU_PRE 32      // weights that a thread of it fetches at once
#define GU_STEP_THREADS (2 * GU_CH * GU_SLICES)
#define GU_THREADS 128

__device__ __forceinline__ float gu_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float gu_gelu(float z) {   // z sigmoid(2 t) = z (1 + tanh(t)) / 2, t = sqrt(2 / pi) (z + 0.044715 z^3)
    return z * gu_sigmoid(1.5957691216057308f * z * fmaf(0.044715f * z, z, 1.0f));
}
// the token's decay and what it adds, of its raw gates with their biases
__device__ __forceinline__ void gu_token(float zr, float zi, float ld, float u, float& a, float& in) {
    const float la = ld * gu_sigmoid(zr);
    a = expf(la);
    in = sqrtf(-expm1f(2.0f * la)) * (gu_sigmoid(zi) * u);
}

// grid (channel parts of a block, blocks, tokens / GU_TOK).  w: [blocks][m][2 m] (input channel before output column; the r
// columns before the i columns).  A thread forms one gate (r or i) of one of the CTA's channels over its slice of the input
// channels, for GU_TOK tokens; the slices' shares are added in their order, and a thread per (channel, token) updates the state.
// A slice's weights are all fetched at once, the first ones while the kernel before this one still runs.  (What earlier kernels
// write carries no __restrict__: the compiler may move loads through such const pointers ahead of the wait.)
template <typename T, typename TW>
__global__ void __launch_bounds__(GU_STEP_THREADS)
gated_unit_step_kernel(const T* u, const TW* __restrict__ w, const float* __restrict__ bias,
                       const float* __restrict__ log_decay, const T* y, size_t y_stride, const float* __restrict__ y_bias,
                       float* state, size_t state_stride, T* out, const int* __restrict__ tok_seq,
                       const int* __restrict__ seq_slots, int n_rows, int n, int m) {
    extern __shared__ __align__(16) float us[];   // [m][GU_TOK]
    __shared__ __align__(16) float part[GU_SLICES][2 * GU_CH][GU_TOK + 4];   // rows 48 bytes apart: 16-byte stores of eight lanes cover all banks
    pdl_trigger();
    const int blk = blockIdx.y, t0 = blockIdx.z * GU_TOK, ch0 = blockIdx.x * GU_CH;
    const int slice = threadIdx.x / (2 * GU_CH), gk = threadIdx.x % (2 * GU_CH), side = gk / GU_CH, k = gk % GU_CH;
    const bool has = ch0 + k < m;
    const int N = 2 * m;
    const TW* wc = w + (size_t)blk * m * N + side * m + ch0 + k;
    // the slice's input channels: GU_PRE of every GU_PRE * GU_SLICES
    TW cur[GU_PRE];
    auto fetch = [&](int k0) {
        if (!has || k0 >= m) return;
        if (k0 + GU_PRE <= m) {
#pragma unroll
            for (int j = 0; j < GU_PRE; ++j) cur[j] = wc[(size_t)(k0 + j) * N];
        } else {
#pragma unroll
            for (int j = 0; j < GU_PRE; ++j)
                if (k0 + j < m) cur[j] = wc[(size_t)(k0 + j) * N];
        }
    };
    fetch(slice * GU_PRE);
    // who updates what afterwards: threads 0 .. GU_CH * GU_TOK - 1, channels in neighbouring lanes
    const int uk = threadIdx.x % GU_CH, ut = (threadIdx.x / GU_CH) % GU_TOK, t = t0 + ut;
    const bool updates = threadIdx.x < GU_CH * GU_TOK && ch0 + uk < m && t < n_rows;
    const int c = blk * m + ch0 + uk;
    float br = 0.f, bi = 0.f, ld = 0.f, yb = 0.f, S = 0.f, yv = 0.f;
    int slot = -1;
    if (updates) {
        const int seq = tok_seq[t];
        if (seq >= 0) slot = seq_slots[seq];
        br = bias[(size_t)blk * N + ch0 + uk]; bi = bias[(size_t)blk * N + m + ch0 + uk];
        ld = log_decay[c]; yb = y_bias[c];
    }
    pdl_wait();
    for (int e = threadIdx.x; e < m * GU_TOK; e += GU_STEP_THREADS) {   // consecutive threads along the channels
        const int tu = e / m, i = e % m;
        us[i * GU_TOK + tu] = t0 + tu < n_rows ? to_f32(u[(size_t)(t0 + tu) * n + (size_t)blk * m + i]) : 0.f;
    }
    if (slot >= 0) {
        S = state[(size_t)slot * state_stride + c];
        yv = to_f32(y[(size_t)t * y_stride + c]);
    }
    __syncthreads();
    float acc[GU_TOK];
#pragma unroll
    for (int q = 0; q < GU_TOK; ++q) acc[q] = 0.f;
    auto take = [&](int i, TW wk) {
        const float wv = to_f32(wk);
        const float4 a0 = *reinterpret_cast<const float4*>(&us[i * GU_TOK]);
        const float4 a1 = *reinterpret_cast<const float4*>(&us[i * GU_TOK + 4]);
        acc[0] = fmaf(wv, a0.x, acc[0]); acc[1] = fmaf(wv, a0.y, acc[1]);
        acc[2] = fmaf(wv, a0.z, acc[2]); acc[3] = fmaf(wv, a0.w, acc[3]);
        acc[4] = fmaf(wv, a1.x, acc[4]); acc[5] = fmaf(wv, a1.y, acc[5]);
        acc[6] = fmaf(wv, a1.z, acc[6]); acc[7] = fmaf(wv, a1.w, acc[7]);
    };
    for (int k0 = slice * GU_PRE; k0 < m; k0 += GU_PRE * GU_SLICES) {
        if (k0 != slice * GU_PRE) fetch(k0);
        if (!has) continue;
        if (k0 + GU_PRE <= m) {
#pragma unroll
            for (int j = 0; j < GU_PRE; ++j) {
                take(k0 + j, cur[j]);
                if (j % 4 == 3) asm volatile("" ::: "memory");   // a few reads of shared memory ahead, not all of them
            }
        } else {
#pragma unroll
            for (int j = 0; j < GU_PRE; ++j)
                if (k0 + j < m) take(k0 + j, cur[j]);
        }
    }
    st4(&part[slice][gk][0], make_float4(acc[0], acc[1], acc[2], acc[3]));
    st4(&part[slice][gk][4], make_float4(acc[4], acc[5], acc[6], acc[7]));
    __syncthreads();
    if (slot < 0) return;
    float zr = br, zi = bi;
#pragma unroll
    for (int q = 0; q < GU_SLICES; ++q) { zr += part[q][uk][ut]; zi += part[q][GU_CH + uk][ut]; }
    float a, in;
    gu_token(zr, zi, ld, us[(ch0 + uk) * GU_TOK + ut], a, in);
    S = fmaf(a, S, in);
    state[(size_t)slot * state_stride + c] = S;
    out[(size_t)t * n + c] = from_f32<T>(S * gu_gelu(yv + yb));
}

extern "C" int odin_gated_unit_step(const void* u, int dtype, const void* w, int w_dtype, const float* bias,
                                    const float* log_decay, const void* y, long long y_stride, const float* y_bias,
                                    float* state, long long state_stride, void* out, const int* tok_seq, const int* seq_slots,
                                    int n_rows, int n, int blocks, void* stream) {
    if (n_rows <= 0) return 0;
    if (n <= 0 || blocks <= 0 || blocks > 65535 || n % blocks != 0) return ODIN_ERR_BAD_ARG;
    const int m = n / blocks;
    const size_t smem = (size_t)m * GU_TOK * sizeof(float);
    if (smem > 160 * 1024 || (n_rows + GU_TOK - 1) / GU_TOK > 65535) return ODIN_ERR_UNSUPPORTED;
    const dim3 grid((m + GU_CH - 1) / GU_CH, blocks, (n_rows + GU_TOK - 1) / GU_TOK);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, TW)                                                                                                    \
    do {                                                                                                             \
        if (smem > 20 * 1024) {                                                                                      \
            cudaError_t e = cudaFuncSetAttribute(gated_unit_step_kernel<T, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        odin_launch(gated_unit_step_kernel<T, TW>, grid, dim3(GU_STEP_THREADS), smem, s, (const T*)u, (const TW*)w, bias, log_decay, \
                    (const T*)y, (size_t)y_stride, y_bias, state, (size_t)state_stride, (T*)out, tok_seq, seq_slots, n_rows, n, m); \
    } while (0)
    if (dtype == ODIN_BF16 && w_dtype == ODIN_BF16) GO(bf16, bf16);
    else if (dtype == ODIN_F32 && w_dtype == ODIN_F32) GO(float, float);
    else if (dtype == ODIN_BF16 && w_dtype == ODIN_F32) GO(bf16, float);
    else return ODIN_ERR_UNSUPPORTED;
#undef GO
    ODIN_LAUNCH_CHECK();
    return 0;
}

// ------------------------------------------------------------ prompts
struct UnitScan {
    const void* u; const void* y; void* out; size_t y_stride;   // u, out: [rows][n]; y: its columns of a wider row
    float* raw; const float* bias;                              // [rows][2 n] (the first pass leaves decays and inputs in it), [2 n]
    const float* log_decay; const float* y_bias;
    float* state; size_t state_stride;
    float* s_own; float* d_own; float* s_first;                 // [sequences * n_blocks][n] twice, [sequences][n]
    const int* seq_start; const int* seq_slots;
    int n, m, block_len, n_blocks;
};

#define GU_OWN 0     // first pass: every block's own state and the product of its decays
#define GU_OUT 1     // second pass: the state at the block's start out of those, the outputs, the sequence's state
#define GU_ONE 2     // one block: everything at once

// One thread per channel and block of tokens, channels in neighbouring lanes.  The first pass turns the raw gates in place into
// (decay, what is added) for the second; its first block starts from the sequence's state, which it also keeps in s_first,
// because the second pass's last block writes the state while its first may still run.
template <typename T, int PASS>
__global__ void __launch_bounds__(GU_THREADS)
gated_unit_scan_kernel(UnitScan p) {
    pdl_trigger();
    const int b = blockIdx.x / p.n_blocks, blk = blockIdx.x % p.n_blocks;
    const int c = blockIdx.y * GU_THREADS + threadIdx.x;
    const int seq0 = p.seq_start[b], seq1 = p.seq_start[b + 1], slot = p.seq_slots[b];
    const int row0 = seq0 + blk * p.block_len, row1 = min(seq1, row0 + p.block_len);
    const int at = (c / p.m) * 2 * p.m + c % p.m;
    constexpr bool GATES = PASS != GU_OUT, OUT = PASS != GU_OWN;
    float br = 0.f, bi = 0.f, ld = 0.f, yb = 0.f;
    if (c < p.n) {
        if (GATES) { br = p.bias[at]; bi = p.bias[at + p.m]; ld = p.log_decay[c]; }
        if (OUT) yb = p.y_bias[c];
    }
    pdl_wait();
    if (row1 <= row0 || c >= p.n) return;   // an empty (padding) sequence owns no state
    float S = 0.f, D = 1.f;
    if (PASS == GU_OUT) {
        if (blk == 0) S = p.s_first[(size_t)b * p.n + c];
        constexpr int CB = 8;   // the loads of eight blocks go out together
        for (int k0 = 0; k0 < blk; k0 += CB) {
            float own[CB], dec[CB];
#pragma unroll
            for (int q = 0; q < CB; ++q) {
                own[q] = 0.f;
                dec[q] = 1.f;
                if (k0 + q < blk) {
                    const size_t item = (size_t)b * p.n_blocks + k0 + q;
                    own[q] = p.s_own[item * p.n + c];
                    dec[q] = k0 + q == 0 ? 0.f : p.d_own[item * p.n + c];   // the first block's state has the sequence's in it
                }
            }
#pragma unroll
            for (int q = 0; q < CB; ++q) S = fmaf(dec[q], S, own[q]);
        }
    } else if (blk == 0) {
        S = p.state[(size_t)slot * p.state_stride + c];
        if (PASS == GU_OWN) p.s_first[(size_t)b * p.n + c] = S;
    }
    constexpr int U = 8;        // the loads of eight tokens go out together, and before the eight tokens before them are worked on
    float z0[U], z1[U], uv[U], yv[U], n0[U], n1[U], nu[U], ny[U];
    auto fetch = [&](int t0, float (&r0)[U], float (&r1)[U], float (&ru)[U], float (&ry)[U]) {
#pragma unroll
        for (int q = 0; q < U; ++q) {
            r0[q] = r1[q] = ru[q] = ry[q] = 0.f;
            if (t0 + q < row1) {
                const size_t r = (size_t)(t0 + q);
                r0[q] = p.raw[r * 2 * p.n + at];
                r1[q] = p.raw[r * 2 * p.n + at + p.m];
                if (GATES) ru[q] = to_f32(((const T*)p.u)[r * p.n + c]);
                if (OUT) ry[q] = to_f32(((const T*)p.y)[r * p.y_stride + c]);
            }
        }
    };
    fetch(row0, z0, z1, uv, yv);
    for (int t0 = row0; t0 < row1; t0 += U) {
        if (t0 + U < row1) fetch(t0 + U, n0, n1, nu, ny);
        float av[U], in[U];
#pragma unroll
        for (int q = 0; q < U; ++q) {
            if (GATES) gu_token(z0[q] + br, z1[q] + bi, ld, uv[q], av[q], in[q]);
            else { av[q] = z0[q]; in[q] = z1[q]; }
        }
#pragma unroll
        for (int q = 0; q < U; ++q) {
            if (t0 + q >= row1) break;
            const size_t r = (size_t)(t0 + q);
            S = fmaf(av[q], S, in[q]);
            if (OUT) {
                ((T*)p.out)[r * p.n + c] = from_f32<T>(S * gu_gelu(yv[q] + yb));
            } else {
                D *= av[q];
                p.raw[r * 2 * p.n + at] = av[q];
                p.raw[r * 2 * p.n + at + p.m] = in[q];
            }
        }
#pragma unroll
        for (int q = 0; q < U; ++q) { z0[q] = n0[q]; z1[q] = n1[q]; uv[q] = nu[q]; yv[q] = ny[q]; }
    }
    if (OUT) {
        if (row1 == seq1) p.state[(size_t)slot * p.state_stride + c] = S;
    } else {
        p.s_own[(size_t)blockIdx.x * p.n + c] = S;
        p.d_own[(size_t)blockIdx.x * p.n + c] = D;
    }
}

extern "C" int odin_gated_unit_scan(const void* u, int dtype, float* raw, const float* bias, const float* log_decay,
                                    const void* y, long long y_stride, const float* y_bias, float* state,
                                    long long state_stride, void* out, const int* seq_start, const int* seq_slots, int n_seqs,
                                    int n, int blocks, int block_len, int n_blocks, float* s_own, float* d_own, float* s_first,
                                    void* stream) {
    if (n_seqs <= 0) return 0;
    if (n <= 0 || blocks <= 0 || n % blocks != 0 || block_len <= 0 || n_blocks <= 0) return ODIN_ERR_BAD_ARG;
    if (n_blocks > 1 && (s_own == nullptr || d_own == nullptr || s_first == nullptr)) return ODIN_ERR_BAD_ARG;
    if ((long long)n_seqs * n_blocks > 2147483647LL || (n + GU_THREADS - 1) / GU_THREADS > 65535) return ODIN_ERR_UNSUPPORTED;
    UnitScan p{u, y, out, (size_t)y_stride, raw, bias, log_decay, y_bias, state, (size_t)state_stride, s_own, d_own, s_first,
               seq_start, seq_slots, n, n / blocks, block_len, n_blocks};
    const dim3 grid((unsigned)(n_seqs * n_blocks), (n + GU_THREADS - 1) / GU_THREADS), threads(GU_THREADS);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype != ODIN_BF16 && dtype != ODIN_F32) return ODIN_ERR_UNSUPPORTED;
    const bool half = dtype == ODIN_BF16;
    if (n_blocks == 1) {
        odin_launch(half ? gated_unit_scan_kernel<bf16, GU_ONE> : gated_unit_scan_kernel<float, GU_ONE>, grid, threads, 0, s, p);
        ODIN_LAUNCH_CHECK();
        return 0;
    }
    odin_launch(half ? gated_unit_scan_kernel<bf16, GU_OWN> : gated_unit_scan_kernel<float, GU_OWN>, grid, threads, 0, s, p);
    ODIN_LAUNCH_CHECK();
    odin_launch(half ? gated_unit_scan_kernel<bf16, GU_OUT> : gated_unit_scan_kernel<float, GU_OUT>, grid, threads, 0, s, p);
    ODIN_LAUNCH_CHECK();
    return 0;
}
