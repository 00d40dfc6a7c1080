// A real-gated linear recurrent unit: one state number per channel.  Per token, with zr and zi the raw gates (products of
// the channel's block of u, without their biases) and ld = -sharpness * softplus(lam) of the channel:
//
//   r = sigmoid(zr + br);   i = sigmoid(zi + bi);   log a = ld * r;   S = a S + sqrt(1 - a^2) i u;   out = S * gelu_tanh(y + by)
//
//   step   one token per sequence: the block's gate products, the update and the output in one kernel;
//   scan   prompts and pieces of prompts: the raw gates come from a product per block; every sequence's rows are cut into
//          blocks of tokens, one kernel leaves each block's own state and decay, a second carries them to the block's start
//          and walks the block's tokens once more with their outputs.
//
// Gates, decays, exponentials and the state are 32-bit.  sqrt(1 - a^2) is taken of -expm1(2 log a), which keeps its digits
// where a is close to 1.  Raw gates and their biases lie block by block: [r of the block's m channels | i of them].
#include "common.cuh"

#define GU_CH 64       // channels of a CTA of the step kernel
#define GU_TOK 8       // tokens of a CTA of the step kernel
#define GU_PRE 32      // weights that a thread of it fetches ahead
#define GU_THREADS 128

__device__ __forceinline__ float gu_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gu_gelu(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// the token's decay and what it adds, of its raw gates with their biases
__device__ __forceinline__ void gu_token(float zr, float zi, float ld, float u, float& a, float& in) {
    const float la = ld * gu_sigmoid(zr);
    a = expf(la);
    in = sqrtf(-expm1f(2.0f * la)) * (gu_sigmoid(zi) * u);
}

// grid (channel parts of a block, blocks, tokens / GU_TOK).  w: [blocks][m][2 m] (input channel before output column; the r
// columns before the i columns).  Thread k < GU_CH forms the r gate of the CTA's channel k, thread GU_CH + k its i gate, each
// over the input channels in ascending order; then every thread takes one channel's update for half of the tokens.
template <typename T, typename TW>
__global__ void __launch_bounds__(GU_THREADS)
gated_unit_step_kernel(const T* __restrict__ u, const TW* __restrict__ w, const float* __restrict__ bias,
                       const float* __restrict__ log_decay, const T* __restrict__ y, size_t y_stride,
                       const float* __restrict__ y_bias, float* __restrict__ state, size_t state_stride, T* __restrict__ out,
                       const int* __restrict__ tok_seq, const int* __restrict__ seq_slots, int n_rows, int n, int m) {
    extern __shared__ __align__(16) float us[];   // [m][GU_TOK]
    __shared__ float z[2][GU_TOK][GU_CH];
    pdl_trigger();
    const int blk = blockIdx.y, t0 = blockIdx.z * GU_TOK, ch0 = blockIdx.x * GU_CH;
    const int side = threadIdx.x / GU_CH, k = threadIdx.x % GU_CH;
    const bool has = ch0 + k < m;
    const int col = side * m + ch0 + k, N = 2 * m;
    const TW* wc = w + (size_t)blk * m * N + col;
    TW cur[GU_PRE], nxt[GU_PRE];
    auto fetch = [&](TW (&dst)[GU_PRE], int k0) {
        if (!has) return;
#pragma unroll
        for (int j = 0; j < GU_PRE; ++j)
            if (k0 + j < m) dst[j] = wc[(size_t)(k0 + j) * N];
    };
    fetch(cur, 0);
    const int c = blk * m + ch0 + k;              // the channel of the whole row
    float b = 0.f, ld = 0.f, yb = 0.f;
    int slot[GU_TOK / 2];
    if (has) { b = bias[(size_t)blk * N + col]; ld = log_decay[c]; yb = y_bias[c]; }
#pragma unroll
    for (int q = 0; q < GU_TOK / 2; ++q) {
        const int t = t0 + side * (GU_TOK / 2) + q;
        const int seq = t < n_rows ? tok_seq[t] : -1;
        slot[q] = seq >= 0 ? seq_slots[seq] : -1;
    }
    pdl_wait();
    {   // sixteen threads per token
        const int tu = threadIdx.x / (GU_THREADS / GU_TOK), l = threadIdx.x % (GU_THREADS / GU_TOK);
        for (int i = l; i < m; i += GU_THREADS / GU_TOK)
            us[i * GU_TOK + tu] = t0 + tu < n_rows ? to_f32(u[(size_t)(t0 + tu) * n + (size_t)blk * m + i]) : 0.f;
    }
    float S[GU_TOK / 2], yv[GU_TOK / 2];
#pragma unroll
    for (int q = 0; q < GU_TOK / 2; ++q) {
        S[q] = yv[q] = 0.f;
        if (has && slot[q] >= 0) {
            S[q] = state[(size_t)slot[q] * state_stride + c];
            yv[q] = to_f32(y[(size_t)(t0 + side * (GU_TOK / 2) + q) * y_stride + c]);
        }
    }
    __syncthreads();
    float acc[GU_TOK];
#pragma unroll
    for (int q = 0; q < GU_TOK; ++q) acc[q] = 0.f;
    for (int k0 = 0; k0 < m; k0 += GU_PRE) {
        fetch(nxt, k0 + GU_PRE);
#pragma unroll
        for (int j = 0; j < GU_PRE; ++j)
            if (has && k0 + j < m) {
                const float wv = to_f32(cur[j]);
                const float4 a0 = *reinterpret_cast<const float4*>(&us[(k0 + j) * GU_TOK]);
                const float4 a1 = *reinterpret_cast<const float4*>(&us[(k0 + j) * GU_TOK + 4]);
                acc[0] = fmaf(wv, a0.x, acc[0]); acc[1] = fmaf(wv, a0.y, acc[1]);
                acc[2] = fmaf(wv, a0.z, acc[2]); acc[3] = fmaf(wv, a0.w, acc[3]);
                acc[4] = fmaf(wv, a1.x, acc[4]); acc[5] = fmaf(wv, a1.y, acc[5]);
                acc[6] = fmaf(wv, a1.z, acc[6]); acc[7] = fmaf(wv, a1.w, acc[7]);
            }
#pragma unroll
        for (int j = 0; j < GU_PRE; ++j) cur[j] = nxt[j];
    }
#pragma unroll
    for (int q = 0; q < GU_TOK; ++q) z[side][q][k] = acc[q] + b;
    __syncthreads();
    if (!has) return;
#pragma unroll
    for (int q = 0; q < GU_TOK / 2; ++q) {
        if (slot[q] < 0) continue;
        const int tq = side * (GU_TOK / 2) + q;
        float a, in;
        gu_token(z[0][tq][k], z[1][tq][k], ld, us[(ch0 + k) * GU_TOK + tq], a, in);
        const float s = fmaf(a, S[q], in);
        state[(size_t)slot[q] * state_stride + c] = s;
        out[(size_t)(t0 + tq) * n + c] = from_f32<T>(s * gu_gelu(yv[q] + yb));
    }
}

extern "C" int odin_gated_unit_step(const void* u, int dtype, const void* w, int w_dtype, const float* bias,
                                    const float* log_decay, const void* y, long long y_stride, const float* y_bias,
                                    float* state, long long state_stride, void* out, const int* tok_seq, const int* seq_slots,
                                    int n_rows, int n, int blocks, void* stream) {
    if (n_rows <= 0) return 0;
    if (n <= 0 || blocks <= 0 || blocks > 65535 || n % blocks != 0) return ODIN_ERR_BAD_ARG;
    const int m = n / blocks;
    const size_t smem = (size_t)m * GU_TOK * sizeof(float);
    if (smem > 200 * 1024 || (n_rows + GU_TOK - 1) / GU_TOK > 65535) return ODIN_ERR_UNSUPPORTED;
    const dim3 grid((m + GU_CH - 1) / GU_CH, blocks, (n_rows + GU_TOK - 1) / GU_TOK);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, TW)                                                                                                    \
    do {                                                                                                             \
        if (smem > 40 * 1024) {                                                                                      \
            cudaError_t e = cudaFuncSetAttribute(gated_unit_step_kernel<T, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        odin_launch(gated_unit_step_kernel<T, TW>, grid, dim3(GU_THREADS), smem, s, (const T*)u, (const TW*)w, bias, log_decay, \
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
    const float* raw; const float* bias;                        // [rows][2 n], [2 n]
    const float* log_decay; const float* y_bias;
    float* state; size_t state_stride;
    float* s_own; float* d_own; float* s_first;                 // [sequences * n_blocks][n] twice, [sequences][n]
    const int* seq_start; const int* seq_slots;
    int n, m, block_len, n_blocks;
};

// One thread per channel and block of tokens, channels in neighbouring lanes.  OUT false: the block's state from zeros (the
// first block: from the sequence's state, which it also keeps in s_first, because the last block writes the state while the
// first may still run) and the product of its decays; the last block is left to the second pass.  OUT true: the state at the
// block's start out of those, the tokens once more, their outputs, and after the last block the sequence's state.
template <typename T, bool OUT>
__global__ void __launch_bounds__(GU_THREADS)
gated_unit_scan_kernel(UnitScan p) {
    pdl_trigger();
    const int b = blockIdx.x / p.n_blocks, blk = blockIdx.x % p.n_blocks;
    const int c = blockIdx.y * GU_THREADS + threadIdx.x;
    const int seq0 = p.seq_start[b], seq1 = p.seq_start[b + 1], slot = p.seq_slots[b];
    const int row0 = seq0 + blk * p.block_len, row1 = min(seq1, row0 + p.block_len);
    const int at = (c / p.m) * 2 * p.m + c % p.m;
    float br = 0.f, bi = 0.f, ld = 0.f, yb = 0.f;
    if (c < p.n) { br = p.bias[at]; bi = p.bias[at + p.m]; ld = p.log_decay[c]; yb = p.y_bias[c]; }
    pdl_wait();
    if (row1 <= row0 || c >= p.n) return;   // an empty (padding) sequence owns no state
    float S = 0.f, D = 1.f;
    if (OUT) {
        if (blk == 0) S = p.n_blocks > 1 ? p.s_first[(size_t)b * p.n + c] : p.state[(size_t)slot * p.state_stride + c];
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
                    dec[q] = k0 + q == 0 ? 0.f : p.d_own[item * p.n + c];
                }
            }
#pragma unroll
            for (int q = 0; q < CB; ++q) S = fmaf(dec[q], S, own[q]);
        }
    } else if (blk == 0) {
        S = p.state[(size_t)slot * p.state_stride + c];
        p.s_first[(size_t)b * p.n + c] = S;
    }
    if (!OUT && row1 == seq1) return;
    constexpr int U = 8;        // the loads of eight tokens go out together
    for (int t0 = row0; t0 < row1; t0 += U) {
        float zr[U], zi[U], uv[U], yv[U];
#pragma unroll
        for (int q = 0; q < U; ++q) {
            zr[q] = zi[q] = uv[q] = yv[q] = 0.f;
            if (t0 + q < row1) {
                const size_t r = (size_t)(t0 + q);
                zr[q] = p.raw[r * 2 * p.n + at];
                zi[q] = p.raw[r * 2 * p.n + at + p.m];
                uv[q] = to_f32(((const T*)p.u)[r * p.n + c]);
                if (OUT) yv[q] = to_f32(((const T*)p.y)[r * p.y_stride + c]);
            }
        }
        float av[U], in[U];
#pragma unroll
        for (int q = 0; q < U; ++q) gu_token(zr[q] + br, zi[q] + bi, ld, uv[q], av[q], in[q]);
#pragma unroll
        for (int q = 0; q < U; ++q) {
            if (t0 + q >= row1) break;
            S = fmaf(av[q], S, in[q]);
            if (OUT) ((T*)p.out)[(size_t)(t0 + q) * p.n + c] = from_f32<T>(S * gu_gelu(yv[q] + yb));
            else D *= av[q];
        }
    }
    if (OUT) {
        if (row1 == seq1) p.state[(size_t)slot * p.state_stride + c] = S;
    } else {
        p.s_own[(size_t)blockIdx.x * p.n + c] = S;
        p.d_own[(size_t)blockIdx.x * p.n + c] = D;
    }
}

extern "C" int odin_gated_unit_scan(const void* u, int dtype, const float* raw, const float* bias, const float* log_decay,
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
    const dim3 grid((unsigned)(n_seqs * n_blocks), (n + GU_THREADS - 1) / GU_THREADS);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype != ODIN_BF16 && dtype != ODIN_F32) return ODIN_ERR_UNSUPPORTED;
    if (n_blocks > 1) {
        if (dtype == ODIN_BF16) odin_launch(gated_unit_scan_kernel<bf16, false>, grid, dim3(GU_THREADS), 0, s, p);
        else odin_launch(gated_unit_scan_kernel<float, false>, grid, dim3(GU_THREADS), 0, s, p);
        ODIN_LAUNCH_CHECK();
    }
    if (dtype == ODIN_BF16) odin_launch(gated_unit_scan_kernel<bf16, true>, grid, dim3(GU_THREADS), 0, s, p);
    else odin_launch(gated_unit_scan_kernel<float, true>, grid, dim3(GU_THREADS), 0, s, p);
    ODIN_LAUNCH_CHECK();
    return 0;
}
