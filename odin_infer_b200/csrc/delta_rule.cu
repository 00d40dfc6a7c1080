// The gated delta rule: a recurrence over a matrix-valued state S (key channel x value channel) per head whose write
// corrects what the state already answers to the token's key.  With unit keys k and queries q (q also times a factor),
// one decay g = exp(-exp(A) softplus(a + bias)) and one write strength beta = sigmoid(b) per head and token:
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// A column of S meets the other columns nowhere, so columns are spread over lanes and CTAs as in the linear recurrences
// (recurrent.cu): column j belongs to four lanes of a warp, each holding a quarter of the key channels in registers, and a
// sequence's tokens are walked in order.  Both sums over the channels are formed in one pass over the state as it was
// before the token, S^T k = g (S_old^T k) and o = g (S_old^T q) + (q . k) u, and keys and queries stay as they come from
// the projections: their unit norms are numbers per token (r_k, r_q) that multiply the sums.
//
// Long prompts in blocks: within a block the state is S_t = M_t S_in + L_t, where L_t is the walk from zeros and M_t, the
// product of the block's steps g (1 - beta k k^T), is the walk from the unit matrix with values of zero: its columns are walked
// as dk further columns.  Their outputs are M_t^T q_t, which is what a token's output needs of the state at the block's
// start.  A second kernel carries the state from block to block (S_in(next) = M S_in + L), a third adds (M_t^T q_t)^T S_in
// to every token's output.
//
// Everything is 32-bit.  Multiply-adds run two channels at a time (fma.rn.f32x2: each half rounds as a single fma does).
#include "recurrence_blocks.cuh"

typedef unsigned long long f32x2;   // two 32-bit floats of neighbouring channels, the first in the low half

__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float sum2(f32x2 v) {
    float a, b;
    unpack2(v, a, b);
    return a + b;
}

struct DeltaParams {
    RecParams r;                              // q, k, v and g (raw decay input a, [rows, H]); c0 = A, c1 = the decay's bias, [H] each
    const float* beta; long long beta_stride; // raw write strengths b, [rows, H]
    float unit_eps;                           // inside the root of the unit norms
    float* m_loc;                             // [sequences * n_blocks][H][dk][dk]: a block's M
};

// What a token asks of the walk beside its vectors.
struct __align__(16) TokenNumbers { float g, beta, rk, rq, kq; };

template <int SL, bool BLOCKS>
__global__ void __launch_bounds__(REC_COLS * REC_SPLIT)
delta_rule_kernel(DeltaParams dp) {
    const RecParams& p = dp.r;
    constexpr int NK = SL * REC_SPLIT;             // key channels the registers hold (dk <= NK)
    constexpr int TOK = NK > 128 ? 8 : 16;
    constexpr int NKP = NK + 4 * REC_SPLIT;        // the four parts of a warp read different banks (see recurrent.cu)
    constexpr bool KEEP_K = SL <= 32;              // the key's channels stay in registers between the sums and the update
    __shared__ __align__(16) float sq[TOK][NKP], sk[TOK][NKP];
    __shared__ float sv[TOK][REC_COLS];
    __shared__ float s_a[TOK], s_b[TOK];
    __shared__ TokenNumbers s_n[TOK];
    pdl_trigger();
    const int b = BLOCKS ? blockIdx.x / p.n_blocks : blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int ccols = blockDim.x / REC_SPLIT;      // columns of this CTA
    const int z_state = (p.dv + ccols - 1) / ccols;
    const bool is_m = BLOCKS && (int)blockIdx.z >= z_state;   // this CTA walks columns of M
    const int n_cols = is_m ? p.dk : p.dv;
    const int col0 = (is_m ? (int)blockIdx.z - z_state : (int)blockIdx.z) * ccols;
    const int part = lane >> 3, cj = warp * 8 + (lane & 7), j = col0 + cj;
    const int dk = p.dk;
    const int seq_end = p.seq_start[b + 1];
    const int row0 = p.seq_start[b] + (BLOCKS ? (int)(blockIdx.x % p.n_blocks) * p.block_len : 0);
    const int row1 = BLOCKS ? min(seq_end, row0 + p.block_len) : seq_end;
    const int slot = p.seq_slots[b];
    const int qc = (head / p.heads_per_group) * dk;           // the head's columns of q and k
    const float decay_rate = expf(p.c0.at(head)), decay_bias = p.c1.at(head);
    const int tok = max(1, min(TOK, REC_FETCH * (int)blockDim.x / NK));
    pdl_wait();
    if (row1 <= row0) return;  // an empty (padding) sequence owns no state
    const bool owns = j < n_cols;
    const int i0 = part * SL;
    float* st = !BLOCKS ? p.state + (size_t)slot * p.state_stride + (size_t)head * dk * p.dv + j
                : is_m  ? dp.m_loc + ((size_t)blockIdx.x * p.H + head) * dk * dk + j
                        : p.s_loc + ((size_t)blockIdx.x * p.H + head) * dk * p.dv + j;
    f32x2 S[SL / 2];
#pragma unroll
    for (int i = 0; i < SL; i += 2) {
        float v[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int ch = i0 + i + e;
            v[e] = 0.f;
            if (!BLOCKS) { if (owns && ch < dk) v[e] = st[(size_t)ch * p.dv]; }
            else if (is_m && ch == j) v[e] = 1.f;
        }
        S[i / 2] = pack2(v[0], v[1]);
    }
    float* out = is_m ? p.qp + (size_t)head * dk + j : p.o + (size_t)head * p.dv + j;
    const size_t out_stride = is_m ? (size_t)p.H * dk : (size_t)p.o_stride;

    float rq[REC_FETCH], rk[REC_FETCH], rv[REC_FETCH], ra = 0.f, rb = 0.f;
    auto fetch = [&](int t0, int nt) {
        if ((int)threadIdx.x < nt) {
            ra = p.g[(size_t)(t0 + threadIdx.x) * p.g_stride + head];
            rb = dp.beta[(size_t)(t0 + threadIdx.x) * dp.beta_stride + head];
        }
#pragma unroll
        for (int f = 0; f < REC_FETCH; ++f) {
            const int e = threadIdx.x + f * blockDim.x;
            rq[f] = rk[f] = rv[f] = 0.f;   // channels beyond dk: nothing in, nothing kept
            if (e < nt * NK) {
                const int u = e / NK, i = e % NK;
                if (i < dk) {
                    rq[f] = p.q[(size_t)(t0 + u) * p.q_stride + qc + i];
                    rk[f] = p.k[(size_t)(t0 + u) * p.k_stride + qc + i];
                }
            }
            if (!is_m && e < nt * ccols) {
                const int u = e / ccols, c = col0 + e % ccols;
                if (c < p.dv) rv[f] = p.v[(size_t)(t0 + u) * p.v_stride + (size_t)head * p.dv + c];
            }
        }
    };
    fetch(row0, min(tok, row1 - row0));
    for (int t0 = row0; t0 < row1; t0 += tok) {
        const int nt = min(tok, row1 - t0);
        __syncthreads();   // the tokens before have been walked
        if ((int)threadIdx.x < nt) { s_a[threadIdx.x] = ra; s_b[threadIdx.x] = rb; }
#pragma unroll
        for (int f = 0; f < REC_FETCH; ++f) {
            const int e = threadIdx.x + f * blockDim.x;
            if (e < nt * NK) {
                const int u = e / NK, i = e % NK, ip = i + (i / SL) * 4;
                sq[u][ip] = rq[f]; sk[u][ip] = rk[f];
            }
            if (e < nt * ccols) sv[e / ccols][e % ccols] = rv[f];
        }
        __syncthreads();
        if (t0 + tok < row1) fetch(t0 + tok, min(tok, row1 - t0 - tok));
        for (int u = warp; u < nt; u += n_warps) {   // a warp per token: its unit norms, its decay, its write strength
            float qq = 0.f, kk = 0.f, qk = 0.f;
            for (int i = lane; i < NK; i += 32) {
                const int ip = i + (i / SL) * 4;
                const float qv = sq[u][ip], kv = sk[u][ip];
                qq = fmaf(qv, qv, qq); kk = fmaf(kv, kv, kk); qk = fmaf(qv, kv, qk);
            }
            qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
            if (lane == 0) {
                TokenNumbers n;
                n.rq = p.q_scale / sqrtf(qq + dp.unit_eps);
                n.rk = 1.0f / sqrtf(kk + dp.unit_eps);
                n.kq = qk * n.rq * n.rk;
                const float z = s_a[u] + decay_bias;
                n.g = expf(-decay_rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
                n.beta = 1.0f / (1.0f + expf(-s_b[u]));
                s_n[u] = n;
            }
        }
        __syncthreads();
        for (int u = 0; u < nt; ++u) {
            const TokenNumbers n = s_n[u];
            const float* kr = &sk[u][i0 + part * 4];
            const float* qr = &sq[u][i0 + part * 4];
            f32x2 kreg[KEEP_K ? SL / 2 : 1];
            f32x2 ka0 = 0ull, ka1 = 0ull, qa0 = 0ull, qa1 = 0ull;
#pragma unroll
            for (int i = 0; i < SL; i += 4) {
                const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(kr + i);
                const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(qr + i);
                if (KEEP_K) { kreg[KEEP_K ? i / 2 : 0] = k4.x; kreg[KEEP_K ? i / 2 + 1 : 0] = k4.y; }
                ka0 = fma2(k4.x, S[i / 2], ka0);
                ka1 = fma2(k4.y, S[i / 2 + 1], ka1);
                qa0 = fma2(q4.x, S[i / 2], qa0);
                qa1 = fma2(q4.y, S[i / 2 + 1], qa1);
            }
            float ks = sum2(add2(ka0, ka1)), qs = sum2(add2(qa0, qa1));
            ks += __shfl_xor_sync(0xffffffffu, ks, 8);
            qs += __shfl_xor_sync(0xffffffffu, qs, 8);
            ks += __shfl_xor_sync(0xffffffffu, ks, 16);
            qs += __shfl_xor_sync(0xffffffffu, qs, 16);
            const float w = n.beta * (sv[u][cj] - n.g * (n.rk * ks));
            if (owns && part == 0) out[(size_t)(t0 + u) * out_stride] = fmaf(n.kq, w, n.g * (n.rq * qs));
            const float kw = n.rk * w;
            const f32x2 w2 = pack2(kw, kw), g2 = pack2(n.g, n.g);
#pragma unroll
            for (int i = 0; i < SL; i += 4) {
                if (KEEP_K) {
                    S[i / 2] = fma2(kreg[KEEP_K ? i / 2 : 0], w2, mul2(g2, S[i / 2]));
                    S[i / 2 + 1] = fma2(kreg[KEEP_K ? i / 2 + 1 : 0], w2, mul2(g2, S[i / 2 + 1]));
                } else {
                    const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(kr + i);
                    S[i / 2] = fma2(k4.x, w2, mul2(g2, S[i / 2]));
                    S[i / 2 + 1] = fma2(k4.y, w2, mul2(g2, S[i / 2 + 1]));
                }
            }
        }
    }
    const size_t pitch = is_m ? (size_t)dk : (size_t)p.dv;
#pragma unroll
    for (int i = 0; i < SL; i += 2) {
        float v[2];
        unpack2(S[i / 2], v[0], v[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e)
            if (owns && i0 + i + e < dk) st[(size_t)(i0 + i + e) * pitch] = v[e];
    }
}

// The state from block to block, 32 columns per CTA: S_in(first) = the sequence's state, S_in(next) = M S_in + L.  s_loc (L)
// is overwritten with S_in, the last S becomes the sequence's state.  Shared memory: the 32 columns of S_in [dk][32] and 32
// columns of M [8 ROWS][32 + 4], the next 32 waiting in registers meanwhile; a warp forms ROWS rows of the product (rows
// warp + 8 r), a lane its column of them.  Sums run over M's columns in their order, even and odd ones apart.
#define DC_COLS 32
#define DC_K 32
template <int ROWS>
__global__ void __launch_bounds__(256)
delta_carry_kernel(DeltaParams dp) {
    const RecParams& p = dp.r;
    extern __shared__ __align__(16) float dc_smem[];
    constexpr int MP = DC_K + 4;
    const int dkp = (p.dk + DC_K - 1) / DC_K * DC_K;          // S rows, zeros beyond dk
    float* Ss = dc_smem;                                      // [dkp][DC_COLS]
    float* Ms = dc_smem + (size_t)dkp * DC_COLS;              // [8 ROWS][MP]
    pdl_trigger();
    const int b = blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int col = blockIdx.z * DC_COLS + lane;
    const int row0 = p.seq_start[b], row1 = p.seq_start[b + 1];
    const int slot = p.seq_slots[b];
    pdl_wait();
    if (row1 <= row0) return;
    const bool owns = col < p.dv;
    const int dk = p.dk, n = (row1 - row0 + p.block_len - 1) / p.block_len, n_k = dkp / DC_K;
    float* st = p.state + (size_t)slot * p.state_stride + (size_t)head * dk * p.dv + col;
    float S[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int i = warp + 8 * r;
        S[r] = (owns && i < dk) ? st[(size_t)i * p.dv] : 0.f;
    }
    for (int i = warp; i < dkp; i += 8)
        if (i >= 8 * ROWS) Ss[i * DC_COLS + lane] = 0.f;
    float mreg[ROWS];
    auto fetch_m = [&](int c, int kk) {
        const float* m = dp.m_loc + (((size_t)b * p.n_blocks + c) * p.H + head) * (size_t)dk * dk + kk * DC_K + lane;
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const int i = warp + 8 * r;
            mreg[r] = (i < dk && kk * DC_K + lane < dk) ? __ldg(m + (size_t)i * dk) : 0.f;
        }
    };
    fetch_m(0, 0);
    for (int c = 0; c < n; ++c) {
        float* loc = p.s_loc + (((size_t)b * p.n_blocks + c) * p.H + head) * (size_t)dk * p.dv + col;
        float own[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const int i = warp + 8 * r;
            own[r] = 0.f;
            if (owns && i < dk) {
                own[r] = loc[(size_t)i * p.dv];
                loc[(size_t)i * p.dv] = S[r];
            }
            if (i < dkp) Ss[i * DC_COLS + lane] = S[r];
        }
        f32x2 acc[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) acc[r] = 0ull;
        for (int kk = 0; kk < n_k; ++kk) {
            __syncthreads();   // the columns of M before have been read (and, the first time, S_in is being written)
#pragma unroll
            for (int r = 0; r < ROWS; ++r) Ms[(warp + 8 * r) * MP + lane] = mreg[r];
            __syncthreads();
            if (kk + 1 < n_k) fetch_m(c, kk + 1);
            else if (c + 1 < n) fetch_m(c + 1, 0);
#pragma unroll
            for (int k = 0; k < DC_K; k += 4) {
                const float* sp = Ss + (kk * DC_K + k) * DC_COLS + lane;
                const f32x2 s01 = pack2(sp[0], sp[DC_COLS]), s23 = pack2(sp[2 * DC_COLS], sp[3 * DC_COLS]);
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    const ulonglong2 m4 = *reinterpret_cast<const ulonglong2*>(&Ms[(warp + 8 * r) * MP + k]);
                    acc[r] = fma2(m4.x, s01, acc[r]);
                    acc[r] = fma2(m4.y, s23, acc[r]);
                }
            }
        }
        __syncthreads();       // S_in has been read by everyone
#pragma unroll
        for (int r = 0; r < ROWS; ++r) S[r] = own[r] + sum2(acc[r]);
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int i = warp + 8 * r;
        if (owns && i < dk) st[(size_t)i * p.dv] = S[r];
    }
}

extern "C" int odin_delta_rule(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                               long long v_stride, const float* a, long long a_stride, const float* beta,
                               long long beta_stride, const void* A, const void* a_bias, int c_dtype, float* o,
                               long long o_stride, float* state, long long state_stride, const int* seq_start,
                               const int* seq_slots, int n_seqs, int H, int dk, int dv, int heads_per_group, float q_scale,
                               float unit_eps, int block_len, int n_blocks, float* qp, float* s_loc, float* m_loc,
                               void* stream) {
    if (n_seqs <= 0) return 0;
    if (block_len < 0 || (block_len > 0 && (n_blocks <= 0 || qp == nullptr || s_loc == nullptr || m_loc == nullptr ||
                                            (long long)n_seqs * n_blocks > 2147483647LL)))
        return ODIN_ERR_BAD_ARG;
    if (H <= 0 || dk <= 0 || dk > REC_MAX_DK || dv <= 0 || dv > 1024 || H > 65535) return ODIN_ERR_UNSUPPORTED;
    if (heads_per_group <= 0 || H % heads_per_group != 0) return ODIN_ERR_BAD_ARG;
    DeltaParams dp = {};
    RecParams& p = dp.r;
    p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride;
    p.g = a; p.g_stride = a_stride; dp.beta = beta; dp.beta_stride = beta_stride;
    p.c0 = VecRef{A, c_dtype == ODIN_BF16}; p.c1 = VecRef{a_bias, c_dtype == ODIN_BF16};
    p.o = o; p.o_stride = o_stride; p.state = state; p.state_stride = state_stride;
    p.seq_start = seq_start; p.seq_slots = seq_slots; p.H = H; p.dk = dk; p.dv = dv;
    p.heads_per_group = heads_per_group; p.q_scale = q_scale; dp.unit_eps = unit_eps;
    p.block_len = block_len; p.n_blocks = n_blocks; p.qp = qp; p.s_loc = s_loc; dp.m_loc = m_loc;
    const bool blocks = block_len > 0;
    const int n_items = blocks ? n_seqs * n_blocks : n_seqs;
    cudaStream_t s = (cudaStream_t)stream;
    // columns per CTA: as the linear recurrences choose them
    int cols = (dv < REC_COLS ? dv : REC_COLS);
    cols = (cols + 7) / 8 * 8;
    const int extra = blocks ? dk : 0;
    while (cols > 32 && (cols / 2) % 8 == 0 &&
           (long long)n_items * H * ((dv + cols - 1) / cols + (extra + cols - 1) / cols) < 2 * 148) cols /= 2;
    const int sl = dk <= 16 ? 4 : dk <= 32 ? 8 : dk <= 48 ? 12 : dk <= 64 ? 16 : dk <= 96 ? 24 : dk <= 128 ? 32 : 64;
    if (cols * REC_SPLIT * REC_FETCH < sl * REC_SPLIT) cols = (sl / REC_FETCH + 7) / 8 * 8;
    const int threads = cols * REC_SPLIT;      // a warp per eight columns
    dim3 grid(n_items, H, (dv + cols - 1) / cols + (extra + cols - 1) / cols);
#define GO(SL)                                                                                         \
    do {                                                                                               \
        if (blocks) odin_launch(delta_rule_kernel<SL, true>, grid, dim3(threads), 0, s, dp);           \
        else odin_launch(delta_rule_kernel<SL, false>, grid, dim3(threads), 0, s, dp);                 \
    } while (0)
    if (dk <= 16) GO(4);
    else if (dk <= 32) GO(8);
    else if (dk <= 48) GO(12);
    else if (dk <= 64) GO(16);
    else if (dk <= 96) GO(24);
    else if (dk <= 128) GO(32);
    else GO(64);
#undef GO
    ODIN_LAUNCH_CHECK();
    if (!blocks) return 0;
    const dim3 cgrid(n_seqs, H, (dv + DC_COLS - 1) / DC_COLS);
#define CARRY(ROWS)                                                                                                       \
    do {                                                                                                                  \
        const size_t smem = ((size_t)((dk + DC_K - 1) / DC_K * DC_K) * DC_COLS + (size_t)8 * (ROWS) * (DC_K + 4)) * sizeof(float); \
        if (smem > 48 * 1024) {                                                                                           \
            cudaError_t e = cudaFuncSetAttribute(delta_carry_kernel<ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                          \
        }                                                                                                                 \
        odin_launch(delta_carry_kernel<ROWS>, cgrid, dim3(256), smem, s, dp);                                             \
    } while (0)
    if (dk <= 32) CARRY(4);
    else if (dk <= 64) CARRY(8);
    else if (dk <= 96) CARRY(12);
    else if (dk <= 128) CARRY(16);
    else CARRY(32);
#undef CARRY
    ODIN_LAUNCH_CHECK();
    return launch_recurrence_carry_out(p, n_items, s);
}
