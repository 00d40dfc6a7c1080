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
// Long prompts in chunks of 64 tokens: the writes w_t of a chunk solve a unit lower triangular system whose right hand side
// is linear in the state at the chunk's start (the "WY" form of a product of rank-one corrections), so that everything but
// one small product per chunk and column can be formed for all chunks at once.  With G_t the sum of the logarithms of the
// decays of a chunk's tokens up to t, S_0 the state at its start, and k, q the unit vectors (q with its factor):
//
//     (I + A) w = diag(beta) V - diag(beta exp(G)) K S_0,       A[t, s] = beta_t exp(G_t - G_s) (k_t . k_s)  for s < t
//     o = diag(exp(G)) Q S_0 + P w,                             P[t, s] = exp(G_t - G_s) (q_t . k_s)         for s <= t
//     S_end = exp(G_last) S_0 + K^T diag(exp(G_last - G)) w
//
// Three kernels: (1) per chunk and head A, P, and the two solutions U = (I + A)^-1 diag(beta) V and
// W = (I + A)^-1 diag(beta exp(G)) K; (2) per sequence, head and 16 columns, chunk after chunk, w = U - W S_0 and the next
// S_0; (3) per chunk and head the outputs.  All exponents are differences that are never positive.
//
// Everything is 32-bit.  The walk's multiply-adds run two channels at a time (fma.rn.f32x2: each half rounds as a single
// fma does).
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

__device__ __forceinline__ ulonglong2 ld2x2(const float* p) { return *reinterpret_cast<const ulonglong2*>(p); }

struct DeltaParams {
    RecParams r;                              // q, k, v and g (raw decay input a, [rows, H]); c0 = A, c1 = the decay's bias, [H] each
    const float* beta; long long beta_stride; // raw write strengths b, [rows, H]
    float unit_eps;                           // inside the root of the unit norms
};

// One token's decay (as a logarithm) and write strength.
__device__ __forceinline__ float delta_log_decay(float a, float bias, float rate) {
    const float z = a + bias;
    return -rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}
__device__ __forceinline__ float delta_beta(float b) { return 1.0f / (1.0f + expf(-b)); }

// What a token asks of the walk beside its vectors.
struct __align__(16) TokenNumbers { float g, beta, rk, rq, kq; };

template <int SL>
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
    const int b = blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int ccols = blockDim.x / REC_SPLIT;      // columns of this CTA
    const int col0 = (int)blockIdx.z * ccols;
    const int part = lane >> 3, cj = warp * 8 + (lane & 7), j = col0 + cj;
    const int dk = p.dk;
    const int row0 = p.seq_start[b], row1 = p.seq_start[b + 1];
    const int slot = p.seq_slots[b];
    const int qc = (head / p.heads_per_group) * dk;           // the head's columns of q and k
    const float decay_rate = expf(p.c0.at(head)), decay_bias = p.c1.at(head);
    const int tok = max(1, min(TOK, REC_FETCH * (int)blockDim.x / NK));
    if (row1 <= row0) { pdl_wait(); return; }  // an empty (padding) sequence owns no state
    const bool owns = j < p.dv;
    const int i0 = part * SL;
    float* st = p.state + (size_t)slot * p.state_stride + (size_t)head * dk * p.dv + j;
    // no other kernel of a step touches this layer's state: it is fetched while the kernel before this one still runs
    f32x2 S[SL / 2];
    const bool whole = owns && i0 + SL <= dk;   // every channel of this lane exists: its loads go out together
    {
        float v[SL];
        const float* sr = st + (size_t)i0 * p.dv;
        if (whole) {
#pragma unroll
            for (int i = 0; i < SL; ++i) v[i] = sr[(size_t)i * p.dv];
        } else {
#pragma unroll
            for (int i = 0; i < SL; ++i) v[i] = (owns && i0 + i < dk) ? sr[(size_t)i * p.dv] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < SL; i += 2) S[i / 2] = pack2(v[i], v[i + 1]);
    }
    pdl_wait();
    float* out = p.o + (size_t)head * p.dv + j;

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
            if (e < nt * ccols) {
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
                n.g = expf(delta_log_decay(s_a[u], decay_bias, decay_rate));
                n.beta = delta_beta(s_b[u]);
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
            if (owns && part == 0) out[(size_t)(t0 + u) * p.o_stride] = fmaf(n.kq, w, n.g * (n.rq * qs));
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
#pragma unroll
    for (int i = 0; i < SL; i += 2) {
        float v[2];
        unpack2(S[i / 2], v[0], v[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e)
            if (owns && i0 + i + e < dk) st[(size_t)(i0 + i + e) * p.dv] = v[e];
    }
}

// ------------------------------------------------------------ chunks of 64 tokens
#define DC_TOK 64     // tokens of a chunk
#define DC_COLS 16    // columns of S per CTA of the kernel that carries the state
#define DC_OCOLS 64   // columns per CTA of the kernel that forms the outputs
#define DC_P (DC_TOK + 4)   // row length of P and of A
struct DeltaChunks {
    int n_chunks;      // most chunks that a sequence of the step brings
    // Where a chunk's scratch lies: sequence b's chunks from seq_start[b] / 64 + b on, which no other sequence's reach, so that
    // the scratch grows with the step's rows and not with the longest sequence times the sequences ("items" below).
    __device__ __forceinline__ static int place(const RecParams& p, int b, int chunk) { return p.seq_start[b] / 64 + b + chunk; }
    int vec;           // rows of q and k are whole 16-byte pieces
    int dkp, dvp;      // dk and dv rounded up to multiples of 4 and of 16: the scratch rows' lengths, zeros beyond dk and dv
    // every matrix lies in memory as the kernels hold it in shared memory (rows of dkp + 4 or of 68 where lanes read rows side by
    // side), so that a copy is one run of 16-byte pieces
    float* kt;         // [items][H][64][dkp]      k_t exp(G_last - G_t)
    float* qt;         // [items][H][64][dkp + 4]  q_t exp(G_t)
    float* w;          // [items][H][64][dkp + 4]  W
    float* u;          // [items][H][dvp / 16][64][16]  U, then the writes w
    float* pm;         // [items][H][64][68]       P
    float* s_in;       // [items][H][dkp][dvp] the state at the chunk's start
    float* g_last;     // [items][H]           exp(G_last)
};

__device__ __forceinline__ void cp_async16(float* smem, const float* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
// n floats (a multiple of 4) by all threads of the CTA
__device__ __forceinline__ void cp_run(float* smem, const float* gmem, int n) {
    for (int e = threadIdx.x * 4; e < n; e += blockDim.x * 4) cp_async16(smem + e, gmem + e);
}
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// (1) grid (items, H).  Shared memory: K and Q [64][dkp + 4] (Q's place later holds solved rows), A transposed [64][68],
// numbers per token.
__global__ void __launch_bounds__(256, 2)
delta_chunk_prepare_kernel(DeltaParams dp, DeltaChunks c) {
    const RecParams& p = dp.r;
    extern __shared__ __align__(16) float cs_smem[];
    const int ld = c.dkp + 4, dk = p.dk;
    float* Ks = cs_smem;
    float* Qs = Ks + DC_TOK * ld;
    float* At = Qs + max(DC_TOK * ld, 32 * 256);   // At[s][t]
    constexpr int AP = DC_P;
    float* beta = At + DC_TOK * AP;
    float* G = beta + DC_TOK;                 // first the logarithms of the decays, then their running sum
    float* bg = G + DC_TOK;                   // beta exp(G)
    pdl_trigger();
    const int item = blockIdx.x, head = blockIdx.y, b = item / c.n_chunks, tid = threadIdx.x;
    const int lane = tid & 31, warp = tid >> 5;
    const int row0 = p.seq_start[b] + (item % c.n_chunks) * DC_TOK;
    const int nt = min(DC_TOK, p.seq_start[b + 1] - row0);
    const float rate = expf(p.c0.at(head)), bias = p.c1.at(head);
    const int qc = (head / p.heads_per_group) * dk;
    pdl_wait();
    if (nt <= 0) return;
    // the rows of q and k as they are: all their loads go out together (in pieces of 16 bytes where the rows allow it)
    for (int t = warp; t < DC_TOK; t += 8) {
        const float* qr = p.q + (size_t)(row0 + t) * p.q_stride + qc;
        const float* kr = p.k + (size_t)(row0 + t) * p.k_stride + qc;
        if (c.vec && t < nt) {
            for (int i = lane * 4; i < dk; i += 128) { cp_async16(Qs + t * ld + i, qr + i); cp_async16(Ks + t * ld + i, kr + i); }
        } else {
            for (int i = lane; i < c.dkp; i += 32) {
                const bool in = t < nt && i < dk;
                Qs[t * ld + i] = in ? qr[i] : 0.f;
                Ks[t * ld + i] = in ? kr[i] : 0.f;
            }
        }
    }
    cp_commit();
    if (tid < DC_TOK) {   // rows beyond the sequence: nothing is written, nothing decays
        beta[tid] = tid < nt ? delta_beta(dp.beta[(size_t)(row0 + tid) * dp.beta_stride + head]) : 0.f;
        G[tid] = tid < nt ? delta_log_decay(p.g[(size_t)(row0 + tid) * p.g_stride + head], bias, rate) : 0.f;
    }
    cp_wait<0>();
    __syncthreads();
    // a warp per token: the unit norms
    for (int t = warp; t < DC_TOK; t += 8) {
        float qq = 0.f, kk = 0.f;
        for (int i = lane; i < c.dkp; i += 32) {
            const float qv = Qs[t * ld + i], kv = Ks[t * ld + i];
            qq = fmaf(qv, qv, qq); kk = fmaf(kv, kv, kk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk);
        const float rq = p.q_scale / sqrtf(qq + dp.unit_eps), rk = 1.0f / sqrtf(kk + dp.unit_eps);
        for (int i = lane; i < c.dkp; i += 32) { Qs[t * ld + i] *= rq; Ks[t * ld + i] *= rk; }
    }
    if (warp == 0) {      // running sum of 64 logarithms, two to a lane
        const float a0 = G[2 * lane], a1 = G[2 * lane + 1];
        float s = a0 + a1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += v;
        }
        const float before = __shfl_up_sync(0xffffffffu, s, 1);
        const float base = lane > 0 ? before : 0.f;
        G[2 * lane] = base + a0;
        G[2 * lane + 1] = base + a0 + a1;
        bg[2 * lane] = beta[2 * lane] * expf(base + a0);
        bg[2 * lane + 1] = beta[2 * lane + 1] * expf(base + a0 + a1);
    }
    __syncthreads();
    // k_t . k_s and q_t . k_s: a thread takes rows t = ty + 16 i and s = tx + 16 j
    const int ty = tid >> 4, tx = tid & 15;
    f32x2 kk[4][4], qk[4][4];                 // even and odd channels' sums
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) kk[i][j] = qk[i][j] = 0ull;
    for (int k = 0; k < c.dkp; k += 4) {
        ulonglong2 bs[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) bs[j] = ld2x2(Ks + (tx + 16 * j) * ld + k);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const ulonglong2 ka = ld2x2(Ks + (ty + 16 * i) * ld + k), qa = ld2x2(Qs + (ty + 16 * i) * ld + k);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                kk[i][j] = fma2(ka.x, bs[j].x, kk[i][j]); kk[i][j] = fma2(ka.y, bs[j].y, kk[i][j]);
                qk[i][j] = fma2(qa.x, bs[j].x, qk[i][j]); qk[i][j] = fma2(qa.y, bs[j].y, qk[i][j]);
            }
        }
    }
    const size_t ih = (size_t)DeltaChunks::place(p, b, item % c.n_chunks) * p.H + head;
    float* pm = c.pm + ih * DC_TOK * DC_P;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = ty + 16 * i, s = tx + 16 * j;
            const float ratio = s <= t ? expf(G[t] - G[s]) : 0.f;
            At[s * AP + t] = s < t ? beta[t] * ratio * sum2(kk[i][j]) : 0.f;
            pm[t * DC_P + s] = ratio * sum2(qk[i][j]);
        }
    __syncthreads();
    const float g_last = G[DC_TOK - 1];
    if (tid == 0) c.g_last[ih] = expf(g_last);
    // q and k as the other kernels want them
    float* kt = c.kt + ih * DC_TOK * c.dkp;
    float* qt = c.qt + ih * DC_TOK * ld;
    for (int t = warp; t < DC_TOK; t += 8) {
        const float fk = expf(g_last - G[t]), fq = expf(G[t]);
        for (int i = lane; i < c.dkp; i += 32) {
            kt[t * c.dkp + i] = Ks[t * ld + i] * fk;
            qt[t * ld + i] = Qs[t * ld + i] * fq;
        }
    }
    __syncthreads();   // Q is done with
    // The two triangular systems: a thread solves for a column, 32 rows at a time; once x_s is known it leaves the later rows
    // of its half at once, and the second half takes the first one's 32 values off before it is solved.
    float* wo = c.w + ih * DC_TOK * ld;
    float* uo = c.u + ih * DC_TOK * c.dvp;
    float* X = Qs + tid;                       // [32][256]: this thread's column of the first half
    for (int col = tid; col < c.dkp + c.dvp; col += 256) {
        const bool is_k = col < c.dkp;
        const int cc = is_k ? col : col - c.dkp;
        float* dst = is_k ? wo + cc : uo + (size_t)(cc / DC_COLS) * DC_TOK * DC_COLS + cc % DC_COLS;
        const int pitch = is_k ? ld : DC_COLS;
        const float* vr = p.v + (size_t)row0 * p.v_stride + (size_t)head * p.dv + cc;
#pragma unroll 1
        for (int h0 = 0; h0 < DC_TOK; h0 += 32) {
            f32x2 x[16];                       // rows h0 + 2 i and h0 + 2 i + 1
            if (is_k) {
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const int t = h0 + 2 * i;
                    x[i] = pack2(Ks[t * ld + cc] * bg[t], Ks[(t + 1) * ld + cc] * bg[t + 1]);
                }
            } else {
                float v[32];                   // all loads first (rows beyond the sequence read its last row, and beta is zero there)
                const bool in = cc < p.dv;
#pragma unroll
                for (int t = 0; t < 32; ++t) v[t] = in ? __ldg(vr + (size_t)min(h0 + t, nt - 1) * p.v_stride) : 0.f;
#pragma unroll
                for (int i = 0; i < 16; ++i)
                    x[i] = pack2(v[2 * i] * beta[h0 + 2 * i], v[2 * i + 1] * beta[h0 + 2 * i + 1]);
            }
            if (h0 > 0) {
#pragma unroll 2
                for (int s = 0; s < 32; ++s) {
                    const float xs = -X[s * 256];
                    const f32x2 xs2 = pack2(xs, xs);
                    const float* ar = At + s * AP + 32;
#pragma unroll
                    for (int i = 0; i < 16; i += 2) {
                        const ulonglong2 a = ld2x2(ar + 2 * i);
                        x[i] = fma2(a.x, xs2, x[i]);
                        x[i + 1] = fma2(a.y, xs2, x[i + 1]);
                    }
                }
            }
            const float* ah = At + h0 * AP + h0;
#pragma unroll
            for (int s = 0; s < 31; ++s) {
                float lo, hi;
                unpack2(x[s / 2], lo, hi);
                const float xs = (s & 1) ? -hi : -lo;
                const f32x2 xs2 = pack2(xs, xs);
#pragma unroll
                for (int i = (s + 1) / 4 * 2; i < 16; i += 2) {   // A is zero up to and with t = s: solved rows stay as they are
                    const ulonglong2 a = ld2x2(ah + s * AP + 2 * i);
                    if (2 * i + 1 > s) x[i] = fma2(a.x, xs2, x[i]);
                    x[i + 1] = fma2(a.y, xs2, x[i + 1]);
                }
            }
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float v[2];
                unpack2(x[i], v[0], v[1]);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    dst[(h0 + 2 * i + e) * pitch] = v[e];
                    if (h0 == 0) X[(2 * i + e) * 256] = v[e];
                }
            }
        }
    }
}

// (2) grid (sequences, H, dvp / 16), 512 threads.  w = U - W S: each quarter of the CTA takes a quarter of the channels, a
// thread four tokens by two columns; S <- g S + kt^T w: a quarter of the tokens each, a thread four channels by four columns
// (RK times).  The quarters' sums meet in shared memory and are added in the order of the quarters.  The state lives in the
// registers of all threads (one channel by four columns, RK times) and, transposed, in shared memory.  W of the next chunk
// arrives while S is updated, kt and U while W S is formed.
template <int RK>
__global__ void __launch_bounds__(512)
delta_chunk_carry_kernel(DeltaParams dp, DeltaChunks c) {
    const RecParams& p = dp.r;
    extern __shared__ __align__(16) float cs_smem[];
    const int ld = c.dkp + 4, dk = p.dk;
    float* Wb = cs_smem;                       // [64][ld]
    float* Kb = Wb + DC_TOK * ld;              // [64][dkp]
    float* Ub = Kb + DC_TOK * c.dkp;           // [64][16]
    float* St = Ub + DC_TOK * DC_COLS;         // [16][ld]
    float* Red = St + DC_COLS * ld;            // [4][16 RK][128]
    pdl_trigger();
    const int b = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * DC_COLS, tid = threadIdx.x;
    const int row0 = p.seq_start[b], n_new = p.seq_start[b + 1] - row0;
    const int slot = p.seq_slots[b];
    const int quarter = tid >> 7, lid = tid & 127;
    pdl_wait();
    if (n_new <= 0) return;
    const int n = (n_new + DC_TOK - 1) / DC_TOK, n4 = c.dkp / 4, place0 = DeltaChunks::place(p, b, 0);
    auto base = [&](int ch) { return ((size_t)place0 + ch) * p.H + head; };
    auto load_w = [&](int ch) {
        cp_run(Wb, c.w + base(ch) * DC_TOK * ld, DC_TOK * ld);
        cp_commit();
    };
    auto load_ku = [&](int ch) {
        cp_run(Kb, c.kt + base(ch) * DC_TOK * c.dkp, DC_TOK * c.dkp);
        cp_run(Ub, c.u + base(ch) * DC_TOK * c.dvp + (size_t)blockIdx.z * DC_TOK * DC_COLS, DC_TOK * DC_COLS);
        cp_commit();
    };
    load_w(0);
    load_ku(0);
    // S: channels (kg + 32 r) 4 + quarter, columns 4 cg .. + 3; its update: channels (kg + 32 r) 4 .. + 3, the same columns
    const int cg = lid & 3, kg = lid >> 2;
    float S[RK][4];
    float* st = p.state + (size_t)slot * p.state_stride + (size_t)head * dk * p.dv;
#pragma unroll
    for (int r = 0; r < RK; ++r) {
        const int k = (kg + 32 * r) * 4 + quarter;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int col = col0 + cg * 4 + j;
            S[r][j] = (k < dk && col < p.dv) ? st[(size_t)k * p.dv + col] : 0.f;
            if (k < c.dkp) St[(cg * 4 + j) * ld + k] = S[r][j];
        }
    }
    const int cp = lid & 7, tg = lid >> 3;     // W S: columns cp and cp + 8, tokens tg + 16 i
    const int k_lo = n4 * quarter / 4 * 4, k_hi = n4 * (quarter + 1) / 4 * 4;
    for (int ch = 0; ch < n; ++ch) {
        const float g = c.g_last[base(ch)];
        float* si = c.s_in + base(ch) * (size_t)c.dkp * c.dvp + col0 + cg * 4;   // what this chunk's tokens look at
#pragma unroll
        for (int r = 0; r < RK; ++r) {
            const int k = (kg + 32 * r) * 4 + quarter;
            if (k < c.dkp) st4(si + (size_t)k * c.dvp, make_float4(S[r][0], S[r][1], S[r][2], S[r][3]));
        }
        cp_wait<1>();
        __syncthreads();                       // W is there, and S in shared memory
        f32x2 acc[4][2];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0ull;
#pragma unroll 4
        for (int k = k_lo; k < k_hi; k += 4) {
            const ulonglong2 s0 = ld2x2(St + cp * ld + k), s1 = ld2x2(St + (cp + 8) * ld + k);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const ulonglong2 w = ld2x2(Wb + (tg + 16 * i) * ld + k);
                acc[i][0] = fma2(w.x, s0.x, acc[i][0]); acc[i][1] = fma2(w.x, s1.x, acc[i][1]);
                acc[i][0] = fma2(w.y, s0.y, acc[i][0]); acc[i][1] = fma2(w.y, s1.y, acc[i][1]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            Red[(quarter * 8 + 2 * i) * 128 + lid] = sum2(acc[i][0]);
            Red[(quarter * 8 + 2 * i + 1) * 128 + lid] = sum2(acc[i][1]);
        }
        cp_wait<0>();
        __syncthreads();                       // kt and U are there, W has been read
        {
            float* uo = c.u + base(ch) * DC_TOK * c.dvp + (size_t)blockIdx.z * DC_TOK * DC_COLS;
#pragma unroll
            for (int j = 0; j < 2; ++j) {      // this thread adds up the pair (token tg + 16 quarter, column cp + 8 j)
                const int at = (2 * quarter + j) * 128 + lid, e = (tg + 16 * quarter) * DC_COLS + cp + 8 * j;
                const float w = Ub[e] - (((Red[at] + Red[8 * 128 + at]) + Red[16 * 128 + at]) + Red[24 * 128 + at]);
                Ub[e] = w;
                uo[e] = w;
            }
        }
        if (ch + 1 < n) load_w(ch + 1);
        __syncthreads();                       // the writes are there
        f32x2 d[RK][4][2];                     // pairs of columns
#pragma unroll
        for (int r = 0; r < RK; ++r)
#pragma unroll
            for (int i = 0; i < 4; ++i) d[r][i][0] = d[r][i][1] = 0ull;
#pragma unroll 8
        for (int t = quarter * 16; t < quarter * 16 + 16; ++t) {
            const ulonglong2 u4 = ld2x2(Ub + t * DC_COLS + cg * 4);
#pragma unroll
            for (int r = 0; r < RK; ++r) {
                const int k = (kg + 32 * r) * 4;
                if (k >= c.dkp) continue;
                const float4 k4 = ld4(Kb + t * c.dkp + k);
                const f32x2 kv[4] = {pack2(k4.x, k4.x), pack2(k4.y, k4.y), pack2(k4.z, k4.z), pack2(k4.w, k4.w)};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    d[r][i][0] = fma2(kv[i], u4.x, d[r][i][0]);
                    d[r][i][1] = fma2(kv[i], u4.y, d[r][i][1]);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < RK; ++r)
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    float lo, hi;
                    unpack2(d[r][i][j], lo, hi);
                    Red[((quarter * RK + r) * 16 + i * 4 + 2 * j) * 128 + lid] = lo;
                    Red[((quarter * RK + r) * 16 + i * 4 + 2 * j + 1) * 128 + lid] = hi;
                }
        __syncthreads();                       // kt and the writes have been read
        if (ch + 1 < n) load_ku(ch + 1);
#pragma unroll
        for (int r = 0; r < RK; ++r) {
            const int k = (kg + 32 * r) * 4 + quarter;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int at = (r * 16 + quarter * 4 + j) * 128 + lid;
                constexpr int Q = RK * 16 * 128;
                S[r][j] = fmaf(g, S[r][j], ((Red[at] + Red[Q + at]) + Red[2 * Q + at]) + Red[3 * Q + at]);
                if (k < c.dkp) St[(cg * 4 + j) * ld + k] = S[r][j];
            }
        }
    }
#pragma unroll
    for (int r = 0; r < RK; ++r)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int k = (kg + 32 * r) * 4 + quarter, col = col0 + cg * 4 + j;
            if (k < dk && col < p.dv) st[(size_t)k * p.dv + col] = S[r][j];
        }
}

// (3) grid (items, H, columns / 64): o = qt S_in + P w, 64 tokens by 64 columns, four by four to a thread.
__global__ void __launch_bounds__(256, 2)
delta_chunk_output_kernel(DeltaParams dp, DeltaChunks c) {
    const RecParams& p = dp.r;
    extern __shared__ __align__(16) float cs_smem[];
    const int ld = c.dkp + 4;
    float* Qs = cs_smem;                        // [64][ld]
    float* Ss = Qs + DC_TOK * ld;               // [dkp][64]
    float* Ps = Ss + (size_t)c.dkp * DC_OCOLS;  // [64][68]
    float* Us = Ps + DC_TOK * DC_P;             // [64][64]
    pdl_trigger();
    const int item = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * DC_OCOLS, tid = threadIdx.x;
    const int b = item / c.n_chunks;
    const int row0 = p.seq_start[b] + (item % c.n_chunks) * DC_TOK;
    const int nt = min(DC_TOK, p.seq_start[b + 1] - row0);
    pdl_wait();
    if (nt <= 0) return;
    const size_t ih = (size_t)DeltaChunks::place(p, b, item % c.n_chunks) * p.H + head;
    const int nc4 = min(DC_OCOLS, c.dvp - col0) / 4;
    cp_run(Qs, c.qt + ih * DC_TOK * ld, DC_TOK * ld);
    const float* si = c.s_in + ih * (size_t)c.dkp * c.dvp + col0;
    for (int e = tid; e < c.dkp * (DC_OCOLS / 4); e += 256)
        if ((e & 15) < nc4) cp_async16(Ss + e * 4, si + (size_t)(e >> 4) * c.dvp + (e & 15) * 4);
    cp_commit();
    cp_run(Ps, c.pm + ih * DC_TOK * DC_P, DC_TOK * DC_P);
    const float* us = c.u + ih * DC_TOK * c.dvp + (size_t)(col0 / DC_COLS) * DC_TOK * DC_COLS;
    for (int e = tid; e < DC_TOK * (DC_OCOLS / 4); e += 256)   // token e / 16, columns 4 (e % 16) .. + 3: a piece of tile (e % 16) / 4
        if ((e & 15) < nc4) cp_async16(Us + e * 4, us + ((size_t)((e & 15) >> 2) * DC_TOK + (e >> 4)) * DC_COLS + (e & 3) * 4);
    cp_commit();
    const int ty = tid >> 4, tx = tid & 15;
    f32x2 acc[4][2];                            // pairs of columns
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0ull;
    auto product = [&](const float* A, int lda, const float* B, int K) {
#pragma unroll 2
        for (int k = 0; k < K; k += 4) {
            ulonglong2 b4[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) b4[e] = ld2x2(B + (k + e) * DC_OCOLS + tx * 4);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float4 a4 = ld4(A + (ty + 16 * i) * lda + k);
                const f32x2 a[4] = {pack2(a4.x, a4.x), pack2(a4.y, a4.y), pack2(a4.z, a4.z), pack2(a4.w, a4.w)};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[i][0] = fma2(a[e], b4[e].x, acc[i][0]);
                    acc[i][1] = fma2(a[e], b4[e].y, acc[i][1]);
                }
            }
        }
    };
    cp_wait<1>();
    __syncthreads();
    if (tx < nc4) product(Qs, ld, Ss, c.dkp);
    cp_wait<0>();
    __syncthreads();
    if (tx < nc4) product(Ps, DC_P, Us, DC_TOK);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty + 16 * i;
        if (t >= nt) continue;
        float* o = p.o + (size_t)(row0 + t) * p.o_stride + (size_t)head * p.dv;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            float v[2];
            unpack2(acc[i][j], v[0], v[1]);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int col = col0 + tx * 4 + 2 * j + e;
                if (tx < nc4 && col < p.dv) o[col] = v[e];
            }
        }
    }
}

template <typename... A>
static int set_smem(void (*kern)(A...), size_t bytes) {
    if (bytes > 227 * 1024) return ODIN_ERR_UNSUPPORTED;
    if (bytes <= 48 * 1024) return 0;
    return (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

// Floats of scratch that the chunked form needs for a step of T rows.
extern "C" long long odin_delta_rule_scratch(int T, int n_seqs, int H, int dk, int dv) {
    const long long n_items = (long long)T / DC_TOK + n_seqs + 1;
    const long long dkp = (dk + 3) / 4 * 4, dvp = (dv + 15) / 16 * 16;
    return n_items * H * (DC_TOK * (3 * dkp + 8) + DC_TOK * dvp + (long long)DC_TOK * DC_P + dkp * dvp + 4);
}

// n_chunks 0: the walk; else the most chunks of 64 tokens that a sequence of this step brings, with scratch as above
// (16-byte aligned).
extern "C" int odin_delta_rule(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                               long long v_stride, const float* a, long long a_stride, const float* beta,
                               long long beta_stride, const void* A, const void* a_bias, int c_dtype, float* o,
                               long long o_stride, float* state, long long state_stride, const int* seq_start,
                               const int* seq_slots, int n_seqs, int H, int dk, int dv, int heads_per_group, float q_scale,
                               float unit_eps, int T, int n_chunks, float* scratch, void* stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || dk <= 0 || dk > REC_MAX_DK || dv <= 0 || dv > 1024 || H > 65535) return ODIN_ERR_UNSUPPORTED;
    if (heads_per_group <= 0 || H % heads_per_group != 0 || n_chunks < 0) return ODIN_ERR_BAD_ARG;
    DeltaParams dp = {};
    RecParams& p = dp.r;
    p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride;
    p.g = a; p.g_stride = a_stride; dp.beta = beta; dp.beta_stride = beta_stride;
    p.c0 = VecRef{A, c_dtype == ODIN_BF16}; p.c1 = VecRef{a_bias, c_dtype == ODIN_BF16};
    p.o = o; p.o_stride = o_stride; p.state = state; p.state_stride = state_stride;
    p.seq_start = seq_start; p.seq_slots = seq_slots; p.H = H; p.dk = dk; p.dv = dv;
    p.heads_per_group = heads_per_group; p.q_scale = q_scale; dp.unit_eps = unit_eps;
    cudaStream_t s = (cudaStream_t)stream;
    if (n_chunks > 0) {
        const long long n_items = (long long)n_seqs * n_chunks;
        if (scratch == nullptr || (((uintptr_t)scratch) & 15) != 0 || n_items > 2147483647LL) return ODIN_ERR_BAD_ARG;
        DeltaChunks c;
        c.vec = dk % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && ((((uintptr_t)q) | ((uintptr_t)k)) & 15) == 0;
        c.n_chunks = n_chunks; c.dkp = (dk + 3) / 4 * 4; c.dvp = (dv + 15) / 16 * 16;
        const size_t ih = ((size_t)T / DC_TOK + n_seqs + 1) * H;
        const size_t ld = c.dkp + 4;
        c.kt = scratch; c.qt = c.kt + ih * DC_TOK * c.dkp; c.w = c.qt + ih * DC_TOK * ld;
        c.u = c.w + ih * DC_TOK * ld; c.pm = c.u + ih * DC_TOK * c.dvp; c.s_in = c.pm + ih * DC_TOK * DC_P;
        c.g_last = c.s_in + ih * (size_t)c.dkp * c.dvp;
        const size_t q_or_x = DC_TOK * ld > 32 * 256 ? DC_TOK * ld : 32 * 256;
        const size_t smem1 = (DC_TOK * ld + q_or_x + DC_TOK * DC_P + 3 * DC_TOK) * sizeof(float);
        const int rk = dk <= 128 ? 1 : 2;
        const size_t smem2 = (DC_TOK * ld + (size_t)DC_TOK * c.dkp + DC_TOK * DC_COLS + DC_COLS * ld + (size_t)4 * 16 * rk * 128) * sizeof(float);
        const size_t smem3 = (DC_TOK * ld + (size_t)c.dkp * DC_OCOLS + DC_TOK * DC_P + DC_TOK * DC_OCOLS) * sizeof(float);
        int rc;
        if ((rc = set_smem(delta_chunk_prepare_kernel, smem1)) || (rc = set_smem(delta_chunk_output_kernel, smem3)) ||
            (rc = rk == 1 ? set_smem(delta_chunk_carry_kernel<1>, smem2) : set_smem(delta_chunk_carry_kernel<2>, smem2)))
            return rc;
        odin_launch(delta_chunk_prepare_kernel, dim3((unsigned)n_items, H), dim3(256), smem1, s, dp, c);
        ODIN_LAUNCH_CHECK();
        const dim3 cgrid(n_seqs, H, c.dvp / DC_COLS);
        if (rk == 1) odin_launch(delta_chunk_carry_kernel<1>, cgrid, dim3(512), smem2, s, dp, c);
        else odin_launch(delta_chunk_carry_kernel<2>, cgrid, dim3(512), smem2, s, dp, c);
        ODIN_LAUNCH_CHECK();
        odin_launch(delta_chunk_output_kernel, dim3((unsigned)n_items, H, (c.dvp + DC_OCOLS - 1) / DC_OCOLS), dim3(256), smem3, s, dp, c);
        ODIN_LAUNCH_CHECK();
        return 0;
    }
    // columns per CTA: as the linear recurrences choose them
    int cols = (dv < REC_COLS ? dv : REC_COLS);
    cols = (cols + 7) / 8 * 8;
    while (cols > 32 && (cols / 2) % 8 == 0 && (long long)n_seqs * H * ((dv + cols - 1) / cols) < 2 * 148) cols /= 2;
    const int sl = dk <= 16 ? 4 : dk <= 32 ? 8 : dk <= 48 ? 12 : dk <= 64 ? 16 : dk <= 96 ? 24 : dk <= 128 ? 32 : 64;
    if (cols * REC_SPLIT * REC_FETCH < sl * REC_SPLIT) cols = (sl / REC_FETCH + 7) / 8 * 8;
    const dim3 grid(n_seqs, H, (dv + cols - 1) / cols), block(cols * REC_SPLIT);   // a warp per eight columns
    if (dk <= 16) odin_launch(delta_rule_kernel<4>, grid, block, 0, s, dp);
    else if (dk <= 32) odin_launch(delta_rule_kernel<8>, grid, block, 0, s, dp);
    else if (dk <= 48) odin_launch(delta_rule_kernel<12>, grid, block, 0, s, dp);
    else if (dk <= 64) odin_launch(delta_rule_kernel<16>, grid, block, 0, s, dp);
    else if (dk <= 96) odin_launch(delta_rule_kernel<24>, grid, block, 0, s, dp);
    else if (dk <= 128) odin_launch(delta_rule_kernel<32>, grid, block, 0, s, dp);
    else odin_launch(delta_rule_kernel<64>, grid, block, 0, s, dp);
    ODIN_LAUNCH_CHECK();
    return 0;
}
