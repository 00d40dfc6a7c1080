// Linear attention with one fixed decay w per head on long prompts,
//
//     S_t = w S_(t-1) + k_t v_t^T          o_t = S_t^T q_t          (q, k and v optionally through SiLU)
//
// in blocks of 128 tokens, everything but the state's way from block to block as products of tiles.  With t and s counted from
// a block's start and S_0 the state there:
//
//     o_t = w^(t+1) S_0^T q_t + sum_{s <= t} w^(t-s) (q_t . k_s) v_s          S_end = w^n S_0 + sum_t w^(n-1-t) k_t v_t^T
//
// Three kernels: (1) per block, head and tile of the state what the block itself adds; (2) the state from block to block;
// (3) per 64 tokens, head and tile of columns the outputs.  All exponents of w are >= 0.  Everything is 32-bit; the
// multiply-adds run two columns at a time (fma.rn.f32x2: each half rounds as a single fma does).
#include "common.cuh"

#define DB_TOK 128     // tokens of a block
#define DB_HALF 64     // tokens of a tile of outputs
#define DB_P (DB_HALF + 4)
#define DB_STAGE 32    // tokens that the first kernel holds in shared memory at once

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 db_pack(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void db_unpack(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 db_fma(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ ulonglong2 db_ld(const float* p) { return *reinterpret_cast<const ulonglong2*>(p); }

struct DecayBlocks {
    const float* q; const float* k; const float* v; long long q_stride, k_stride, v_stride;
    const float* decay; float* o; long long o_stride; float* state; long long state_stride;
    const int* seq_start; const int* seq_slots;
    int H, dk, dv, n_blocks, silu, vec;       // vec: rows of q, k, v and of the states are whole 16-byte pieces
    float* s;                                 // [sequences * n_blocks][H][dk][dv]: what a block adds, then the state at its start
};

__device__ __forceinline__ float db_act(float x, int silu) { return silu ? __fdividef(x, 1.0f + expf(-x)) : x; }

// rows [0, n_rows) of `rows` x `cols` (cols a multiple of 4) from gmem (row stride in elements) into shared memory rows of
// `pitch`, through SiLU where asked, row r times scale[r] where given; rows beyond n_rows and columns beyond n_cols are zeros
__device__ __forceinline__ void db_stage(float* dst, int pitch, const float* src, long long stride, int rows, int n_rows, int cols,
                                         int n_cols, int silu, int vec, const float* scale) {
    const int per = cols / 4;
    constexpr int U = 4;   // a thread's loads of four pieces go out together
    for (int e0 = threadIdx.x; e0 < rows * per; e0 += blockDim.x * U) {
        float4 x[U];
#pragma unroll
        for (int q = 0; q < U; ++q) {
            const int e = e0 + q * blockDim.x, r = e / per, c = (e % per) * 4;
            x[q] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (e >= rows * per || r >= n_rows) continue;
            const float* g = src + (size_t)r * stride + c;
            if (vec && c + 4 <= n_cols) x[q] = ld4(g);
            else {
                if (c < n_cols) x[q].x = g[0];
                if (c + 1 < n_cols) x[q].y = g[1];
                if (c + 2 < n_cols) x[q].z = g[2];
                if (c + 3 < n_cols) x[q].w = g[3];
            }
        }
#pragma unroll
        for (int q = 0; q < U; ++q) {
            const int e = e0 + q * blockDim.x, r = e / per, c = (e % per) * 4;
            if (e >= rows * per) continue;
            if (silu) x[q] = make_float4(db_act(x[q].x, 1), db_act(x[q].y, 1), db_act(x[q].z, 1), db_act(x[q].w, 1));
            if (scale != nullptr) { const float f = scale[r]; x[q].x *= f; x[q].y *= f; x[q].z *= f; x[q].w *= f; }
            st4(dst + r * pitch + c, x[q]);
        }
    }
}

// (1) grid (items, H, key tiles of 128 x column tiles of 64): own[i][j] = sum_t w^(n-1-t) k_t[i] v_t[j].
__global__ void __launch_bounds__(256, 2)
decay_own_kernel(DecayBlocks p) {
    __shared__ __align__(16) float Ks[DB_STAGE][128], Vs[DB_STAGE][64];
    __shared__ float f[DB_STAGE];
    pdl_trigger();
    const int item = blockIdx.x, head = blockIdx.y, b = item / p.n_blocks;
    const int k_tiles = (p.dk + 127) / 128;
    const int i0 = (blockIdx.z % k_tiles) * 128, j0 = (blockIdx.z / k_tiles) * 64;
    const int row0 = p.seq_start[b] + (item % p.n_blocks) * DB_TOK;
    const int n = min(DB_TOK, p.seq_start[b + 1] - row0);
    const float w = p.decay[head];
    pdl_wait();
    if (n <= 0) return;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;   // rows ty 8 .. + 7, columns tx 4 .. + 3
    const int nk = min(128, p.dk - i0), nv = min(64, p.dv - j0);
    f32x2 acc[8][2];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = 0ull;
    for (int t0 = 0; t0 < n; t0 += DB_STAGE) {
        const int m = min(DB_STAGE, n - t0);
        __syncthreads();
        if (threadIdx.x < DB_STAGE) f[threadIdx.x] = threadIdx.x < m ? powf(w, (float)(n - 1 - t0 - threadIdx.x)) : 0.f;
        __syncthreads();
        db_stage(&Ks[0][0], 128, p.k + (size_t)(row0 + t0) * p.k_stride + (size_t)head * p.dk + i0, p.k_stride, DB_STAGE, m, 128, nk, p.silu, p.vec, f);
        db_stage(&Vs[0][0], 64, p.v + (size_t)(row0 + t0) * p.v_stride + (size_t)head * p.dv + j0, p.v_stride, DB_STAGE, m, 64, nv, p.silu, p.vec, nullptr);
        __syncthreads();
#pragma unroll 4
        for (int t = 0; t < DB_STAGE; ++t) {
            const ulonglong2 v2 = db_ld(&Vs[t][tx * 4]);
            const float4 a = ld4(&Ks[t][ty * 8]), c = ld4(&Ks[t][ty * 8 + 4]);
            const float kk[8] = {a.x, a.y, a.z, a.w, c.x, c.y, c.z, c.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const f32x2 k2 = db_pack(kk[i], kk[i]);
                acc[i][0] = db_fma(k2, v2.x, acc[i][0]);
                acc[i][1] = db_fma(k2, v2.y, acc[i][1]);
            }
        }
    }
    float* s = p.s + ((size_t)item * p.H + head) * p.dk * p.dv;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int r = i0 + ty * 8 + i, c = j0 + tx * 4;
        if (r >= p.dk) continue;
        float x[4];
        db_unpack(acc[i][0], x[0], x[1]);
        db_unpack(acc[i][1], x[2], x[3]);
        if (p.vec && c + 4 <= p.dv) st4(s + (size_t)r * p.dv + c, make_float4(x[0], x[1], x[2], x[3]));
        else
            for (int e = 0; e < 4; ++e)
                if (c + e < p.dv) s[(size_t)r * p.dv + c + e] = x[e];
    }
}

// (2) a thread per element of a head's state: s of every block <- the state at its start, the last one to the sequence's state.
__global__ void __launch_bounds__(256)
decay_carry_kernel(DecayBlocks p) {
    pdl_trigger();
    const int b = blockIdx.x, head = blockIdx.y;
    const int e = blockIdx.z * blockDim.x + threadIdx.x;
    const int row0 = p.seq_start[b], rows = p.seq_start[b + 1] - row0, slot = p.seq_slots[b];
    const float w = p.decay[head];
    pdl_wait();
    if (rows <= 0 || e >= p.dk * p.dv) return;
    float* st = p.state + (size_t)slot * p.state_stride + (size_t)head * p.dk * p.dv + e;
    const int n = (rows + DB_TOK - 1) / DB_TOK;
    const float full = powf(w, (float)DB_TOK), last = powf(w, (float)(rows - (n - 1) * DB_TOK));
    const size_t per_item = (size_t)p.H * p.dk * p.dv;
    float* at = p.s + (size_t)b * p.n_blocks * per_item + (size_t)head * p.dk * p.dv + e;
    float S = *st;
    constexpr int CB = 8;   // the loads of eight blocks go out together
    for (int c0 = 0; c0 < n; c0 += CB) {
        float own[CB];
#pragma unroll
        for (int u = 0; u < CB; ++u) own[u] = c0 + u < n ? at[(size_t)(c0 + u) * per_item] : 0.f;
#pragma unroll
        for (int u = 0; u < CB; ++u)
            if (c0 + u < n) {
                at[(size_t)(c0 + u) * per_item] = S;
                S = fmaf(c0 + u + 1 < n ? full : last, S, own[u]);
            }
    }
    *st = S;
}

// (3) grid (items x 2, H, column tiles of 64 NJ): 64 tokens by 64 NJ columns, a thread four tokens by four columns (NJ times).
// Shared memory: Q [64][dkp + 4]; one place for a block of K [64][dkp + 4], of V or of the state [64][64 NJ]; P [64][68]; powers.
template <int NJ>
__global__ void __launch_bounds__(256, 2)
decay_out_kernel(DecayBlocks p) {
    extern __shared__ __align__(16) float db_smem[];
    constexpr int CT = 64 * NJ;
    const int dkp = (p.dk + 3) / 4 * 4, ld = dkp + 4;
    float* Qs = db_smem;
    float* Bs = Qs + DB_HALF * ld;
    float* Ps = Bs + DB_HALF * max(ld, CT);
    float* pw = Ps + DB_HALF * DB_P;          // w^0 .. w^128
    pdl_trigger();
    const int item = blockIdx.x >> 1, half = blockIdx.x & 1, head = blockIdx.y, b = item / p.n_blocks;
    const int block0 = p.seq_start[b] + (item % p.n_blocks) * DB_TOK, row0 = block0 + half * DB_HALF;
    const int n = min(DB_HALF, p.seq_start[b + 1] - row0);
    const int j0 = blockIdx.z * CT, nv = min(CT, p.dv - j0);
    const float w = p.decay[head];
    pdl_wait();
    if (n <= 0) return;
    const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
    if (tid <= DB_TOK) pw[tid] = powf(w, (float)tid);
    db_stage(Qs, ld, p.q + (size_t)row0 * p.q_stride + (size_t)head * p.dk, p.q_stride, DB_HALF, n, dkp, p.dk, p.silu, p.vec, nullptr);
    f32x2 acc[4][2 * NJ];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2 * NJ; ++j) acc[i][j] = 0ull;
    // acc[i][..] += sum over r < n_r of A[ty 4 + i][r] B[r][..]; A's rows are pitch apart
    auto product = [&](const float* A, int pitch, int n_r) {
#pragma unroll 2
        for (int r = 0; r < n_r; r += 4) {
            float4 a[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = ld4(A + (ty * 4 + i) * pitch + r);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                ulonglong2 v2[NJ];
#pragma unroll
                for (int j = 0; j < NJ; ++j) v2[j] = db_ld(Bs + (r + e) * CT + j * 64 + tx * 4);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float av = e == 0 ? a[i].x : e == 1 ? a[i].y : e == 2 ? a[i].z : a[i].w;
                    const f32x2 a2 = db_pack(av, av);
#pragma unroll
                    for (int j = 0; j < NJ; ++j) {
                        acc[i][2 * j] = db_fma(a2, v2[j].x, acc[i][2 * j]);
                        acc[i][2 * j + 1] = db_fma(a2, v2[j].y, acc[i][2 * j + 1]);
                    }
                }
            }
        }
    };
    // the state at the block's start, 64 key channels at a time
    const float* s_in = p.s + ((size_t)item * p.H + head) * p.dk * p.dv + j0;
    for (int i0 = 0; i0 < p.dk; i0 += DB_HALF) {
        __syncthreads();
        db_stage(Bs, CT, s_in + (size_t)i0 * p.dv, p.dv, DB_HALF, min(DB_HALF, p.dk - i0), CT, nv, 0, p.vec, nullptr);
        __syncthreads();
        product(Qs + i0, ld, min(DB_HALF, dkp - i0));
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float g = pw[half * DB_HALF + ty * 4 + i + 1];
        const f32x2 g2 = db_pack(g, g);
#pragma unroll
        for (int j = 0; j < 2 * NJ; ++j) acc[i][j] = db_fma(g2, acc[i][j], 0ull);
    }
    // the block's own tokens, 64 at a time
    for (int sb = 0; sb <= half; ++sb) {
        const int s0 = block0 + sb * DB_HALF, m = min(DB_HALF, p.seq_start[b + 1] - s0);
        __syncthreads();
        db_stage(Bs, ld, p.k + (size_t)s0 * p.k_stride + (size_t)head * p.dk, p.k_stride, DB_HALF, m, dkp, p.dk, p.silu, p.vec, nullptr);
        __syncthreads();
        {   // rows t = ty + 16 i, columns s = tx + 16 j: even and odd channels' sums
            f32x2 qk[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) qk[i][j] = 0ull;
            for (int k = 0; k < dkp; k += 4) {
                ulonglong2 ks[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) ks[j] = db_ld(Bs + (tx + 16 * j) * ld + k);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const ulonglong2 qa = db_ld(Qs + (ty + 16 * i) * ld + k);
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        qk[i][j] = db_fma(qa.x, ks[j].x, qk[i][j]);
                        qk[i][j] = db_fma(qa.y, ks[j].y, qk[i][j]);
                    }
                }
            }
            const int ahead = (half - sb) * DB_HALF;   // positions that a row lies further on than a column of the same number
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int back = ahead + ty + 16 * i - (tx + 16 * j);
                    float lo, hi;
                    db_unpack(qk[i][j], lo, hi);
                    Ps[(ty + 16 * i) * DB_P + tx + 16 * j] = back >= 0 ? pw[back] * (lo + hi) : 0.f;
                }
        }
        __syncthreads();
        db_stage(Bs, CT, p.v + (size_t)s0 * p.v_stride + (size_t)head * p.dv + j0, p.v_stride, DB_HALF, m, CT, nv, p.silu, p.vec, nullptr);
        __syncthreads();
        product(Ps, DB_P, DB_HALF);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int c = j * 64 + tx * 4;
            float x[4];
            db_unpack(acc[i][2 * j], x[0], x[1]);
            db_unpack(acc[i][2 * j + 1], x[2], x[3]);
            float* o = p.o + (size_t)(row0 + t) * p.o_stride + (size_t)head * p.dv + j0 + c;
            if (p.vec && c + 4 <= nv) st4(o, make_float4(x[0], x[1], x[2], x[3]));
            else
                for (int e = 0; e < 4; ++e)
                    if (c + e < nv) o[e] = x[e];
        }
    }
}

extern "C" int odin_decay_blocks(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                                 long long v_stride, const float* decay, float* o, long long o_stride, float* state,
                                 long long state_stride, const int* seq_start, const int* seq_slots, int n_seqs, int H, int dk,
                                 int dv, int silu, int n_blocks, float* scratch, void* stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || dk <= 0 || dv <= 0 || n_blocks <= 0 || scratch == nullptr) return ODIN_ERR_BAD_ARG;
    if (dk > 256 || H > 65535 || (long long)n_seqs * n_blocks > 1073741823LL) return ODIN_ERR_UNSUPPORTED;
    const bool vec = (dk % 4 == 0) && (dv % 4 == 0) && (q_stride % 4 == 0) && (k_stride % 4 == 0) && (v_stride % 4 == 0) && (o_stride % 4 == 0) &&
                     ((((uintptr_t)q) | ((uintptr_t)k) | ((uintptr_t)v) | ((uintptr_t)o) | ((uintptr_t)scratch)) & 15) == 0;
    DecayBlocks p{q, k, v, q_stride, k_stride, v_stride, decay, o, o_stride, state, state_stride, seq_start, seq_slots,
                  H, dk, dv, n_blocks, silu, vec ? 1 : 0, scratch};
    cudaStream_t s = (cudaStream_t)stream;
    const int items = n_seqs * n_blocks;
    odin_launch(decay_own_kernel, dim3(items, H, ((dk + 127) / 128) * ((dv + 63) / 64)), dim3(256), 0, s, p);
    ODIN_LAUNCH_CHECK();
    odin_launch(decay_carry_kernel, dim3(n_seqs, H, (dk * dv + 255) / 256), dim3(256), 0, s, p);
    ODIN_LAUNCH_CHECK();
    const int ld = (dk + 3) / 4 * 4 + 4, nj = dv > 64 ? 2 : 1;
    const size_t smem = sizeof(float) * (size_t)(DB_HALF * ld + DB_HALF * (ld > 64 * nj ? ld : 64 * nj) + DB_HALF * DB_P + DB_TOK + 1);
    auto kern = nj == 2 ? decay_out_kernel<2> : decay_out_kernel<1>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    odin_launch(kern, dim3(items * 2, H, (dv + 64 * nj - 1) / (64 * nj)), dim3(256), smem, s, p);
    ODIN_LAUNCH_CHECK();
    return 0;
}
