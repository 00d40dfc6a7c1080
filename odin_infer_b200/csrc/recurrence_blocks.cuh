// What the recurrences over a matrix-valued state per head share (recurrent.cu, delta_rule.cu): their parameters, and the
// kernel that adds to every token's output what the state at the start of its block of tokens contributes.
#pragma once
#include "common.cuh"

// Threads that share a column of S: each owns a quarter of the key channels.  (Sixteen lanes per column, a quarter of
// the registers each, walked a prompt of 2,048 tokens a fifth faster and made a decode step three to four times slower:
// four times the threads for the same work.)
#define REC_SPLIT 4
#define REC_MAX_DK 256
#define REC_COLS 128    // columns of S that one CTA covers at most
#define REC_FETCH 4     // elements of each input that a thread fetches ahead per block of tokens

struct RecParams {
    const float* q; long long q_stride;   // [rows, H*dk] projections (32-bit), row strides in elements
    const float* k; long long k_stride;   // REC_BONUS and REC_FIXED
    const float* g; long long g_stride;   // the raw decay / forget gate (REC_FIXED: unused)
    const float* v; long long v_stride;   // [rows, H*dv]
    VecRef c0, c1;                        // per (head, key channel): REC_BONUS w0 and u; REC_GATED bias and lower bound; REC_FIXED: c0 per head
    float* o; long long o_stride;         // [rows, H*dv]
    float* state; long long state_stride; // per slot: [H][dk][dv] floats
    const int* seq_start; const int* seq_slots;
    int H, dk, dv;
    float q_scale;        // REC_GLA: factor on q
    int heads_per_group;  // REC_SSD: heads that share one q and one k (their columns: group * dk)
    // the token shift's memory: after the step the sequence's last row of h goes to its state
    const void* shift_src; int shift_is_bf16; float* shift_state; long long shift_stride; int width;
    // Blocks of tokens (block_len > 0): a CTA walks one block of one sequence from a state of zeros and leaves
    // the block's own state in s_loc, the product of the block's decays per key channel in d_tot, and per token
    // q times the decays since the block's start in qp; two small kernels then carry the state from block to block
    // and add what each block's incoming state contributes to its tokens' outputs.
    int block_len, n_blocks;
    float* qp;     // [rows, H*dk]
    float* s_loc;  // [sequences * n_blocks][H][dk][dv]
    float* d_tot;  // [sequences * n_blocks][H*dk]
};

// o[t, head, :] += (q_t * decays since the block's start)^T S_in(block): 64 (or 32) tokens by 32 columns per CTA pass.
// Shared memory: the incoming state's 32 columns [dk][32], then (dk a multiple of four) 64 tokens' q [64][dk], which the
// CTA fetches with loads that all go out together; a warp then takes eight tokens and reads four channels of a token's q
// in one broadcast.  Every sum runs over the channels in their order, whichever path computes it.
#define CARRY_OUT_TOK 64
__global__ void __launch_bounds__(256)
recurrence_carry_out_kernel(RecParams p) {
    extern __shared__ __align__(16) float co_smem[];
    float (*tile)[32] = reinterpret_cast<float (*)[32]>(co_smem);
    float* qsm = co_smem + (size_t)p.dk * 32;
    pdl_trigger();
    const int item = blockIdx.x, head = blockIdx.y;
    const int b = item / p.n_blocks;
    const int lane = threadIdx.x & 31, lane_t = threadIdx.x >> 5;
    const int col = blockIdx.z * 32 + lane;
    const int seq_end = p.seq_start[b + 1];
    const int row0 = p.seq_start[b] + (item % p.n_blocks) * p.block_len;
    const int row1 = min(seq_end, row0 + p.block_len);
    pdl_wait();
    if (row1 <= row0) return;
    const float* sin = p.s_loc + ((size_t)item * p.H + head) * p.dk * p.dv;
    for (int e = threadIdx.x; e < p.dk * 32; e += blockDim.x) {
        const int i = e >> 5, c = blockIdx.z * 32 + (e & 31);
        tile[i][e & 31] = c < p.dv ? sin[(size_t)i * p.dv + c] : 0.f;
    }
    const size_t qs = (size_t)p.H * p.dk;
    if ((p.dk & 3) == 0) {
        const int dk4 = p.dk >> 2;
        for (int tb = row0; tb < row1; tb += CARRY_OUT_TOK) {
            __syncthreads();   // the pass before has read its q (and, the first time, the tile is there after the next one)
            for (int e = threadIdx.x; e < CARRY_OUT_TOK * dk4; e += blockDim.x) {
                const int u = e / dk4, c4 = e % dk4;
                if (tb + u < row1)
                    reinterpret_cast<float4*>(qsm)[e] =
                        __ldg(reinterpret_cast<const float4*>(p.qp + (size_t)(tb + u) * qs + (size_t)head * p.dk) + c4);
            }
            __syncthreads();
            const int t0 = tb + lane_t * 8;
            const int nt = min(8, row1 - t0);
            if (nt <= 0) continue;
            float acc[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) acc[u] = 0.f;
            const float* qw = qsm + (size_t)lane_t * 8 * p.dk;
            for (int i = 0; i < p.dk; i += 4) {
                const float s0 = tile[i][lane], s1 = tile[i + 1][lane], s2 = tile[i + 2][lane], s3 = tile[i + 3][lane];
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    if (u < nt) {
                        const float4 q4 = *reinterpret_cast<const float4*>(qw + u * p.dk + i);
                        acc[u] = fmaf(q4.x, s0, acc[u]);
                        acc[u] = fmaf(q4.y, s1, acc[u]);
                        acc[u] = fmaf(q4.z, s2, acc[u]);
                        acc[u] = fmaf(q4.w, s3, acc[u]);
                    }
            }
            if (col < p.dv) {
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    if (u < nt) p.o[(size_t)(t0 + u) * p.o_stride + (size_t)head * p.dv + col] += acc[u];
            }
        }
        return;
    }
    __syncthreads();
    for (int t0 = row0 + lane_t * 4; t0 < row1; t0 += 32) {   // a warp takes four tokens at a time
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const float* qrow = p.qp + (size_t)t0 * qs + (size_t)head * p.dk;
        for (int i = 0; i < p.dk; ++i) {
            const float sv = tile[i][lane];
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (t0 + u < row1) acc[u] = fmaf(__ldg(qrow + u * qs + i), sv, acc[u]);
        }
        if (col < p.dv) {
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (t0 + u < row1) p.o[(size_t)(t0 + u) * p.o_stride + (size_t)head * p.dv + col] += acc[u];
        }
    }
}

static inline int launch_recurrence_carry_out(const RecParams& p, int n_items, cudaStream_t s) {
    const size_t co_smem = (size_t)p.dk * 32 * sizeof(float) + ((p.dk & 3) == 0 ? (size_t)CARRY_OUT_TOK * p.dk * sizeof(float) : 0);
    if (co_smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(recurrence_carry_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)co_smem);
        if (e != cudaSuccess) return (int)e;
    }
    odin_launch(recurrence_carry_out_kernel, dim3(n_items, p.H, (p.dv + 31) / 32), dim3(256), co_smem, s, p);
    ODIN_LAUNCH_CHECK();
    return 0;
}
