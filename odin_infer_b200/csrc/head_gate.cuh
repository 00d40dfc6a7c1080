// A sigmoid gate per token and head, or per token and element, for the epilogues of products that leave a head's outputs.
#pragma once
#include "common.cuh"

struct HeadGate {
    const void* p;             // null: no gate
    int is_bf16, n_split;
    long long split_stride, row_stride;
    int per_element;           // 0: one number per head (column h of a token's row); else the row has a number per element
    int aligned4;              // per element: four neighbouring numbers may be read at once (columns in multiples of four)
    __device__ __forceinline__ float sigmoid_at(int t, int col) const {
        float z = 0.f;
        for (int s = 0; s < n_split; ++s) {
            const size_t at = (size_t)s * split_stride + (size_t)t * row_stride + col;
            z += is_bf16 ? __bfloat162float(((const bf16*)p)[at]) : ((const float*)p)[at];
        }
        return 1.0f / (1.0f + expf(-z));
    }
    // the head's factor (1 where there is none, or one per element)
    __device__ __forceinline__ float factor(int t, int h) const {
        return (p == nullptr || per_element) ? 1.0f : sigmoid_at(t, h);
    }
    // element n of head h (N elements a head)
    __device__ __forceinline__ float element(int t, int h, int n, int N) const {
        return (p == nullptr || !per_element) ? 1.0f : sigmoid_at(t, h * N + n);
    }
    // one column of TOK tokens from t0 on (those before T)
    template <int TOK>
    __device__ __forceinline__ void columns(int t0, int T, int col, float (&f)[TOK]) const {
#pragma unroll
        for (int u = 0; u < TOK; ++u) f[u] = 0.f;
        for (int s = 0; s < n_split; ++s) {
#pragma unroll
            for (int u = 0; u < TOK; ++u) {
                const size_t at = (size_t)s * split_stride + (size_t)(t0 + u) * row_stride + col;
                if (t0 + u < T) f[u] += is_bf16 ? __bfloat162float(((const bf16*)p)[at]) : ((const float*)p)[at];
            }
        }
#pragma unroll
        for (int u = 0; u < TOK; ++u) f[u] = 1.0f / (1.0f + expf(-f[u]));
    }
    // 32 columns from col on, loads together (aligned4)
    __device__ __forceinline__ void sigmoid32(int t, int col, float (&f)[32]) const {
#pragma unroll
        for (int q = 0; q < 32; ++q) f[q] = 0.f;
        for (int s = 0; s < n_split; ++s) {
            const size_t at = (size_t)s * split_stride + (size_t)t * row_stride + col;
#pragma unroll
            for (int q = 0; q < 32; q += 4) {
                const float4 v = is_bf16 ? ld4((const bf16*)p + at + q) : ld4((const float*)p + at + q);
                f[q] += v.x; f[q + 1] += v.y; f[q + 2] += v.z; f[q + 3] += v.w;
            }
        }
#pragma unroll
        for (int q = 0; q < 32; ++q) f[q] = __fdividef(1.0f, 1.0f + __expf(-f[q]));
    }
};

static inline HeadGate make_head_gate(const void* gate, int dtype, int splits, long long ss, long long rs, int per_element) {
    const bool a4 = (ss % 4 == 0) && (rs % 4 == 0) && (((uintptr_t)gate) & 15) == 0;
    return HeadGate{gate, dtype == ODIN_BF16, splits, ss, rs, per_element, a4 ? 1 : 0};
}
