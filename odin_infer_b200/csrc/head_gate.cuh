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
    __device__ __forceinline__ float4 sigmoid4_at(int t, int col) const {
        float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < n_split; ++s) {
            const size_t at = (size_t)s * split_stride + (size_t)t * row_stride + col;
            const float4 v = is_bf16 ? ld4((const bf16*)p + at) : ld4((const float*)p + at);
            z.x += v.x; z.y += v.y; z.z += v.z; z.w += v.w;
        }
        return make_float4(1.0f / (1.0f + expf(-z.x)), 1.0f / (1.0f + expf(-z.y)), 1.0f / (1.0f + expf(-z.z)), 1.0f / (1.0f + expf(-z.w)));
    }
};

static inline HeadGate make_head_gate(const void* gate, int dtype, int splits, long long ss, long long rs, int per_element) {
    const bool a4 = (ss % 4 == 0) && (rs % 4 == 0) && (((uintptr_t)gate) & 15) == 0;
    return HeadGate{gate, dtype == ODIN_BF16, splits, ss, rs, per_element, a4 ? 1 : 0};
}
