// A sigmoid gate per token and head, for the epilogues of products that leave a head's outputs.
#pragma once
#include "common.cuh"

struct HeadGate {
    const void* p;             // null: no gate
    int is_bf16, n_split;
    long long split_stride, row_stride;
    __device__ __forceinline__ float factor(int t, int h) const {
        if (p == nullptr) return 1.0f;
        float z = 0.f;
        for (int s = 0; s < n_split; ++s) {
            const size_t at = (size_t)s * split_stride + (size_t)t * row_stride + h;
            z += is_bf16 ? __bfloat162float(((const bf16*)p)[at]) : ((const float*)p)[at];
        }
        return 1.0f / (1.0f + expf(-z));
    }
};
