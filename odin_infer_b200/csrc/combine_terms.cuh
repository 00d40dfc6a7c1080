// An update of the residual that is a sum of terms: what the kernels that add such updates take.
#pragma once
#include "common.cuh"

#define COMBINE_MAX_TERMS 4
// scale * row_scale[r] * f(sum of the parts + bias), f the identity or norm_w * v / sqrt(mean(v^2) + norm_eps) over the row
struct CombineTerm {
    const void* p; int is_bf16; int n_split; long long split_stride;
    float scale; const float* row_scale; VecRef norm_w; float norm_eps; VecRef bias;
};
struct CombineArgs { CombineTerm t[COMBINE_MAX_TERMS]; int n; };

// all_bits collects what must be a multiple of 16 for four elements to move at a time
static inline int fill_combine_args(CombineArgs& a, uintptr_t& all_bits, int n_terms, const void* const* ptrs, const int* dtypes,
                                    const int* n_splits, const long long* split_strides, const float* scales,
                                    const float* const* row_scales, const void* const* norm_ws, const int* norm_w_dtypes,
                                    const float* norm_eps, const void* const* biases, const int* bias_dtypes) {
    if (n_terms < 0 || n_terms > COMBINE_MAX_TERMS) return ODIN_ERR_BAD_ARG;
    a.n = n_terms;
    for (int i = 0; i < n_terms; ++i) {
        if (dtypes[i] != ODIN_BF16 && dtypes[i] != ODIN_F32) return ODIN_ERR_UNSUPPORTED;
        a.t[i].p = ptrs[i]; a.t[i].is_bf16 = dtypes[i] == ODIN_BF16; a.t[i].n_split = n_splits[i];
        a.t[i].split_stride = split_strides[i]; a.t[i].scale = scales[i]; a.t[i].row_scale = row_scales[i];
        a.t[i].norm_w = VecRef{norm_ws[i], norm_w_dtypes[i] == ODIN_BF16}; a.t[i].norm_eps = norm_eps[i];
        a.t[i].bias = VecRef{biases[i], bias_dtypes[i] == ODIN_BF16};
        all_bits |= (uintptr_t)ptrs[i] | (uintptr_t)norm_ws[i] | (uintptr_t)biases[i] | (uintptr_t)(split_strides[i] * 4);
    }
    return 0;
}
