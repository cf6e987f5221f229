// What the kernels that sum a token's experts share.
#pragma once
#include "common.cuh"

// The weights of a token's choices that stand for the identity (router outputs n_real and above), added up.
__device__ __forceinline__ float moe_identity_weight(const int* __restrict__ experts, const float* __restrict__ weights, int t,
                                                     int top, int n_real) {
    float w = 0.f;
    for (int k = 0; k < top; ++k)
        if (__ldcg(experts + (size_t)t * top + k) >= n_real) w += __ldcg(weights + (size_t)t * top + k);
    return w;
}
