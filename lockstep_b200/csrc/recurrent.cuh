// What the sources of mixers with a carried state share.
#pragma once

#include "common.cuh"

constexpr int MAX_TAPS = 16;      // taps of a short convolution whose inputs are carried

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
