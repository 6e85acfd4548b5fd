// What the two files of the generalised delta rule share: its bounds and its element-wise functions.
#pragma once
#include "common.cuh"

namespace celeg_b200 {

constexpr int kDeltaMaxDim = 256;
constexpr float kDecaySpan = 0.60653065971263342f;             // e^(-1/2)

__device__ __forceinline__ float sigmoid_of(float x) { return 1.0f / (1.0f + expf(-x)); }
// 1 + expm1: a decay close to one is then its nearest float, without a bias that thousands of steps would add up
__device__ __forceinline__ float channel_decay(float z) { return 1.0f + expm1f(-kDecaySpan * sigmoid_of(z)); }

}  // namespace celeg_b200
