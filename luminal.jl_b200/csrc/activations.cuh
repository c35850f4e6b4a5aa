// Activations of the layered decoders' epilogues and recurrences, in float32.
#pragma once
#include <cuda_runtime.h>

namespace lmb {

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float gelu_tanh_f32(float x) {
  return 0.5f * x * (1.0f + tanhf(0.79788456f * (x + 0.044715f * x * x * x)));
}
// logarithm of a decay: -exp(a) softplus(x + b)
__device__ __forceinline__ float log_decay_f32(float x, float a, float b) { return -expf(a) * softplus_f32(x + b); }

}  // namespace lmb
