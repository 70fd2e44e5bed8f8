// Sizes and scalar pieces of the gated delta rule, shared by its kernels (see delta.cu for the rule).
#pragma once
#include "act_io.cuh"

namespace mlora {

struct DeltaDims {
  int heads, kv_heads, dim, vdim;  // sizes as stored: multiples of 8
  int vdim_true;                   // columns the norm's mean goes over
  float q_scale;
};

constexpr int kMaxTaps = 8;

// silu of a value that is stored as A: fast exponential and division where the result is rounded to 16 bits anyway.
template <typename A>
__device__ __forceinline__ float silu(float z) {
  if constexpr (sizeof(A) == 2) return __fdividef(z, 1.f + __expf(-z));
  return z / (1.f + expf(-z));
}
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float step_size(float b) { return 1.f / (1.f + expf(-b)); }
__device__ __forceinline__ float log_decay(float a, float A_log, float dt_bias) { return -expf(A_log) * softplus(a + dt_bias); }

// Size checks common to the entry points; MLORA_OK or an error.
int check_delta_dims(const char* who, const DeltaDims& d, int C, int taps);

}  // namespace mlora
