// Residual add + dynamic tanh norm, beside residual_rmsnorm: out = tanh(alpha * res) * w + b needs no row statistics, so
// the kernel is one pass.  It also takes over the end of a mixture-of-experts layer: the weighted sum of a token's expert
// rows is added to the residual here instead of by a kernel of its own.
#include "act_io.cuh"

namespace mlora {
namespace {

template <typename A>
struct DytArgs {
  const A* delta;        // [T, H] or NULL
  const A* expert_rows;  // [pairs, H] rows in expert order, or NULL
  const int32_t* pos;    // [T, top] row of pair (t, k)
  const float* weight;   // [T, top]
  int top;
  float* res;            // [T, H]
  const int32_t* rows;   // NULL: every row; else output row i is residual row rows[i]
  const bf16 *w, *b, *alpha;
  A* out;
  int H;
};

template <typename A>
__global__ void __launch_bounds__(256) residual_dyt_kernel(DytArgs<A> a) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t orow = blockIdx.x, row = a.rows ? (size_t)a.rows[orow] : orow;
  const float alpha = __bfloat162float(*a.alpha);
  for (int k = threadIdx.x * 8; k < a.H; k += 256 * 8) {
    float v[8], w[8], b[8];
    load8(a.res + row * a.H + k, v);
    load8(a.w + k, w);
    load8(a.b + k, b);
    if (a.delta) {
      float d[8];
      load8(a.delta + row * a.H + k, d);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] += d[i];
    }
    if (a.expert_rows) {
      for (int j = 0; j < a.top; ++j) {
        float d[8];
        const float wt = a.weight[row * a.top + j];
        load8(a.expert_rows + (size_t)a.pos[row * a.top + j] * a.H + k, d);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = fmaf(wt, d[i], v[i]);
      }
    }
    if (a.delta || a.expert_rows) store8(a.res + row * a.H + k, v);
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = fmaf(tanhf(alpha * v[i]), w[i], b[i]);
    store8(a.out + orow * a.H + k, o);
  }
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_residual_dyt(const void* d_delta, const void* d_expert_rows, const int32_t* d_pos, const float* d_weight,
                                  int32_t top, float* d_res, const int32_t* d_rows, const void* d_w, const void* d_b,
                                  const void* d_alpha, void* d_out, int32_t T, int32_t H, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && H > 0 && H % 8 == 0, "residual_dyt: H must be a positive multiple of 8 (H=%d)", H);
  MLORA_REQUIRE(d_res && d_w && d_b && d_alpha && d_out, "residual_dyt: null pointer");
  MLORA_REQUIRE(!d_expert_rows || (d_pos && d_weight && top > 0), "residual_dyt: expert rows need positions and weights");
  MLORA_REQUIRE(aligned16(d_delta) && aligned16(d_expert_rows) && aligned16(d_res) && aligned16(d_w) && aligned16(d_b) && aligned16(d_out),
                "residual_dyt: pointers must be 16-byte aligned");
  if (T == 0) return MLORA_OK;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    DytArgs<A> a{(const A*)d_delta, (const A*)d_expert_rows, d_pos, d_weight, top, d_res, d_rows, (const bf16*)d_w,
                 (const bf16*)d_b, (const bf16*)d_alpha, (A*)d_out, H};
    launch_pdl_if(pdl_enabled_norm(), residual_dyt_kernel<A>, T, 256, 0, (cudaStream_t)stream, a);
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("residual_dyt_kernel");
  return MLORA_OK;
}
