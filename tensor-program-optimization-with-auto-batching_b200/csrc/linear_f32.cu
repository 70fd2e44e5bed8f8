// Projections in true 32-bit: y = x W^T with fp32 operands on the CUDA cores, plain or grouped (see mlora_grouped_linear
// for the groups).  The path of models loaded in float32; 64 x 64 output tiles, 4 x 4 per thread.
#include "linear.cuh"

namespace mlora {
namespace {

constexpr int kFT = 64, kFK = 16;

struct F32Args {
  const float* x;
  int64_t ldx;
  const float* W;  // [groups, out, in]
  float* y;
  int64_t ldy;
  const int32_t* table;
  const int32_t* gather;
  int T, in, out, x_cols, y_cols, act;
  const float* gate;
  int64_t ld_gate;
};

__global__ void __launch_bounds__(256) linear_f32_kernel(F32Args a) {
  __shared__ float xs[kFK][kFT + 4], ws[kFK][kFT + 4];
  pdl_launch_dependents();
  pdl_wait();
  int group, row0, rows;
  if (a.table != nullptr) {
    if ((int)blockIdx.y >= a.table[0]) return;
    const int32_t* e = a.table + 4 + 4 * blockIdx.y;
    group = e[0], row0 = e[1], rows = e[2];
  } else {
    group = blockIdx.z, row0 = blockIdx.y * kFT, rows = min(kFT, a.T - row0);
  }
  const int o0 = blockIdx.x * kFT, tid = threadIdx.x;
  const float* W = a.W + (size_t)group * a.out * a.in;
  const float* x = a.x + (size_t)group * a.x_cols;
  const int lr = tid >> 2, lk = (tid & 3) * 4;  // row and first k this thread loads of either tile
  int xrow = -1;
  if (lr < rows) xrow = a.gather ? a.gather[row0 + lr] : row0 + lr;
  const int tx = tid & 15, ty = tid >> 4;  // outputs o0 + tx + 16 j, rows ty * 4 + i
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.in; k0 += kFK) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = k0 + lk + e;
      xs[lk + e][lr] = (xrow >= 0 && k < a.in) ? x[(size_t)xrow * a.ldx + k] : 0.f;
      ws[lk + e][lr] = (o0 + lr < a.out && k < a.in) ? W[(size_t)(o0 + lr) * a.in + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = xs[k][ty * 4 + i], wv[i] = ws[k][tx + 16 * i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) continue;
    const float g = a.gate ? 1.f / (1.f + expf(-a.gate[(size_t)(row0 + r) * a.ld_gate + group])) : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int o = o0 + tx + 16 * j;
      if (o < a.out) a.y[(size_t)(row0 + r) * a.ldy + (size_t)group * a.y_cols + o] = act_one(acc[i][j], a.act) * g;
    }
  }
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_linear_f32(const float* d_x, int64_t ldx, int32_t x_cols, const int32_t* d_gather, const float* d_W,
                                float* d_y, int64_t ldy, int32_t y_cols, const int32_t* d_tiles, int32_t max_tiles,
                                int32_t n_groups, int32_t T, int32_t in, int32_t out, int32_t flags, const float* d_gate,
                                int64_t ld_gate, void* stream) {
  MLORA_REQUIRE(T >= 0 && in > 0 && out > 0 && n_groups > 0 && n_groups <= 65535, "linear_f32: bad sizes");
  MLORA_REQUIRE(d_x && d_W && d_y, "linear_f32: null pointer");
  MLORA_REQUIRE(!(flags & ~(MLORA_ACT_RELU2 | MLORA_ACT_GELU)) && flags != (MLORA_ACT_RELU2 | MLORA_ACT_GELU),
                "linear_f32: flags hold at most one activation");
  MLORA_REQUIRE(!d_gather || d_tiles, "linear_f32: a gather list needs a tile table");
  const int ty = d_tiles ? max_tiles : (T + kFT - 1) / kFT;
  if (ty <= 0) return MLORA_OK;
  MLORA_REQUIRE(ty <= 65535, "linear_f32: too many row tiles (%d)", ty);
  F32Args a{d_x, ldx, d_W, d_y, ldy, d_tiles, d_gather, T, in, out, x_cols, y_cols, flags, d_gate, ld_gate};
  launch_pdl(linear_f32_kernel, dim3((out + kFT - 1) / kFT, ty, d_tiles ? 1 : n_groups), 256, 0, (cudaStream_t)stream, a);
  count_launch();
  MLORA_CHECK_LAUNCH("linear_f32_kernel");
  return MLORA_OK;
}
