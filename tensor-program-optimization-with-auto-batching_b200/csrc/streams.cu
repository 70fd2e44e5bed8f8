// Hyper-connections and layer norm, beside residual_rmsnorm and residual_dyt: the residual is not one row but `n` streams,
// mixed by a small matrix when a sublayer hands its result back, and read by the next sublayer as a weighted sum.  One
// launch does both ends -- the result of the sublayer before into the streams, the weighted sum and its layer norm for the
// sublayer after -- so that every stream is read and written once per sublayer.
//
// One CTA per row; a thread keeps the streams of eight columns in registers while it mixes them, the weighted sum of the
// row stays in shared memory for the two passes of the norm (mean, then squared deviations).
#include "act_io.cuh"

namespace mlora {
namespace {

constexpr int kMaxStreams = 16;

template <typename A>
struct StreamsArgs {
  const A* delta;         // [T, H] result of the sublayer before, or NULL: nothing is mixed
  const float* src;       // streams before: row pitch ld_src, stream s at + s * src_stream (0: all streams are one row)
  int64_t ld_src, src_stream;
  float* dst;             // streams after [T][n][H], or NULL: not stored
  const float* back;      // with delta: [n] what every stream gets of it, then [n, n] the mix, a row per old stream
  const float* read;      // [n_read] weights of the sum that is normalised
  const int32_t* rows;    // NULL: every row; else output row i is row rows[i]
  const bf16* w;
  float eps;
  A* out;
  int n, n_read;          // n_read = n, or (n = 1) the weights of streams that are all the one row
  int H, width;           // H: pitch of all rows (a multiple of 8); width: columns that count
};

__device__ __forceinline__ float cta_sum(float v, float* sm /*[33]*/) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (lane == 0) sm[w] = v;
  __syncthreads();
  float t = lane < nw ? sm[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

// N streams, or (N = 0) any number up to kMaxStreams.
template <typename A, int N>
__global__ void __launch_bounds__(512) residual_streams_norm_kernel(StreamsArgs<A> a) {
  constexpr int kN = N ? N : kMaxStreams;
  extern __shared__ float s_u[];  // [H]
  __shared__ float sm[33];
  __shared__ float s_back[kN * (kN + 1)], s_read[kN];
  pdl_launch_dependents();
  pdl_wait();
  const int n = N ? N : a.n;
  const size_t orow = blockIdx.x, row = a.rows ? (size_t)a.rows[orow] : orow;
  if (a.delta)
    for (int i = threadIdx.x; i < n * (n + 1); i += blockDim.x) s_back[i] = a.back[i];
  if constexpr (N == 1) {
    if (threadIdx.x == 0) {
      float r = 0.f;
      for (int i = 0; i < a.n_read; ++i) r += a.read[i];
      s_read[0] = r;
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) s_read[i] = a.read[i];
  }
  __syncthreads();
  float sum = 0.f;
  for (int k = threadIdx.x * 8; k < a.H; k += blockDim.x * 8) {
    float x[kN][8], u[8];
#pragma unroll
    for (int s = 0; s < kN; ++s) {
      if (s > 0 && a.src_stream == 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[s][i] = x[0][i];
      } else if (s < n) {
        load8(a.src + row * a.ld_src + s * a.src_stream + k, x[s]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) u[i] = 0.f;
    if (a.delta) {
      float d[8];
      load8(a.delta + row * a.H + k, d);
#pragma unroll
      for (int t = 0; t < kN; ++t) {
        if (t >= n) break;
        float y[8];
        const float b = s_back[t], r = s_read[t];
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = b * d[i];
#pragma unroll
        for (int s = 0; s < kN; ++s) {
          if (s >= n) break;
          const float m = s_back[n + s * n + t];
#pragma unroll
          for (int i = 0; i < 8; ++i) y[i] = fmaf(m, x[s][i], y[i]);
        }
        if (a.dst) store8(a.dst + (row * n + t) * a.H + k, y);
#pragma unroll
        for (int i = 0; i < 8; ++i) u[i] = fmaf(r, y[i], u[i]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < kN; ++s) {
        if (s >= n) break;
        const float r = s_read[s];
#pragma unroll
        for (int i = 0; i < 8; ++i) u[i] = fmaf(r, x[s][i], u[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (k + i < a.width) sum += u[i];
    store8(s_u + k, u);
  }
  const float mean = cta_sum(sum, sm) / (float)a.width;
  float sq = 0.f;
  for (int k = threadIdx.x * 8; k < a.H; k += blockDim.x * 8) {  // (a thread reads back what it wrote)
    float u[8];
    load8(s_u + k, u);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (k + i < a.width) sq = fmaf(u[i] - mean, u[i] - mean, sq);
  }
  const float inv = 1.f / sqrtf(cta_sum(sq, sm) / (float)a.width + a.eps);
  for (int k = threadIdx.x * 8; k < a.H; k += blockDim.x * 8) {
    float u[8], w[8];
    load8(s_u + k, u);
    load8(a.w + k, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) u[i] = k + i < a.width ? (u[i] - mean) * inv * w[i] : 0.f;
    store8(a.out + orow * a.H + k, u);
  }
}

template <typename A>
int launch_streams(const StreamsArgs<A>& a, int T, cudaStream_t st) {
  int threads = (a.H / 8 + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  const size_t smem = (size_t)a.H * 4;
  const auto go = [&](auto kernel) {
    if (smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return fail(MLORA_ECUDA, "residual_streams_layernorm: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    }
    launch_pdl_if(pdl_enabled_norm(), kernel, T, threads, smem, st, a);
    count_launch();
    MLORA_CHECK_LAUNCH("residual_streams_norm_kernel");
    return (int)MLORA_OK;
  };
  switch (!a.delta && a.src_stream == 0 ? 1 : a.n) {  // (untouched streams: one row, the sum of the weights)
    case 1: return go(residual_streams_norm_kernel<A, 1>);
    case 2: return go(residual_streams_norm_kernel<A, 2>);
    case 3: return go(residual_streams_norm_kernel<A, 3>);
    case 4: return go(residual_streams_norm_kernel<A, 4>);
    default: return go(residual_streams_norm_kernel<A, 0>);
  }
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_residual_streams_layernorm(const void* d_delta, const float* d_src, int64_t ld_src, int64_t src_stream,
                                                float* d_dst, const float* d_back, const float* d_read, const int32_t* d_rows,
                                                const void* d_w, float eps, void* d_out, int32_t T, int32_t n, int32_t H,
                                                int32_t width, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && H > 0 && H % 8 == 0 && width > 0 && width <= H, "residual_streams_layernorm: H must be a positive multiple of 8, width within it (H=%d, width=%d)", H, width);
  MLORA_REQUIRE(n > 0 && n <= kMaxStreams, "residual_streams_layernorm: 1 to %d streams (got %d)", kMaxStreams, n);
  MLORA_REQUIRE(H <= 48 * 1024, "residual_streams_layernorm: rows of up to 49152 columns (got %d)", H);
  MLORA_REQUIRE(d_src && d_read && d_w && d_out && (!d_delta || d_back), "residual_streams_layernorm: null pointer");
  MLORA_REQUIRE(ld_src >= H && ld_src % 4 == 0 && src_stream >= 0 && src_stream % 4 == 0, "residual_streams_layernorm: bad pitches");
  MLORA_REQUIRE(aligned16(d_delta) && aligned16(d_src) && aligned16(d_dst) && aligned16(d_w) && aligned16(d_out),
                "residual_streams_layernorm: pointers must be 16-byte aligned");
  if (T == 0) return MLORA_OK;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    StreamsArgs<A> a{(const A*)d_delta, d_src, ld_src, src_stream, d_dst, d_back, d_read, d_rows, (const bf16*)d_w, eps,
                     (A*)d_out, n, n, H, width};
    return launch_streams(a, T, (cudaStream_t)stream);
  };
  return f32 ? launch(0.f) : launch(bf16());
}
