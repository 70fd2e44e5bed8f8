// Mixture-of-experts bookkeeping on the device: per token the `top` experts with the largest router logits and the softmax
// over exactly those logits, and the grouping of all (token, expert) pairs by expert that the grouped projections read.
//
//   decode sizes: one launch for everything, router included -- a CTA per token computes its logits and chooses, the last
//   one to finish groups the pairs;
//   prompt passes: route (choice, and the pairs' ranks inside their CTA), scan, scatter.
// Either way pairs of one expert stay in token order, so the grouping is deterministic.
#include "act_io.cuh"

namespace mlora {
namespace {

constexpr int kMoeMaxExperts = 1024;
constexpr int kDecodeTokens = 64;    // one-launch form: tokens
constexpr int kDecodePairs = 1024;   //                  and pairs
constexpr int kLocalPairs = 4096;    // pairs of one CTA of the route kernel

// One warp: experts and weights of one token, in order of decreasing logit, lower index first among equals.  `z(e)` is the
// logit of expert e; lane l keeps those of experts l, l + 32, ... in R registers.
template <int R, typename F>
__device__ __forceinline__ void route_token(F z, int E, int top, int32_t* __restrict__ idx, float* __restrict__ wt) {
  const int lane = threadIdx.x & 31;
  float v[R];
#pragma unroll
  for (int r = 0; r < R; ++r) v[r] = lane + 32 * r < E ? z(lane + 32 * r) : -INFINITY;
  unsigned taken = 0;  // bit r: register r has been chosen (or does not exist)
#pragma unroll
  for (int r = 0; r < R; ++r)
    if (lane + 32 * r >= E) taken |= 1u << r;
  float z0 = 0.f, sum = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (!(taken >> r & 1) && (bi == 0x7fffffff || v[r] > best)) best = v[r], bi = lane + 32 * r;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (oi != 0x7fffffff && (bi == 0x7fffffff || ov > best || (ov == best && oi < bi))) best = ov, bi = oi;
    }
    bi = __shfl_sync(0xffffffffu, bi, 0);  // (one view of the choice, NaN logits included)
    best = __shfl_sync(0xffffffffu, best, 0);
    if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
    if (k == 0) z0 = best;
    const float w = expf(best - z0);
    sum += w;
    if (lane == 0) idx[k] = bi, wt[k] = w;
  }
  __syncwarp();
  for (int k = lane; k < top; k += 32) wt[k] /= sum;
}
template <typename F>
__device__ __forceinline__ void route_any(F z, int E, int top, int32_t* __restrict__ idx, float* __restrict__ wt) {
  if (E <= 64)
    route_token<2>(z, E, top, idx, wt);
  else if (E <= 256)
    route_token<8>(z, E, top, idx, wt);
  else
    route_token<32>(z, E, top, idx, wt);
}

struct PlanOut {
  int32_t* idx;    // [T * top] expert of pair (t, k)
  float* wt;       // [T * top]
  int32_t* pos;    // [T * top] row of the pair in expert order
  int32_t* rows;   // [T * top] token of a row in expert order
  int32_t* tiles;  // [4 + 4 * max_tiles]: count, 0, 0, 0, then (expert, first row, rows, 0)
};

// Exclusive sums over the experts of their rows and of their tiles, by one warp; writes the tile count.
__device__ __forceinline__ void scan_experts(const int* s_cnt, int* s_off, int* s_tile, int E, int tile_rows, int32_t* n_tiles) {
  const int lane = threadIdx.x & 31;
  int rows = 0, tiles = 0;
  for (int e0 = 0; e0 < E; e0 += 32) {
    const int e = e0 + lane, c = e < E ? s_cnt[e] : 0, nt = (c + tile_rows - 1) / tile_rows;
    int a = c, b = nt;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const int pa = __shfl_up_sync(0xffffffffu, a, d), pb = __shfl_up_sync(0xffffffffu, b, d);
      if (lane >= d) a += pa, b += pb;
    }
    if (e < E) s_off[e] = rows + a - c, s_tile[e] = tiles + b - nt;
    rows += __shfl_sync(0xffffffffu, a, 31);
    tiles += __shfl_sync(0xffffffffu, b, 31);
  }
  if (lane == 0) *n_tiles = tiles;
}
__device__ __forceinline__ void write_tiles(const int* s_cnt, const int* s_off, const int* s_tile, int E, int tile_rows, int32_t* tiles) {
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    for (int r = 0, i = s_tile[e]; r < s_cnt[e]; r += tile_rows, ++i)
      reinterpret_cast<int4*>(tiles)[1 + i] = make_int4(e, s_off[e] + r, min(tile_rows, s_cnt[e] - r), 0);
}

// CTA = token.  z = W h + bias in fp32 (two experts per warp at a time), choice by warp 0; the last CTA groups.
constexpr int kDecodeThreads = 1024;

template <typename A>
__global__ void __launch_bounds__(kDecodeThreads, 1) moe_decode_kernel(const A* __restrict__ h, int64_t ldh, const A* __restrict__ W,
                                                                       int in, const float* __restrict__ bias, int T, int E, int top,
                                                                       int tile_rows, PlanOut o, int32_t* __restrict__ ticket) {
  __shared__ float s_z[kMoeMaxExperts];
  __shared__ int s_cnt[kMoeMaxExperts], s_off[kMoeMaxExperts], s_tile[kMoeMaxExperts];
  __shared__ int s_e[kDecodePairs];
  __shared__ int s_last;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n = T * top;
  const A* x = h + (size_t)t * ldh;
  for (int e0 = warp * 2; e0 < E; e0 += kDecodeThreads / 16) {
    const bool two = e0 + 1 < E;
    const A* w0 = W + (size_t)e0 * in;
    const A* w1 = two ? w0 + in : w0;
    float a0 = 0.f, a1 = 0.f;
#pragma unroll 4
    for (int k = lane * 8; k < in; k += 256) {
      float xv[8], u[8], v[8];
      load8(x + k, xv);
      load8(w0 + k, u);
      load8(w1 + k, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) a0 = fmaf(xv[i], u[i], a0), a1 = fmaf(xv[i], v[i], a1);
    }
    a0 = warp_sum(a0);
    a1 = warp_sum(a1);
    if (lane == 0) {
      s_z[e0] = a0 + bias[e0];
      if (two) s_z[e0 + 1] = a1 + bias[e0 + 1];
    }
  }
  __syncthreads();
  if (warp == 0) {
    route_any([&](int e) { return s_z[e]; }, E, top, o.idx + (size_t)t * top, o.wt + (size_t)t * top);
    __threadfence();
    __syncwarp();
    if (lane == 0) s_last = atomicAdd(ticket, 1) == T - 1;
  }
  __syncthreads();
  if (!s_last) return;
  if (tid == 0) *ticket = 0;  // ready for the next call
  __threadfence();
  for (int i = tid; i < n; i += kDecodeThreads) s_e[i] = __ldcg(o.idx + i);
  for (int e = tid; e < E; e += kDecodeThreads) s_cnt[e] = 0;
  __syncthreads();
  for (int i = tid; i < n; i += kDecodeThreads) atomicAdd(&s_cnt[s_e[i]], 1);
  __syncthreads();
  if (warp == 0) scan_experts(s_cnt, s_off, s_tile, E, tile_rows, o.tiles);
  __syncthreads();
  write_tiles(s_cnt, s_off, s_tile, E, tile_rows, o.tiles);
  // row of pair i = first row of its expert + pairs of the same expert before it
  for (int i = tid; i < n; i += kDecodeThreads) {
    const int e = s_e[i];
    int before = 0;
#pragma unroll 8
    for (int j = 0; j < i; ++j) before += s_e[j] == e;
    const int p = s_off[e] + before;
    o.pos[i] = p;
    o.rows[p] = i / top;
  }
}

// Prompt passes.  CTA c: tokens [c * per, ...); hist[e * CTAs + c] = its pairs of expert e; rank (in o.pos) = place of a pair
// among the CTA's pairs of its expert.
__global__ void __launch_bounds__(256) moe_route_kernel(const float* __restrict__ logits, int64_t ld, const float* __restrict__ bias,
                                                        int T, int E, int top, int per, PlanOut o, int32_t* __restrict__ hist) {
  __shared__ int s_e[kLocalPairs];
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * per, n = (min(T, t0 + per) - t0) * top, warp = threadIdx.x >> 5;
  for (int t = t0 + warp; t < min(T, t0 + per); t += 8) {
    const float* z = logits + (size_t)t * ld;
    route_any([&](int e) { return z[e] + bias[e]; }, E, top, o.idx + (size_t)t * top, o.wt + (size_t)t * top);
    __syncwarp();
    for (int k = threadIdx.x & 31; k < top; k += 32) s_e[(t - t0) * top + k] = o.idx[(size_t)t * top + k];
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256) {
    int c = 0;
#pragma unroll 8
    for (int i = 0; i < n; ++i)
      if (s_e[i] == e) o.pos[(size_t)t0 * top + i] = c++;
    hist[(size_t)e * gridDim.x + blockIdx.x] = c;
  }
}

// One CTA: hist[e][c] becomes the first row of CTA c's pairs of expert e; the tile table.
__global__ void __launch_bounds__(1024) moe_scan_kernel(int32_t* __restrict__ hist, int n_cta, int E, int tile_rows, PlanOut o) {
  __shared__ int s_cnt[kMoeMaxExperts], s_off[kMoeMaxExperts], s_tile[kMoeMaxExperts];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = warp; e < E; e += 32) {
    int total = 0;
    for (int c = lane; c < n_cta; c += 32) total += hist[(size_t)e * n_cta + c];
    total = __reduce_add_sync(0xffffffffu, total);
    if (lane == 0) s_cnt[e] = total;
  }
  __syncthreads();
  if (warp == 0) scan_experts(s_cnt, s_off, s_tile, E, tile_rows, o.tiles);
  __syncthreads();
  write_tiles(s_cnt, s_off, s_tile, E, tile_rows, o.tiles);
  for (int e = warp; e < E; e += 32) {
    int run = s_off[e];
    for (int c0 = 0; c0 < n_cta; c0 += 32) {
      const int c = c0 + lane, v = c < n_cta ? hist[(size_t)e * n_cta + c] : 0;
      int a = v;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int p = __shfl_up_sync(0xffffffffu, a, d);
        if (lane >= d) a += p;
      }
      if (c < n_cta) hist[(size_t)e * n_cta + c] = run + a - v;
      run += __shfl_sync(0xffffffffu, a, 31);
    }
  }
}

__global__ void __launch_bounds__(256) moe_scatter_kernel(const int32_t* __restrict__ first, int n, int n_cta, int top, int per, PlanOut o) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const int t = i / top, p = first[(size_t)o.idx[i] * n_cta + t / per] + o.pos[i];
  o.pos[i] = p;
  o.rows[p] = t;
}

// (8 warps: a token or a few each)
int tokens_per_cta(int top) { return kLocalPairs / top < 32 ? kLocalPairs / top : 32; }

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" size_t mlora_moe_plan_workspace(int32_t T, int32_t E, int32_t top) {
  if (T <= 0 || E <= 0 || top <= 0 || top > E || E > kMoeMaxExperts) return 256;
  const int per = tokens_per_cta(top);
  return 256 + (size_t)((T + per - 1) / per) * E * sizeof(int32_t);
}

#define MOE_CHECK(what)                                                                                                        \
  MLORA_REQUIRE(T >= 0 && E > 0 && E <= kMoeMaxExperts && top > 0 && top <= E && tile_rows > 0,                                \
                what ": bad sizes T=%d experts=%d (at most %d) top=%d", T, E, kMoeMaxExperts, top);                            \
  MLORA_REQUIRE(d_bias && d_expert && d_weight && d_pos && d_rows && d_tiles && aligned16(d_tiles) && d_work,                  \
                what ": null or unaligned pointer");                                                                           \
  MLORA_REQUIRE((int64_t)T * top <= 0x7fffffff, what ": too many (token, expert) pairs");                                      \
  MLORA_REQUIRE(work_bytes >= mlora_moe_plan_workspace(T, E, top), what ": workspace of %zu bytes needed, %zu given",           \
                mlora_moe_plan_workspace(T, E, top), work_bytes)

extern "C" int mlora_moe_plan(const float* d_logits, int64_t ld, const float* d_bias, int32_t T, int32_t E, int32_t top,
                              int32_t tile_rows, int32_t* d_expert, float* d_weight, int32_t* d_pos, int32_t* d_rows,
                              int32_t* d_tiles, void* d_work, size_t work_bytes, void* stream) {
  MOE_CHECK("moe_plan");
  MLORA_REQUIRE(d_logits && ld >= E, "moe_plan: null logits or pitch below the number of experts");
  if (T == 0) return MLORA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const PlanOut o{d_expert, d_weight, d_pos, d_rows, d_tiles};
  const int n = T * top, per = tokens_per_cta(top), n_cta = (T + per - 1) / per;
  int32_t* hist = (int32_t*)((uint8_t*)d_work + 256);
  launch_pdl_if(pdl_enabled_norm(), moe_route_kernel, n_cta, 256, 0, st, d_logits, ld, d_bias, T, E, top, per, o, hist);
  launch_pdl_if(pdl_enabled_norm(), moe_scan_kernel, 1, 1024, 0, st, hist, n_cta, E, tile_rows, o);
  launch_pdl_if(pdl_enabled_norm(), moe_scatter_kernel, (n + 255) / 256, 256, 0, st, hist, n, n_cta, top, per, o);
  count_launch(3);
  MLORA_CHECK_LAUNCH("moe_plan");
  return MLORA_OK;
}

extern "C" uint32_t mlora_moe_decode_fits(int32_t T, int32_t top) {
  return T > 0 && T <= kDecodeTokens && top > 0 && (int64_t)T * top <= kDecodePairs ? 1u : 0u;
}

extern "C" int mlora_moe_route_plan(const void* d_h, int64_t ldh, const void* d_W, int32_t in, const float* d_bias, int32_t T,
                                    int32_t E, int32_t top, int32_t tile_rows, int32_t* d_expert, float* d_weight,
                                    int32_t* d_pos, int32_t* d_rows, int32_t* d_tiles, void* d_work, size_t work_bytes,
                                    int32_t f32, void* stream) {
  MOE_CHECK("moe_route_plan");
  MLORA_REQUIRE(T == 0 || mlora_moe_decode_fits(T, top), "moe_route_plan: at most %d tokens and %d pairs", kDecodeTokens, kDecodePairs);
  MLORA_REQUIRE(d_h && d_W && in > 0 && in % 8 == 0 && ldh % 8 == 0 && aligned16(d_h) && aligned16(d_W),
                "moe_route_plan: h and W 16-byte aligned, in and ldh multiples of 8");
  if (T == 0) return MLORA_OK;
  const PlanOut o{d_expert, d_weight, d_pos, d_rows, d_tiles};
  if (f32)
    launch_pdl_if(pdl_enabled_norm(), moe_decode_kernel<float>, T, kDecodeThreads, 0, (cudaStream_t)stream, (const float*)d_h, ldh,
                  (const float*)d_W, in, d_bias, T, E, top, tile_rows, o, (int32_t*)d_work);
  else
    launch_pdl_if(pdl_enabled_norm(), moe_decode_kernel<bf16>, T, kDecodeThreads, 0, (cudaStream_t)stream, (const bf16*)d_h, ldh,
                  (const bf16*)d_W, in, d_bias, T, E, top, tile_rows, o, (int32_t*)d_work);
  count_launch();
  MLORA_CHECK_LAUNCH("moe_decode_kernel");
  return MLORA_OK;
}
