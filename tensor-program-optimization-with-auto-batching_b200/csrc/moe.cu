// Mixture-of-experts bookkeeping on the device: per token the `top` experts with the largest router logits and the softmax
// over exactly those logits, and the grouping of all (token, expert) pairs by expert that the grouped projections read.
//
//   plan_small  one CTA does everything when there are few pairs (decode steps);
//   route, then the framework's stable bucket sort with the expert as the key, then finish: prompt passes.
// Either way pairs of one expert stay in token order, so the grouping is deterministic.
#include <cfloat>

#include "common.cuh"

namespace mlora {
namespace {

constexpr int kMoeThreads = 1024;
constexpr int kMoeSmall = 2048;      // pairs one CTA handles by itself
constexpr int kMoeMaxExperts = 1024;

// One warp: experts and weights of one token.  Selected in order of decreasing logit, lower index first among equals.
__device__ __forceinline__ void route_token(const float* __restrict__ z, const float* __restrict__ bias, int E, int top,
                                            int32_t* __restrict__ idx, float* __restrict__ wt) {
  const int lane = threadIdx.x & 31;
  float last = INFINITY, z0 = 0.f, sum = 0.f;
  int last_i = -1;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = z[e] + bias[e];
      const bool after = v < last || (v == last && e > last_i);  // not chosen yet
      if (after && (bi == 0x7fffffff || v > best)) best = v, bi = e;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (oi != 0x7fffffff && (bi == 0x7fffffff || ov > best || (ov == best && oi < bi))) best = ov, bi = oi;
    }
    if (bi == 0x7fffffff) bi = k < E ? k : 0, best = -INFINITY;  // (only with NaN logits: stay in range)
    if (k == 0) z0 = best;
    const float w = expf(best - z0);
    sum += w;
    if (lane == 0) idx[k] = bi, wt[k] = w;
    last = best;
    last_i = bi;
  }
  __syncwarp();
  for (int k = lane; k < top; k += 32) wt[k] /= sum;
}

struct PlanOut {
  int32_t* idx;    // [T * top] expert of pair (t, k)
  float* wt;       // [T * top]
  int32_t* pos;    // [T * top] row of the pair in expert order
  int32_t* rows;   // [T * top] token of a row in expert order
  int32_t* tiles;  // [4 + 4 * max_tiles]: count, 0, 0, 0, then (expert, first row, rows, 0)
};

__global__ void __launch_bounds__(kMoeThreads) moe_plan_small_kernel(const float* __restrict__ logits, int64_t ld,
                                                                     const float* __restrict__ bias, int T, int E, int top,
                                                                     int tile_rows, PlanOut o) {
  __shared__ int s_e[kMoeSmall];
  __shared__ int s_cnt[kMoeMaxExperts], s_off[kMoeMaxExperts], s_tile[kMoeMaxExperts];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n = T * top;
  for (int t = warp; t < T; t += kMoeThreads / 32) {
    route_token(logits + (size_t)t * ld, bias, E, top, o.idx + (size_t)t * top, o.wt + (size_t)t * top);
    __syncwarp();
    for (int k = lane; k < top; k += 32) s_e[t * top + k] = o.idx[(size_t)t * top + k];
  }
  for (int e = tid; e < E; e += kMoeThreads) s_cnt[e] = 0;
  __syncthreads();
  for (int i = tid; i < n; i += kMoeThreads) atomicAdd(&s_cnt[s_e[i]], 1);
  __syncthreads();
  // exclusive sums over the experts of their rows and of their tiles (one warp)
  if (warp == 0) {
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
    if (lane == 0) o.tiles[0] = tiles;
  }
  __syncthreads();
  for (int e = tid; e < E; e += kMoeThreads)
    for (int r = 0, i = s_tile[e]; r < s_cnt[e]; r += tile_rows, ++i)
      reinterpret_cast<int4*>(o.tiles)[1 + i] = make_int4(e, s_off[e] + r, min(tile_rows, s_cnt[e] - r), 0);
  // row of pair i = first row of its expert + pairs of the same expert before it
  for (int i = tid; i < n; i += kMoeThreads) {
    const int e = s_e[i];
    int before = 0;
    for (int j = 0; j < i; ++j) before += s_e[j] == e;
    const int p = s_off[e] + before;
    o.pos[i] = p;
    o.rows[p] = i / top;
  }
}

__global__ void __launch_bounds__(256) moe_route_kernel(const float* __restrict__ logits, int64_t ld,
                                                        const float* __restrict__ bias, int T, int E, int top,
                                                        int32_t* __restrict__ idx, float* __restrict__ wt) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < T) route_token(logits + (size_t)t * ld, bias, E, top, idx + (size_t)t * top, wt + (size_t)t * top);
}

// perm / segments: the bucket sort's outputs.  CTA 0 writes the tile table as well.
__global__ void __launch_bounds__(256) moe_finish_kernel(const int32_t* __restrict__ perm, const int32_t* __restrict__ seg_off,
                                                         const int32_t* __restrict__ seg_expert,
                                                         const int32_t* __restrict__ counts, int n, int top, int tile_rows,
                                                         PlanOut o) {
  __shared__ int s_first[kMoeMaxExperts];
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i < n) {
    const int p = perm[i];
    o.pos[p] = i;
    o.rows[i] = p / top;
  }
  if (blockIdx.x != 0) return;
  const int n_seg = counts[0];
  if (threadIdx.x < 32) {
    int tiles = 0;
    for (int s0 = 0; s0 < n_seg; s0 += 32) {
      const int s = s0 + threadIdx.x;
      const int nt = s < n_seg ? (seg_off[s + 1] - seg_off[s] + tile_rows - 1) / tile_rows : 0;
      int b = nt;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int pb = __shfl_up_sync(0xffffffffu, b, d);
        if ((int)threadIdx.x >= d) b += pb;
      }
      if (s < n_seg) s_first[s] = tiles + b - nt;
      tiles += __shfl_sync(0xffffffffu, b, 31);
    }
    if (threadIdx.x == 0) o.tiles[0] = tiles;
  }
  __syncthreads();
  for (int s = threadIdx.x; s < n_seg; s += 256) {
    const int a = seg_off[s], c = seg_off[s + 1] - a;
    for (int r = 0, j = s_first[s]; r < c; r += tile_rows, ++j)
      reinterpret_cast<int4*>(o.tiles)[1 + j] = make_int4(seg_expert[s], a + r, min(tile_rows, c - r), 0);
  }
}

size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" size_t mlora_moe_plan_workspace(int32_t T, int32_t E, int32_t top) {
  const int64_t n = (int64_t)T * top;
  if (T <= 0 || E <= 0 || top <= 0 || n <= kMoeSmall || n > 0x7fffffff) return 0;
  return 3 * align256(4 * (size_t)n) + 3 * align256(4 * (size_t)(E + 2)) + 256 +
         align256(mlora_bucket_sort_workspace((int32_t)n, 1, E));
}

extern "C" int mlora_moe_plan(const float* d_logits, int64_t ld, const float* d_bias, int32_t T, int32_t E, int32_t top,
                              int32_t tile_rows, int32_t* d_expert, float* d_weight, int32_t* d_pos, int32_t* d_rows,
                              int32_t* d_tiles, void* d_work, size_t work_bytes, void* stream) {
  MLORA_REQUIRE(T >= 0 && E > 0 && E <= kMoeMaxExperts && top > 0 && top <= E && tile_rows > 0 && ld >= E,
                "moe_plan: bad sizes T=%d experts=%d (at most %d) top=%d", T, E, kMoeMaxExperts, top);
  MLORA_REQUIRE(d_logits && d_bias && d_expert && d_weight && d_pos && d_rows && d_tiles && aligned16(d_tiles),
                "moe_plan: null or unaligned pointer");
  MLORA_REQUIRE((int64_t)T * top <= 0x7fffffff, "moe_plan: too many (token, expert) pairs");
  if (T == 0) return MLORA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const PlanOut o{d_expert, d_weight, d_pos, d_rows, d_tiles};
  const int n = T * top;
  if (n <= kMoeSmall) {
    launch_pdl(moe_plan_small_kernel, 1, kMoeThreads, 0, st, d_logits, ld, d_bias, T, E, top, tile_rows, o);
    count_launch();
    MLORA_CHECK_LAUNCH("moe_plan_small_kernel");
    return MLORA_OK;
  }
  const size_t need = mlora_moe_plan_workspace(T, E, top);
  MLORA_REQUIRE(d_work && work_bytes >= need, "moe_plan: workspace of %zu bytes needed, %zu given", need, work_bytes);
  uint8_t* w = (uint8_t*)d_work;
  auto take = [&](size_t bytes) {
    uint8_t* p = w;
    w += align256(bytes);
    return (int32_t*)p;
  };
  int32_t* perm = take(4 * (size_t)n);
  int32_t* s_tid = take(4 * (size_t)n);
  int32_t* s_wid = take(4 * (size_t)n);
  int32_t* seg_off = take(4 * (size_t)(E + 2));
  int32_t* seg_tid = take(4 * (size_t)(E + 2));
  int32_t* seg_wid = take(4 * (size_t)(E + 2));
  int32_t* counts = take(256);
  launch_pdl(moe_route_kernel, (T + 7) / 8, 256, 0, st, d_logits, ld, d_bias, T, E, top, d_expert, d_weight);
  count_launch();
  MLORA_CHECK_LAUNCH("moe_route_kernel");
  const int rc = mlora_bucket_sort(nullptr, d_expert, n, 1, E, 0, perm, s_tid, s_wid, seg_off, seg_tid, seg_wid, counts, w,
                                   mlora_bucket_sort_workspace(n, 1, E), stream);
  if (rc != MLORA_OK) return rc;
  launch_pdl(moe_finish_kernel, (n + 255) / 256, 256, 0, st, perm, seg_off, seg_wid, counts, n, top, tile_rows, o);
  count_launch();
  MLORA_CHECK_LAUNCH("moe_finish_kernel");
  return MLORA_OK;
}
