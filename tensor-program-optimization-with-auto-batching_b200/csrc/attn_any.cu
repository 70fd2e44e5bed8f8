// Attention pieces beside the Llama ones: queries and keys that get a bias, are rotated on part of a head and then divided
// by their root mean square, keys that are their own values, and a plain attention kernel for any head size and for 32-bit
// caches (the tensor-core and streaming kernels take bf16 heads of 64 and 128).
#include <cmath>

#include "act_io.cuh"

namespace mlora {
namespace {

constexpr int kMaxPerLane = 16;  // columns of a head per lane: heads of up to 512

template <typename A>
struct RotArgs {
  const A* x;            // rows of [q heads | k heads], dim columns each
  int64_t ld;
  const float* bias;     // [(Hq + Hkv) * dim] or NULL
  const float* inv_freq; // [rot / 2]
  int rot, dim, pad;     // rotated columns, head size, head size as stored
  float eps, q_scale;
  A* q_out;              // [T, Hq * pad]
  A *k_pages, *v_pages;  // [page][Hkv][page_size][pad]
  const int32_t* bt;
  int max_pages;
  const int32_t *row_slot, *row_pos;
  int Hq, Hkv, page_size;
};

// V neighbouring values as one access.
template <typename A, int V>
struct Pack {
  A v[V];
};
template <>
struct __align__(4) Pack<bf16, 2> {
  bf16 v[2];
};
template <>
struct __align__(8) Pack<float, 2> {
  float v[2];
};
template <>
struct __align__(8) Pack<bf16, 4> {
  bf16 v[4];
};
template <>
struct __align__(16) Pack<float, 4> {
  float v[4];
};

// CTA (row, part of the heads): sines and cosines of its position once, then a warp per head, two heads at a time.  Lane:
// columns V (lane + 32 j).  y = rotate(x + bias); y / rms(y): queries times q_scale to q_out, keys to their page; a key as it
// was before rotation and norm goes to the value pages.
template <typename A, int V, int NP>
__global__ void __launch_bounds__(256) rotate_rms_append_kernel(RotArgs<A> a) {
  typedef Pack<A, V> P;
  extern __shared__ __align__(16) float s_cs[];  // [rot / 2] cosines, then sines
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, half = a.rot / 2;
  const int pos = a.row_pos[t];
  const int pidx = pos / a.page_size;
  const bool store = pos >= 0 && pidx < a.max_pages;
  const A* row = a.x + (size_t)t * a.ld;
  const int page = store ? a.bt[(size_t)a.row_slot[t] * a.max_pages + pidx] : 0;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * a.inv_freq[i], &sn, &cs);
    s_cs[i] = cs;
    s_cs[half + i] = sn;
  }
  __syncthreads();
  const int heads = a.Hq + a.Hkv, step = gridDim.y * (blockDim.x >> 5);
  for (int h0 = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5); h0 < heads; h0 += 2 * step) {
    P raw[2][NP], other[2][NP];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int h = h0 + u * step;
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int d = V * (lane + 32 * j);
        if (h >= heads || d >= a.dim) continue;
        raw[u][j] = *reinterpret_cast<const P*>(row + (size_t)h * a.dim + d);
        if (d < a.rot) other[u][j] = *reinterpret_cast<const P*>(row + (size_t)h * a.dim + (d < half ? d + half : d - half));
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int h = h0 + u * step;
      if (h >= heads) break;
      typedef Pack<float, V> F;
      const float* b = a.bias ? a.bias + (size_t)h * a.dim : nullptr;
      float x[NP][V], y[NP][V], ss = 0.f;
#pragma unroll
      for (int j = 0; j < NP; ++j) {  // (a lane's V columns lie on one side of the half, inside or outside of the rotated part)
        const int d = V * (lane + 32 * j);
#pragma unroll
        for (int e = 0; e < V; ++e) x[j][e] = y[j][e] = 0.f;
        if (d >= a.dim) continue;
        F bd{}, bo{}, cs, sn;
        const int i = d < half ? d : d - half;
        if (b) bd = *reinterpret_cast<const F*>(b + d);
        if (b && d < a.rot) bo = *reinterpret_cast<const F*>(b + (d < half ? d + half : i));
        if (d < a.rot) cs = *reinterpret_cast<const F*>(s_cs + i), sn = *reinterpret_cast<const F*>(s_cs + half + i);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          x[j][e] = y[j][e] = to_f32(raw[u][j].v[e]) + bd.v[e];
          if (d < a.rot) {
            const float z = (to_f32(other[u][j].v[e]) + bo.v[e]) * (d < half ? -sn.v[e] : sn.v[e]);
            y[j][e] = fmaf(x[j][e], cs.v[e], z);
          }
          ss = fmaf(y[j][e], y[j][e], ss);
        }
      }
      const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
      const bool is_q = h < a.Hq;
      const float f = is_q ? inv * a.q_scale : inv;
      const size_t at = is_q ? ((size_t)t * a.Hq + h) * a.pad
                             : (((size_t)page * a.Hkv + (h - a.Hq)) * a.page_size + pos % a.page_size) * a.pad;
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int d = V * (lane + 32 * j);
        if (d >= a.pad || (!is_q && !store)) continue;
        P o, v;
#pragma unroll
        for (int e = 0; e < V; ++e) o.v[e] = from_f32<A>(y[j][e] * f), v.v[e] = from_f32<A>(x[j][e]);
        *reinterpret_cast<P*>((is_q ? a.q_out : a.k_pages) + at + d) = o;
        if (!is_q) *reinterpret_cast<P*>(a.v_pages + at + d) = v;
      }
    }
  }
}

template <typename A>
struct AnyArgs {
  const A* q;  // [T, Hq * D]
  const A *k_pages, *v_pages;
  const int32_t* bt;
  int max_pages;
  const int32_t *row_slot, *row_pos;
  int Hq, Hkv, D, page_size, chunk;
  float scale;
  const float* sink;
  A* out;
  int64_t ld_out;
};

constexpr int kAnyKeys = 64;  // keys per step
constexpr int kAnyAcc = 4;    // columns per thread: heads of up to 512

// CTA (row, head), 128 threads: scores of 64 keys at a time (one warp per key, lanes over the head), online softmax that
// starts from the sink, sums with the threads over the head.
template <typename A>
__global__ void __launch_bounds__(128) paged_attn_any_kernel(AnyArgs<A> a) {
  __shared__ float s_p[kAnyKeys];
  __shared__ float s_m, s_l, s_corr;
  extern __shared__ float s_q[];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = a.D;
  const int kvh = h / (a.Hq / a.Hkv), pos = a.row_pos[t];
  const int n = min(pos + 1, a.max_pages * a.page_size);
  const int lo = (a.chunk > 0 && pos > 0) ? pos - pos % a.chunk : 0;
  const int32_t* table = a.bt + (size_t)a.row_slot[t] * a.max_pages;
  const A* q = a.q + ((size_t)t * a.Hq + h) * D;
  for (int k = tid; k < D; k += 128) s_q[k] = to_f32(q[k]);
  if (tid == 0) s_m = a.sink ? a.sink[h] : -INFINITY, s_l = a.sink ? 1.f : 0.f;
  float acc[kAnyAcc];
#pragma unroll
  for (int i = 0; i < kAnyAcc; ++i) acc[i] = 0.f;
  __syncthreads();
  const auto key_at = [&](int j) {
    return (((size_t)table[j / a.page_size] * a.Hkv + kvh) * a.page_size + j % a.page_size) * D;
  };
  for (int k0 = lo; k0 < n; k0 += kAnyKeys) {
    const int m = min(kAnyKeys, n - k0);
    for (int j = warp; j < m; j += 4) {
      const A* c = a.k_pages + key_at(k0 + j);
      float s = 0.f;
      for (int k = lane; k < D; k += 32) s = fmaf(s_q[k], to_f32(c[k]), s);
      s = warp_sum(s);
      if (lane == 0) s_p[j] = s * a.scale;
    }
    __syncthreads();
    if (warp == 0) {
      const float x = lane < m ? s_p[lane] : -INFINITY, y = lane + 32 < m ? s_p[lane + 32] : -INFINITY;
      const float m_old = s_m, m_new = fmaxf(m_old, warp_max(fmaxf(x, y)));
      const float px = lane < m ? expf(x - m_new) : 0.f, py = lane + 32 < m ? expf(y - m_new) : 0.f;
      const float sum = warp_sum(px + py);
      s_p[lane] = px;
      s_p[lane + 32] = py;
      __syncwarp();
      if (lane == 0) {
        s_corr = expf(m_old - m_new);  // (exp(-inf) = 0 at the first step without a sink)
        s_l = s_l * s_corr + sum;
        s_m = m_new;
      }
    }
    __syncthreads();
    const float corr = s_corr;
#pragma unroll
    for (int i = 0; i < kAnyAcc; ++i) acc[i] *= corr;
    for (int j = 0; j < m; ++j) {
      const A* v = a.v_pages + key_at(k0 + j);
      const float p = s_p[j];
#pragma unroll
      for (int i = 0; i < kAnyAcc; ++i)
        if (tid + i * 128 < D) acc[i] = fmaf(p, to_f32(v[tid + i * 128]), acc[i]);
    }
    __syncthreads();
  }
  const float inv = n > lo ? 1.f / s_l : 0.f;
#pragma unroll
  for (int i = 0; i < kAnyAcc; ++i)
    if (tid + i * 128 < D) a.out[(size_t)t * a.ld_out + (size_t)h * D + tid + i * 128] = from_f32<A>(acc[i] * inv);
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_rotate_rms_append(const void* d_x, int64_t ld, const float* d_bias, const float* d_inv_freq, int32_t rot,
                                       int32_t dim, int32_t pad, float eps, float q_scale, void* d_q, void* d_k_pages,
                                       void* d_v_pages, const int32_t* d_block_table, int32_t max_pages,
                                       const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, int32_t Hq, int32_t Hkv,
                                       int32_t page_size, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && Hq > 0 && Hkv > 0 && page_size > 0 && max_pages > 0, "rotate_rms_append: bad sizes");
  MLORA_REQUIRE(dim > 0 && dim <= pad && pad <= 32 * kMaxPerLane && rot >= 0 && rot % 2 == 0 && rot <= dim,
                "rotate_rms_append: heads of up to %d, an even number of rotated columns within (dim=%d, rot=%d)", 32 * kMaxPerLane, dim, rot);
  MLORA_REQUIRE(ld >= (int64_t)(Hq + Hkv) * dim, "rotate_rms_append: row pitch");
  MLORA_REQUIRE(d_x && d_q && d_k_pages && d_v_pages && d_block_table && d_row_slot && d_row_pos && (!rot || d_inv_freq),
                "rotate_rms_append: null pointer");
  if (T == 0) return MLORA_OK;
  // two or four columns per access where halves and heads allow it; few rows: the heads spread over more CTAs
  const bool two = dim % 2 == 0 && rot % 4 == 0 && pad % 2 == 0 && ld % 2 == 0;
  const bool four = dim % 4 == 0 && rot % 8 == 0 && pad % 4 == 0 && ld % 4 == 0 && aligned16(d_x) && aligned16(d_bias) &&
                    aligned16(d_q) && aligned16(d_k_pages) && aligned16(d_v_pages);
  const int heads = Hq + Hkv, threads = T >= 1024 ? 256 : 64;
  const int parts = T >= 1024 ? 1 : (heads + 3) / 4;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    RotArgs<A> a{(const A*)d_x, ld, d_bias, d_inv_freq, rot, dim, pad, eps, q_scale, (A*)d_q, (A*)d_k_pages, (A*)d_v_pages,
                 d_block_table, max_pages, d_row_slot, d_row_pos, Hq, Hkv, page_size};
    const auto go = [&](auto kernel) {
      launch_pdl_if(pdl_enabled_attn(), kernel, dim3(T, parts), threads, (size_t)rot * 4, (cudaStream_t)stream, a);
    };
    if (four && pad <= 128) go(rotate_rms_append_kernel<A, 4, 1>);
    else if (two && pad <= 64) go(rotate_rms_append_kernel<A, 2, 1>);
    else if (two && pad <= 128) go(rotate_rms_append_kernel<A, 2, 2>);
    else if (two) go(rotate_rms_append_kernel<A, 2, kMaxPerLane / 2>);
    else go(rotate_rms_append_kernel<A, 1, kMaxPerLane>);
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("rotate_rms_append_kernel");
  return MLORA_OK;
}

extern "C" int mlora_paged_attention_any(const void* d_q, const void* d_k_pages, const void* d_v_pages,
                                         const int32_t* d_block_table, int32_t max_pages, const int32_t* d_row_slot,
                                         const int32_t* d_row_pos, int32_t T, int32_t Hq, int32_t Hkv, int32_t D,
                                         int32_t page_size, float scale, int32_t chunk, const float* d_sink, void* d_out,
                                         int64_t ld_out, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && Hq > 0 && Hkv > 0 && Hq % Hkv == 0 && Hq <= 65535 && page_size > 0 && max_pages > 0,
                "paged_attention_any: bad sizes");
  MLORA_REQUIRE(D > 0 && D <= 128 * kAnyAcc, "paged_attention_any: heads of up to %d (got %d)", 128 * kAnyAcc, D);
  MLORA_REQUIRE(chunk >= 0 && ld_out >= (int64_t)Hq * D, "paged_attention_any: bad chunk or pitch");
  MLORA_REQUIRE(d_q && d_k_pages && d_v_pages && d_block_table && d_row_slot && d_row_pos && d_out, "paged_attention_any: null pointer");
  if (T == 0) return MLORA_OK;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    AnyArgs<A> a{(const A*)d_q, (const A*)d_k_pages, (const A*)d_v_pages, d_block_table, max_pages, d_row_slot, d_row_pos,
                 Hq, Hkv, D, page_size, chunk, scale, d_sink, (A*)d_out, ld_out};
    launch_pdl(paged_attn_any_kernel<A>, dim3(T, Hq), 128, (size_t)D * 4, (cudaStream_t)stream, a);
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("paged_attn_any_kernel");
  return MLORA_OK;
}
