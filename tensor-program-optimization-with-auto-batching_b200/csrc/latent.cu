// Latent attention over a paged cache of compressed rows: one vector c of kv_rank values per token and layer, from which
// every head's key (W_uk c) and value (W_uv c) follow.  Here: normalise-and-append, the copy of cached latents into
// consecutive rows (for prompt passes that expand keys and values), and attention in latent space on the CUDA cores.
//
// In latent space a score is (W_uk^T q) . c and a head's result W_uv (sum_j p_j c_j): the caller applies W_uk^T to the
// queries before and W_uv to the sums after, and the cache is read as it is, once for all heads of a CTA.
#include <cfloat>

#include "act_io.cuh"
#include "latent.cuh"

namespace mlora {
namespace {

// One warp per row: c = x / sqrt(mean(x^2) + eps) * w, written to the row's place in the pages; columns up to the cache
// pitch are zero.
template <typename A>
__global__ void __launch_bounds__(256) latent_append_kernel(const A* __restrict__ x, int64_t ld, int R, const bf16* __restrict__ w,
                                                            float eps, A* __restrict__ pages, int pitch, int page_size,
                                                            const int32_t* __restrict__ bt, int max_pages,
                                                            const int32_t* __restrict__ row_slot,
                                                            const int32_t* __restrict__ row_pos, int T) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  const int pos = row_pos[t];
  if (pos < 0 || pos / page_size >= max_pages) return;
  const A* xr = x + (size_t)t * ld;
  float ss = 0.f;
  for (int k = lane; k < R; k += 32) {
    const float v = to_f32(xr[k]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)R + eps);
  const int page = bt[(size_t)row_slot[t] * max_pages + pos / page_size];
  A* c = pages + (size_t)page * page_size * pitch;
  for (int k = lane; k < pitch; k += 32)
    c[latent_offset(pos % page_size, k, pitch)] = from_f32<A>(k < R ? to_f32(xr[k]) * inv * to_f32(w[k]) : 0.f);
}

// CTA (page p, segment s): rows [base, base + page_size) of the dense copy = page p of the segment's sequence.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* __restrict__ pages, int vec_per_page,
                                                            const int32_t* __restrict__ bt, int max_pages, int page_size,
                                                            const int4* __restrict__ segs, uint4* __restrict__ out) {
  const int4 sg = segs[blockIdx.y];  // (slot, first row, tokens, 0)
  const int p = blockIdx.x;
  if (p * page_size >= sg.z || p >= max_pages) return;
  const uint4* src = pages + (size_t)bt[(size_t)sg.x * max_pages + p] * vec_per_page;
  uint4* dst = out + ((size_t)sg.y / page_size + p) * vec_per_page;
  const int per_row = vec_per_page / page_size;  // 16-byte chunks of a row
  for (int i = threadIdx.x; i < vec_per_page; i += 128) {
    const int row = i / per_row, c = i - row * per_row;
    dst[i] = src[latent_offset(row, c * 8, per_row * 8) >> 3];
  }
}

constexpr int kLaKeys = 64;   // keys per step
constexpr int kLaMaxAcc = 16;  // latent columns per thread: kv_rank <= 128 * 16

// CTA (row, head), 128 threads: scores of 64 keys at a time (one warp per key, lanes over the rank), online softmax,
// latent sums with the threads over the rank.
template <typename A>
__global__ void __launch_bounds__(128) latent_attn_kernel(const A* __restrict__ qa, int64_t q_pitch, const A* __restrict__ pages,
                                                          int R, int pitch, int page_size, const int32_t* __restrict__ bt,
                                                          int max_pages, const int32_t* __restrict__ row_slot,
                                                          const int32_t* __restrict__ row_pos, int H, float scale,
                                                          A* __restrict__ out) {
  __shared__ float s_p[kLaKeys];
  __shared__ float s_m, s_l, s_corr;
  extern __shared__ float s_q[];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t row = (size_t)t * H + h;
  const int n = min(row_pos[t] + 1, max_pages * page_size);
  const int32_t* table = bt + (size_t)row_slot[t] * max_pages;
  for (int k = tid; k < R; k += 128) s_q[k] = to_f32(qa[row * q_pitch + k]);
  if (tid == 0) s_m = -INFINITY, s_l = 0.f;
  float acc[kLaMaxAcc];
#pragma unroll
  for (int i = 0; i < kLaMaxAcc; ++i) acc[i] = 0.f;
  __syncthreads();
  for (int k0 = 0; k0 < n; k0 += kLaKeys) {
    const int m = min(kLaKeys, n - k0);
    for (int j = warp; j < m; j += 4) {
      const A* c = pages + (size_t)table[(k0 + j) / page_size] * page_size * pitch;
      const int r = (k0 + j) % page_size;
      float s = 0.f;
      for (int k = lane; k < R; k += 32) s = fmaf(s_q[k], to_f32(c[latent_offset(r, k, pitch)]), s);
      s = warp_sum(s);
      if (lane == 0) s_p[j] = s * scale;
    }
    __syncthreads();
    if (warp == 0) {
      const float a = lane < m ? s_p[lane] : -INFINITY, b = lane + 32 < m ? s_p[lane + 32] : -INFINITY;
      const float m_old = s_m, m_new = fmaxf(m_old, warp_max(fmaxf(a, b)));
      const float pa = lane < m ? expf(a - m_new) : 0.f, pb = lane + 32 < m ? expf(b - m_new) : 0.f;
      const float sum = warp_sum(pa + pb);
      s_p[lane] = pa;
      s_p[lane + 32] = pb;
      __syncwarp();
      if (lane == 0) {
        s_corr = expf(m_old - m_new);  // (exp(-inf) = 0 at the first step)
        s_l = s_l * s_corr + sum;
        s_m = m_new;
      }
    }
    __syncthreads();
    const float corr = s_corr;
#pragma unroll
    for (int i = 0; i < kLaMaxAcc; ++i) acc[i] *= corr;
    for (int j = 0; j < m; ++j) {
      const A* c = pages + (size_t)table[(k0 + j) / page_size] * page_size * pitch;
      const int r = (k0 + j) % page_size;
      const float p = s_p[j];
#pragma unroll
      for (int i = 0; i < kLaMaxAcc; ++i)
        if (tid + i * 128 < R) acc[i] = fmaf(p, to_f32(c[latent_offset(r, tid + i * 128, pitch)]), acc[i]);
    }
    __syncthreads();
  }
  const float inv = n > 0 ? 1.f / s_l : 0.f;
#pragma unroll
  for (int i = 0; i < kLaMaxAcc; ++i)
    if (tid + i * 128 < q_pitch) out[row * q_pitch + tid + i * 128] = from_f32<A>(tid + i * 128 < R ? acc[i] * inv : 0.f);
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_latent_append(const void* d_x, int64_t ld, int32_t R, const void* d_w, float eps, void* d_pages,
                                   int32_t pitch, int32_t page_size, const int32_t* d_block_table, int32_t max_pages,
                                   const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && R > 0 && pitch >= R && pitch % 64 == 0 && page_size > 0 && page_size % 8 == 0 && max_pages > 0 && ld >= R,
                "latent_append: bad sizes (pitch a multiple of 64, page size of 8)");
  MLORA_REQUIRE(d_x && d_w && d_pages && d_block_table && d_row_slot && d_row_pos, "latent_append: null pointer");
  if (T == 0) return MLORA_OK;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    launch_pdl_if(pdl_enabled_norm(), latent_append_kernel<A>, (T + 7) / 8, 256, 0, (cudaStream_t)stream, (const A*)d_x, ld, R, (const bf16*)d_w, eps,
                  (A*)d_pages, pitch, page_size, d_block_table, max_pages, d_row_slot, d_row_pos, T);
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("latent_append_kernel");
  return MLORA_OK;
}

extern "C" int mlora_latent_gather(const void* d_pages, int32_t pitch, int32_t page_size, const int32_t* d_block_table,
                                   int32_t max_pages, const int32_t* d_segs, int32_t n_segs, int32_t max_tokens, void* d_out,
                                   void* stream) {
  MLORA_REQUIRE(n_segs >= 0 && n_segs <= 65535 && pitch > 0 && pitch % 64 == 0 && page_size > 0 && page_size % 8 == 0 && max_tokens >= 0, "latent_gather: bad sizes");
  MLORA_REQUIRE(d_pages && d_block_table && d_segs && d_out && aligned16(d_pages) && aligned16(d_segs) && aligned16(d_out),
                "latent_gather: null or unaligned pointer");
  if (n_segs == 0 || max_tokens == 0) return MLORA_OK;
  latent_gather_kernel<<<dim3((max_tokens + page_size - 1) / page_size, n_segs), 128, 0, (cudaStream_t)stream>>>(
      (const uint4*)d_pages, pitch * page_size / 8, d_block_table, max_pages, page_size, (const int4*)d_segs, (uint4*)d_out);
  count_launch();
  MLORA_CHECK_LAUNCH("latent_gather_kernel");
  return MLORA_OK;
}

extern "C" int mlora_latent_attention_simt(const void* d_qa, int64_t q_pitch, const void* d_pages, int32_t R, int32_t pitch,
                                           int32_t page_size, const int32_t* d_block_table, int32_t max_pages,
                                           const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, int32_t H, float scale,
                                           void* d_out, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && H > 0 && H <= 65535 && R > 0 && pitch >= R && pitch % 64 == 0 && q_pitch >= R && page_size > 0 && page_size % 8 == 0 && max_pages > 0,
                "latent_attention_simt: bad sizes");
  MLORA_REQUIRE(q_pitch <= 128 * kLaMaxAcc, "latent_attention_simt: kv_rank up to %d (row pitch %lld)", 128 * kLaMaxAcc, (long long)q_pitch);
  MLORA_REQUIRE(d_qa && d_pages && d_block_table && d_row_slot && d_row_pos && d_out, "latent_attention_simt: null pointer");
  if (T == 0) return MLORA_OK;
  if (f32)
    launch_pdl(latent_attn_kernel<float>, dim3(T, H), 128, R * 4, (cudaStream_t)stream, (const float*)d_qa, q_pitch,
               (const float*)d_pages, R, pitch, page_size, d_block_table, max_pages, d_row_slot, d_row_pos, H, scale, (float*)d_out);
  else
    launch_pdl(latent_attn_kernel<bf16>, dim3(T, H), 128, R * 4, (cudaStream_t)stream, (const bf16*)d_qa, q_pitch,
               (const bf16*)d_pages, R, pitch, page_size, d_block_table, max_pages, d_row_slot, d_row_pos, H, scale, (bf16*)d_out);
  count_launch();
  MLORA_CHECK_LAUNCH("latent_attn_kernel");
  return MLORA_OK;
}
