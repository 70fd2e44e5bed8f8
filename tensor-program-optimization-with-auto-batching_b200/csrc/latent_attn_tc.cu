// Attention in latent space on the 5th-generation tensor cores: one query row at a time (decode steps, short portions of a
// prompt) against the paged latents, for up to 32 heads of the row in one CTA -- the latents of a key are read once for all
// of them, as key and as value.
//
// CTA = (row, split of its keys, group of HG heads).  Keys are the M dimension, heads the N dimension:
//   S^T [128 keys x HG]          = C [128 x R] . Qa^T [R x HG]      A = the latents as the pages hold them, K-major
//   O^T [R x HG] (128 at a time) += C^T [R x 128] . P^T [128 x HG]  A = the same shared memory, now MN-major: the rank is
//                                                                    the contiguous dimension, no transpose is made
// so a head count of 32 wastes nothing, and both products read one copy of C.  Roles: warp 0 brings pages by TMA into a
// ring of slots of 128 keys x 128 latent columns, warp 1 issues the MMAs, warps 2..5 (one thread per key = TMEM lane) do
// the softmax in fp32.  The running maximum of a head is moved only when a block exceeds it by more than 2^8, and only then
// are the sums in TMEM rescaled; the row sums stay per thread until the end.  A slot is refilled as soon as the O^T
// product of its 128 columns has retired, so the ring keeps streaming across blocks.
//
// With several splits a CTA leaves unnormalised fp32 sums, its maxima and row sums, and a small kernel joins them.
// Every wait is bounded; a CTA that gives up sets the status word and leaves its outputs undefined.
#include <math.h>

#include <atomic>

#include "common.cuh"
#include "tc_ptx.cuh"

namespace mlora {
namespace {

constexpr int kKeys = 128;                     // keys per block
constexpr int kSubTile = kKeys * 128;          // [128 keys][64 columns] bf16
constexpr int kSlot = 2 * kSubTile;            // 128 columns
constexpr int kLtThreads = 192;
constexpr int kMaxChunks = 4;                  // kv_rank up to 512
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRescale = 8.f;                // (log2) how far scores may exceed the reference maximum

struct LtArgs {
  const int32_t* block_table;
  int max_pages, page_size, n_page_rows;       // n_page_rows: rows of the page tensor (the first row that does not exist)
  const int32_t *row_slot, *row_pos;
  int H, R, q_pitch, n_chunks, n_slots, n_splits;
  float scale_log2;
  bf16* out;                                   // [T, H, q_pitch]
  float* part;                                 // [T, H, n_splits, q_pitch] unnormalised sums
  float2* ml;                                  // [T, H, n_splits] (reference maximum, row sum)
  int32_t* status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ uint64_t desc_mn(uint32_t saddr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);
  d |= (uint64_t)(lbo >> 4) << 16;
  d |= (uint64_t)(sbo >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

template <int N>
__device__ __forceinline__ void tmem_ld(uint32_t addr, float (&v)[32]) {
  if constexpr (N == 32) tmem_ld32(addr, v); else tmem_ld16(addr, v);
}
template <int N>
__device__ __forceinline__ void tmem_st(uint32_t addr, const float (&v)[32]) {
  const uint32_t* r = reinterpret_cast<const uint32_t*>(v);
  if constexpr (N == 32)
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,"
        "%30,%31,%32};" ::"r"(addr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
        "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]),
        "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]),
        "r"(r[31])
        : "memory");
  else
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(addr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
        "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}

// Reduces N values per lane over the warp's lanes: afterwards lane l holds in v[0] the result of value l % N.
template <int N, typename F>
__device__ __forceinline__ void reduce_scatter(float (&v)[32], F f) {
  const int lane = threadIdx.x & 31;
  if constexpr (N == 16) {
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = f(v[i], __shfl_xor_sync(0xffffffffu, v[i], 16));
  }
#pragma unroll
  for (int off = N / 2; off >= 1; off >>= 1) {
    const bool up = (lane & off) != 0;
#pragma unroll
    for (int j = 0; j < off; ++j) {
      const float send = up ? v[j] : v[j + off], keep = up ? v[j + off] : v[j];
      v[j] = f(keep, __shfl_xor_sync(0xffffffffu, send, off));
    }
  }
}

template <int HG>
__global__ void __launch_bounds__(kLtThreads, 1) latent_attn_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                       const __grid_constant__ CUtensorMap map_c, LtArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* sq = ring + a.n_slots * kSlot;               // queries: sub-tiles [HG][64 columns]
  uint8_t* sp = sq + 2 * a.n_chunks * HG * 128;         // probabilities: sub-tiles [HG][64 keys]
  __shared__ uint64_t full_bar[8], empty_bar[8], q_bar, s_bar, p_bar, o_bar;
  __shared__ uint32_t tmem_slot;
  __shared__ int s_abort, s_changed;
  __shared__ float s_red[4][HG];
  __shared__ __align__(16) float s_m[HG], s_f[HG];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = blockIdx.x, split = blockIdx.y, head0 = blockIdx.z * HG;
  const int heads = min(HG, a.H - head0);
  pdl_launch_dependents();
  pdl_wait();
  const int n_keys = min(a.row_pos[t] + 1, a.max_pages * a.page_size);
  const int blocks = (n_keys + kKeys - 1) / kKeys, per = (blocks + a.n_splits - 1) / a.n_splits;
  const int b0 = min(split * per, blocks), b1 = min(b0 + per, blocks);
  const size_t out_row = (size_t)t * a.H + head0;

  if (b0 >= b1) {  // no keys for this CTA (a padding row, or more splits than blocks)
    if (a.n_splits == 1) {
      for (int i = tid; i < heads * a.q_pitch; i += kLtThreads) a.out[out_row * a.q_pitch + i] = __float2bfloat16_rn(0.f);
    } else if (tid < heads) {
      a.ml[(out_row + tid) * a.n_splits + split] = make_float2(-INFINITY, 0.f);
    }
    return;
  }

  if (tid == 0) {
    s_abort = 0;
    for (int i = 0; i < a.n_slots; ++i) {
      mbar_init(&full_bar[i], 1);
      mbar_init(&empty_bar[i], 1);
    }
    mbar_init(&q_bar, 1);
    mbar_init(&s_bar, 1);
    mbar_init(&p_bar, 128);
    mbar_init(&o_bar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_c);
  }
  if (tid < HG) s_m[tid] = -INFINITY;
  if (warp == 1) tmem_alloc(&tmem_slot, 256);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = tmem_slot, tmem_o = tmem_s + 32;  // S^T: HG columns; O^T: HG columns per 128 of the rank

  if (warp == 0) {
    // ---- producer ------------------------------------------------------------------------------------------------
    if (lane == 0) mbar_expect_tx(&q_bar, 2 * a.n_chunks * HG * 128);
    __syncwarp();
    if (lane < 2 * a.n_chunks) tma_load_2d(sq + lane * HG * 128, &map_q, lane * 64, (int)out_row, &q_bar);
    const int32_t* bt = a.block_table + (size_t)a.row_slot[t] * a.max_pages;
    const int ppb = kKeys / a.page_size, half = lane & 1, p = lane >> 1;  // one (page, column half) per lane
    const int n_pages = (n_keys + a.page_size - 1) / a.page_size;
    auto row_of = [&](int b) {  // rows past the last page read as zeros
      const int pg = b * ppb + p;
      return p < ppb && pg < n_pages ? bt[pg] * a.page_size : a.n_page_rows;
    };
    int n = 0, next = row_of(b0);
    bool ok = true;
    for (int b = b0; b < b1 && ok; ++b) {
      const int row = next;
      if (b + 1 < b1) next = row_of(b + 1);
      for (int j = 0; j < a.n_chunks; ++j, ++n) {
        const int s = n % a.n_slots;
        if (lane == 0) {
          ok = mbar_wait(&empty_bar[s], ((n / a.n_slots) & 1) ^ 1, &s_abort);
          if (ok) mbar_expect_tx(&full_bar[s], kSlot);
        }
        ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
        if (!ok) break;
        if (p < ppb)
          tma_load_2d(ring + s * kSlot + half * kSubTile + p * a.page_size * 128, &map_c, j * 128 + half * 64, row, &full_bar[s]);
      }
    }
    if (!ok) s_abort = 1;
  } else if (warp == 1) {
    // ---- MMA issue -----------------------------------------------------------------------------------------------
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(128, HG), idesc_o = make_idesc(128, HG) | (1u << 15);  // O^T: A is MN-major
      bool ok = mbar_wait(&q_bar, 0, &s_abort);
      int n = 0;
      for (int b = b0; b < b1 && ok; ++b) {
        const uint32_t par = (b - b0) & 1;
        for (int j = 0; j < a.n_chunks && ok; ++j) {
          const int s = (n + j) % a.n_slots;
          ok = mbar_wait(&full_bar[s], ((n + j) / a.n_slots) & 1, &s_abort);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const uint64_t ad = make_smem_desc(smem_u32(ring + s * kSlot + h * kSubTile));
            const uint64_t bd = make_smem_desc(smem_u32(sq + (2 * j + h) * HG * 128));
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_bf16(tmem_s, ad + 2 * k, bd + 2 * k, idesc_s, (j | h | k) ? 1u : 0u);
          }
        }
        if (!ok) break;
        umma_commit(&s_bar);
        ok = mbar_wait(&p_bar, par, &s_abort);
        if (!ok) break;
        tc_fence_after();
        for (int j = 0; j < a.n_chunks; ++j) {
          const int s = (n + j) % a.n_slots;
          const uint32_t c = smem_u32(ring + s * kSlot);
#pragma unroll
          for (int k = 0; k < 8; ++k)  // 16 keys = 2048 bytes of a sub-tile
            umma_bf16(tmem_o + j * HG, desc_mn(c + k * 2048, kSubTile, 1024),
                      make_smem_desc(smem_u32(sp + (k >> 2) * HG * 128)) + 2 * (k & 3), idesc_o, (b > b0 || k > 0) ? 1u : 0u);
          umma_commit(&empty_bar[s]);
        }
        n += a.n_chunks;
      }
      if (!ok) s_abort = 1;
      umma_commit(&o_bar);
    }
    __syncwarp();
  } else {
    // ---- softmax: thread = key of the block ------------------------------------------------------------------------
    const int q = warp & 3, kl = q * 32 + lane;
    const uint32_t lane_base = (uint32_t)(q * 32) << 16;
    float lp[HG];
#pragma unroll
    for (int i = 0; i < HG; ++i) lp[i] = 0.f;
    bool ok = true;
    for (int b = b0; b < b1; ++b) {
      ok = mbar_wait(&s_bar, (b - b0) & 1, &s_abort);  // every MMA issued before has retired as well: sp and O^T are free
      if (!ok) s_abort = 1;
      tc_fence_after();
      const bool valid = b * kKeys + kl < n_keys;
      float s[32], mx[32];
      tmem_ld<HG>(tmem_s + lane_base, s);
#pragma unroll
      for (int i = 0; i < HG; ++i) {
        s[i] = valid ? s[i] * a.scale_log2 : -INFINITY;
        mx[i] = s[i];
      }
      reduce_scatter<HG>(mx, [](float x, float y) { return fmaxf(x, y); });
      if (lane < HG) s_red[q][lane] = mx[0];
      if (kl == 0) s_changed = 0;
      epi_bar_sync();
      if (kl < HG) {
        const float bm = fmaxf(fmaxf(s_red[0][kl], s_red[1][kl]), fmaxf(s_red[2][kl], s_red[3][kl]));
        const float old = s_m[kl];
        float f = 1.f;
        if (bm > old + kRescale || old == -INFINITY) {
          f = ex2(old - bm);  // (0 at the first block)
          if (bm == -INFINITY) f = 1.f;  // (every score -inf: nothing to scale)
          else s_m[kl] = bm;
          s_changed = 1;
        }
        s_f[kl] = f;
      }
      epi_bar_sync();
      if (s_changed && b > b0) {
#pragma unroll
        for (int i = 0; i < HG; ++i) lp[i] *= s_f[i];
        for (int j = 0; j < a.n_chunks; ++j) {
          float o[32];
          tmem_ld<HG>(tmem_o + j * HG + lane_base, o);
#pragma unroll
          for (int i = 0; i < HG; ++i) o[i] *= s_f[i];
          tmem_st<HG>(tmem_o + j * HG + lane_base, o);
        }
      }
      uint8_t* pd = sp + (kl >> 6) * HG * 128 + (kl & 7) * 2;
      const int cx = (kl & 63) >> 3;
#pragma unroll
      for (int i = 0; i < HG; ++i) {
        const float m = s_m[i];
        const float pr = valid ? ex2(s[i] - (m == -INFINITY ? 0.f : m)) : 0.f;
        lp[i] += pr;
        *reinterpret_cast<bf16*>(pd + i * 128 + ((cx ^ (i & 7)) << 4)) = __float2bfloat16_rn(pr);
      }
      if (!valid) {
        // latents of keys that do not exist (whatever the last page holds there): their probability is 0, but 0 * NaN is not
        for (int j = 0; j < a.n_chunks; ++j) {
          uint8_t* c = ring + (((b - b0) * a.n_chunks + j) % a.n_slots) * kSlot + kl * 128;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            reinterpret_cast<uint4*>(c)[i] = make_uint4(0u, 0u, 0u, 0u);
            reinterpret_cast<uint4*>(c + kSubTile)[i] = make_uint4(0u, 0u, 0u, 0u);
          }
        }
      }
      tc_fence_before();
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      mbar_arrive(&p_bar);
    }
    if (!mbar_wait(&o_bar, 0, &s_abort)) s_abort = 1;
    tc_fence_after();
    // row sums over the 128 threads, head by head
    float sum[32];
#pragma unroll
    for (int i = 0; i < HG; ++i) sum[i] = lp[i];
    reduce_scatter<HG>(sum, [](float x, float y) { return x + y; });
    if (lane < HG) s_red[q][lane] = sum[0];
    epi_bar_sync();
    if (kl < HG) {
      const float l = (s_red[0][kl] + s_red[1][kl]) + (s_red[2][kl] + s_red[3][kl]);
      s_f[kl] = a.n_splits == 1 ? (l > 0.f ? 1.f / l : 0.f) : 1.f;
      if (a.n_splits > 1 && kl < heads) a.ml[(out_row + kl) * a.n_splits + split] = make_float2(s_m[kl], l);
    }
    epi_bar_sync();
    for (int j = 0; j < a.n_chunks; ++j) {
      float o[32];
      tmem_ld<HG>(tmem_o + j * HG + lane_base, o);
      const int r = j * 128 + kl;
#pragma unroll
      for (int i = 0; i < HG; ++i) {
        if (i < heads) {
          const size_t row = out_row + i;
          if (a.n_splits == 1)
            a.out[row * a.q_pitch + r] = __float2bfloat16_rn(o[i] * s_f[i]);
          else
            a.part[(row * a.n_splits + split) * a.q_pitch + r] = o[i];
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (s_abort) {
    if (tid == 0 && a.status) atomicOr(a.status, 1);
    for (int i = 0; i < 64; ++i) __nanosleep(1000);  // copies still in flight land before the CTA's shared memory goes
  }
  if (warp == 1) tmem_dealloc(tmem_s, 256);
}

// Joins the splits of one (row, head): weights 2^(m_s - max m), then one division.
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part, const float2* __restrict__ ml, int n_splits,
                                                           int q_pitch, bf16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, ml[row * n_splits + s].x);
  for (int s = 0; s < n_splits; ++s) {
    const float2 v = ml[row * n_splits + s];
    if (v.y > 0.f) l += v.y * ex2(v.x - m);
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int r = threadIdx.x * 4; r < q_pitch; r += 128 * 4) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < n_splits; ++s) {
      const float2 v = ml[row * n_splits + s];
      if (!(v.y > 0.f)) continue;
      const float w = ex2(v.x - m) * inv;
      const float4 x = *reinterpret_cast<const float4*>(part + (row * n_splits + s) * q_pitch + r);
      o.x = fmaf(w, x.x, o.x), o.y = fmaf(w, x.y, o.y), o.z = fmaf(w, x.z, o.z), o.w = fmaf(w, x.w, o.w);
    }
    uint2 pk;
    *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(o.x, o.y);
    *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(o.z, o.w);
    *reinterpret_cast<uint2*>(out + row * q_pitch + r) = pk;
  }
}

int head_group(int H) { return H <= 16 ? 16 : 32; }

// Splits of a row's keys: the count that finishes first when every CTA has an SM to itself, with about one block's time
// of fixed cost per CTA.
int pick_splits(int T, int H, int max_keys) {
  int dev = 0, sms = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const long long ctas = (long long)T * ((H + head_group(H) - 1) / head_group(H));
  const int blocks = (max_keys + kKeys - 1) / kKeys;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 32 && s <= blocks; ++s) {
    const double waves = (double)((ctas * s + sms - 1) / sms);
    const double cost = waves * ((blocks + s - 1) / s + 1.5) + (s > 1 ? 1.0 : 0.0);
    if (cost < best_cost - 1e-9) best_cost = cost, best = s;
  }
  return best;
}

template <int HG>
int launch_lt(const CUtensorMap& mq, const CUtensorMap& mc, const LtArgs& a, int T, cudaStream_t st) {
  const int smem = a.n_slots * kSlot + 2 * a.n_chunks * HG * 128 + 2 * HG * 128 + 1024;
  static std::atomic<unsigned long long> attr_done{0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!((attr_done.load(std::memory_order_acquire) >> (dev & 63)) & 1ull)) {
    cudaError_t e = cudaFuncSetAttribute(latent_attn_tc_kernel<HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
    if (e != cudaSuccess) return fail(MLORA_ECUDA, "latent_attention: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    attr_done.fetch_or(1ull << (dev & 63), std::memory_order_release);
  }
  launch_pdl_if(pdl_enabled_attn(), latent_attn_tc_kernel<HG>, dim3(T, a.n_splits, (a.H + HG - 1) / HG), kLtThreads, smem, st, mq, mc, a);
  count_launch();
  MLORA_CHECK_LAUNCH("latent_attn_tc_kernel");
  return MLORA_OK;
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" uint32_t mlora_latent_attention_splits(int32_t T, int32_t H, int32_t max_keys) {
  return T > 0 && H > 0 && max_keys > 0 ? (uint32_t)pick_splits(T, H, max_keys) : 1u;
}

extern "C" size_t mlora_latent_attention_workspace(int32_t T, int32_t H, int32_t q_pitch, int32_t n_splits) {
  if (n_splits <= 1) return 0;
  return (size_t)T * H * n_splits * ((size_t)q_pitch * sizeof(float) + sizeof(float2));
}

extern "C" int mlora_latent_attention(const void* d_qa, int64_t q_pitch, const void* d_pages, int32_t n_pages_total, int32_t R,
                                      int32_t pitch, int32_t page_size, const int32_t* d_block_table, int32_t max_pages,
                                      const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, int32_t H, float scale,
                                      int32_t n_splits, void* d_out, void* d_work, size_t work_bytes, int32_t* d_status,
                                      void* stream) {
  MLORA_REQUIRE(T >= 0 && H > 0 && R > 0 && R <= kMaxChunks * 128 && pitch >= R && pitch % 8 == 0 && max_pages > 0 && n_pages_total > 0,
                "latent_attention: bad sizes (kv_rank up to %d, cache pitch a multiple of 8)", kMaxChunks * 128);
  MLORA_REQUIRE(page_size == 16 || page_size == 32, "latent_attention: page size 16 or 32 (got %d)", page_size);
  const int n_chunks = (R + 127) / 128;
  MLORA_REQUIRE(q_pitch == n_chunks * 128, "latent_attention: rows of qa and out have kv_rank rounded up to 128 columns (got %lld)", (long long)q_pitch);
  MLORA_REQUIRE(d_qa && d_pages && d_block_table && d_row_slot && d_row_pos && d_out && aligned16(d_qa) && aligned16(d_pages) &&
                    aligned16(d_out) && (int64_t)n_pages_total * page_size < 0x7fffffff && (int64_t)T * H < 0x7fffffff,
                "latent_attention: null or unaligned pointer, or too many rows");
  MLORA_REQUIRE(n_splits >= 1 && n_splits <= 65535, "latent_attention: bad n_splits %d", n_splits);
  const size_t need = mlora_latent_attention_workspace(T, H, (int32_t)q_pitch, n_splits);
  MLORA_REQUIRE(!need || (d_work && aligned16(d_work) && work_bytes >= need), "latent_attention: workspace of %zu bytes needed, %zu given", need, work_bytes);
  if (T == 0) return MLORA_OK;
  const int HG = head_group(H);
  CUtensorMap mq, mc;
  int rc = make_map(&mq, d_qa, (long long)T * H, (int)q_pitch, q_pitch, HG, 64);
  if (rc) return rc;
  rc = make_map(&mc, d_pages, (long long)n_pages_total * page_size, pitch, pitch, page_size, 64);
  if (rc) return rc;
  LtArgs a{};
  a.block_table = d_block_table;
  a.max_pages = max_pages;
  a.page_size = page_size;
  a.n_page_rows = n_pages_total * page_size;
  a.row_slot = d_row_slot;
  a.row_pos = d_row_pos;
  a.H = H;
  a.R = R;
  a.q_pitch = (int)q_pitch;
  a.n_chunks = n_chunks;
  const int fixed = 2 * n_chunks * HG * 128 + 2 * HG * 128 + 1024;
  a.n_slots = (224 * 1024 - fixed) / kSlot;
  if (a.n_slots > 8) a.n_slots = 8;
  if (a.n_slots > 2 * n_chunks) a.n_slots = 2 * n_chunks;
  a.n_splits = n_splits;
  a.scale_log2 = scale * kLog2e;
  a.out = (bf16*)d_out;
  a.part = (float*)d_work;
  a.ml = (float2*)((float*)d_work + (size_t)T * H * n_splits * q_pitch);
  a.status = d_status;
  rc = HG == 16 ? launch_lt<16>(mq, mc, a, T, (cudaStream_t)stream) : launch_lt<32>(mq, mc, a, T, (cudaStream_t)stream);
  if (rc || n_splits == 1) return rc;
  launch_pdl(latent_merge_kernel, (unsigned)(T * H), 128, 0, (cudaStream_t)stream, a.part, a.ml, n_splits, (int)q_pitch, (bf16*)d_out);
  count_launch();
  MLORA_CHECK_LAUNCH("latent_merge_kernel");
  return MLORA_OK;
}
