// Attention in latent space on the 5th-generation tensor cores: one query row at a time (decode steps, short portions of a
// prompt) against the paged latents, for up to 32 heads of the row in one CTA -- the latents of a key are read once for all
// of them, as key and as value.
//
// CTA = (row, split of its keys, group of HG heads), 64 keys per block:
//   S [heads x 64]          = Qa [heads x R] . C^T            A = the queries, in TMEM (lane = head), B = the latents as the
//                                                             pages hold them, K-major
//   O^T [R x HG] (by 128)  += C^T [R x 64] . P^T [64 x HG]    A = the same shared memory, now MN-major (the rank is the
//                                                             contiguous dimension: no transpose is made), B = P
// so both products read one copy of C, and a head is a TMEM lane for the softmax: one thread per head walks its 64 scores,
// no value crosses lanes.  The scores and the probabilities are double buffered: the scores of block b + 1 are computed
// while the softmax of block b runs, and the ring of blocks keeps streaming.  A page lies in memory as the operand image
// (latent.cuh) and arrives as one bulk copy: with a TMA box per 64 columns (2 KB) the copies' issue rate was the bound.  The
// running maximum of a head is moved only when a block exceeds it by more than 2^8; only then do all four output warps
// rescale the sums in TMEM, on request.
//
// Roles: warp 0 copies, warp 1 MMA issue, warp 4 (TMEM lanes 0..31) softmax, warps 2..5 rescaling and output.
// With several splits a CTA leaves unnormalised fp32 sums, its maxima and row sums, and a small kernel joins them.
// Every wait is bounded; a CTA that gives up sets the status word and leaves its outputs undefined.
#include <math.h>

#include <atomic>

#include "latent.cuh"
#include "tc_ptx.cuh"

namespace mlora {
namespace {

constexpr int kKeys = 64;                      // keys per block
constexpr int kMaxSlots = 8;                   // blocks in the ring
constexpr int kLtThreads = 192;
constexpr int kMaxChunks = 4;                  // kv_rank up to 512
constexpr int kTmemCols = 512;                 // S: 2 x 64, O^T: 4 x 32, queries: 256
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRescale = 8.f;                // (log2) how far scores may exceed the reference maximum

struct LtArgs {
  const int32_t* block_table;
  int max_pages, page_size;
  const uint8_t* pages;
  const int32_t *row_slot, *row_pos;
  const bf16* qa;                              // [T, H, q_pitch]
  int H, R, pitch, q_pitch, n_chunks, n_slots, n_splits;
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

template <int HG>
__global__ void __launch_bounds__(kLtThreads, 1) latent_attn_tc_kernel(LtArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int slot_bytes = kKeys * a.pitch * 2;           // a block: row groups of 8 keys, slices of 64 columns
  uint8_t* sp = ring + a.n_slots * slot_bytes;               // probabilities: two buffers [HG][64 keys]
  __shared__ uint64_t full_bar[kMaxSlots], empty_bar[kMaxSlots], q_bar, s_bar[2], p_bar[2], o_bar[2], cmd_bar, ack_bar;
  __shared__ uint32_t tmem_slot;
  __shared__ int s_abort, s_end;
  __shared__ __align__(16) float s_f[32];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = blockIdx.x, split = blockIdx.y, head0 = blockIdx.z * HG;
  const int heads = min(HG, a.H - head0);
  pdl_launch_dependents();
  pdl_wait();
  const int n_keys = min(a.row_pos[t] + 1, a.max_pages * a.page_size);
  const int blocks = (n_keys + kKeys - 1) / kKeys, per = (blocks + a.n_splits - 1) / a.n_splits;
  const int b0 = min(split * per, blocks), nb = min(b0 + per, blocks) - b0;
  const size_t out_row = (size_t)t * a.H + head0;

  if (nb <= 0) {  // no keys for this CTA (a padding row, or more splits than blocks)
    if (a.n_splits == 1) {
      for (int i = tid; i < heads * a.q_pitch; i += kLtThreads) a.out[out_row * a.q_pitch + i] = __float2bfloat16_rn(0.f);
    } else if (tid < heads) {
      a.ml[(out_row + tid) * a.n_splits + split] = make_float2(-INFINITY, 0.f);
    }
    return;
  }

  if (tid == 0) {
    s_abort = s_end = 0;
    for (int i = 0; i < a.n_slots; ++i) {
      mbar_init(&full_bar[i], 1);
      mbar_init(&empty_bar[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_bar[i], 1);
      mbar_init(&p_bar[i], 32);
      mbar_init(&o_bar[i], 1);
    }
    mbar_init(&q_bar, 32);
    mbar_init(&cmd_bar, 32);
    mbar_init(&ack_bar, 128);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(&tmem_slot, kTmemCols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = tmem_slot, tmem_o = tmem_s + 128, tmem_q = tmem_s + 256;

  if (warp == 0) {
    // ---- producer: one page per lane -------------------------------------------------------------------------------
    const int32_t* bt = a.block_table + (size_t)a.row_slot[t] * a.max_pages;
    const int ppb = kKeys / a.page_size, page_bytes = a.page_size * a.pitch * 2;
    const int n_pages = (n_keys + a.page_size - 1) / a.page_size;
    auto page_of = [&](int b) {
      const int pg = (b0 + b) * ppb + lane;
      return b < nb && lane < ppb && pg < n_pages ? bt[pg] : -1;
    };
    int s = 0, next = page_of(0), next2 = page_of(1);
    uint32_t par = 1;
    bool ok = true;
    for (int b = 0; b < nb && ok; ++b) {
      const int page = next;
      next = next2;
      next2 = page_of(b + 2);
      const int valid = __popc(__ballot_sync(0xffffffffu, page >= 0));
      if (lane == 0) {
        ok = mbar_wait(&empty_bar[s], par, &s_abort);
        if (ok) mbar_expect_tx(&full_bar[s], valid * page_bytes);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (ok && page >= 0) bulk_load(ring + s * slot_bytes + lane * page_bytes, a.pages + (size_t)page * page_bytes, page_bytes, &full_bar[s]);
      if (++s == a.n_slots) s = 0, par ^= 1;
    }
    if (!ok) s_abort = 1;
  } else if (warp == 1) {
    // ---- MMA issue -----------------------------------------------------------------------------------------------
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc(128, kKeys), idesc_o = make_idesc(128, HG) | (1u << 15);  // O^T: A is MN-major
      bool ok = mbar_wait(&q_bar, 0, &s_abort);
      tc_fence_after();
      const int group = 16 * a.pitch, slices = a.pitch / 64;  // bytes of 8 keys
      // K-major operand (keys x 64 columns of a slice): row groups `group` bytes apart instead of adjacent
      auto desc_k = [&](uint32_t addr) { return (make_smem_desc(addr) & ~((uint64_t)0x3FFF << 32)) | ((uint64_t)(group >> 4) << 32); };
      int s_s = 0, s_o = 0;  // ring positions of the two products
      uint32_t par = 0;
      auto scores = [&](int b) {
        if (!mbar_wait(&full_bar[s_s], par, &s_abort)) return false;
        tc_fence_after();
        for (int j = 0; j < slices; ++j) {
          const uint64_t bd = desc_k(smem_u32(ring + s_s * slot_bytes + j * 1024));
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ta(tmem_s + (b & 1) * kKeys, tmem_q + j * 32 + k * 8, bd + 2 * k, idesc_s, (j | k) ? 1u : 0u);
        }
        if (++s_s == a.n_slots) s_s = 0, par ^= 1;
        umma_commit(&s_bar[b & 1]);
        return true;
      };
      ok = ok && scores(0);
      for (int b = 0; b < nb && ok; ++b) {
        if (b + 1 < nb) ok = scores(b + 1);  // (the softmax has read the scores of block b - 1: its probabilities came)
        ok = ok && mbar_wait(&p_bar[b & 1], (b >> 1) & 1, &s_abort);
        if (!ok) break;
        tc_fence_after();
        const uint64_t pd = make_smem_desc(smem_u32(sp + (b & 1) * HG * 128));
        for (int j = 0; j < a.n_chunks; ++j) {
          // 128 of the rank = two slices, 1 KB apart.  (Where the rank ends in the first of them, the second reads the next
          // row group's first slice: those sums are not stored.)
          const uint32_t c = smem_u32(ring + s_o * slot_bytes + j * 2048);
#pragma unroll
          for (int k = 0; k < 4; ++k)  // 16 keys = two row groups
            umma_bf16(tmem_o + j * 32, make_smem_desc_mn(c + k * 2 * group, 1024, group), pd + 2 * k, idesc_o, (b | k) ? 1u : 0u);
        }
        umma_commit(&empty_bar[s_o]);
        umma_commit(&o_bar[b & 1]);
        if (++s_o == a.n_slots) s_o = 0;
      }
      if (!ok) s_abort = 1;
    }
    __syncwarp();
  } else {
    const int q = warp & 3;
    const uint32_t lane_base = (uint32_t)(q * 32) << 16;
    bool ok = true;
    auto rescale = [&]() {  // this warp's quarter of O^T, every head by its factor
      for (int j = 0; j < a.n_chunks; ++j) {
        float o[32];
        tmem_ld<HG>(tmem_o + j * 32 + lane_base, o);
#pragma unroll
        for (int i = 0; i < HG; ++i) o[i] *= s_f[i];
        tmem_st<HG>(tmem_o + j * 32 + lane_base, o);
      }
      tc_fence_before();
    };
    uint32_t n_cmd = 0;
    if (q == 0) {
      // ---- softmax: thread = head ------------------------------------------------------------------------------------
      const bool live = lane < heads;
      {
        // queries -> TMEM, 32 columns (64 values) at a time
        const uint4* src = reinterpret_cast<const uint4*>(a.qa + (out_row + (live ? lane : 0)) * a.q_pitch);
        for (int c = 0; c < 2 * a.n_chunks; ++c) {
          uint4 w[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) w[i] = live ? __ldg(src + c * 8 + i) : make_uint4(0u, 0u, 0u, 0u);
          tmem_st<32>(tmem_q + c * 32, *reinterpret_cast<const float(*)[32]>(w));
        }
        tc_fence_before();
        mbar_arrive(&q_bar);
      }
      float m = -INFINITY, l = 0.f;
      for (int b = 0; b < nb; ++b) {
        if (!mbar_wait(&s_bar[b & 1], (b >> 1) & 1, &s_abort)) s_abort = 1;
        tc_fence_after();
        float s0[32], s1[32];
        tmem_ld32(tmem_s + (b & 1) * kKeys, s0);
        tmem_ld32(tmem_s + (b & 1) * kKeys + 32, s1);
        const int valid = n_keys - (b0 + b) * kKeys;  // keys of this block that exist (>= 64: all)
        float mx0 = -INFINITY, mx1 = -INFINITY;
        if (valid >= kKeys) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            s0[i] *= a.scale_log2, s1[i] *= a.scale_log2;
            mx0 = fmaxf(mx0, s0[i]), mx1 = fmaxf(mx1, s1[i]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            s0[i] = i < valid ? s0[i] * a.scale_log2 : -INFINITY, s1[i] = i + 32 < valid ? s1[i] * a.scale_log2 : -INFINITY;
            mx0 = fmaxf(mx0, s0[i]), mx1 = fmaxf(mx1, s1[i]);
          }
        }
        const float mx = fmaxf(mx0, mx1);
        float f = 1.f;
        if (live && mx > -INFINITY && (m == -INFINITY || mx > m + kRescale)) {
          f = ex2(m - mx);  // (0 while nothing has been seen)
          m = mx;
          l *= f;
        }
        if (b > 0 && __any_sync(0xffffffffu, f != 1.f)) {
          // every product issued so far must have retired before the sums are touched
          if (!mbar_wait(&o_bar[(b - 1) & 1], ((b - 1) >> 1) & 1, &s_abort)) s_abort = 1;
          tc_fence_after();
          s_f[lane] = f;
          __syncwarp();
          mbar_arrive(&cmd_bar);
          rescale();
          mbar_arrive(&ack_bar);
          if (!mbar_wait(&ack_bar, n_cmd & 1, &s_abort)) s_abort = 1;
          ++n_cmd;
        }
        const float base = m == -INFINITY ? 0.f : m;
        float l0 = 0.f, l1 = 0.f;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s0[i] = ex2(s0[i] - base), s1[i] = ex2(s1[i] - base);
          l0 += s0[i], l1 += s1[i];
        }
        l += l0 + l1;
        // the product of block b - 2 has read this buffer
        if (b >= 2 && !mbar_wait(&o_bar[b & 1], ((b >> 1) & 1) ^ 1, &s_abort)) s_abort = 1;
        if (lane < HG) {
          uint8_t* pr = sp + (b & 1) * HG * 128 + lane * 128;
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float f0[8] = {s0[8 * c], s0[8 * c + 1], s0[8 * c + 2], s0[8 * c + 3], s0[8 * c + 4], s0[8 * c + 5], s0[8 * c + 6], s0[8 * c + 7]};
            const float f1[8] = {s1[8 * c], s1[8 * c + 1], s1[8 * c + 2], s1[8 * c + 3], s1[8 * c + 4], s1[8 * c + 5], s1[8 * c + 6], s1[8 * c + 7]};
            *reinterpret_cast<uint4*>(pr + ((c ^ (lane & 7)) << 4)) = pack8(f0);
            *reinterpret_cast<uint4*>(pr + (((c + 4) ^ (lane & 7)) << 4)) = pack8(f1);
          }
        }
        if (valid < kKeys) {
          // latents of keys that do not exist (whatever the last page holds there, and pages that were not copied): their probability is 0, but 0 * NaN is
          // not.  The scores of this block have been computed, so its pages have landed.
          uint4* c = reinterpret_cast<uint4*>(ring + (b % a.n_slots) * slot_bytes);
          const int per_group = a.pitch;  // 16-byte chunks of 8 keys: [slice][key][8]
          for (int i = (valid >> 3) * per_group + lane; i < 8 * per_group; i += 32)
            if (i >= ((valid + 7) >> 3) * per_group || ((i >> 3) & 7) >= (valid & 7)) c[i] = make_uint4(0u, 0u, 0u, 0u);
        }
        tc_fence_before();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        mbar_arrive(&p_bar[b & 1]);
      }
      if (!mbar_wait(&o_bar[(nb - 1) & 1], ((nb - 1) >> 1) & 1, &s_abort)) s_abort = 1;
      s_f[lane] = a.n_splits == 1 ? (l > 0.f ? 1.f / l : 0.f) : 1.f;
      if (a.n_splits > 1 && live) a.ml[(out_row + lane) * a.n_splits + split] = make_float2(m, l);
      if (lane == 0) s_end = 1;
      __syncwarp();
      mbar_arrive(&cmd_bar);
    } else {
      // ---- the other output warps: rescale on request, until the sums are complete -------------------------------------
      while (true) {
        ok = mbar_wait(&cmd_bar, n_cmd & 1, &s_abort);
        if (!ok || *(volatile int*)&s_end) break;
        tc_fence_after();
        rescale();
        mbar_arrive(&ack_bar);
        if (!mbar_wait(&ack_bar, n_cmd & 1, &s_abort)) break;  // nobody is a request ahead of the others
        ++n_cmd;
      }
      if (!ok) s_abort = 1;
    }
    tc_fence_after();
    if (!*(volatile int*)&s_abort) {
      for (int j = 0; j < a.n_chunks; ++j) {
        float o[32];
        tmem_ld<HG>(tmem_o + j * 32 + lane_base, o);
        const int r = j * 128 + q * 32 + lane;
#pragma unroll
        for (int i = 0; i < HG; ++i) {
          if (i < heads) {
            const size_t row = out_row + i;
            if (a.n_splits == 1)
              a.out[row * a.q_pitch + r] = __float2bfloat16_rn(r < a.R ? o[i] * s_f[i] : 0.f);
            else
              a.part[(row * a.n_splits + split) * a.q_pitch + r] = r < a.R ? o[i] : 0.f;
          }
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
  if (warp == 1) tmem_dealloc(tmem_s, kTmemCols);
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

// Splits of a row's keys: the count that finishes first when every CTA has an SM to itself, with about three blocks'
// time of fixed cost per CTA.
int pick_splits(int T, int H, int max_keys) {
  int dev = 0, sms = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const long long ctas = (long long)T * ((H + head_group(H) - 1) / head_group(H));
  const int blocks = (max_keys + kKeys - 1) / kKeys;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 32 && s <= blocks; ++s) {
    const double waves = (double)((ctas * s + sms - 1) / sms);
    const double cost = waves * ((blocks + s - 1) / s + 3.0) + (s > 1 ? 2.0 : 0.0);
    if (cost < best_cost - 1e-9) best_cost = cost, best = s;
  }
  return best;
}

template <int HG>
int launch_lt(const LtArgs& a, int T, cudaStream_t st) {
  const int smem = a.n_slots * kKeys * a.pitch * 2 + 2 * HG * 128 + 1024;
  static std::atomic<unsigned long long> attr_done{0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!((attr_done.load(std::memory_order_acquire) >> (dev & 63)) & 1ull)) {
    cudaError_t e = cudaFuncSetAttribute(latent_attn_tc_kernel<HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
    if (e != cudaSuccess) return fail(MLORA_ECUDA, "latent_attention: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    attr_done.fetch_or(1ull << (dev & 63), std::memory_order_release);
  }
  launch_pdl_if(pdl_enabled_attn(), latent_attn_tc_kernel<HG>, dim3(T, a.n_splits, (a.H + HG - 1) / HG), kLtThreads, smem, st, a);
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
  const int n_chunks = (R + 127) / 128;
  MLORA_REQUIRE(T >= 0 && H > 0 && R > 0 && R <= kMaxChunks * 128 && pitch >= R && pitch % 64 == 0 && pitch <= n_chunks * 128 && max_pages > 0 && n_pages_total > 0,
                "latent_attention: bad sizes (kv_rank up to %d, cache pitch a multiple of 64)", kMaxChunks * 128);
  MLORA_REQUIRE(page_size == 16 || page_size == 32, "latent_attention: page size 16 or 32 (got %d)", page_size);
  MLORA_REQUIRE(q_pitch == n_chunks * 128, "latent_attention: rows of qa and out have kv_rank rounded up to 128 columns (got %lld)", (long long)q_pitch);
  MLORA_REQUIRE(d_qa && d_pages && d_block_table && d_row_slot && d_row_pos && d_out && aligned16(d_qa) && aligned16(d_pages) &&
                    aligned16(d_out) && (int64_t)n_pages_total * page_size < 0x7fffffff && (int64_t)T * H < 0x7fffffff,
                "latent_attention: null or unaligned pointer, or too many rows");
  MLORA_REQUIRE(n_splits >= 1 && n_splits <= 65535, "latent_attention: bad n_splits %d", n_splits);
  const size_t need = mlora_latent_attention_workspace(T, H, (int32_t)q_pitch, n_splits);
  MLORA_REQUIRE(!need || (d_work && aligned16(d_work) && work_bytes >= need), "latent_attention: workspace of %zu bytes needed, %zu given", need, work_bytes);
  if (T == 0) return MLORA_OK;
  const int HG = head_group(H);
  LtArgs a{};
  a.block_table = d_block_table;
  a.max_pages = max_pages;
  a.page_size = page_size;
  a.pages = (const uint8_t*)d_pages;
  a.R = R;
  a.pitch = pitch;
  a.row_slot = d_row_slot;
  a.row_pos = d_row_pos;
  a.qa = (const bf16*)d_qa;
  a.H = H;
  a.q_pitch = (int)q_pitch;
  a.n_chunks = n_chunks;
  a.n_slots = (224 * 1024 - 2 * HG * 128 - 1024) / (kKeys * pitch * 2);
  if (a.n_slots > kMaxSlots) a.n_slots = kMaxSlots;
  a.n_splits = n_splits;
  a.scale_log2 = scale * kLog2e;
  a.out = (bf16*)d_out;
  a.part = (float*)d_work;
  a.ml = (float2*)((float*)d_work + (size_t)T * H * n_splits * q_pitch);
  a.status = d_status;
  const int rc = HG == 16 ? launch_lt<16>(a, T, (cudaStream_t)stream) : launch_lt<32>(a, T, (cudaStream_t)stream);
  if (rc || n_splits == 1) return rc;
  launch_pdl_if(pdl_enabled_norm(), latent_merge_kernel, (unsigned)(T * H), 128, 0, (cudaStream_t)stream, a.part, a.ml, n_splits, (int)q_pitch, (bf16*)d_out);
  count_launch();
  MLORA_CHECK_LAUNCH("latent_merge_kernel");
  return MLORA_OK;
}
