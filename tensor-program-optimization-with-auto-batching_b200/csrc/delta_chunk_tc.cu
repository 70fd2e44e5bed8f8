// The gated delta rule over whole prompts on the 5th-generation tensor cores: 64 tokens at a time instead of one.
//
// With c_1 .. c_64 the decays of a chunk, C_i = c_1 ... c_i, S the state before it and b_i the steps, the rule of delta.cu
// unrolled over the chunk reads (i, j tokens; K, Q, V, W the rows k_i, q_i, v_i, w_i)
//
//   W = T R             T = (1 + L)^-1,  L_ij = b_i (C_i / C_j) (k_i . k_j) for j < i,    R_i = b_i (v_i - C_i S^T k_i)
//   out_i = C_i S^T q_i + sum_j A_ij w_j                                  A_ij = (C_i / C_j) (q_i . k_j) for j <= i
//   S' = C_64 S + sum_j (C_64 / C_j) k_j w_j^T
//
// (the compact form of a product of Householder-like factors.)  T and A depend on keys, queries and decays only:
// delta_chunk_prepare computes them for all chunks of all heads at once; delta_chunk then walks the chunks of a (head,
// sequence) one after the other, four products each, with the state in registers.
//
// Precision: the rule is kept in 32-bit.  A tensor-core operand holds 8 significant bits (bf16), so every fp32 factor is
// split into three bf16 planes h + m + l (24 bits) and a product of two such factors is the sum of the six plane products
// that matter, accumulated in fp32.  Keys and queries enter as they come out of the convolution, which is bf16 already: one
// plane, exact; their lengths, decays and steps are fp32 scalars per token, applied outside the products.  C_i / C_j is
// exp of a difference of summed logarithms, the sums kept as two floats each.
//
// Layout: lane of TMEM = column v of the state, so that every product has M = 128 = vdim and the thread that owns lane v can
// write the next product's A operand (R, W: into TMEM; S: into shared memory) without any exchange.
#include <math.h>

#include "delta.cuh"
#include "tc_ptx.cuh"

namespace mlora {
namespace {

constexpr int kC = 64;                   // tokens per chunk
constexpr int kSub = 128 * 64 * 2;       // one [128 x 64] bf16 operand tile
constexpr int kPlane = kC * kC * 2;      // one plane of T or A: [64 x 64] bf16 = a K-major operand with 128-byte rows
constexpr int kScal = 1280;              // per chunk: float4 per token, then C_64
constexpr int kRec = 6 * kPlane + kScal; // what prepare leaves per (chunk, head)

struct ChunkArgs {
  const bf16* xc;      // [T, C] after convolution and silu
  const bf16* x;       // projected rows
  int64_t ld;
  int C, taps, b_col, a_col;
  const float *A_log, *dt_bias;
  DeltaDims d;
  const int4* segs;    // (slot, first row, rows, position of the first row)
  float* state;        // [slot][heads][dim][vdim]
  bf16* ring;          // [slot][taps][C]
  float* out;          // [T, heads * vdim]
  uint8_t* rec;
  int32_t* status;
};

// Record of chunk c of segment s (rows / 64 + s never collide: a segment has at most rows / 64 + 1 chunks).
__device__ __forceinline__ uint8_t* record(const ChunkArgs& a, const int4& seg, int s, int c, int h) {
  return a.rec + ((size_t)(seg.y / kC + s + c) * a.d.heads + h) * kRec;
}

// f = h + m + l, each of eight values rounded to bf16.
__device__ __forceinline__ void split8(const float (&f)[8], uint32_t (&p)[3][4]) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float a = f[2 * i], b = f[2 * i + 1];
#pragma unroll
    for (int k = 0; k < 3; ++k) {
      const __nv_bfloat162 r = __floats2bfloat162_rn(a, b);
      p[k][i] = *reinterpret_cast<const uint32_t*>(&r);
      a -= __low2float(r);
      b -= __high2float(r);
    }
  }
}

// ---- per (chunk, head): T, A and the tokens' scalars ---------------------------------------------------------------------
constexpr int kPrepThreads = 160;  // warps 0..3: one thread per row of [K; Q]; warp 4: loads and MMA
constexpr int kLPitch = kC + 4;

template <int NK>
constexpr int prep_smem() {
  return (NK * kSub > 3 * kPlane ? NK * kSub : 3 * kPlane) + kC * kLPitch * 4 + 1024;
}

template <int NK>
__global__ void __launch_bounds__(kPrepThreads) delta_chunk_prepare_kernel(const __grid_constant__ CUtensorMap map, ChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* s_kq = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  float* s_L = reinterpret_cast<float*>(s_kq + (NK * kSub > 3 * kPlane ? NK * kSub : 3 * kPlane));  // [64][kLPitch]
  __shared__ uint64_t kbar, dbar;
  __shared__ uint32_t tmem_slot;
  __shared__ int s_abort;
  __shared__ float s_inv[128], s_hi[kC], s_lo[kC], s_b[kC];
  __shared__ double s_first;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.x, c = blockIdx.y, s = blockIdx.z;
  const int4 seg = a.segs[s];
  const int n = min(kC, seg.z - c * kC);
  if (n <= 0) return;
  const DeltaDims d = a.d;
  const int kh = h / (d.heads / d.kv_heads), r0 = seg.y + c * kC;
  uint8_t* rec = record(a, seg, s, c, h);
  if (tid == 0) {
    s_abort = 0;
    mbar_init(&kbar, 1);
    mbar_init(&dbar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    tma_prefetch_desc(&map);
  }
  if (warp == 4) tmem_alloc(&tmem_slot, 64);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  pdl_launch_dependents();  // (not before this CTA has its TMEM: the next kernel allocates all of it)
  pdl_wait();
  bool ok = true;
  if (warp == 4) {
    if (lane == 0) {
      mbar_expect_tx(&kbar, NK * kSub);
#pragma unroll
      for (int j = 0; j < NK; ++j) {
        tma_load_2d(s_kq + j * kSub, &map, (d.kv_heads + kh) * d.dim + j * 64, r0, &kbar);
        tma_load_2d(s_kq + j * kSub + kSub / 2, &map, kh * d.dim + j * 64, r0, &kbar);
      }
      ok = mbar_wait(&kbar, 0, &s_abort);
      if (ok) {
        constexpr uint32_t idesc = make_idesc(128, kC);
#pragma unroll
        for (int j = 0; j < NK; ++j) {
          const uint64_t desc = make_smem_desc(smem_u32(s_kq + j * kSub));  // A: all 128 rows; B: the keys, its first 64
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_bf16(tmem, desc + 2 * k, desc + 2 * k, idesc, (j | k) ? 1u : 0u);
        }
        umma_commit(&dbar);
      } else {
        s_abort = 1;
      }
    }
    __syncwarp();
  } else {
    if (tid < kC) {  // steps; logarithms of the decays summed over the chunk
      double v = 0.;
      float b = 0.f;
      if (tid < n) {
        const bf16* row = a.x + (size_t)(r0 + tid) * a.ld;
        b = step_size(__bfloat162float(row[a.b_col + h]));
        v = log_decay(__bfloat162float(row[a.a_col + h]), a.A_log[h], a.dt_bias[h]);
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double y = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += y;
      }
      if (tid == 31) s_first = v;
      asm volatile("bar.sync 2, 64;" ::: "memory");
      if (warp == 1) v += s_first;
      const float hi = (float)v;
      s_hi[tid] = hi;
      s_lo[tid] = (float)(v - (double)hi);
      s_b[tid] = b;
    }
    if (!mbar_wait(&kbar, 0, &s_abort)) ok = false, s_abort = 1;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NK; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) {  // (a swizzled row stays inside its own 128 bytes)
        float f[8];
        unpack8(*reinterpret_cast<const uint4*>(s_kq + j * kSub + tid * 128 + ((i ^ (tid & 7)) << 4)), f);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(f[e], f[e], ss);
      }
    s_inv[tid] = (tid < kC ? 1.f : d.q_scale) / sqrtf(ss + 1e-6f);
  }
  __syncthreads();
  if (warp < 4) {
    if (!mbar_wait(&dbar, 0, &s_abort)) ok = false, s_abort = 1;
    tc_fence_after();
    const int t = tid & (kC - 1);
    const bool is_k = tid < kC;
    const float hi = s_hi[t], lo = s_lo[t], mine = s_inv[tid] * (is_k ? s_b[t] : 1.f);
    const uint32_t addr = tmem + ((uint32_t)(warp * 32) << 16);
#pragma unroll
    for (int c0 = 0; c0 < kC; c0 += 32) {
      float g[32];
      tmem_ld32(addr + c0, g);
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const int j = c0 + i;
        const bool in = is_k ? j < t : j <= t;
        g[i] = in ? g[i] * (mine * s_inv[j]) * expf((hi - s_hi[j]) + (lo - s_lo[j])) : 0.f;
      }
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (is_k) {
          *reinterpret_cast<float4*>(s_L + t * kLPitch + c0 + q * 8) = make_float4(g[q * 8], g[q * 8 + 1], g[q * 8 + 2], g[q * 8 + 3]);
          *reinterpret_cast<float4*>(s_L + t * kLPitch + c0 + q * 8 + 4) = make_float4(g[q * 8 + 4], g[q * 8 + 5], g[q * 8 + 6], g[q * 8 + 7]);
        } else {
          float f[8];
          uint32_t p[3][4];
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = g[q * 8 + e];
          split8(f, p);
#pragma unroll
          for (int k = 0; k < 3; ++k)
            *reinterpret_cast<uint4*>(rec + (3 + k) * kPlane + t * 128 + ((((c0 >> 3) + q) ^ (t & 7)) << 4)) =
                make_uint4(p[k][0], p[k][1], p[k][2], p[k][3]);
        }
      }
    }
    if (is_k) {
      const float C = expf(hi + lo);
      const float4 v = make_float4(s_b[t] * C * s_inv[t], s_b[t], C * s_inv[kC + t], s_inv[t] * expf((s_hi[kC - 1] - hi) + (s_lo[kC - 1] - lo)));
      reinterpret_cast<float4*>(rec + 6 * kPlane)[t] = v;
      if (t == kC - 1) *reinterpret_cast<float*>(rec + 6 * kPlane + kC * 16) = C;
    }
    tc_fence_before();
  }
  __syncthreads();
  // T, a column per thread, by forward substitution; planes into shared memory (over K and Q, which the MMAs have read)
  if (tid < kC) {
    float x[kC];
#pragma unroll
    for (int i = 0; i < kC; ++i) {
      float s0 = i == tid ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
      for (int j = 0; j + 4 <= (i + 3) / 4 * 4; j += 4) {  // (L is zero from its diagonal on)
        const float4 l = *reinterpret_cast<const float4*>(s_L + i * kLPitch + j);
        s0 = fmaf(-l.x, x[j], s0);
        if (j + 1 < i) s1 = fmaf(-l.y, x[j + 1], s1);
        if (j + 2 < i) s2 = fmaf(-l.z, x[j + 2], s2);
        if (j + 3 < i) s3 = fmaf(-l.w, x[j + 3], s3);
      }
      x[i] = (s0 + s1) + (s2 + s3);
      float r = x[i];
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const bf16 v = __float2bfloat16_rn(r);
        r -= __bfloat162float(v);
        *reinterpret_cast<bf16*>(s_kq + k * kPlane + i * 128 + (((tid >> 3) ^ (i & 7)) << 4) + (tid & 7) * 2) = v;
      }
    }
  }
  __syncthreads();
  for (int i = tid; i < 3 * kPlane / 16; i += kPrepThreads) reinterpret_cast<uint4*>(rec)[i] = reinterpret_cast<const uint4*>(s_kq)[i];
  if (!ok && a.status) atomicOr(a.status, 1);
  if (warp == 4) tmem_dealloc(tmem, 64);
}

// ---- the walk over the chunks ------------------------------------------------------------------------------------------------
constexpr int kWalkThreads = 288;  // warps 0..7: lane v of the state, half of its columns / of the tokens; warp 8: loads, MMA
constexpr uint32_t kD1 = 0, kD2 = 128, kD4 = 192, kRW = 320, kWt = 416;  // TMEM columns: S^T [K; Q], T R then A W, K^T W, planes

template <int NK>
constexpr int walk_smem() { return 5 * NK * kSub + 6 * kPlane + 4 * kScal + 1024; }

// (The issue loop's descriptors are sums of one base and constants: recomputed per chunk, not kept in registers across it.)
__device__ __forceinline__ uint64_t opaque(uint64_t v) {
  asm volatile("" : "+l"(v));
  return v;
}

// Six products of two factors in three planes each, smallest first, added to what dst holds if `add`: A in TMEM, B [64 x 64]
// in shared memory.
__device__ __forceinline__ void umma_planes(uint32_t dst, uint32_t a, const uint8_t* b, bool add) {
  constexpr uint32_t idesc = make_idesc(128, kC);
  constexpr int pa[6] = {2, 1, 0, 1, 0, 0}, pb[6] = {0, 1, 2, 0, 1, 0};
  const uint64_t first = opaque(make_smem_desc(smem_u32(b)));
#pragma unroll
  for (int p = 0; p < 6; ++p) {
    const uint64_t desc = first + pb[p] * (kPlane >> 4);
#pragma unroll
    for (int k = 0; k < 4; ++k) umma_bf16_ta(dst, a + pa[p] * 32 + k * 8, desc + 2 * k, idesc, (add || p || k) ? 1u : 0u);
  }
}

// Eight values of this lane into the three planes at TMEM column `at` (4 columns each, planes 32 apart).
__device__ __forceinline__ void store_planes(uint32_t at, const float (&f)[8]) {
  uint32_t p[3][4];
  split8(f, p);
#pragma unroll
  for (int k = 0; k < 3; ++k)
    asm volatile("tcgen05.st.sync.aligned.32x32b.x4.b32 [%0], {%1,%2,%3,%4};" ::"r"(at + k * 32), "r"(p[k][0]), "r"(p[k][1]),
                 "r"(p[k][2]), "r"(p[k][3])
                 : "memory");
}
__device__ __forceinline__ void tmem_store_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

template <int NK>
__global__ void __launch_bounds__(kWalkThreads, 1) delta_chunk_kernel(const __grid_constant__ CUtensorMap map, ChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* s_S = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* s_kq = s_S + 3 * NK * kSub;   // two buffers
  uint8_t* s_T = s_kq + 2 * NK * kSub;
  uint8_t* s_A = s_T + 3 * kPlane;
  uint8_t* s_sc = s_A + 3 * kPlane;      // four buffers
  __shared__ uint64_t kq_bar[2], sc_bar[4], t_bar, a_bar, d_bar[4];
  __shared__ uint32_t tmem_slot;
  __shared__ int s_abort;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const DeltaDims d = a.d;
  const int h = blockIdx.y, s = blockIdx.z, col0 = blockIdx.x * 128;
  const int4 seg = a.segs[s];
  const int slot = seg.x, r0 = seg.y, n = seg.z, pos0 = seg.w, nc = (n + kC - 1) / kC;
  if (n <= 0) return;
  const int kh = h / (d.heads / d.kv_heads);
  if (tid == 0) {
    s_abort = 0;
    for (int i = 0; i < 2; ++i) mbar_init(&kq_bar[i], 1);
    for (int i = 0; i < 4; ++i) mbar_init(&sc_bar[i], 1);
    for (int i = 0; i < 4; ++i) mbar_init(&d_bar[i], 1);
    mbar_init(&t_bar, 1);
    mbar_init(&a_bar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    tma_prefetch_desc(&map);
  }
  if (warp == 8) tmem_alloc(&tmem_slot, 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  pdl_launch_dependents();
  pdl_wait();
  bool ok = true;
  const auto wait = [&](uint64_t* bar, uint32_t par) {
    if (!mbar_wait(bar, par, &s_abort)) ok = false, s_abort = 1;
  };

  if (warp == 8) {
    const int q_col = kh * d.dim, k_col = (d.kv_heads + kh) * d.dim;
    const auto load_kq = [&](int c) {
      uint64_t* bar = &kq_bar[c & 1];
      uint8_t* dst = s_kq + (c & 1) * NK * kSub;
      mbar_expect_tx(bar, NK * kSub);
#pragma unroll
      for (int j = 0; j < NK; ++j) {
        tma_load_2d(dst + j * kSub, &map, k_col + j * 64, r0 + c * kC, bar);
        tma_load_2d(dst + j * kSub + kSub / 2, &map, q_col + j * 64, r0 + c * kC, bar);
      }
      mbar_expect_tx(&sc_bar[c & 3], kScal);
      bulk_load(s_sc + (c & 3) * kScal, record(a, seg, s, c, h) + 6 * kPlane, kScal, &sc_bar[c & 3]);
    };
    const auto load_planes = [&](int c, int which, uint8_t* dst, uint64_t* bar) {
      mbar_expect_tx(bar, 3 * kPlane);
      bulk_load(dst, record(a, seg, s, c, h) + which * 3 * kPlane, 3 * kPlane, bar);
    };
    if (lane == 0) {
      load_kq(0);
      load_planes(0, 0, s_T, &t_bar);
      load_planes(0, 1, s_A, &a_bar);
      if (nc > 1) load_kq(1);
    }
    __syncwarp();
    for (int c = 0; c < nc; ++c) {
      const uint8_t* kq = s_kq + (c & 1) * NK * kSub;
      if (__syncthreads_or(!ok)) break;  // (1) the state's planes are there
      if (lane == 0) {
        wait(&kq_bar[c & 1], (c >> 1) & 1);
        tc_fence_after();
        constexpr uint32_t idesc = make_idesc(128, 128);
        const uint64_t a0 = opaque(make_smem_desc(smem_u32(s_S))), b0 = opaque(make_smem_desc(smem_u32(kq)));
#pragma unroll
        for (int p = 2; p >= 0; --p)
#pragma unroll
          for (int j = 0; j < NK; ++j) {
            const uint64_t ad = a0 + (p * NK + j) * (kSub >> 4), bd = b0 + j * (kSub >> 4);
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_bf16(tmem + kD1, ad + 2 * k, bd + 2 * k, idesc, (p < 2 || j || k) ? 1u : 0u);
          }
        umma_commit(&d_bar[0]);
      }
      __syncwarp();
      __syncthreads();  // (2) R is there
      if (lane == 0) {
        wait(&t_bar, c & 1);
        tc_fence_after();
        umma_planes(tmem + kD2, tmem + kRW, s_T, false);
        umma_commit(&d_bar[1]);
      }
      __syncwarp();
      __syncthreads();  // (3) W is there
      if (lane == 0) {
        tc_fence_after();
        constexpr uint32_t idesc = make_idesc(128, 64 * NK) | (1u << 16);  // B: keys as loaded, [token][dim], the dimension contiguous
        const uint64_t b0 = opaque(make_smem_desc_mn(smem_u32(kq), kSub, 1024));
#pragma unroll
        for (int p = 2; p >= 0; --p)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ta(tmem + kD4, tmem + kWt + p * 32 + k * 8, b0 + k * (2048 >> 4), idesc,
                         (p < 2 || k) ? 1u : 0u);
        umma_commit(&d_bar[3]);
        wait(&a_bar, c & 1);
        umma_planes(tmem + kD2, tmem + kRW, s_A, true);  // onto C_i S^T q_i
        umma_commit(&d_bar[2]);
        // what these products have read is free again
        wait(&d_bar[3], c & 1);
        if (c + 1 < nc) load_planes(c + 1, 0, s_T, &t_bar);
        if (c + 2 < nc) load_kq(c + 2);
        wait(&d_bar[2], c & 1);
        if (c + 1 < nc) load_planes(c + 1, 1, s_A, &a_bar);
      }
      __syncwarp();
    }
    __syncthreads();  // the walk's end
    if (s_abort && lane == 0) {  // gave up: what is still being copied gets a bounded chance to land before the memory goes
      int none = 0;
      for (int i = 0; i < 2; ++i) mbar_wait(&kq_bar[i], 0, &none);
      mbar_wait(&t_bar, 0, &none);
      mbar_wait(&a_bar, 0, &none);
    }
  } else {
    const int half = warp >> 2, v = (warp & 3) * 32 + lane;  // this thread's lane of TMEM = column of the state
    const uint32_t base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const bool live = col0 + v < d.vdim;
    constexpr int kCols = 32 * NK;
    float S[kCols];  // rows half * kCols + i of column v
    float* state = a.state + (((size_t)slot * d.heads + h) * d.dim + half * kCols) * d.vdim + col0 + v;
    {
      const float* p = state;
#pragma unroll
      for (int i = 0; i < kCols; ++i) {
        S[i] = (live && pos0 > 0) ? *p : 0.f;
        p += d.vdim;
        asm volatile("" : "+l"(p));  // (one pointer that moves on, not an offset per element kept in registers)
      }
    }
    const bf16* vin = a.xc + (size_t)(r0 + half * 32) * a.C + 2 * d.kv_heads * d.dim + h * d.vdim + col0 + v;
    float* out = a.out + ((size_t)(r0 + half * 32) * d.heads + h) * d.vdim + col0 + v;
    bf16 vv[32];
    const auto fetch_v = [&](int c) {
      const bf16* p = vin + (size_t)c * kC * a.C;
      const int m = live ? n - c * kC - half * 32 : 0;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        vv[i] = i < m ? *p : __float2bfloat16_rn(0.f);
        p += a.C;
        asm volatile("" : "+l"(p));
      }
    };
    const auto store_state = [&]() {  // planes of S as K-major operand tiles
#pragma unroll
      for (int q = 0; q < kCols / 8; ++q) {
        float f[8];
        uint32_t p[3][4];
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = S[q * 8 + e];
        split8(f, p);
        const int col = half * kCols + q * 8;
        const int at = (col >> 6) * kSub + v * 128 + ((((col & 63) >> 3) ^ (v & 7)) << 4);
#pragma unroll
        for (int k = 0; k < 3; ++k) *reinterpret_cast<uint4*>(s_S + k * NK * kSub + at) = make_uint4(p[k][0], p[k][1], p[k][2], p[k][3]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    };
    const auto write_out = [&](int c) {
      wait(&d_bar[2], c & 1);
      tc_fence_after();
      float y[32];
      tmem_ld32(base + kD2 + half * 32, y);
      float* p = out + (size_t)c * kC * d.heads * d.vdim;
      const int m = live ? n - c * kC - half * 32 : 0;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        if (i < m) *p = y[i];
        p += (size_t)d.heads * d.vdim;
        asm volatile("" : "+l"(p));
      }
    };
    store_state();
    fetch_v(0);
    for (int c = 0; c < nc; ++c) {
      const float4* sc = reinterpret_cast<const float4*>(s_sc + (c & 3) * kScal) + half * 32;
      tc_fence_before();
      if (__syncthreads_or(!ok)) break;  // (1)
      if (c > 0) write_out(c - 1);
      wait(&sc_bar[c & 3], (c >> 2) & 1);
      wait(&d_bar[0], c & 1);
      tc_fence_after();
      {
        float ks[32];
        tmem_ld32(base + kD1 + half * 32, ks);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float r[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float4 x = sc[q * 8 + e];
            r[e] = fmaf(-x.x, ks[q * 8 + e], x.y * __bfloat162float(vv[q * 8 + e]));
          }
          store_planes(base + kRW + half * 16 + q * 4, r);
        }
        tmem_store_wait();
      }
      if (c + 1 < nc) fetch_v(c + 1);
      tc_fence_before();
      __syncthreads();  // (2)
      wait(&d_bar[1], c & 1);
      tc_fence_after();
      {
        float w[32];
        tmem_ld32(base + kD2 + half * 32, w);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float r[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) r[e] = w[q * 8 + e] * sc[q * 8 + e].w;
          store_planes(base + kWt + half * 16 + q * 4, r);
#pragma unroll
          for (int e = 0; e < 8; ++e) r[e] = w[q * 8 + e];
          store_planes(base + kRW + half * 16 + q * 4, r);
        }
        tmem_ld32(base + kD1 + 64 + half * 32, w);  // what A W is added to
#pragma unroll
        for (int i = 0; i < 32; ++i) w[i] *= sc[i].z;
        tmem_st<32>(base + kD2 + half * 32, w);
      }
      tc_fence_before();
      __syncthreads();  // (3)
      const float C = *reinterpret_cast<const float*>(s_sc + (c & 3) * kScal + kC * 16);
      wait(&d_bar[3], c & 1);
      tc_fence_after();
#pragma unroll
      for (int g = 0; g < NK; ++g) {
        float y[32];
        tmem_ld32(base + kD4 + half * kCols + g * 32, y);
#pragma unroll
        for (int i = 0; i < 32; ++i) S[g * 32 + i] = fmaf(C, S[g * 32 + i], y[i]);
      }
      if (c + 1 < nc) store_state();
    }
    if (ok) write_out(nc - 1);
#pragma unroll
    for (int i = 0; i < kCols; ++i) {
      if (live) *state = S[i];
      state += d.vdim;
      asm volatile("" : "+l"(state));
    }
    // the ring: every channel once (q and k by the first head that uses them and the first column part)
    const int q_col = kh * d.dim, k_col = (d.kv_heads + kh) * d.dim, v_col = 2 * d.kv_heads * d.dim + h * d.vdim + col0;
    const bool owns_qk = blockIdx.x == 0 && h % (d.heads / d.kv_heads) == 0;
    for (int t = max(0, n - a.taps); t < n; ++t) {
      const bf16* row = a.x + (size_t)(r0 + t) * a.ld;
      bf16* dst = a.ring + ((size_t)slot * a.taps + (pos0 + t) % a.taps) * a.C;
      if (owns_qk && half == 0)
        for (int i = v; i < d.dim; i += 128) dst[q_col + i] = row[q_col + i];
      if (owns_qk && half == 1)
        for (int i = v; i < d.dim; i += 128) dst[k_col + i] = row[k_col + i];
      if (live && half == 0) dst[v_col + v] = row[v_col + v];
    }
    if (!ok && a.status) atomicOr(a.status, 1);
    tc_fence_before();
    __syncthreads();  // the walk's end
  }
  if (warp == 8) tmem_dealloc(tmem, 512);
}

template <int NK>
int launch_chunks(const CUtensorMap& map, const ChunkArgs& a, int n_segs, int max_rows, cudaStream_t st) {
  cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem<NK>());
  if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, walk_smem<NK>());
  if (e != cudaSuccess) return fail(MLORA_ECUDA, "delta_chunk: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  launch_pdl(delta_chunk_prepare_kernel<NK>, dim3(a.d.heads, (max_rows + kC - 1) / kC, n_segs), kPrepThreads, prep_smem<NK>(), st, map, a);
  launch_pdl(delta_chunk_kernel<NK>, dim3((a.d.vdim + 127) / 128, a.d.heads, n_segs), kWalkThreads, walk_smem<NK>(), st, map, a);
  count_launch(2);
  MLORA_CHECK_LAUNCH("delta_chunk_kernel");
  return MLORA_OK;
}

}  // namespace
}  // namespace mlora

using namespace mlora;

extern "C" size_t mlora_delta_chunk_workspace(int32_t T, int32_t n_segs, int32_t heads) {
  if (T <= 0 || n_segs <= 0 || heads <= 0) return 0;
  return (size_t)(T / kC + n_segs + 1) * heads * kRec;
}

extern "C" int mlora_delta_chunk(const void* d_xc, const void* d_x, int64_t ld, int32_t C, int32_t taps, int32_t b_col, int32_t a_col,
                                 const float* d_A_log, const float* d_dt_bias, int32_t heads, int32_t kv_heads, int32_t dim,
                                 int32_t vdim, float q_scale, const int32_t* d_segs, int32_t n_segs, int32_t T, int32_t max_rows,
                                 float* d_state, void* d_ring, float* d_out, void* d_work, size_t work_bytes, int32_t* d_status,
                                 void* stream) {
  const DeltaDims d{heads, kv_heads, dim, vdim, vdim, q_scale};
  const int rc = check_delta_dims("delta_chunk", d, C, taps);
  if (rc) return rc;
  MLORA_REQUIRE(dim == 64 || dim == 128, "delta_chunk: dim 64 or 128 (got %d)", dim);
  MLORA_REQUIRE(n_segs >= 0 && n_segs <= 65535 && T >= 0 && max_rows >= 0 && max_rows <= T && (max_rows + kC - 1) / kC <= 65535 &&
                    ld >= C && b_col >= 0 && a_col >= 0 && b_col + heads <= ld && a_col + heads <= ld,
                "delta_chunk: bad sizes");
  MLORA_REQUIRE(d_xc && d_x && d_A_log && d_dt_bias && d_segs && d_state && d_ring && d_out && d_work, "delta_chunk: null pointer");
  MLORA_REQUIRE(aligned16(d_xc) && aligned16(d_segs) && aligned16(d_work), "delta_chunk: pointers must be 16-byte aligned");
  if (n_segs == 0 || max_rows == 0) return MLORA_OK;
  if (work_bytes < mlora_delta_chunk_workspace(T, n_segs, heads))
    return fail(MLORA_ESIZE, "delta_chunk: workspace of %zu bytes needed, %zu given", mlora_delta_chunk_workspace(T, n_segs, heads), work_bytes);
  CUtensorMap map;
  const int rm = make_map(&map, d_xc, T, C, C, kC, 64);
  if (rm) return rm;
  ChunkArgs a{(const bf16*)d_xc, (const bf16*)d_x, ld, C, taps, b_col, a_col, d_A_log, d_dt_bias, d, (const int4*)d_segs, d_state,
              (bf16*)d_ring, d_out, (uint8_t*)d_work, d_status};
  return dim == 64 ? launch_chunks<1>(map, a, n_segs, max_rows, (cudaStream_t)stream)
                   : launch_chunks<2>(map, a, n_segs, max_rows, (cudaStream_t)stream);
}
