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
// split into three bf16 planes h + m + l (24 bits, exactly) and a product of two such factors is the sum of the six plane products
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
constexpr int kScal = 1040;              // per chunk: four values per token (arrays of 64 floats), then C_64
constexpr int kScKey = 0, kScStep = kC, kScQuery = 2 * kC, kScEnd = 3 * kC, kScAll = 4 * kC;  // b C_i / |k|, b, C_i / |q|, C_64 / (C_i |k|), C_64
constexpr int kRec = 6 * kPlane + 1280;  // what prepare leaves per (chunk, head)

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

// f = h + m + l exactly: the upper 16 bits of f are the bf16 h, of f - h the bf16 m, and what is left has at most eight bits.
// (Cut off, not rounded: masks and subtractions instead of conversions.)
__device__ __forceinline__ void split8(const float (&f)[8], uint32_t (&p)[3][4]) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float a = f[2 * i], b = f[2 * i + 1];
#pragma unroll
    for (int k = 0; k < 3; ++k) {
      const uint32_t ua = __float_as_uint(a), ub = __float_as_uint(b);
      p[k][i] = __byte_perm(ua, ub, 0x7632);
      if (k < 2) a -= __uint_as_float(ua & 0xffff0000u), b -= __uint_as_float(ub & 0xffff0000u);
    }
  }
}

__device__ __forceinline__ float f4(const float4& v, int e) { return e == 0 ? v.x : e == 1 ? v.y : e == 2 ? v.z : v.w; }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ---- per (chunk, head): T, A and the tokens' scalars ---------------------------------------------------------------------
constexpr int kPrepThreads = 160;  // warps 0..3: one thread per row of [K; Q]; warp 4: loads and MMA
constexpr int kLPitch = kC + 4, kBPitch = 32 + 4;

template <int NK>
constexpr int prep_kq() { return NK * kSub > 3 * kPlane ? NK * kSub : 3 * kPlane; }
template <int NK>
constexpr int prep_smem() { return prep_kq<NK>() + 3 * kPlane + 3 * 32 * kBPitch * 4 + 1024; }  // K and Q, then A's planes; L, then T's planes; blocks

// Columns 8 q .. 8 q + 7 of a row of T or A as planes of a K-major operand tile.
__device__ __forceinline__ void write_chunk(uint8_t* planes, int row, int q, const float (&f)[8]) {
  uint32_t p[3][4];
  split8(f, p);
#pragma unroll
  for (int k = 0; k < 3; ++k)
    *reinterpret_cast<uint4*>(planes + k * kPlane + row * 128 + ((q ^ (row & 7)) << 4)) = make_uint4(p[k][0], p[k][1], p[k][2], p[k][3]);
}
template <int N>
__device__ __forceinline__ void write_row(uint8_t* planes, int row, int q0, const float (&f)[N]) {
#pragma unroll
  for (int q = 0; q < N / 8; ++q) {
    float e[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) e[i] = f[q * 8 + i];
    write_chunk(planes, row, q0 + q, e);
  }
}
// Eight neighbouring sums over 32 products: a[i] is this thread's, at stride `step`; rows of b are shared by its warp.
__device__ __forceinline__ void dot32(const float* a, int step, const float* b, float (&y)[8]) {
#pragma unroll
  for (int e = 0; e < 8; ++e) y[e] = 0.f;
#pragma unroll
  for (int i = 0; i < 32; ++i) {
    const float x = a[i * step];
    const float4 u = *reinterpret_cast<const float4*>(b + i * kBPitch), w = *reinterpret_cast<const float4*>(b + i * kBPitch + 4);
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = fmaf(x, f4(u, e), y[e]), y[4 + e] = fmaf(x, f4(w, e), y[4 + e]);
  }
}
__device__ __forceinline__ void bulk_store(void* dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(smem_u32(src)), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

template <int NK>
__global__ void __launch_bounds__(kPrepThreads, 3) delta_chunk_prepare_kernel(const __grid_constant__ CUtensorMap map, ChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* s_kq = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* s_T = s_kq + prep_kq<NK>();
  float* s_L = reinterpret_cast<float*>(s_T);  // [64][kLPitch], transposed: row j holds L_ij of all i
  float* s_T1 = reinterpret_cast<float*>(s_T + 3 * kPlane);  // [32][kBPitch] each: T's upper left block,
  float* s_T2 = s_T1 + 32 * kBPitch;                         // its lower right block, transposed,
  float* s_Y = s_T2 + 32 * kBPitch;                          // L's lower left block times the first
  __shared__ uint64_t kbar, dbar;
  __shared__ uint32_t tmem_slot;
  __shared__ int s_abort;
  __shared__ __align__(16) float s_inv[128], s_hi[kC], s_lo[kC];
  __shared__ float s_b[kC];
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
    if (tid < kC) {  // steps; logarithms (to base 2) of the decays summed over the chunk
      double v = 0.;
      float b = 0.f;
      if (tid < n) {
        const bf16* row = a.x + (size_t)(r0 + tid) * a.ld;
        b = step_size(__bfloat162float(row[a.b_col + h]));
        v = (double)log_decay(__bfloat162float(row[a.a_col + h]), a.A_log[h], a.dt_bias[h]) * 1.4426950408889634;
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
    float ss[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < NK; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) {  // (a swizzled row stays inside its own 128 bytes)
        float f[8];
        unpack8(*reinterpret_cast<const uint4*>(s_kq + j * kSub + tid * 128 + ((i ^ (tid & 7)) << 4)), f);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss[e & 3] = fmaf(f[e], f[e], ss[e & 3]);
      }
    s_inv[tid] = (tid < kC ? 1.f : d.q_scale) / sqrtf((ss[0] + ss[1]) + (ss[2] + ss[3]) + 1e-6f);
  }
  __syncthreads();
  if (warp < 4) {
    if (!mbar_wait(&dbar, 0, &s_abort)) ok = false, s_abort = 1;
    tc_fence_after();
    const int t = tid & (kC - 1);
    const bool is_k = tid < kC;
    const float2 cum = make_float2(s_hi[t], s_lo[t]);
    const float mine = s_inv[tid] * (is_k ? s_b[t] : 1.f);
    const uint32_t addr = tmem + ((uint32_t)(warp * 32) << 16);
    float g[kC];
    tmem_ld32(addr, *reinterpret_cast<float(*)[32]>(g));
    tmem_ld32(addr + 32, *reinterpret_cast<float(*)[32]>(g + 32));
    tc_fence_before();
    const int last = is_k ? t - 1 : t;  // last column that is not zero
#pragma unroll
    for (int j = 0; j < kC; j += 4) {
      const float4 hi = *reinterpret_cast<const float4*>(s_hi + j), lo = *reinterpret_cast<const float4*>(s_lo + j);
      const float4 inv = *reinterpret_cast<const float4*>(s_inv + j);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        g[j + e] = j + e <= last ? g[j + e] * (mine * f4(inv, e)) * ex2((cum.x - f4(hi, e)) + (cum.y - f4(lo, e))) : 0.f;
    }
    if (is_k) {
#pragma unroll
      for (int j = 0; j < kC; ++j) s_L[j * kLPitch + t] = g[j];
      const float C = ex2(cum.x + cum.y);
      const float2 end = make_float2(s_hi[kC - 1], s_lo[kC - 1]);
      float* sc = reinterpret_cast<float*>(rec + 6 * kPlane);
      sc[kScKey + t] = s_b[t] * C * s_inv[t];
      sc[kScStep + t] = s_b[t];
      sc[kScQuery + t] = C * s_inv[kC + t];
      sc[kScEnd + t] = s_inv[t] * ex2((end.x - cum.x) + (end.y - cum.y));
      if (t == kC - 1) sc[kScAll] = C;
      asm volatile("bar.sync 2, 64;" ::: "memory");
      // T = (1 + L)^-1 in blocks of 32: each warp a row per lane of its diagonal block, from X (1 + L) = 1, last column first
      const float* L = s_L + warp * 32 * (kLPitch + 1);
      float x[32];
#pragma unroll
      for (int j = 31; j >= 0; --j) {
        // (four sums; the value found last comes in last, so that little waits for it)
        float y[4] = {j == lane ? 1.f : 0.f, 0.f, 0.f, 0.f}, l_next = 0.f;
#pragma unroll
        for (int i = 28; i >= (j + 1) / 4 * 4; i -= 4) {
          const float4 l = *reinterpret_cast<const float4*>(L + j * kLPitch + i);
#pragma unroll
          for (int e = 3; e >= 0; --e) {
            if (i + e > j + 1) y[e] = fmaf(-f4(l, e), x[i + e], y[e]);
            if (i + e == j + 1) l_next = f4(l, e);
          }
        }
        const float rest = (y[0] + y[1]) + (y[2] + y[3]);
        x[j] = j < 31 ? fmaf(-l_next, x[(j + 1) & 31], rest) : rest;
      }
      if (warp == 0) {
#pragma unroll
        for (int j = 0; j < 32; j += 4) *reinterpret_cast<float4*>(s_T1 + lane * kBPitch + j) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
      } else {
#pragma unroll
        for (int j = 0; j < 32; ++j) s_T2[j * kBPitch + lane] = x[j];
      }
#pragma unroll
      for (int j = 0; j < 32; ++j) g[j] = x[j];
    } else {
      write_row(s_kq, t, 0, g);  // (over K and Q, which the MMAs have read)
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    asm volatile("bar.sync 3, 128;" ::: "memory");
    if (tid == kC) bulk_store(rec + 3 * kPlane, s_kq, 3 * kPlane);
    float y[8];  // the block below the first: minus the second times L's times the first; eight columns per warp
    dot32(s_L + 32 + lane, kLPitch, s_T1 + warp * 8, y);
#pragma unroll
    for (int e = 0; e < 8; ++e) s_Y[lane * kBPitch + warp * 8 + e] = y[e];
    asm volatile("bar.sync 3, 128;" ::: "memory");  // L has been read: T's planes take its place
    dot32(s_T2 + lane, kBPitch, s_Y + warp * 8, y);
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] = -y[e];
    write_chunk(s_T, 32 + lane, warp, y);
    if (is_k) {
      float x[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) x[j] = g[j];
      write_row(s_T, t, warp * 4, x);
    } else if (warp == 2) {
      const float zero[32] = {};
      write_row(s_T, lane, 4, zero);
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("bar.sync 3, 128;" ::: "memory");
    if (tid == kC) {
      bulk_store(rec, s_T, 3 * kPlane);
      bulk_wait_all0();
    }
  }
  if (!ok && a.status) atomicOr(a.status, 1);
  __syncthreads();
  if (warp == 4) tmem_dealloc(tmem, 64);
}

// ---- the walk over the chunks ------------------------------------------------------------------------------------------------
constexpr int kParts = 4;                          // groups of four warps: each has a quarter of the tokens, or of the state's rows
constexpr int kWalkThreads = kParts * 128 + 32;    // thread of a group = lane of TMEM = column v of the state; last warp: loads, MMA
constexpr int kTok = kC / kParts;
constexpr uint32_t kD1 = 0, kD2 = 128, kD4 = 192, kRW = 320, kWt = 416;  // TMEM columns: S^T [K; Q], T R then A W, K^T W, planes

template <int NK>
constexpr int walk_smem() { return 5 * NK * kSub + 6 * kPlane + kSub + 2 * kScal + 128; }
static_assert(walk_smem<2>() <= 232448, "shared memory of a CTA");

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

// 16 values of this lane into the three planes at TMEM column `at` (8 columns each, planes 32 apart).
__device__ __forceinline__ void store_planes(uint32_t at, const float (&f)[kTok]) {
  static_assert(kTok == 16, "");
  uint32_t p[2][3][4];
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    float e[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) e[i] = f[q * 8 + i];
    split8(e, p[q]);
  }
#pragma unroll
  for (int k = 0; k < 3; ++k)
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(at + k * 32), "r"(p[0][k][0]),
                 "r"(p[0][k][1]), "r"(p[0][k][2]), "r"(p[0][k][3]), "r"(p[1][k][0]), "r"(p[1][k][1]), "r"(p[1][k][2]),
                 "r"(p[1][k][3])
                 : "memory");
}
__device__ __forceinline__ void tmem_store_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// S^T times keys and queries [128 x dim]: the state's three planes, smallest first.
template <int NK>
__device__ __forceinline__ void umma_state(uint32_t dst, const uint8_t* s, const uint8_t* kq) {
  constexpr uint32_t idesc = make_idesc(128, 2 * kC);
  const uint64_t a0 = opaque(make_smem_desc(smem_u32(s))), b0 = opaque(make_smem_desc(smem_u32(kq)));
#pragma unroll
  for (int p = 2; p >= 0; --p)
#pragma unroll
    for (int j = 0; j < NK; ++j) {
      const uint64_t ad = a0 + (p * NK + j) * (kSub >> 4), bd = b0 + j * (kSub >> 4);
#pragma unroll
      for (int k = 0; k < 4; ++k) umma_bf16(dst, ad + 2 * k, bd + 2 * k, idesc, (p < 2 || j || k) ? 1u : 0u);
    }
}

template <int NK>
__global__ void __launch_bounds__(kWalkThreads, 1) delta_chunk_kernel(const __grid_constant__ CUtensorMap map, ChunkArgs a) {
  extern __shared__ __align__(1024) uint8_t s_S[];  // (nothing static: all of the SM's shared memory is spoken for)
  uint8_t* s_kq = s_S + 3 * NK * kSub;   // two buffers
  uint8_t* s_T = s_kq + 2 * NK * kSub;
  uint8_t* s_A = s_T + 3 * kPlane;
  uint8_t* s_v = s_A + 3 * kPlane;       // values [2][64 tokens][64 columns]
  uint8_t* s_sc = s_v + kSub;            // two buffers
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_sc + 2 * kScal);
  uint64_t *kq_bar = bars, *sc_bar = bars + 2, *d_bar = bars + 4, &t_bar = bars[8], &a_bar = bars[9], &v_bar = bars[10];
  uint32_t& tmem_slot = *reinterpret_cast<uint32_t*>(bars + 11);
  int& s_abort = *reinterpret_cast<int*>(bars + 12);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const DeltaDims d = a.d;
  const int h = blockIdx.y, s = blockIdx.z, col0 = blockIdx.x * 128;
  const int4 seg = a.segs[s];
  const int slot = seg.x, r0 = seg.y, n = seg.z, pos0 = seg.w, nc = (n + kC - 1) / kC;
  if (n <= 0) return;
  if (smem_u32(s_S) & 1023) {  // (swizzled operand tiles)
    if (tid == 0 && a.status) atomicOr(a.status, 2);
    return;
  }
  const int kh = h / (d.heads / d.kv_heads);
  if (tid == 0) {
    s_abort = 0;
    for (int i = 0; i < 11; ++i) mbar_init(&bars[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    tma_prefetch_desc(&map);
  }
  if (warp == 4 * kParts) tmem_alloc(&tmem_slot, 512);
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

  if (warp == 4 * kParts) {
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
    };
    const auto load_sc = [&](int c) {
      mbar_expect_tx(&sc_bar[c & 1], kScal);
      bulk_load(s_sc + (c & 1) * kScal, record(a, seg, s, c, h) + 6 * kPlane, kScal, &sc_bar[c & 1]);
    };
    const auto load_v = [&](int c) {
      mbar_expect_tx(&v_bar, kSub);
      const int x = 2 * d.kv_heads * d.dim + h * d.vdim + col0;
      tma_load_2d(s_v, &map, x, r0 + c * kC, &v_bar);
      tma_load_2d(s_v + kSub / 2, &map, x + 64, r0 + c * kC, &v_bar);
    };
    const auto load_planes = [&](int c, int which, uint8_t* dst, uint64_t* bar) {
      mbar_expect_tx(bar, 3 * kPlane);
      bulk_load(dst, record(a, seg, s, c, h) + which * 3 * kPlane, 3 * kPlane, bar);
    };
    if (lane == 0) {
      load_kq(0);
      load_sc(0);
      load_v(0);
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
        umma_state<NK>(tmem + kD1, s_S, kq);
        umma_commit(&d_bar[0]);
        if (c + 1 < nc) load_sc(c + 1);  // (its buffer was last read before the barrier above)
      }
      __syncwarp();
      __syncthreads();  // (2) R is there
      if (lane == 0) {
        wait(&t_bar, c & 1);
        tc_fence_after();
        umma_planes(tmem + kD2, tmem + kRW, s_T, false);
        umma_commit(&d_bar[1]);
        if (c + 1 < nc) load_v(c + 1);
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
      mbar_wait(&v_bar, 0, &none);
      for (int i = 0; i < 2; ++i) mbar_wait(&sc_bar[i], 0, &none);
    }
  } else {
    const int part = warp >> 2, v = (warp & 3) * 32 + lane;  // this thread's lane of TMEM = column of the state
    const uint32_t base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const bool live = col0 + v < d.vdim;
    constexpr int kCols = 64 * NK / kParts;
    float S[kCols];  // rows part * kCols + i of column v
    float* state = a.state + (((size_t)slot * d.heads + h) * d.dim + part * kCols) * d.vdim + col0 + v;
    {
      const float* p = state;
#pragma unroll
      for (int i = 0; i < kCols; ++i) {
        S[i] = (live && pos0 > 0) ? *p : 0.f;
        p += d.vdim;
        asm volatile("" : "+l"(p));  // (one pointer that moves on, not an offset per element kept in registers)
      }
    }
    float* out = a.out + ((size_t)(r0 + part * kTok) * d.heads + h) * d.vdim + col0 + v;
    const auto store_state = [&]() {  // planes of S as K-major operand tiles
#pragma unroll
      for (int q = 0; q < kCols / 8; ++q) {
        float f[8];
        uint32_t p[3][4];
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = S[q * 8 + e];
        split8(f, p);
        const int col = part * kCols + q * 8;
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
      tmem_ld16(base + kD2 + part * kTok, y);
      float* p = out + (size_t)c * kC * d.heads * d.vdim;
      const int m = live ? n - c * kC - part * kTok : 0;
#pragma unroll
      for (int i = 0; i < kTok; ++i) {
        if (i < m) *p = y[i];
        p += (size_t)d.heads * d.vdim;
        asm volatile("" : "+l"(p));
      }
    };
    const uint8_t* my_v = s_v + (v >> 6) * (kSub / 2) + part * kTok * 128 + (v & 7) * 2;  // (16 tokens: row i of a group of 8 is i % 8)
    store_state();
    for (int c = 0; c < nc; ++c) {
      const float* sc = reinterpret_cast<const float*>(s_sc + (c & 1) * kScal) + part * kTok;
      float y[32], f[kTok];
      tc_fence_before();
      if (__syncthreads_or(!ok)) break;  // (1)
      if (c > 0) write_out(c - 1);
      wait(&sc_bar[c & 1], (c >> 1) & 1);
      wait(&v_bar, c & 1);
      wait(&d_bar[0], c & 1);
      tc_fence_after();
      tmem_ld16(base + kD1 + part * kTok, y);
      if (live) {
#pragma unroll
        for (int i = 0; i < kTok; i += 4) {
          const float4 k = *reinterpret_cast<const float4*>(sc + kScKey + i), b = *reinterpret_cast<const float4*>(sc + kScStep + i);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const uint32_t val = *reinterpret_cast<const uint16_t*>(my_v + (i + e) * 128 + (((v >> 3) ^ (i + e)) & 7) * 16);
            f[i + e] = fmaf(-f4(k, e), y[i + e], f4(b, e) * __uint_as_float(val << 16));
          }
        }
      } else {
#pragma unroll
        for (int i = 0; i < kTok; ++i) f[i] = 0.f;
      }
      store_planes(base + kRW + part * (kTok / 2), f);
      tmem_store_wait();
      tc_fence_before();
      __syncthreads();  // (2)
      wait(&d_bar[1], c & 1);
      tc_fence_after();
      tmem_ld16(base + kD2 + part * kTok, y);
#pragma unroll
      for (int i = 0; i < kTok; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(sc + kScEnd + i);
#pragma unroll
        for (int e = 0; e < 4; ++e) f[i + e] = y[i + e] * f4(x, e);
      }
      store_planes(base + kWt + part * (kTok / 2), f);
#pragma unroll
      for (int i = 0; i < kTok; ++i) f[i] = y[i];
      store_planes(base + kRW + part * (kTok / 2), f);
      tmem_ld16(base + kD1 + 64 + part * kTok, y);  // what A W is added to
#pragma unroll
      for (int i = 0; i < kTok; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(sc + kScQuery + i);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i + e] *= f4(x, e);
      }
      tmem_st<16>(base + kD2 + part * kTok, y);
      tc_fence_before();
      __syncthreads();  // (3)
      const float C = reinterpret_cast<const float*>(s_sc + (c & 1) * kScal)[kScAll];
      wait(&d_bar[3], c & 1);
      tc_fence_after();
#pragma unroll
      for (int g = 0; g < kCols / 16; ++g) {
        tmem_ld16(base + kD4 + part * kCols + g * 16, y);
#pragma unroll
        for (int i = 0; i < 16; ++i) S[g * 16 + i] = fmaf(C, S[g * 16 + i], y[i]);
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
      if (owns_qk && part == 0)
        for (int i = v; i < d.dim; i += 128) dst[q_col + i] = row[q_col + i];
      if (owns_qk && part == 1)
        for (int i = v; i < d.dim; i += 128) dst[k_col + i] = row[k_col + i];
      if (live && part == 0) dst[v_col + v] = row[v_col + v];
    }
    if (!ok && a.status) atomicOr(a.status, 1);
    tc_fence_before();
    __syncthreads();  // the walk's end
  }
  if (warp == 4 * kParts) tmem_dealloc(tmem, 512);
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
