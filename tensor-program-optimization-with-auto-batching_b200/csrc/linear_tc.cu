// Host side of the weight-streaming tensor-core projection (the kernel is in linear_tc.cuh): how a projection is dealt to
// the CTAs, weight and adapter pre-packing, launches.
#include <stdlib.h>

#include <atomic>

#include "linear_tc.cuh"

namespace mlora {
namespace {

// ---- host side -------------------------------------------------------------------------------------
struct Plan {
  int bn, row_tiles, tok_tiles, k_blocks, grid, per_cta, wave_gt, wave_full, wave_ch, wave_ch_last, wave_lanes;
};

// min_waves: whole-tile mode needs at least this many tiles per CTA, so that the unfilled last wave costs little.
Plan plan_for(int bn, int min_waves, int T, int in, int out) {
  Plan pl;
  pl.bn = bn;
  pl.row_tiles = (out + BM - 1) / BM;
  pl.tok_tiles = (T + pl.bn - 1) / pl.bn;
  pl.k_blocks = (in + BK - 1) / BK;
  const long long total = (long long)pl.row_tiles * pl.tok_tiles * pl.k_blocks;
  long long grid = sm_count();
  pl.wave_gt = pl.wave_full = pl.wave_ch = pl.wave_ch_last = pl.wave_lanes = 0;
  const long long n_tiles = (long long)pl.row_tiles * pl.tok_tiles;
  if (pl.tok_tiles >= 4 && n_tiles >= min_waves * grid) {
    // Waves of (token tiles x row tiles).
    static const int lane_form = [] {
      const char* e = getenv("MLORA_WAVE_LANES");
      return e ? atoi(e) : 1;
    }();
    if (lane_form) {
      // Lane form.  Token tiles per group: the group's token rows are what the CTAs re-read from L2 row tile after row
      // tile, so they should stay resident next to the weight tiles in flight (<= 48 MB of the 126 MB).  Among the
      // sizes that fit, the one with the fewest steps (groups x row tiles per lane); fewer groups on ties (each group
      // streams the weights once).
      long long best = -1;
      for (int d = 1; d <= 48 && d <= pl.tok_tiles && d <= (int)grid; ++d) {
        if (d > 1 && (double)d * pl.bn * in * 2.0 > 48e6) break;
        const int lanes = (int)grid / d;
        const int steps = (pl.row_tiles + lanes - 1) / lanes;
        const int groups = (pl.tok_tiles + d - 1) / d;
        const long long cost = (long long)groups * steps;
        if (best < 0 || cost <= best) {
          best = cost;
          pl.wave_gt = d;
          pl.wave_lanes = lanes;
          pl.wave_ch = steps;
          pl.wave_full = groups;
        }
      }
      pl.wave_ch_last = 0;
      pl.per_cta = pl.wave_full * pl.wave_ch * pl.k_blocks;
      pl.grid = (int)grid;
      return pl;
    }
    // Chunk form: the tiles of a group, token tile major / row tile minor, cut into equal contiguous chunks.  Token tiles
    // per group: the group's token rows should stay L2-resident (<= 56 MB), and row_tiles * group should fill whole
    // rounds of the grid (the slots beyond it idle); among the sizes that fit, the one that wastes the fewest slots.
    int gt = 1;
    double best = 2.0;
    for (int d = 1; d <= 48 && d <= pl.tok_tiles; ++d) {
      if (d > 1 && (double)d * pl.bn * in * 2.0 > 56e6) break;
      const long long tiles = (long long)pl.row_tiles * d;
      const long long slots = (tiles + grid - 1) / grid * grid;
      const double waste = (double)(slots - tiles) / (double)slots;
      if (waste <= best + 1e-9) {
        best = waste;
        gt = d;
      }
    }
    pl.wave_gt = gt;
    pl.wave_full = pl.tok_tiles / pl.wave_gt;
    const int gt_last = pl.tok_tiles - pl.wave_full * pl.wave_gt;
    pl.wave_ch = (int)(((long long)pl.row_tiles * pl.wave_gt + grid - 1) / grid);
    pl.wave_ch_last = (int)(((long long)pl.row_tiles * gt_last + grid - 1) / grid);
    pl.per_cta = (pl.wave_full * pl.wave_ch + pl.wave_ch_last) * pl.k_blocks;
    pl.grid = (int)grid;
    return pl;
  }
  // at least 4 k-blocks (64 KB of weights) per CTA, so tiny problems do not pay for 148 partial tiles
  if (grid > (total + 3) / 4) grid = (total + 3) / 4;
  if (grid < 1) grid = 1;
  pl.per_cta = (int)((total + grid - 1) / grid);
  pl.grid = (int)((total + pl.per_cta - 1) / pl.per_cta);
  return pl;
}

// 256-token tiles where whole tiles fill the grid at least three times over (prompt passes of thousands of rows): a
// 128 x 128 tile moves 64 KB through shared memory per 256 tensor-pipe cycles, twice what a shared memory delivers;
// 128 x 256 moves 96 KB per 512.  Switch: MLORA_TILE256=0 keeps 128-token tiles.
bool tile256_enabled() {
  static const bool on = [] {
    const char* e = getenv("MLORA_TILE256");
    return !(e && e[0] == '0');
  }();
  return on;
}

Plan make_plan(int T, int in, int out) {
  if (T >= 1024 && tile256_enabled()) {
    Plan big = plan_for(256, 3, T, in, out);
    if (big.wave_gt > 0) return big;
  }
  return plan_for(pick_bn(T), 8, T, in, out);
}

template <int BN>
int launch(const LinearArgs& a, const Plan& pl, void* work, cudaStream_t st) {
  using C = Cfg<BN>;
  CUtensorMap mw, mx;
  int rc = make_map(&mx, a.x, a.T, a.in, a.ldx, BN);
  if (rc) return rc;
  if (a.flags & MLORA_W_PACKED) {
    mw = mx;  // unused by the kernel
  } else {
    rc = make_map(&mw, a.W, a.out, a.in, a.in, BM);
    if (rc) return rc;
  }
  TcParams p;
  p.a = a;
  // LoRA expand: on the tensor cores when the rank pitch is 16/32/64/128 and every module boundary
  // is a multiple of the 128-row tile; else on CUDA cores in the epilogue (needs pitch <= 64)
  p.lora_mode = 0;
  p.lora_sub = 16;
  p.n_sub = 1;
  CUtensorMap mb = mw;
  if (a.u != nullptr) {
    bool aligned_mods = true;
    for (int m = 1; m < a.n_mod; ++m) aligned_mods = aligned_mods && (a.mod_off[m] % BM == 0);
    const bool pitch_ok = a.r_max == 16 || a.r_max == 32 || a.r_max == 64 || a.r_max == 128;
    if (pitch_ok && aligned_mods) {
      p.lora_mode = 2;
      p.lora_sub = a.r_max < 64 ? a.r_max : 64;
      p.n_sub = a.r_max / p.lora_sub;
      if (!(a.flags & MLORA_B_PACKED)) {
        rc = make_map(&mb, a.B_all, (long long)a.n_adapters * a.out, a.r_max, a.r_max, BM, p.lora_sub);
        if (rc) return rc;
      }
    } else {
      if (a.flags & MLORA_B_PACKED)
        return fail(MLORA_EINVAL, "linear: a packed B_all needs rank pitch 16/32/64/128 and tile-aligned modules");
      if (a.r_max > 64) return fail(MLORA_EINVAL, "linear: rank pitch %d needs tile-aligned modules", a.r_max);
      p.lora_mode = 1;
    }
  }
  p.k_blocks = pl.k_blocks;
  p.row_tiles = pl.row_tiles;
  p.n_tiles = pl.row_tiles * pl.tok_tiles;
  p.tok_tiles = pl.tok_tiles;
  p.wave_gt = pl.wave_gt;
  p.wave_full = pl.wave_full;
  p.wave_ch = pl.wave_ch;
  p.wave_ch_last = pl.wave_ch_last;
  p.wave_lanes = pl.wave_lanes;
  p.per_cta = pl.per_cta;
  // output through TMA when the tensor satisfies its alignment rules (16-byte base and row pitch)
  CUtensorMap my = mx;
  {
    const bool f32 = (a.flags & MLORA_OUT_F32) != 0, silu = (a.flags & MLORA_SILU_MUL) != 0;
    const int es = f32 ? 4 : 2, cols = silu ? a.out / 2 : a.out;
    p.tma_store = !(BN >= 128 && f32) && aligned16(a.y) && (a.ldy * es) % 16 == 0 && (cols * es) % 16 == 0;
    if (p.tma_store) {
      rc = make_out_map(&my, a.y, a.T, cols, a.ldy, BN < 32 ? BN : 32, silu ? BM / 2 : BM, f32);
      if (rc) return rc;
    }
  }
  p.prefetch = 0;  // measured: an L2 prefetch stream ahead of the ring slows the kernel down on B200
  p.status = (int32_t*)work;
  p.tickets = (int32_t*)((uint8_t*)work + kHeaderBytes);
  p.partials = (float*)((uint8_t*)work + kHeaderBytes + kMaxGrid * 4);
  // the shared-memory opt-in is a per-device attribute of each instantiation
  static std::atomic<unsigned long long> attr_done{0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!((attr_done.load(std::memory_order_acquire) >> (dev & 63)) & 1ull)) {
    cudaError_t e = cudaFuncSetAttribute(linear_tc_kernel<BN, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(linear_tc_kernel<BN, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(linear_tc_kernel<BN, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
    if (e != cudaSuccess) return fail(MLORA_ECUDA, "linear: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    attr_done.fetch_or(1ull << (dev & 63), std::memory_order_release);
  }
  if constexpr (BN <= 32) {
    if (a.nf.res != nullptr || a.nf.sumsq_in != nullptr) {
      if (p.lora_mode == 1) return fail(MLORA_EINVAL, "linear_norm: the LoRA expand of this call runs on CUDA cores (rank pitch / module alignment)");
      static std::atomic<unsigned long long> nf_attr_done{0};
      if (!((nf_attr_done.load(std::memory_order_acquire) >> (dev & 63)) & 1ull)) {
        cudaError_t e = cudaFuncSetAttribute(linear_tc_kernel<BN, 0, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
        if (e == cudaSuccess)
          e = cudaFuncSetAttribute(linear_tc_kernel<BN, 2, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
        if (e != cudaSuccess) return fail(MLORA_ECUDA, "linear: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
        nf_attr_done.fetch_or(1ull << (dev & 63), std::memory_order_release);
      }
      if (p.lora_mode == 2 || (a.flags & MLORA_SHARE_LORA_KERNEL))
        launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 2, true>, pl.grid, kThreads, C::kSmemBytes, st, mw, mx, mb, my, p);
      else
        launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 0, true>, pl.grid, kThreads, C::kSmemBytes, st, mw, mx, mb, my, p);
      count_launch();
      MLORA_CHECK_LAUNCH("linear_tc_kernel");
      return MLORA_OK;
    }
  }
  if (p.lora_mode == 1)
    launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 1>, pl.grid, kThreads, C::kSmemBytes, st, mw, mx, mb, my, p);
  else if (p.lora_mode == 2 || (a.flags & MLORA_SHARE_LORA_KERNEL))
    launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 2>, pl.grid, kThreads, C::kSmemBytes, st, mw, mx, mb, my, p);
  else
    launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 0>, pl.grid, kThreads, C::kSmemBytes, st, mw, mx, mb, my, p);
  count_launch();
  MLORA_CHECK_LAUNCH("linear_tc_kernel");
  return MLORA_OK;
}

// Repacks W [out, in] into tiles [row_tile][k_block][128 rows][64 k] whose bytes are the
// shared-memory image the MMA reads: row r of a tile at r*128 bytes, its 16-byte chunk c at
// ((c ^ (r & 7)) * 16) (128-byte swizzle).  Rows / columns past the matrix are zero.
__global__ void __launch_bounds__(256) pack_weight_kernel(const bf16* __restrict__ W, int out, int in, int k_blocks,
                                                          uint4* __restrict__ Wp) {
  const size_t tile = blockIdx.x;  // row_tile * k_blocks + kb
  const int row_tile = (int)(tile / k_blocks), kb = (int)(tile % k_blocks);
  for (int idx = threadIdx.x; idx < BM * 8; idx += blockDim.x) {
    const int r = idx >> 3, c = idx & 7;
    const int row = row_tile * BM + r, k = kb * BK + c * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < out && k < in) v = *reinterpret_cast<const uint4*>(W + (size_t)row * in + k);  // in % 8 == 0
    Wp[tile * (BM * 8) + r * 8 + (c ^ (r & 7))] = v;
  }
}

// Repacks B_all [N, out, r_max] into tiles [slot][row_tile][sub-block][128 rows][lora_sub] whose bytes
// are the shared-memory image of a LoRA stage's A operand: row r at r*rb bytes (rb = 2*lora_sub), its
// 16-byte chunk c at ((c ^ swizzle(r)) * 16), swizzle span = rb.  Rows past `out` are zero.
__global__ void __launch_bounds__(256) pack_lora_b_kernel(const bf16* __restrict__ B, int out, int r_max,
                                                          int row_tiles, int lora_sub, int n_sub,
                                                          uint4* __restrict__ Bp) {
  const size_t tile = blockIdx.x;  // (slot * row_tiles + row_tile) * n_sub + sb
  const int sb = (int)(tile % n_sub);
  const size_t sr = tile / n_sub;
  const int row_tile = (int)(sr % row_tiles), slot = (int)(sr / row_tiles);
  const int chunks = lora_sub / 8, rb = lora_sub * 2;
  for (int idx = threadIdx.x; idx < BM * chunks; idx += blockDim.x) {
    const int r = idx / chunks, c = idx - r * chunks;
    const int row = row_tile * BM + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < out) v = *reinterpret_cast<const uint4*>(B + ((size_t)slot * out + row) * r_max + sb * lora_sub + c * 8);
    const int sw = rb == 128 ? (r & 7) : rb == 64 ? ((r >> 1) & 3) : ((r >> 2) & 1);
    Bp[tile * (BM * chunks) + r * chunks + (c ^ sw)] = v;
  }
}

}  // namespace

size_t packed_lora_b_bytes(int n_adapters, int out, int r_max) {
  return (size_t)n_adapters * ((out + BM - 1) / BM) * BM * r_max * 2;
}

int launch_pack_lora_b(const void* B, int n_adapters, int out, int r_max, void* Bp, cudaStream_t st) {
  if (!(r_max == 16 || r_max == 32 || r_max == 64 || r_max == 128))
    return fail(MLORA_EINVAL, "pack_lora_b: rank pitch must be 16, 32, 64 or 128 (got %d)", r_max);
  const int lora_sub = r_max < 64 ? r_max : 64, n_sub = r_max / lora_sub;
  const int row_tiles = (out + BM - 1) / BM;
  const long long tiles = (long long)n_adapters * row_tiles * n_sub;
  if (tiles > 2147483647ll) return fail(MLORA_ESIZE, "pack_lora_b: stack too large");
  pack_lora_b_kernel<<<(unsigned)tiles, 256, 0, st>>>((const bf16*)B, out, r_max, row_tiles, lora_sub, n_sub, (uint4*)Bp);
  count_launch();
  MLORA_CHECK_LAUNCH("pack_lora_b_kernel");
  return MLORA_OK;
}

size_t packed_weight_bytes(int out, int in) {
  return (size_t)((out + BM - 1) / BM) * ((in + BK - 1) / BK) * (BM * BK * 2);
}

int launch_pack_weight(const void* W, int out, int in, void* Wp, cudaStream_t st) {
  const int k_blocks = (in + BK - 1) / BK;
  const long long tiles = (long long)((out + BM - 1) / BM) * k_blocks;
  if (tiles > 2147483647ll) return fail(MLORA_ESIZE, "pack_weight: matrix too large");
  pack_weight_kernel<<<(unsigned)tiles, 256, 0, st>>>((const bf16*)W, out, in, k_blocks, (uint4*)Wp);
  count_launch();
  MLORA_CHECK_LAUNCH("pack_weight_kernel");
  return MLORA_OK;
}

bool linear_tc_supported(const LinearArgs& a) {
  // TMA needs 16-byte aligned bases and row pitches; everything else (ragged K, out, T) is handled by
  // zero-filled out-of-bounds boxes and masked stores.
  const long long tiles = (long long)((a.out + BM - 1) / BM) * ((a.T + 127) / 128);
  return aligned16(a.x) && aligned16(a.W) && (a.ldx * 2) % 16 == 0 && (a.in * 2) % 16 == 0 && (a.u == nullptr || a.r_max % 8 == 0) &&
         (a.u == nullptr || a.r_max <= 64 || a.r_max == 128) &&
         tiles * ((a.in + BK - 1) / BK) < 2000000000ll;
}

// How a projection of this shape is dealt to the CTAs (host-side planning only; no device work).
void linear_tc_plan(int T, int in, int out, int32_t* v) {
  const Plan pl = make_plan(T, in, out);
  v[0] = pl.bn;
  v[1] = pl.grid;
  v[2] = pl.row_tiles;
  v[3] = pl.tok_tiles;
  v[4] = pl.k_blocks;
  v[5] = pl.per_cta;
  v[6] = pl.wave_gt;
  v[7] = pl.wave_lanes;
  v[8] = pl.wave_ch;
  v[9] = pl.wave_full;
  v[10] = pl.wave_ch_last;
  v[11] = 0;
}

size_t linear_tc_workspace(int T, int in, int out) {
  const int bn = T > 0 ? pick_bn(T) : 16;
  return kHeaderBytes + kMaxGrid * 4 + (size_t)kMaxGrid * 2 * bn * BM * sizeof(float);
}

int launch_linear_tc(const LinearArgs& a, void* work, size_t work_bytes, cudaStream_t st) {
  const size_t need = linear_tc_workspace(a.T, a.in, a.out);
  if (work_bytes < need) return fail(MLORA_ESIZE, "linear: workspace of %zu bytes needed, %zu given", need, work_bytes);
  Plan pl = make_plan(a.T, a.in, a.out);
  switch (pl.bn) {
    case 16: return launch<16>(a, pl, work, st);
    case 32: return launch<32>(a, pl, work, st);
    case 64: return launch<64>(a, pl, work, st);
    case 256: return launch<256>(a, pl, work, st);
    default: return launch<128>(a, pl, work, st);
  }
}

}  // namespace mlora
