// Grouped projections on the tensor cores: the weight-streaming kernel of linear_tc.cuh over several weights of one shape,
// each with its own rows (experts of a mixture) or its own column slices (heads).
#include <atomic>

#include "linear_tc.cuh"

namespace mlora {
namespace {

template <int BN>
int launch_grouped(const GroupedArgs& ga, void* work, cudaStream_t st) {
  using C = Cfg<BN>;
  const LinearArgs& a = ga.a;
  CUtensorMap mx;
  int rc = make_map(&mx, a.x, ga.x_rows, ga.x_cols ? (int)a.ldx : a.in, a.ldx, ga.gather ? 1 : BN);
  if (rc) return rc;
  TcParams p = {};
  p.a = a;
  p.row_tiles = (a.out + BM - 1) / BM;
  p.k_blocks = (a.in + BK - 1) / BK;
  p.g.table = ga.table;
  p.g.gather = ga.gather;
  p.g.w_bytes = packed_weight_bytes(a.out, a.in);
  p.g.tiles_per_group = ga.table ? 1 : (a.T + BN - 1) / BN;
  p.g.x_cols = ga.x_cols;
  p.g.y_cols = ga.y_cols;
  p.g.gate = ga.gate;
  p.g.ld_gate = ga.ld_gate;
  p.tok_tiles = ga.table ? 0 : ga.n_groups * p.g.tiles_per_group;
  p.n_tiles = p.row_tiles * p.tok_tiles;
  // whole output chunks by TMA when y allows it (a ragged chunk never goes that way, so the map needs no row count)
  CUtensorMap my = mx;
  p.tma_store = !(a.flags & MLORA_OUT_F32) && aligned16(a.y) && a.ldy % 8 == 0 && ga.y_cols % 8 == 0 && a.out % 8 == 0;
  if (p.tma_store) {
    rc = make_out_map(&my, a.y, 1 << 30, (int)a.ldy, a.ldy, C::kChunk, BM, false);
    if (rc) return rc;
  }
  p.lora_sub = 16;
  p.n_sub = 1;
  p.status = (int32_t*)work;
  p.tickets = (int32_t*)((uint8_t*)work + kHeaderBytes);
  p.partials = (float*)((uint8_t*)work + kHeaderBytes + kMaxGrid * 4);
  static std::atomic<unsigned long long> attr_done{0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!((attr_done.load(std::memory_order_acquire) >> (dev & 63)) & 1ull)) {
    cudaError_t e = cudaFuncSetAttribute(linear_tc_kernel<BN, 0, false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmemBytes);
    if (e != cudaSuccess) return fail(MLORA_ECUDA, "grouped_linear: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    attr_done.fetch_or(1ull << (dev & 63), std::memory_order_release);
  }
  launch_pdl_if(pdl_enabled_gemm(), linear_tc_kernel<BN, 0, false, true>, sm_count(), kThreads, C::kSmemBytes, st, mx, mx, mx, my, p);
  count_launch();
  MLORA_CHECK_LAUNCH("linear_tc_kernel (grouped)");
  return MLORA_OK;
}

}  // namespace

// split tiles (and their partial sums) only exist below 128-row tiles
size_t grouped_tc_workspace(int tile_rows) {
  return kHeaderBytes + kMaxGrid * 4 + (tile_rows >= 128 ? 0 : (size_t)kMaxGrid * 2 * tile_rows * BM * sizeof(float));
}

int launch_grouped_tc(const GroupedArgs& ga, void* work, size_t work_bytes, cudaStream_t st) {
  const size_t need = grouped_tc_workspace(ga.tile_rows);
  if (work_bytes < need) return fail(MLORA_ESIZE, "grouped_linear: workspace of %zu bytes needed, %zu given", need, work_bytes);
  switch (ga.tile_rows) {
    case 16: return launch_grouped<16>(ga, work, st);
    case 32: return launch_grouped<32>(ga, work, st);
    case 64: return launch_grouped<64>(ga, work, st);
    case 128: return launch_grouped<128>(ga, work, st);
    case 256: return launch_grouped<256>(ga, work, st);
  }
  return fail(MLORA_EINVAL, "grouped_linear: rows per tile must be 16, 32, 64, 128 or 256 (got %d)", ga.tile_rows);
}

}  // namespace mlora

using namespace mlora;

extern "C" size_t mlora_grouped_linear_workspace(int32_t tile_rows) { return grouped_tc_workspace(tile_rows); }

extern "C" int mlora_grouped_linear(const void* d_x, int64_t ldx, int32_t x_rows, int32_t x_cols, const int32_t* d_gather,
                                    const void* d_Wp, void* d_y, int64_t ldy, int32_t y_cols, const int32_t* d_tiles,
                                    int32_t n_groups, int32_t T, int32_t tile_rows, int32_t in, int32_t out, int32_t flags,
                                    const void* d_gate, int64_t ld_gate, void* d_work, size_t work_bytes, void* stream) {
  MLORA_REQUIRE(T >= 0 && in > 0 && out > 0 && n_groups > 0 && x_rows >= 0, "grouped_linear: bad sizes");
  MLORA_REQUIRE(in % 8 == 0 && ldx % 8 == 0 && x_cols % 64 == 0, "grouped_linear: in and ldx multiples of 8, x_cols of 64 (in=%d ldx=%lld x_cols=%d)",
                in, (long long)ldx, x_cols);
  MLORA_REQUIRE(x_cols == 0 || in % 64 == 0, "grouped_linear: a column slice per group must be whole k-blocks of 64 (in=%d)", in);
  MLORA_REQUIRE(d_x && d_Wp && d_y && d_work, "grouped_linear: null pointer");
  MLORA_REQUIRE(aligned16(d_x) && aligned16(d_Wp), "grouped_linear: x and the packed weights must be 16-byte aligned");
  MLORA_REQUIRE(!(flags & ~(MLORA_OUT_F32 | MLORA_ACT_RELU2 | MLORA_ACT_GELU)) &&
                    (flags & (MLORA_ACT_RELU2 | MLORA_ACT_GELU)) != (MLORA_ACT_RELU2 | MLORA_ACT_GELU),
                "grouped_linear: flags are MLORA_OUT_F32 and one activation");
  MLORA_REQUIRE(!d_gather || d_tiles, "grouped_linear: a gather list needs a tile table");
  MLORA_REQUIRE(!d_tiles || (aligned16(d_tiles)), "grouped_linear: the tile table must be 16-byte aligned");
  MLORA_REQUIRE(d_tiles || T <= x_rows, "grouped_linear: T=%d rows of %d", T, x_rows);
  const int64_t cols = x_cols ? (int64_t)(n_groups - 1) * x_cols + in : in;
  MLORA_REQUIRE(cols <= ldx, "grouped_linear: the groups' columns exceed the row pitch");
  if ((!d_tiles && T == 0) || x_rows == 0) return MLORA_OK;
  GroupedArgs g{};
  g.a.x = (const bf16*)d_x;
  g.a.ldx = ldx;
  g.a.W = (const bf16*)d_Wp;
  g.a.y = d_y;
  g.a.ldy = ldy;
  g.a.T = T;
  g.a.in = in;
  g.a.out = out;
  g.a.flags = flags | MLORA_W_PACKED;
  g.a.n_mod = 1;
  g.table = d_tiles;
  g.gather = d_gather;
  g.x_rows = x_rows;
  g.n_groups = n_groups;
  g.tile_rows = tile_rows;
  g.x_cols = x_cols;
  g.y_cols = y_cols;
  g.gate = (const bf16*)d_gate;
  g.ld_gate = ld_gate;
  return launch_grouped_tc(g, d_work, work_bytes, (cudaStream_t)stream);
}
