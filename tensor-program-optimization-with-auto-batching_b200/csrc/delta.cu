// Gated delta rule: a matrix M [dim, vdim] per head and sequence instead of a cache of keys.  A token fades it by its decay c,
// corrects what it holds under the key k towards the value v by its step b, and reads the result under the query q:
//
//   M' = c M + k w^T   with   w = b (v - c M^T k),        out = M'^T q
//
// with q, k unit vectors (q scaled), one decay and one step per head and token, and a short causal convolution with silu in
// front of q, k and v.  Sizes, scale, taps and where things lie in a projected row are arguments.
//
//   short_conv     prompt passes: convolution + silu of every row, earlier tokens from the pass or from the ring
//   delta_scan     prompt passes: the recurrence over all rows of a sequence
//   gated_rms      o / rms(o) * w * silu(gate) per head
//   delta_step     one token of every row: all of the above in one launch
//
// The last `taps` inputs of the convolution are kept per sequence in a ring (token p at place p mod taps), one place more
// than the convolution looks back: a token's own input never overwrites one that is still read.  Nothing is read from ring
// or state at position 0, so neither is cleared when a sequence starts.
//
// The recurrence runs in 32-bit on the CUDA cores.  Columns of M are independent of one another: eight lanes share a group
// of four columns, each with every eighth group of four rows, in registers for the whole pass.  M^T k and M^T q are taken
// of the same M in one go, as M'^T q = c M^T q + w (k . q): one reduction over the eight lanes per token.
// Products are done on pairs of rows (fma.rn.f32x2).
#include <cmath>

#include "delta.cuh"
#include "tc_ptx.cuh"

namespace mlora {
namespace {

// Four neighbouring activations as they are stored.
template <typename A>
struct Raw4;
template <>
struct Raw4<bf16> {
  typedef uint2 type;
};
template <>
struct Raw4<float> {
  typedef float4 type;
};
__device__ __forceinline__ void widen4(const uint2& v, float (&f)[4]) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y;
}
__device__ __forceinline__ void widen4(const float4& v, float (&f)[4]) { f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w; }
template <typename A>
__device__ __forceinline__ void load4(const A* p, float (&f)[4]) {
  widen4(*reinterpret_cast<const typename Raw4<A>::type*>(p), f);
}

typedef unsigned long long f32x2;  // two fp32 values in one register pair
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// The part of a state one warp holds: 16 columns, RJ * 32 rows.  Lane l: rows 32 j + 4 (l % 8) + {0..3}, columns
// 4 (l / 8) + {0..3}.
template <int RJ>
struct Tile {
  f32x2 s[RJ][2][4];

  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int j = 0; j < RJ; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[j][0][c] = s[j][1][c] = 0ull;
  }
  // S: [dim][vdim] of this head; c: this lane's first column
  __device__ __forceinline__ void load(const float* S, int dim, int vdim, int row0, int c) {
#pragma unroll
    for (int j = 0; j < RJ; ++j) {
      const int r = 32 * j + row0;
      float4 v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        v[i] = (r < dim && c < vdim) ? *reinterpret_cast<const float4*>(S + (size_t)(r + i) * vdim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        s[j][p][0] = pack2(v[2 * p].x, v[2 * p + 1].x);
        s[j][p][1] = pack2(v[2 * p].y, v[2 * p + 1].y);
        s[j][p][2] = pack2(v[2 * p].z, v[2 * p + 1].z);
        s[j][p][3] = pack2(v[2 * p].w, v[2 * p + 1].w);
      }
    }
  }
  __device__ __forceinline__ void store(float* S, int dim, int vdim, int row0, int c) const {
#pragma unroll
    for (int j = 0; j < RJ; ++j) {
      const int r = 32 * j + row0;
      if (r >= dim || c >= vdim) continue;
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const float2 a = unpack2(s[j][p][0]), b = unpack2(s[j][p][1]), d = unpack2(s[j][p][2]), e = unpack2(s[j][p][3]);
        *reinterpret_cast<float4*>(S + (size_t)(r + 2 * p) * vdim + c) = make_float4(a.x, b.x, d.x, e.x);
        *reinterpret_cast<float4*>(S + (size_t)(r + 2 * p + 1) * vdim + c) = make_float4(a.y, b.y, d.y, e.y);
      }
    }
  }
  // One token.  k, q: this lane's rows.  v: the value of column 4 (l / 8) + l % 4.  Lanes with l % 8 >= 4 return that
  // column's output, the others something else.
  __device__ __forceinline__ float step(const ulonglong2 (&k)[RJ], const ulonglong2 (&q)[RJ], float v, float g, float beta,
                                        float kq, int lane) {
    f32x2 dk[4] = {0ull, 0ull, 0ull, 0ull}, dq[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
    for (int j = 0; j < RJ; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        dk[c] = fma2(s[j][0][c], k[j].x, dk[c]);
        dq[c] = fma2(s[j][0][c], q[j].x, dq[c]);
        dk[c] = fma2(s[j][1][c], k[j].y, dk[c]);
        dq[c] = fma2(s[j][1][c], q[j].y, dq[c]);
      }
    // sums over the eight lanes, left where they are used: lane bit 2 picks k or q, bits 1 and 0 the column
    const bool b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
    float y[4], z[2];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const float2 a = unpack2(dk[c]), b = unpack2(dq[c]);
      const float sk = a.x + a.y, sq = b.x + b.y;
      y[c] = (b2 ? sq : sk) + __shfl_xor_sync(0xffffffffu, b2 ? sk : sq, 4);
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) z[c] = (b1 ? y[c + 2] : y[c]) + __shfl_xor_sync(0xffffffffu, b1 ? y[c] : y[c + 2], 2);
    const float w = g * ((b0 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, b0 ? z[0] : z[1], 1));
    const float u = beta * (v - w);  // (meaningful on the lanes of k)
    const int base = lane & 24;
    const float o = fmaf(__shfl_sync(0xffffffffu, u, base + (lane & 3)), kq, w);
    const f32x2 g2 = pack2(g, g);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const float uc = __shfl_sync(0xffffffffu, u, base + c);
      const f32x2 u2 = pack2(uc, uc);
#pragma unroll
      for (int j = 0; j < RJ; ++j) {
        s[j][0][c] = fma2(k[j].x, u2, mul2(s[j][0][c], g2));
        s[j][1][c] = fma2(k[j].y, u2, mul2(s[j][1][c], g2));
      }
    }
    return o;
  }
};

// ---- prompt passes: convolution ------------------------------------------------------------------------------------
template <typename A>
struct ConvArgs {
  const A* x;        // [T, >= C]
  int64_t ld;
  int C, taps;       // channels (a multiple of 8)
  const float* w;    // [taps][C], row taps - 1 for the token itself
  const A* ring;     // [slot][taps][C]
  const int32_t *row_slot, *row_pos;
  A* out;            // [T, C]
  int T;
};

constexpr int kConvRows = 16;  // rows per thread, walked with the inputs of the last tokens in registers

// Thread: 8 channels x kConvRows rows.  K taps.
template <typename A, int K>
__global__ void __launch_bounds__(128) short_conv_kernel(ConvArgs<A> a) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= a.C) return;
  const int t0 = blockIdx.y * kConvRows, t1 = min(t0 + kConvRows, a.T);
  float w[K][8], h[K][8];  // h[j]: input j tokens back
#pragma unroll
  for (int k = 0; k < K; ++k) load8(a.w + (size_t)k * a.C + c, w[k]);
  int prev_slot = -1, prev_pos = -1;
  for (int t = t0; t < t1; ++t) {
    const int slot = a.row_slot[t], pos = a.row_pos[t];
    if (t == t0 || slot != prev_slot || pos != prev_pos + 1) {
      // first row here, or first row of a sequence: earlier tokens from rows of this pass that go before, else the ring
#pragma unroll
      for (int j = 1; j < K; ++j) {
        const bool in_pass = t >= j && a.row_slot[t - j] == slot && a.row_pos[t - j] == pos - j;
        if (pos - j < 0) {
#pragma unroll
          for (int i = 0; i < 8; ++i) h[j - 1][i] = 0.f;
        } else if (in_pass) {
          load8(a.x + (size_t)(t - j) * a.ld + c, h[j - 1]);
        } else {
          load8(a.ring + ((size_t)slot * K + (pos - j) % K) * a.C + c, h[j - 1]);
        }
      }
    }
    prev_slot = slot, prev_pos = pos;
    // (h[j - 1] holds the input j tokens before the current one: shift, then put the current one first)
#pragma unroll
    for (int j = K - 1; j > 0; --j)
#pragma unroll
      for (int i = 0; i < 8; ++i) h[j][i] = h[j - 1][i];
    load8(a.x + (size_t)t * a.ld + c, h[0]);
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float s = 0.f;
#pragma unroll
      for (int j = K - 1; j >= 0; --j) s = fmaf(w[K - 1 - j][i], h[j][i], s);
      o[i] = silu<A>(s);
    }
    store8(a.out + (size_t)t * a.C + c, o);
  }
}

// ---- prompt passes: recurrence ---------------------------------------------------------------------------------------
template <typename A>
struct ScanArgs {
  const A* xc;       // [T, C]: q [kv_heads, dim] | k [kv_heads, dim] | v [heads, vdim], after convolution and silu
  const A* x;        // the projected rows (what the convolution read), for the ring
  int64_t ld;
  int C, taps, b_col, a_col;  // columns of the step sizes' and the decays' projections in x
  const float *A_log, *dt_bias;
  DeltaDims d;
  const int32_t* segs;  // [n][4]: slot, first row, rows, position of the first row
  float* state;         // [slot][heads][dim][vdim]
  A* ring;              // [slot][taps][C]
  float* out;           // [T, heads * vdim]
};

constexpr int kPer = 2;  // tokens a warp stages per block of tokens

// CTA (column part, head, segment) of NW warps = 16 NW columns.  Tokens go through shared memory in blocks of kPer * NW,
// read from global memory one block ahead.
template <typename A, int RJ, int NW>
__global__ void __launch_bounds__(NW * 32) delta_scan_kernel(ScanArgs<A> a) {
  constexpr int kRows = 32 * RJ, kTok = kPer * NW, kCols = 16 * NW;
  constexpr int kVec = (RJ + 3) / 4;  // groups of four rows a lane stages
  extern __shared__ __align__(16) float smem[];
  float* s_k = smem;                          // [2][kTok][kRows]
  float* s_q = s_k + 2 * kTok * kRows;        // [2][kTok][kRows]
  float* s_v = s_q + 2 * kTok * kRows;        // [2][kTok][kCols]
  float4* s_g = reinterpret_cast<float4*>(s_v + 2 * kTok * kCols);  // [2][kTok]: g, beta, k . q
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const DeltaDims d = a.d;
  const int h = blockIdx.y, kh = h / (d.heads / d.kv_heads), col0 = blockIdx.x * kCols;
  const int4 seg = reinterpret_cast<const int4*>(a.segs)[blockIdx.z];
  const int slot = seg.x, r0 = seg.y, n = seg.z, pos0 = seg.w;
  const int q_col = kh * d.dim, k_col = (d.kv_heads + kh) * d.dim, v_col = 2 * d.kv_heads * d.dim + h * d.vdim + col0;
  const float A_log = a.A_log[h], dt_bias = a.dt_bias[h];

  typedef typename Raw4<A>::type Raw;
  Raw pq[kPer][kVec], pk[kPer][kVec], pv[kPer];
  A pa[kPer], pb[kPer];
  const auto fetch = [&](int t0) {  // (nothing is converted here: the values are not waited for)
#pragma unroll
    for (int e = 0; e < kPer; ++e) {
      const int t = t0 + e * NW + warp;
      const bool in = t < n;
      const A* row = a.xc + (size_t)(r0 + (in ? t : 0)) * a.C;
#pragma unroll
      for (int i = 0; i < kVec; ++i) {
        const int r = 4 * (lane + 32 * i);
        pq[e][i] = pk[e][i] = Raw{};
        if (in && r < d.dim) {
          pq[e][i] = *reinterpret_cast<const Raw*>(row + q_col + r);
          pk[e][i] = *reinterpret_cast<const Raw*>(row + k_col + r);
        }
      }
      pv[e] = Raw{};
      if (in && 4 * lane < kCols && col0 + 4 * lane < d.vdim) pv[e] = *reinterpret_cast<const Raw*>(row + v_col + 4 * lane);
      const A* xr = a.x + (size_t)(r0 + (in ? t : 0)) * a.ld;
      pb[e] = xr[a.b_col + h], pa[e] = xr[a.a_col + h];
    }
  };
  const auto stage = [&](int buf) {  // unit vectors, their product
#pragma unroll
    for (int e = 0; e < kPer; ++e) {
      const int tok = buf * kTok + e * NW + warp;
      float sq = 0.f, sk = 0.f, sx = 0.f, fq[kVec][4], fk[kVec][4], fv[4];
      widen4(pv[e], fv);
#pragma unroll
      for (int i = 0; i < kVec; ++i) {
        widen4(pq[e][i], fq[i]);
        widen4(pk[e][i], fk[i]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          sq = fmaf(fq[i][j], fq[i][j], sq);
          sk = fmaf(fk[i][j], fk[i][j], sk);
          sx = fmaf(fq[i][j], fk[i][j], sx);
        }
      }
      sq = warp_sum(sq), sk = warp_sum(sk), sx = warp_sum(sx);
      const float iq = d.q_scale / sqrtf(sq + 1e-6f), ik = 1.f / sqrtf(sk + 1e-6f);
#pragma unroll
      for (int i = 0; i < kVec; ++i) {
        const int r = 4 * (lane + 32 * i);
        if (r < kRows) {
          *reinterpret_cast<float4*>(s_q + tok * kRows + r) = make_float4(fq[i][0] * iq, fq[i][1] * iq, fq[i][2] * iq, fq[i][3] * iq);
          *reinterpret_cast<float4*>(s_k + tok * kRows + r) = make_float4(fk[i][0] * ik, fk[i][1] * ik, fk[i][2] * ik, fk[i][3] * ik);
        }
      }
      if (4 * lane < kCols) *reinterpret_cast<float4*>(s_v + tok * kCols + 4 * lane) = make_float4(fv[0], fv[1], fv[2], fv[3]);
      if (lane == 0) s_g[tok] = make_float4(expf(log_decay(to_f32(pa[e]), A_log, dt_bias)), step_size(to_f32(pb[e])), sx * iq * ik, 0.f);
    }
  };

  Tile<RJ> tile;
  const int row0 = 4 * (lane & 7), c = 16 * warp + 4 * (lane >> 3);
  float* S = a.state + ((size_t)slot * d.heads + h) * d.dim * d.vdim;
  fetch(0);
  if (pos0 > 0)
    tile.load(S, d.dim, d.vdim, row0, col0 + c);
  else
    tile.zero();
  stage(0);
  __syncthreads();
  const int my_col = c + (lane & 3);
  const bool writes = (lane & 4) && col0 + my_col < d.vdim;
  float* out = a.out + (size_t)r0 * d.heads * d.vdim + (size_t)h * d.vdim + col0 + my_col;
  for (int t0 = 0, buf = 0; t0 < n; t0 += kTok, buf ^= 1) {
    const bool more = t0 + kTok < n;
    if (more) fetch(t0 + kTok);
    const int m = min(kTok, n - t0);
    for (int e = 0; e < m; ++e) {
      const int tok = buf * kTok + e;
      ulonglong2 k[RJ], q[RJ];
#pragma unroll
      for (int j = 0; j < RJ; ++j) {
        k[j] = *reinterpret_cast<const ulonglong2*>(s_k + tok * kRows + 32 * j + row0);
        q[j] = *reinterpret_cast<const ulonglong2*>(s_q + tok * kRows + 32 * j + row0);
      }
      const float4 gb = s_g[tok];
      const float o = tile.step(k, q, s_v[tok * kCols + my_col], gb.x, gb.y, gb.z, lane);
      if (writes) out[(size_t)(t0 + e) * d.heads * d.vdim] = o;
    }
    if (more) stage(buf ^ 1);
    __syncthreads();
  }
  tile.store(S, d.dim, d.vdim, row0, col0 + c);
  // the ring: every channel once (q and k by the first head that uses them and the first column part)
  const bool owns_qk = blockIdx.x == 0 && h % (d.heads / d.kv_heads) == 0;
  for (int t = max(0, n - a.taps); t < n; ++t) {
    const A* row = a.x + (size_t)(r0 + t) * a.ld;
    A* dst = a.ring + ((size_t)slot * a.taps + (pos0 + t) % a.taps) * a.C;
    if (owns_qk)
      for (int i = threadIdx.x; i < d.dim; i += NW * 32) {
        dst[q_col + i] = row[q_col + i];
        dst[k_col + i] = row[k_col + i];
      }
    for (int i = threadIdx.x; i < kCols && col0 + i < d.vdim; i += NW * 32) dst[v_col + i] = row[v_col + i];
  }
}

// ---- prompt passes: norm and gate of the outputs -------------------------------------------------------------------------
template <typename A>
__global__ void __launch_bounds__(256) gated_rms_kernel(const float* __restrict__ o, const A* __restrict__ gate, int64_t ld_gate,
                                                        const float* __restrict__ w, int heads, int vdim, int vdim_true,
                                                        float eps, A* __restrict__ out, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const int t = r / heads, h = r - t * heads;
  const float* x = o + (size_t)r * vdim;
  const A* gt = gate + (size_t)t * ld_gate + (size_t)h * vdim;
  float ss = 0.f;
  for (int i = lane * 4; i < vdim; i += 128) {
    float v[4];
    load4(x + i, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(v[j], v[j], ss);
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim_true + eps);
  for (int i = lane * 4; i < vdim; i += 128) {
    float v[4], g[4], wt[4];
    load4(x + i, v);
    load4(gt + i, g);
    load4(w + i, wt);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = v[j] * inv * wt[j] * silu<A>(g[j]);
    A* dst = out + (size_t)r * vdim + i;
    if constexpr (sizeof(A) == 2) {
      __nv_bfloat162 p[2] = {__floats2bfloat162_rn(v[0], v[1]), __floats2bfloat162_rn(v[2], v[3])};
      *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<uint2*>(p);
    } else {
      *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    }
  }
}

// ---- decode steps ----------------------------------------------------------------------------------------------------------
template <typename A>
struct StepArgs {
  const A* x;        // projected rows: q | k | v as for the scan, and the columns below
  int64_t ld;
  int C, taps, g_col, b_col, a_col;
  const float* conv; // [taps][C]
  const float *A_log, *dt_bias, *norm_w;
  float eps;
  DeltaDims d;
  const int32_t *row_slot, *row_pos;
  float* state;
  A* ring;
  A* out;            // [T, heads * vdim]
  int32_t* status;
};

// Convolution and silu of one head's channels of a new token: out = q [rows] | k [rows] | v [vdim], zero past dim; the token's
// inputs go to the ring (those of q and k by the first head that uses them).
template <typename A>
__device__ __forceinline__ void step_conv(const StepArgs<A>& a, const A* row, A* ring, int h, int pos, int rows, float* out) {
  const int tid = threadIdx.x, threads = blockDim.x, rep = a.d.heads / a.d.kv_heads, kh = h / rep;
  const int q_col = kh * a.d.dim, k_col = (a.d.kv_heads + kh) * a.d.dim, v_col = 2 * a.d.kv_heads * a.d.dim + h * a.d.vdim;
  // convolutions: everything two channels need is requested before the first use
  const int total = 2 * rows + a.d.vdim, back = min(a.taps - 1, pos), now = pos % a.taps;
  for (int i0 = tid; i0 < total; i0 += 2 * threads) {
    float w[2][kMaxTaps], x[2][kMaxTaps];
    A cur[2];
    int chan[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * threads, part = i < rows ? 0 : i < 2 * rows ? 1 : 2, e = i - part * rows;
      const bool there = i < total && (part == 2 || e < a.d.dim);
      chan[u] = there ? (part == 0 ? q_col : part == 1 ? k_col : v_col) + e : -1;
#pragma unroll
      for (int j = 0; j < kMaxTaps; ++j) {
        w[u][j] = x[u][j] = 0.f;
        if (!there || j > back) continue;
        const int at = now - j < 0 ? now - j + a.taps : now - j;
        w[u][j] = a.conv[(size_t)(a.taps - 1 - j) * a.C + chan[u]];
        if (j == 0)
          cur[u] = row[chan[u]];
        else
          x[u][j] = to_f32(ring[(size_t)at * a.C + chan[u]]);
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * threads;
      if (i >= total) break;
      float val = 0.f;
      if (chan[u] >= 0) {
        float sum = 0.f;
#pragma unroll
        for (int j = kMaxTaps - 1; j > 0; --j) sum = fmaf(w[u][j], x[u][j], sum);
        val = silu<float>(fmaf(w[u][0], to_f32(cur[u]), sum));
        if (i >= 2 * rows || h % rep == 0) ring[(size_t)now * a.C + chan[u]] = cur[u];
      }
      out[i] = val;
    }
  }
}

// CTA (head, row), the state in shared memory: one bulk copy in, one out.  Threads over the columns, several parts of the rows.
template <typename A>
__global__ void __launch_bounds__(256, 3) delta_step_bulk_kernel(StepArgs<A> a) {
  extern __shared__ __align__(16) float smem[];
  const DeltaDims d = a.d;
  float* s_S = smem;                   // [dim][vdim]
  float* s_q = s_S + d.dim * d.vdim;   // [dim]
  float* s_k = s_q + d.dim;            // [dim]
  float* s_v = s_k + d.dim;            // [vdim], then the outputs
  float2* s_part = reinterpret_cast<float2*>(s_v + d.vdim);  // [256]
  __shared__ uint64_t bar;
  __shared__ float s_kq;
  __shared__ int s_abort;
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, t = blockIdx.y;
  if (tid == 0) {
    s_abort = 0;
    mbar_init(&bar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  pdl_wait();
  const int slot = a.row_slot[t], pos = a.row_pos[t];
  A* out = a.out + ((size_t)t * d.heads + h) * d.vdim;
  if (pos < 0) {  // padding row
    for (int i = tid; i < d.vdim; i += 256) out[i] = from_f32<A>(0.f);
    return;
  }
  float* S = a.state + ((size_t)slot * d.heads + h) * d.dim * d.vdim;
  const uint32_t bytes = (uint32_t)(d.dim * d.vdim) * 4;
  if (pos > 0) {
    if (tid == 0) {
      mbar_expect_tx(&bar, bytes);
      bulk_load(s_S, S, bytes, &bar);
    }
  } else {
    for (int i = tid; i < d.dim * d.vdim; i += 256) s_S[i] = 0.f;
  }
  const A* row = a.x + (size_t)t * a.ld;
  const float beta = step_size(to_f32(row[a.b_col + h])), g = expf(log_decay(to_f32(row[a.a_col + h]), a.A_log[h], a.dt_bias[h]));
  step_conv(a, row, a.ring + (size_t)slot * a.taps * a.C, h, pos, d.dim, s_q);
  __syncthreads();
  if (warp == 0) {  // unit vectors, their product
    float sq = 0.f, sk = 0.f, sx = 0.f;
    for (int i = lane; i < d.dim; i += 32) {
      const float q = s_q[i], k = s_k[i];
      sq = fmaf(q, q, sq), sk = fmaf(k, k, sk), sx = fmaf(q, k, sx);
    }
    sq = warp_sum(sq), sk = warp_sum(sk), sx = warp_sum(sx);
    const float iq = d.q_scale / sqrtf(sq + 1e-6f), ik = 1.f / sqrtf(sk + 1e-6f);
    for (int i = lane; i < d.dim; i += 32) s_q[i] *= iq, s_k[i] *= ik;
    if (lane == 0) s_kq = sx * iq * ik;
  }
  const bool ok = pos == 0 || mbar_wait(&bar, 0, &s_abort);
  if (__syncthreads_or(!ok)) {  // gave up: nothing is written, the copy gets another bounded chance to land
    if (tid == 0) {
      if (a.status) atomicOr(a.status, 1);
      mbar_wait(&bar, 0, &s_abort);
    }
    __syncthreads();
    return;
  }
  const int width = min((d.vdim + 31) / 32 * 32, 256), parts = 256 / width, col = tid % width, part = tid / width;
  const int per = (d.dim / 4 + parts - 1) / parts * 4, r0 = min(part * per, d.dim), r1 = min(r0 + per, d.dim);
  const bool works = part < parts;
  for (int c0 = 0; c0 < d.vdim; c0 += width) {
    const int v = c0 + col;
    float dk = 0.f, dq = 0.f, o = 0.f;
    if (works && v < d.vdim) {
#pragma unroll 4
      for (int r = r0; r < r1; r += 4) {
        const float4 k = *reinterpret_cast<const float4*>(s_k + r), q = *reinterpret_cast<const float4*>(s_q + r);
        const float a0 = s_S[r * d.vdim + v], a1 = s_S[(r + 1) * d.vdim + v], a2 = s_S[(r + 2) * d.vdim + v], a3 = s_S[(r + 3) * d.vdim + v];
        dk = fmaf(a0, k.x, dk), dq = fmaf(a0, q.x, dq);
        dk = fmaf(a1, k.y, dk), dq = fmaf(a1, q.y, dq);
        dk = fmaf(a2, k.z, dk), dq = fmaf(a2, q.z, dq);
        dk = fmaf(a3, k.w, dk), dq = fmaf(a3, q.w, dq);
      }
    }
    s_part[tid] = make_float2(dk, dq);
    __syncthreads();
    if (works && v < d.vdim) {
      dk = dq = 0.f;
      for (int p = 0; p < parts; ++p) {
        const float2 x = s_part[p * width + col];
        dk += x.x, dq += x.y;
      }
      const float u = beta * (s_v[v] - g * dk);
      o = fmaf(u, s_kq, g * dq);
#pragma unroll 4
      for (int r = r0; r < r1; r += 4) {
        const float4 k = *reinterpret_cast<const float4*>(s_k + r);
        float* x = s_S + r * d.vdim + v;
        x[0] = fmaf(k.x, u, g * x[0]);
        x[d.vdim] = fmaf(k.y, u, g * x[d.vdim]);
        x[2 * d.vdim] = fmaf(k.z, u, g * x[2 * d.vdim]);
        x[3 * d.vdim] = fmaf(k.w, u, g * x[3 * d.vdim]);
      }
    }
    __syncthreads();  // (everybody has read the value and the partial sums)
    if (part == 0 && v < d.vdim) s_v[v] = o;
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  __syncthreads();
  if (tid == 0) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(S), "r"(smem_u32(s_S)), "r"(bytes) : "memory");
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
  }
  float ss = 0.f;
  for (int i = lane; i < d.vdim; i += 32) ss = fmaf(s_v[i], s_v[i], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)d.vdim_true + a.eps);
  for (int i = tid; i < d.vdim; i += 256)
    out[i] = from_f32<A>(s_v[i] * inv * a.norm_w[i] * silu<A>(to_f32(row[a.g_col + h * d.vdim + i])));
  if (tid == 0) bulk_wait_all0();
}

// CTA (head, row), for states beyond shared memory: the tile in registers, eight warps = 128 columns at a time.
template <typename A, int RJ>
__global__ void __launch_bounds__(256) delta_step_kernel(StepArgs<A> a) {
  constexpr int kRows = 32 * RJ;
  extern __shared__ __align__(16) float smem[];
  float* s_q = smem;            // [kRows]
  float* s_k = s_q + kRows;     // [kRows]
  float* s_v = s_k + kRows;     // [vdim]
  float* s_o = s_v + a.d.vdim;  // [vdim]
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x, threads = blockDim.x;
  const DeltaDims d = a.d;
  const int h = blockIdx.x, t = blockIdx.y, rep = d.heads / d.kv_heads, kh = h / rep;
  const int slot = a.row_slot[t], pos = a.row_pos[t];
  A* out = a.out + ((size_t)t * d.heads + h) * d.vdim;
  if (pos < 0) {  // padding row
    for (int i = tid; i < d.vdim; i += threads) out[i] = from_f32<A>(0.f);
    return;
  }
  const int cols = 16 * (threads >> 5), row0 = 4 * (lane & 7), c = 16 * warp + 4 * (lane >> 3);
  float* S = a.state + ((size_t)slot * d.heads + h) * d.dim * d.vdim;
  Tile<RJ> tile;
  if (pos > 0)
    tile.load(S, d.dim, d.vdim, row0, c);
  else
    tile.zero();
  const A* row = a.x + (size_t)t * a.ld;
  A* ring = a.ring + (size_t)slot * a.taps * a.C;
  const float beta = step_size(to_f32(row[a.b_col + h])), g = expf(log_decay(to_f32(row[a.a_col + h]), a.A_log[h], a.dt_bias[h]));
  step_conv(a, row, ring, h, pos, kRows, smem);
  __syncthreads();
  ulonglong2 k[RJ], q[RJ];
  float sq = 0.f, sk = 0.f, sx = 0.f;
#pragma unroll
  for (int j = 0; j < RJ; ++j) {
    k[j] = *reinterpret_cast<const ulonglong2*>(s_k + 32 * j + row0);
    q[j] = *reinterpret_cast<const ulonglong2*>(s_q + 32 * j + row0);
    const float2 k0 = unpack2(k[j].x), k1 = unpack2(k[j].y), q0 = unpack2(q[j].x), q1 = unpack2(q[j].y);
    sk += k0.x * k0.x + k0.y * k0.y + k1.x * k1.x + k1.y * k1.y;
    sq += q0.x * q0.x + q0.y * q0.y + q1.x * q1.x + q1.y * q1.y;
    sx += q0.x * k0.x + q0.y * k0.y + q1.x * k1.x + q1.y * k1.y;
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
    sx += __shfl_xor_sync(0xffffffffu, sx, o);
  }
  const float iq = d.q_scale / sqrtf(sq + 1e-6f), ik = 1.f / sqrtf(sk + 1e-6f), kq = sx * iq * ik;
  const f32x2 iq2 = pack2(iq, iq), ik2 = pack2(ik, ik);
#pragma unroll
  for (int j = 0; j < RJ; ++j) {
    k[j].x = mul2(k[j].x, ik2), k[j].y = mul2(k[j].y, ik2);
    q[j].x = mul2(q[j].x, iq2), q[j].y = mul2(q[j].y, iq2);
  }
  for (int c0 = 0; c0 < d.vdim; c0 += cols) {
    const int my_col = c0 + c + (lane & 3);
    if (c0 > 0) {
      if (pos > 0)
        tile.load(S, d.dim, d.vdim, row0, c0 + c);
      else
        tile.zero();
    }
    const float o = tile.step(k, q, my_col < d.vdim ? s_v[my_col] : 0.f, g, beta, kq, lane);
    if ((lane & 4) && my_col < d.vdim) s_o[my_col] = o;
    tile.store(S, d.dim, d.vdim, row0, c0 + c);
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = lane; i < d.vdim; i += 32) ss = fmaf(s_o[i], s_o[i], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)d.vdim_true + a.eps);
  for (int i = tid; i < d.vdim; i += threads)
    out[i] = from_f32<A>(s_o[i] * inv * a.norm_w[i] * silu<A>(to_f32(row[a.g_col + h * d.vdim + i])));
}

// ---- host --------------------------------------------------------------------------------------------------------------------
template <typename A, int RJ, int NW>
int launch_scan(const ScanArgs<A>& a, int n_segs, cudaStream_t st) {
  constexpr int kTok = kPer * NW;
  constexpr size_t smem = 2 * kTok * (2 * 32 * RJ + 16 * NW) * sizeof(float) + 2 * kTok * sizeof(float4);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<A, RJ, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(MLORA_ECUDA, "delta_scan: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  }
  launch_pdl(delta_scan_kernel<A, RJ, NW>, dim3((a.d.vdim + 16 * NW - 1) / (16 * NW), a.d.heads, n_segs), NW * 32, smem, st, a);
  count_launch();
  MLORA_CHECK_LAUNCH("delta_scan_kernel");
  return MLORA_OK;
}

// Columns per CTA: as many as there are, halved while that leaves SMs without work.
template <typename A, int RJ>
int launch_scan_rows(const ScanArgs<A>& a, int n_segs, cudaStream_t st) {
  int nw = a.d.vdim > 64 ? 8 : a.d.vdim > 32 ? 4 : 2;
  const auto ctas = [&](int w) { return (long long)n_segs * a.d.heads * ((a.d.vdim + 16 * w - 1) / (16 * w)); };
  while (nw > 2 && ctas(nw) < 2 * 148) nw /= 2;
  if (nw == 8) return launch_scan<A, RJ, 8>(a, n_segs, st);
  if (nw == 4) return launch_scan<A, RJ, 4>(a, n_segs, st);
  return launch_scan<A, RJ, 2>(a, n_segs, st);
}

}  // namespace
}  // namespace mlora

namespace mlora {
int check_delta_dims(const char* who, const DeltaDims& d, int C, int taps) {
  MLORA_REQUIRE(d.heads > 0 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.heads <= 65535, "%s: bad head counts", who);
  MLORA_REQUIRE(d.dim > 0 && d.dim % 8 == 0 && d.dim <= 256, "%s: dim a multiple of 8 up to 256 (got %d)", who, d.dim);
  MLORA_REQUIRE(d.vdim > 0 && d.vdim % 8 == 0 && d.vdim <= 4096 && d.vdim_true > 0 && d.vdim_true <= d.vdim,
                "%s: vdim a multiple of 8 up to 4096 (got %d)", who, d.vdim);
  MLORA_REQUIRE(C % 8 == 0 && C >= 2 * d.kv_heads * d.dim + d.heads * d.vdim, "%s: too few channels (%d)", who, C);
  MLORA_REQUIRE(taps > 0 && taps <= kMaxTaps, "%s: 1 to %d taps (got %d)", who, kMaxTaps, taps);
  return MLORA_OK;
}
}  // namespace mlora

using namespace mlora;

extern "C" int mlora_short_conv(const void* d_x, int64_t ld, int32_t C, int32_t taps, const float* d_w, const void* d_ring,
                                const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, void* d_out, int32_t f32,
                                void* stream) {
  MLORA_REQUIRE(T >= 0 && C > 0 && C % 8 == 0 && ld >= C && ld % 8 == 0, "short_conv: channels and pitch must be multiples of 8");
  MLORA_REQUIRE(taps > 0 && taps <= kMaxTaps, "short_conv: 1 to %d taps (got %d)", kMaxTaps, taps);
  MLORA_REQUIRE(d_x && d_w && d_ring && d_row_slot && d_row_pos && d_out, "short_conv: null pointer");
  MLORA_REQUIRE(aligned16(d_x) && aligned16(d_w) && aligned16(d_ring) && aligned16(d_out), "short_conv: pointers must be 16-byte aligned");
  if (T == 0) return MLORA_OK;
  const dim3 grid((C / 8 + 127) / 128, (T + kConvRows - 1) / kConvRows);
  MLORA_REQUIRE(grid.y <= 65535, "short_conv: too many rows (%d)", T);
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    ConvArgs<A> a{(const A*)d_x, ld, C, taps, d_w, (const A*)d_ring, d_row_slot, d_row_pos, (A*)d_out, T};
    const auto go = [&](auto kernel) { launch_pdl(kernel, grid, 128, 0, (cudaStream_t)stream, a); };
    switch (taps) {
      case 1: go(short_conv_kernel<A, 1>); break;
      case 2: go(short_conv_kernel<A, 2>); break;
      case 3: go(short_conv_kernel<A, 3>); break;
      case 4: go(short_conv_kernel<A, 4>); break;
      case 5: go(short_conv_kernel<A, 5>); break;
      case 6: go(short_conv_kernel<A, 6>); break;
      case 7: go(short_conv_kernel<A, 7>); break;
      default: go(short_conv_kernel<A, 8>); break;
    }
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("short_conv_kernel");
  return MLORA_OK;
}

extern "C" int mlora_delta_scan(const void* d_xc, const void* d_x, int64_t ld, int32_t C, int32_t taps, int32_t b_col,
                                int32_t a_col, const float* d_A_log, const float* d_dt_bias, int32_t heads, int32_t kv_heads,
                                int32_t dim, int32_t vdim, float q_scale, const int32_t* d_segs, int32_t n_segs, float* d_state,
                                void* d_ring, float* d_out, int32_t f32, void* stream) {
  const DeltaDims d{heads, kv_heads, dim, vdim, vdim, q_scale};
  const int rc = check_delta_dims("delta_scan", d, C, taps);
  if (rc) return rc;
  MLORA_REQUIRE(n_segs >= 0 && n_segs <= 65535 && ld >= C && b_col >= 0 && a_col >= 0 && b_col + heads <= ld && a_col + heads <= ld,
                "delta_scan: bad sizes");
  MLORA_REQUIRE(d_xc && d_x && d_A_log && d_dt_bias && d_segs && d_state && d_ring && d_out, "delta_scan: null pointer");
  MLORA_REQUIRE(aligned16(d_xc) && aligned16(d_segs) && aligned16(d_state) && aligned16(d_out), "delta_scan: pointers must be 16-byte aligned");
  if (n_segs == 0) return MLORA_OK;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    ScanArgs<A> a{(const A*)d_xc, (const A*)d_x, ld, C, taps, b_col, a_col, d_A_log, d_dt_bias, d, d_segs, d_state, (A*)d_ring, d_out};
    cudaStream_t st = (cudaStream_t)stream;
    if (dim <= 32) return launch_scan_rows<A, 1>(a, n_segs, st);
    if (dim <= 64) return launch_scan_rows<A, 2>(a, n_segs, st);
    if (dim <= 128) return launch_scan_rows<A, 4>(a, n_segs, st);
    return launch_scan_rows<A, 8>(a, n_segs, st);
  };
  return f32 ? launch(0.f) : launch(bf16());
}

extern "C" int mlora_gated_rms(const float* d_o, const void* d_gate, int64_t ld_gate, const float* d_w, int32_t T, int32_t heads,
                               int32_t vdim, int32_t vdim_true, float eps, void* d_out, int32_t f32, void* stream) {
  MLORA_REQUIRE(T >= 0 && heads > 0 && vdim > 0 && vdim % 8 == 0 && vdim_true > 0 && vdim_true <= vdim &&
                    ld_gate >= (int64_t)heads * vdim && ld_gate % 8 == 0 && (int64_t)T * heads < 2147483640ll,
                "gated_rms: bad sizes");
  MLORA_REQUIRE(d_o && d_gate && d_w && d_out, "gated_rms: null pointer");
  MLORA_REQUIRE(aligned16(d_o) && aligned16(d_gate) && aligned16(d_w) && aligned16(d_out), "gated_rms: pointers must be 16-byte aligned");
  if (T == 0) return MLORA_OK;
  const int rows = T * heads;
  if (f32)
    launch_pdl(gated_rms_kernel<float>, (rows + 7) / 8, 256, 0, (cudaStream_t)stream, d_o, (const float*)d_gate, ld_gate, d_w, heads,
               vdim, vdim_true, eps, (float*)d_out, rows);
  else
    launch_pdl(gated_rms_kernel<bf16>, (rows + 7) / 8, 256, 0, (cudaStream_t)stream, d_o, (const bf16*)d_gate, ld_gate, d_w, heads,
               vdim, vdim_true, eps, (bf16*)d_out, rows);
  count_launch();
  MLORA_CHECK_LAUNCH("gated_rms_kernel");
  return MLORA_OK;
}

extern "C" int mlora_delta_step(const void* d_x, int64_t ld, int32_t C, int32_t taps, int32_t g_col, int32_t b_col, int32_t a_col,
                                const float* d_conv, const float* d_A_log, const float* d_dt_bias, const float* d_norm_w, float eps,
                                int32_t heads, int32_t kv_heads, int32_t dim, int32_t vdim, int32_t vdim_true, float q_scale,
                                const int32_t* d_row_slot, const int32_t* d_row_pos, int32_t T, float* d_state, void* d_ring,
                                void* d_out, int32_t* d_status, int32_t f32, void* stream) {
  const DeltaDims d{heads, kv_heads, dim, vdim, vdim_true, q_scale};
  const int rc = check_delta_dims("delta_step", d, C, taps);
  if (rc) return rc;
  MLORA_REQUIRE(T >= 0 && T <= 65535 && ld >= C && g_col >= 0 && b_col >= 0 && a_col >= 0 && b_col + heads <= ld &&
                    a_col + heads <= ld && (int64_t)g_col + heads * vdim <= ld,
                "delta_step: bad sizes");
  MLORA_REQUIRE(d_x && d_conv && d_A_log && d_dt_bias && d_norm_w && d_row_slot && d_row_pos && d_state && d_ring && d_out,
                "delta_step: null pointer");
  MLORA_REQUIRE(aligned16(d_state), "delta_step: the state must be 16-byte aligned");
  if (T == 0) return MLORA_OK;
  const int warps = vdim > 64 ? 8 : vdim > 32 ? 4 : 2;
  const auto launch = [&](auto zero) {
    using A = decltype(zero);
    StepArgs<A> a{(const A*)d_x, ld, C, taps, g_col, b_col, a_col, d_conv, d_A_log, d_dt_bias, d_norm_w, eps, d, d_row_slot,
                  d_row_pos, d_state, (A*)d_ring, (A*)d_out, d_status};
    const auto go = [&](auto kernel, int rj) {
      launch_pdl_if(pdl_enabled_attn(), kernel, dim3(heads, T), warps * 32, (size_t)(64 * rj + 2 * vdim) * 4, (cudaStream_t)stream, a);
    };
    const size_t bulk = ((size_t)dim * vdim + 2 * dim + vdim + 512) * 4;
    if (bulk <= 200 * 1024) {
      if (bulk > 48 * 1024) cudaFuncSetAttribute(delta_step_bulk_kernel<A>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bulk);
      launch_pdl_if(pdl_enabled_attn(), delta_step_bulk_kernel<A>, dim3(heads, T), 256, bulk, (cudaStream_t)stream, a);
      return;
    }
    if (dim <= 32) go(delta_step_kernel<A, 1>, 1);
    else if (dim <= 64) go(delta_step_kernel<A, 2>, 2);
    else if (dim <= 128) go(delta_step_kernel<A, 4>, 4);
    else go(delta_step_kernel<A, 8>, 8);
  };
  if (f32)
    launch(0.f);
  else
    launch(bf16());
  count_launch();
  MLORA_CHECK_LAUNCH("delta_step_kernel");
  return MLORA_OK;
}
