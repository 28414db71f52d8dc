// Gated delta rule with one decay per key channel, over a ragged batch, in fp32.  Per head, with
// the state S [dim, vdim] carried from token to token:
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// The columns of S are independent, so a block takes one (entry, head) and 4 C columns per warp and
// keeps its part of S in registers from the first token of the entry to the last.  Eight lanes
// share C (2 or 4) columns, each holding R of the key channels; more columns per lane save reads
// of shared memory, fewer give more warps.  Both products of a token use the
// decayed state (o = S^T q + (k . q) u), so one reduction over the eight lanes serves them; the
// arithmetic is two-wide packed fp32.  Tokens are staged in shared memory a few ahead.
#include "ragged.cuh"

namespace cb {

using f2 = unsigned long long;     // two packed fp32 values
__device__ __forceinline__ f2 mul_f2(f2 a, f2 b) {
  f2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f2 fma_f2(f2 a, f2 b, f2 c) {
  f2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f2 pack_f2(float lo, float hi) {
  f2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack_f2(f2 a) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(a));
  return r;
}
__device__ __forceinline__ float hsum_f2(f2 a) {
  const float2 r = unpack_f2(a);
  return r.x + r.y;
}
__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}

constexpr int SCAN_WARPS = 4;
constexpr int SCAN_TB = 8;         // tokens per stage
constexpr int SCAN_STAGES = 3;

struct ScanArgs {
  const float* q;      // [kv_heads, rows, DP], DP = dim rounded up to a multiple of 32
  const float* k;      // [kv_heads, rows, DP]
  const float* kq;     // [kv_heads, rows]
  const float* v;      // [rows, heads, vdim]
  const float* g;      // [heads, rows, DP]
  const float* beta;   // [heads, rows]
  float* state;        // [slots, heads, dim, vdim]
  float* o;            // out [rows, heads, vdim]
  int rows, heads, kv_heads, dim, vdim;
  Entries e;
};

template <int R, int C>   // R key channels per lane, a multiple of 4; DP = 8 R
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_kernel(const ScanArgs p) {
  constexpr int DP = 8 * R, SCAN_COLS = SCAN_WARPS * 4 * C;
  constexpr int STAGE = SCAN_TB * (3 * DP + SCAN_COLS + 2);  // floats
  constexpr int THREADS = SCAN_WARPS * 32;
  extern __shared__ __align__(16) float sm[];
  const int e = blockIdx.y, h = blockIdx.x % p.heads, slab = blockIdx.x / p.heads;
  const int hk = h / (p.heads / p.kv_heads);
  const int row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ld = lane & 7;
  const int col_base = slab * SCAN_COLS;
  const int c0 = (warp * 4 + (lane >> 3)) * C;               // first of this lane's columns
  float* st = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dim * p.vdim;
  const float* gq = p.q + (static_cast<size_t>(hk) * p.rows + row0) * DP;
  const float* gk = p.k + (static_cast<size_t>(hk) * p.rows + row0) * DP;
  const float* gg = p.g + (static_cast<size_t>(h) * p.rows + row0) * DP;
  const float* gv = p.v + (static_cast<size_t>(row0) * p.heads + h) * p.vdim + col_base;
  const float* gb = p.beta + static_cast<size_t>(h) * p.rows + row0;
  const float* gkq = p.kq + static_cast<size_t>(hk) * p.rows + row0;
  const int vstride = p.heads * p.vdim;

  // tokens t0 .. t0 + SCAN_TB - 1 into a stage: q, k and g are contiguous blocks
  auto fetch = [&](int stage, int t0) {
    const uint32_t base = smem_u32(sm + stage * STAGE);
    const int n = min(SCAN_TB, len - t0);
    const int at = t0 * DP;
#pragma unroll
    for (int i = threadIdx.x; i < SCAN_TB * DP / 4; i += THREADS) {
      if (i < n * (DP / 4)) {
        cp_async16(base + i * 16, gq + at + i * 4);
        cp_async16(base + (SCAN_TB * DP + i * 4) * 4, gk + at + i * 4);
        cp_async16(base + (2 * SCAN_TB * DP + i * 4) * 4, gg + at + i * 4);
      }
    }
    const uint32_t vb = base + SCAN_TB * 3 * DP * 4;
#pragma unroll
    for (int i = threadIdx.x; i < SCAN_TB * SCAN_COLS; i += THREADS) {
      const int t = i / SCAN_COLS, c = i % SCAN_COLS;
      if (t < n && col_base + c < p.vdim)
        cp_async4(vb + i * 4, gv + static_cast<size_t>(t0 + t) * vstride + c);
    }
    if (threadIdx.x < 2 * SCAN_TB) {
      const int t = threadIdx.x % SCAN_TB;
      if (t < n)
        cp_async4(vb + (SCAN_TB * SCAN_COLS + threadIdx.x) * 4,
                  (threadIdx.x < SCAN_TB ? gb : gkq) + t0 + t);
    }
    cp_async_commit();
  };

  for (int i = 0; i < SCAN_STAGES - 1; ++i) {
    if (i * SCAN_TB < len) fetch(i, i * SCAN_TB);
    else cp_async_commit();
  }
  f2 s[C][R / 2];
  const bool has_state = p.e.pos0[e] > 0;
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col_base + c0 + c;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int d = (i / 2) * 32 + ld * 4 + (i % 2) * 2;
      float x = 0.f, y = 0.f;
      if (has_state && col < p.vdim) {
        if (d < p.dim) x = st[static_cast<size_t>(d) * p.vdim + col];
        if (d + 1 < p.dim) y = st[static_cast<size_t>(d + 1) * p.vdim + col];
      }
      s[c][i] = pack_f2(x, y);
    }
  }
  // the column this lane finishes, and whether it ends with S^T q (else S^T k); see below
  const int my_c = C == 4 ? ((ld >> 1) & 1) * 2 + ((ld >> 2) & 1) : (ld >> 1) & 1;
  const int my = c0 + my_c;
  int stage = 0;
  for (int t0 = 0; t0 < len; t0 += SCAN_TB) {
    cp_async_wait<SCAN_STAGES - 2>();
    __syncthreads();                       // the stage is filled, and the one before it is free
    const int ahead = t0 + (SCAN_STAGES - 1) * SCAN_TB;
    if (ahead < len) fetch((stage + SCAN_STAGES - 1) % SCAN_STAGES, ahead);
    else cp_async_commit();
    const float* sb = sm + stage * STAGE;
    const float* sv = sb + SCAN_TB * 3 * DP;
    const float* ss = sv + SCAN_TB * SCAN_COLS;
    const int n = min(SCAN_TB, len - t0);
    stage = (stage + 1) % SCAN_STAGES;
    for (int t = 0; t < n; ++t) {
      const float* tq = sb + t * DP + ld * 4;
      f2 a[C], b[C];
#pragma unroll
      for (int c = 0; c < C; ++c) a[c] = b[c] = 0ull;
      f2 kk[R / 2];
#pragma unroll
      for (int j = 0; j < R / 4; ++j) {
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(tq + j * 32);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(tq + SCAN_TB * DP + j * 32);
        const ulonglong2 g2 = *reinterpret_cast<const ulonglong2*>(tq + 2 * SCAN_TB * DP + j * 32);
        kk[2 * j] = k2.x;
        kk[2 * j + 1] = k2.y;
#pragma unroll
        for (int c = 0; c < C; ++c) {
          s[c][2 * j] = mul_f2(s[c][2 * j], g2.x);
          s[c][2 * j + 1] = mul_f2(s[c][2 * j + 1], g2.y);
          a[c] = fma_f2(s[c][2 * j], k2.x, a[c]);
          b[c] = fma_f2(s[c][2 * j], q2.x, b[c]);
          a[c] = fma_f2(s[c][2 * j + 1], k2.y, a[c]);
          b[c] = fma_f2(s[c][2 * j + 1], q2.y, b[c]);
        }
      }
      // Sum over the eight lanes, ending with one value per lane: in the first exchange a lane
      // keeps S^T q (odd ld) or S^T k (even), in the next ones a half of the columns it still has.
      const bool odd = ld & 1, hi = ld & 2, top = ld & 4;
      float x[C], y;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float fa = hsum_f2(a[c]), fb = hsum_f2(b[c]);
        x[c] = (odd ? fb : fa) + __shfl_xor_sync(0xffffffffu, odd ? fa : fb, 1);
      }
      if constexpr (C == 4) {
        const float z0 = (hi ? x[2] : x[0]) + __shfl_xor_sync(0xffffffffu, hi ? x[0] : x[2], 2);
        const float z1 = (hi ? x[3] : x[1]) + __shfl_xor_sync(0xffffffffu, hi ? x[1] : x[3], 2);
        y = (top ? z1 : z0) + __shfl_xor_sync(0xffffffffu, top ? z0 : z1, 4);
      } else {
        y = (hi ? x[1] : x[0]) + __shfl_xor_sync(0xffffffffu, hi ? x[0] : x[1], 2);
        y += __shfl_xor_sync(0xffffffffu, y, 4);
      }
      const float beta = ss[t], kq = ss[SCAN_TB + t];
      const float un = beta * (sv[t * SCAN_COLS + my] - y);  // of use on even lanes
      float u_my = 0.f;
#pragma unroll
      for (int c = 0; c < C; ++c) {
        // the even lane that finished column c
        const int src = C == 4 ? ((c >> 1) << 1) | ((c & 1) << 2) : c << 1;
        const float u = __shfl_sync(0xffffffffu, un, (lane & 24) | src);
        if (c == my_c) u_my = u;
        const f2 uu = pack_f2(u, u);
#pragma unroll
        for (int i = 0; i < R / 2; ++i) s[c][i] = fma_f2(kk[i], uu, s[c][i]);
      }
      if (odd && (C == 4 || ld < 4) && col_base + my < p.vdim)
        p.o[(static_cast<size_t>(row0 + t0 + t) * p.heads + h) * p.vdim + col_base + my] = y + kq * u_my;
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col_base + c0 + c;
    if (col >= p.vdim) continue;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int d = (i / 2) * 32 + ld * 4 + (i % 2) * 2;
      const float2 x = unpack_f2(s[c][i]);
      if (d < p.dim) st[static_cast<size_t>(d) * p.vdim + col] = x.x;
      if (d + 1 < p.dim) st[static_cast<size_t>(d + 1) * p.vdim + col] = x.y;
    }
  }
}

// ------------------------------------------------------------------------------ blocks of tokens
// For longer entries four tokens are taken at a time.  With G_j the product of the decays of tokens
// 1 .. j of a block and S the state before it, everything a token needs is linear in S:
//   S'_j^T k_j = S^T (G_j k_j) + sum_{i<j} c_ij u_i      c_ij = sum_d k_i (g_{i+1} .. g_j) k_j
//   o_j        = S^T (G_j q_j) + sum_{i<=j} e_ij u_i     e_ij = sum_d k_i (g_{i+1} .. g_j) q_j
//   S <- G_4 S + sum_j (g_{j+1} .. g_4 k_j) u_j^T
// so the state is read once per block, one reduction over the lanes serves four tokens, and only the
// u_j = beta_j (v_j - S'_j^T k_j) follow one another.  Products of decays only shrink: nothing is
// divided.  delta_block_kernel prepares the vectors and the coefficients, per value head; tokens past
// an entry's end get k = q = 0, g = 1, beta = 0 and change nothing.
constexpr int BLK = 4;
constexpr int BLK_VECS = 3 * BLK + 1;          // G k | G q | G_4 | suffix products times k
constexpr int BLK_SCAL = 20;                   // c (6, by j then i), e (10), beta (4)

struct BlockArgs {
  const float* q;      // as in ScanArgs
  const float* k;
  const float* g;
  const float* beta;
  float* vecs;         // out [heads, groups, BLK_VECS, DP]
  float* scal;         // out [heads, groups, BLK_SCAL]
  int rows, heads, kv_heads, groups;
  Entries e;
  const int* tile_entry;   // [groups / 4] the tiles of 16 tokens of the convolution kernels
  const int* tile_off;
};

template <int NR>      // channels per lane; DP = 32 NR
__global__ void __launch_bounds__(128) delta_block_kernel(const BlockArgs p) {
  constexpr int DP = 32 * NR;
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int h = blockIdx.y, hk = h / (p.heads / p.kv_heads);
  if (unit >= p.groups) return;
  const int e = p.tile_entry[unit / 4], off = p.tile_off[unit / 4] + (unit % 4) * BLK;
  const int row0 = p.e.row0[e] + off, n = p.e.len[e] - off;
  if (n <= 0) return;                          // no scan reads this group
  float k[BLK][NR], q[BLK][NR], g[BLK][NR];
#pragma unroll
  for (int j = 0; j < BLK; ++j) {
    const bool in = j < n;
    const size_t kv = (static_cast<size_t>(hk) * p.rows + row0 + (in ? j : 0)) * DP + lane;
    const size_t hv = (static_cast<size_t>(h) * p.rows + row0 + (in ? j : 0)) * DP + lane;
#pragma unroll
    for (int x = 0; x < NR; ++x) {
      k[j][x] = in ? p.k[kv + 32 * x] : 0.f;
      q[j][x] = in ? p.q[kv + 32 * x] : 0.f;
      g[j][x] = in ? p.g[hv + 32 * x] : 1.f;
    }
  }
  float* out = p.vecs + (static_cast<size_t>(h) * p.groups + unit) * BLK_VECS * DP + lane;
  float c[6] = {}, ee[10] = {};
#pragma unroll
  for (int x = 0; x < NR; ++x) {
    float pre = 1.f, suf = 1.f;
#pragma unroll
    for (int j = 0; j < BLK; ++j) {
      pre *= g[j][x];
      out[j * DP + 32 * x] = pre * k[j][x];
      out[(BLK + j) * DP + 32 * x] = pre * q[j][x];
      // w = k_i (g_{i+1} .. g_j), from i = j down
      float w = 1.f;
#pragma unroll
      for (int i = j; i >= 0; --i) {
        const float kw = k[i][x] * w;
        ee[j * (j + 1) / 2 + i] += kw * q[j][x];
        if (i < j) c[j * (j - 1) / 2 + i] += kw * k[j][x];
        w *= g[i][x];
      }
    }
    out[2 * BLK * DP + 32 * x] = pre;
#pragma unroll
    for (int j = BLK - 1; j >= 0; --j) {
      out[(2 * BLK + 1 + j) * DP + 32 * x] = suf * k[j][x];
      suf *= g[j][x];
    }
  }
#pragma unroll
  for (int i = 0; i < 6; ++i) c[i] = warp_sum(c[i]);
#pragma unroll
  for (int i = 0; i < 10; ++i) ee[i] = warp_sum(ee[i]);
  if (lane == 0) {
    float* sc = p.scal + (static_cast<size_t>(h) * p.groups + unit) * BLK_SCAL;
#pragma unroll
    for (int i = 0; i < 6; ++i) sc[i] = c[i];
#pragma unroll
    for (int i = 0; i < 10; ++i) sc[6 + i] = ee[i];
#pragma unroll
    for (int j = 0; j < BLK; ++j)
      sc[16 + j] = j < n ? p.beta[static_cast<size_t>(h) * p.rows + row0 + j] : 0.f;
  }
}

struct BlockScanArgs {
  const float* vecs;
  const float* scal;
  const float* v;      // [rows, heads, vdim]
  float* state;
  float* o;
  int heads, dim, vdim, groups;
  Entries e;
  const int* tile0;    // [entries] first tile of the entry
};

template <int R, int C>   // R key channels and C (2 or 4) columns per lane
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_blocks_kernel(const BlockScanArgs p) {
  constexpr int DP = 8 * R, COLS = SCAN_WARPS * 4 * C, THREADS = SCAN_WARPS * 32;
  constexpr int STAGE = BLK_VECS * DP + BLK_SCAL + BLK * COLS;   // floats of one block of tokens
  extern __shared__ __align__(16) float sm[];
  const int e = blockIdx.y, h = blockIdx.x % p.heads, slab = blockIdx.x / p.heads;
  const int row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ld = lane & 7;
  const int col_base = slab * COLS, c0 = (warp * 4 + (lane >> 3)) * C;
  float* st = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dim * p.vdim;
  const size_t first = static_cast<size_t>(h) * p.groups + p.tile0[e] * 4;
  const float* gvec = p.vecs + first * BLK_VECS * DP;
  const float* gsc = p.scal + first * BLK_SCAL;
  const float* gv = p.v + (static_cast<size_t>(row0) * p.heads + h) * p.vdim + col_base;
  const int vstride = p.heads * p.vdim;
  const int nb = (len + BLK - 1) / BLK;

  auto fetch = [&](int stage, int b) {
    const uint32_t base = smem_u32(sm + stage * STAGE);
    const float* src = gvec + static_cast<size_t>(b) * BLK_VECS * DP;
#pragma unroll
    for (int i = threadIdx.x; i < BLK_VECS * DP / 4; i += THREADS) cp_async16(base + i * 16, src + i * 4);
    if (threadIdx.x < BLK_SCAL / 4)
      cp_async16(base + (BLK_VECS * DP + threadIdx.x * 4) * 4, gsc + b * BLK_SCAL + threadIdx.x * 4);
    for (int i = threadIdx.x; i < BLK * COLS; i += THREADS) {
      const int t = b * BLK + i / COLS, c = i % COLS;
      const bool in = t < len && col_base + c < p.vdim;
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(
                       base + (BLK_VECS * DP + BLK_SCAL + i) * 4),
                   "l"(in ? gv + static_cast<size_t>(t) * vstride + c : gv), "r"(in ? 4 : 0)
                   : "memory");
    }
    cp_async_commit();
  };
  for (int i = 0; i < SCAN_STAGES - 1; ++i) {
    if (i < nb) fetch(i, i);
    else cp_async_commit();
  }
  f2 s[C][R / 2];
  const bool has_state = p.e.pos0[e] > 0;
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col_base + c0 + c;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int d = (i / 2) * 32 + ld * 4 + (i % 2) * 2;
      float x = 0.f, y = 0.f;
      if (has_state && col < p.vdim) {
        if (d < p.dim) x = st[static_cast<size_t>(d) * p.vdim + col];
        if (d + 1 < p.dim) y = st[static_cast<size_t>(d + 1) * p.vdim + col];
      }
      s[c][i] = pack_f2(x, y);
    }
  }
  // After the reduction lane ld holds both sums of token j_my and of NC = C / 2 columns from c_my on.
  constexpr int NC = C / 2;
  const int j_my = ld & 3, c_my = (ld >> 2) * NC;
  const bool hi_col = ld & 4;
  int stage = 0;
  for (int b = 0; b < nb; ++b) {
    cp_async_wait<SCAN_STAGES - 2>();
    __syncthreads();
    if (b + SCAN_STAGES - 1 < nb) fetch((stage + SCAN_STAGES - 1) % SCAN_STAGES, b + SCAN_STAGES - 1);
    else cp_async_commit();
    const float* sb = sm + stage * STAGE;
    const float* sc = sb + BLK_VECS * DP;
    const float* sv = sc + BLK_SCAL;
    stage = (stage + 1) % SCAN_STAGES;
    const float* tq = sb + ld * 4;
    // S^T (G_j k_j), then S^T (G_j q_j); the first exchange, over lane bit 2, keeps half the columns
    float y[2 * BLK][NC];
#pragma unroll
    for (int w = 0; w < 2 * BLK; ++w) {
      f2 acc[C];
#pragma unroll
      for (int c = 0; c < C; ++c) acc[c] = 0ull;
#pragma unroll
      for (int j = 0; j < R / 4; ++j) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(tq + w * DP + j * 32);
#pragma unroll
        for (int c = 0; c < C; ++c) acc[c] = fma_f2(s[c][2 * j], x.x, acc[c]);
#pragma unroll
        for (int c = 0; c < C; ++c) acc[c] = fma_f2(s[c][2 * j + 1], x.y, acc[c]);
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const float lo = hsum_f2(acc[c]), hi = hsum_f2(acc[NC + c]);
        y[w][c] = (hi_col ? hi : lo) + __shfl_xor_sync(0xffffffffu, hi_col ? lo : hi, 4);
      }
    }
    // bits 1 and 0: half of the tokens each time
    const bool b1 = ld & 2, b0 = ld & 1;
    float a[NC], o[NC], v[NC];
    const float beta = sc[16 + j_my];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      float z[2][2];
#pragma unroll
      for (int m = 0; m < 2; ++m)             // m: S^T k or S^T q
#pragma unroll
        for (int x = 0; x < 2; ++x)
          z[m][x] = (b1 ? y[m * BLK + 2 + x][c] : y[m * BLK + x][c]) +
                    __shfl_xor_sync(0xffffffffu, b1 ? y[m * BLK + x][c] : y[m * BLK + 2 + x][c], 2);
      a[c] = (b0 ? z[0][1] : z[0][0]) + __shfl_xor_sync(0xffffffffu, b0 ? z[0][0] : z[0][1], 1);
      o[c] = (b0 ? z[1][1] : z[1][0]) + __shfl_xor_sync(0xffffffffu, b0 ? z[1][0] : z[1][1], 1);
      v[c] = sv[j_my * COLS + c0 + c_my + c];
    }
    float u[BLK][C];
#pragma unroll
    for (int i = 0; i < BLK; ++i) {
      const float ci = j_my > i ? sc[j_my * (j_my - 1) / 2 + i] : 0.f;
      const float ei = j_my >= i ? sc[6 + j_my * (j_my + 1) / 2 + i] : 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const float un = beta * (v[c] - a[c]);       // final on the lanes of token i
        u[i][c] = __shfl_sync(0xffffffffu, un, (lane & 24) | i);
        u[i][NC + c] = __shfl_sync(0xffffffffu, un, (lane & 24) | 4 | i);
        const float mine = hi_col ? u[i][NC + c] : u[i][c];
        a[c] += ci * mine;
        o[c] += ei * mine;
      }
    }
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
      const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(tq + 2 * BLK * DP + j * 32);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        s[c][2 * j] = mul_f2(s[c][2 * j], g.x);
        s[c][2 * j + 1] = mul_f2(s[c][2 * j + 1], g.y);
      }
#pragma unroll
      for (int i = 0; i < BLK; ++i) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(tq + (2 * BLK + 1 + i) * DP + j * 32);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const f2 uu = pack_f2(u[i][c], u[i][c]);
          s[c][2 * j] = fma_f2(x.x, uu, s[c][2 * j]);
          s[c][2 * j + 1] = fma_f2(x.y, uu, s[c][2 * j + 1]);
        }
      }
    }
    const int t = b * BLK + j_my;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int col = col_base + c0 + c_my + c;
      if (t < len && col < p.vdim)
        p.o[(static_cast<size_t>(row0 + t) * p.heads + h) * p.vdim + col] = o[c];
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col_base + c0 + c;
    if (col >= p.vdim) continue;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      const int d = (i / 2) * 32 + ld * 4 + (i % 2) * 2;
      const float2 x = unpack_f2(s[c][i]);
      if (d < p.dim) st[static_cast<size_t>(d) * p.vdim + col] = x.x;
      if (d + 1 < p.dim) st[static_cast<size_t>(d + 1) * p.vdim + col] = x.y;
    }
  }
}

template <int R, int C>
static int launch_block_scan(const BlockScanArgs& a, int entries, cudaStream_t st) {
  constexpr int cols = SCAN_WARPS * 4 * C;
  const int smem = SCAN_STAGES * (BLK_VECS * 8 * R + BLK_SCAL + BLK * cols) * 4;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_scan_blocks_kernel<R, C>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -4;
    set = true;
  }
  dim3 grid(a.heads * ((a.vdim + cols - 1) / cols), entries);
  delta_scan_blocks_kernel<R, C><<<grid, SCAN_WARPS * 32, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int R>
static int launch_blocks(const BlockArgs& b, const BlockScanArgs& a, int entries, cudaStream_t st) {
  dim3 gb((b.groups + 3) / 4, b.heads);
  delta_block_kernel<R / 4><<<gb, 128, 0, st>>>(b);
  if constexpr (R <= 16) {
    const int wide = a.heads * ((a.vdim + 63) / 64) * entries;   // CTAs with four columns a lane
    if (a.vdim > 32 && wide >= sm_count()) return launch_block_scan<R, 4>(a, entries, st);
  }
  return launch_block_scan<R, 2>(a, entries, st);
}

template <int R, int C>
static int launch_scan_c(const ScanArgs& a, int entries, cudaStream_t st) {
  constexpr int cols = SCAN_WARPS * 4 * C;
  const int smem = SCAN_STAGES * SCAN_TB * (3 * 8 * R + cols + 2) * 4;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(delta_scan_kernel<R, C>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             smem) != cudaSuccess)
      return -4;
    set = true;
  }
  dim3 grid(a.heads * ((a.vdim + cols - 1) / cols), entries);
  delta_scan_kernel<R, C><<<grid, SCAN_WARPS * 32, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int R>
static int launch_scan(const ScanArgs& a, int entries, cudaStream_t st) {
  if constexpr (R <= 16) {
    const int wide = a.heads * ((a.vdim + 63) / 64) * entries;   // blocks with four columns a lane
    if (a.vdim > 32 && wide >= sm_count()) return launch_scan_c<R, 4>(a, entries, st);
  }
  return launch_scan_c<R, 2>(a, entries, st);
}

}  // namespace cb

using namespace cb;

extern "C" int cb_delta_scan(const float* q, const float* k, const float* kq, const float* v,
                             const float* g, const float* beta, float* state, float* o, int rows,
                             int heads, int kv_heads, int dim, int dim_p, int vdim, const int* slot,
                             const int* row0, const int* len, const int* pos0, int entries,
                             void* stream) {
  if (entries <= 0 || entries > 65535 || kv_heads < 1 || heads % kv_heads != 0) return -1;
  if (dim < 1 || dim > 256 || dim_p != (dim + 31) / 32 * 32) return -2;
  ScanArgs a;
  a.q = q; a.k = k; a.kq = kq; a.v = v; a.g = g; a.beta = beta; a.state = state; a.o = o;
  a.rows = rows; a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim;
  a.e.slot = slot; a.e.row0 = row0; a.e.len = len; a.e.pos0 = pos0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (dim_p / 32) {
    case 1: return launch_scan<4>(a, entries, st);
    case 2: return launch_scan<8>(a, entries, st);
    case 3: return launch_scan<12>(a, entries, st);
    case 4: return launch_scan<16>(a, entries, st);
    case 5: return launch_scan<20>(a, entries, st);
    case 6: return launch_scan<24>(a, entries, st);
    case 7: return launch_scan<28>(a, entries, st);
    default: return launch_scan<32>(a, entries, st);
  }
}

// The same in blocks of four tokens, for entries of more than a few: vecs [heads, 4 tiles, 13, dim_p]
// and scal [heads, 4 tiles, 20] are scratch, tile_entry / tile_off [tiles] the 16-token tiles of the
// batch and tile0 [entries] the first tile of every entry.
extern "C" int cb_delta_scan_blocks(const float* q, const float* k, const float* v, const float* g,
                                    const float* beta, float* state, float* o, float* vecs,
                                    float* scal, int rows, int heads, int kv_heads, int dim,
                                    int dim_p, int vdim, const int* slot, const int* row0,
                                    const int* len, const int* pos0, int entries,
                                    const int* tile_entry, const int* tile_off, const int* tile0,
                                    int tiles, void* stream) {
  if (entries <= 0 || entries > 65535 || tiles <= 0 || kv_heads < 1 || heads % kv_heads != 0 ||
      heads > 65535)
    return -1;
  if (dim < 1 || dim > 256 || dim_p != (dim + 31) / 32 * 32) return -2;
  BlockArgs b;
  b.q = q; b.k = k; b.g = g; b.beta = beta; b.vecs = vecs; b.scal = scal; b.rows = rows;
  b.heads = heads; b.kv_heads = kv_heads; b.groups = 4 * tiles;
  b.tile_entry = tile_entry; b.tile_off = tile_off;
  b.e.slot = slot; b.e.row0 = row0; b.e.len = len; b.e.pos0 = pos0;
  BlockScanArgs a;
  a.vecs = vecs; a.scal = scal; a.v = v; a.state = state; a.o = o; a.heads = heads; a.dim = dim;
  a.vdim = vdim; a.groups = b.groups; a.e = b.e; a.tile0 = tile0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (dim_p / 32) {
    case 1: return launch_blocks<4>(b, a, entries, st);
    case 2: return launch_blocks<8>(b, a, entries, st);
    case 3: return launch_blocks<12>(b, a, entries, st);
    case 4: return launch_blocks<16>(b, a, entries, st);
    case 5: return launch_blocks<20>(b, a, entries, st);
    case 6: return launch_blocks<24>(b, a, entries, st);
    case 7: return launch_blocks<28>(b, a, entries, st);
    default: return launch_blocks<32>(b, a, entries, st);
  }
}
