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
