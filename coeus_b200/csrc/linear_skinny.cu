// bf16 linear layers of a decode step: Y[M, N] = act(X[M, K] . W[N, K]^T + bias[N]) with few rows
// (M <= 16), bound by streaming the weights.  The weights are the 16-row operand of mma m16n8k16 and the
// tokens its 8 columns; every lane reads 32 consecutive bytes of a weight row per 64-wide slice
// of K (the contraction index is permuted the same way on both sides, so fragments come straight
// from global memory).  The warps of a CTA split K and add their results through shared memory.
// One launch can run two problems (the two projections of a parallel block read two norms of the
// same stream; the two inner products of factored projections).
#include "ragged.cuh"

namespace cb {

enum : int { SK_NONE = 0, SK_RELU2 = 4, SK_SOFTCAP = 5, SK_GELU_ERF = 6, SK_GLU = 7 };

struct SkinnyProblem {
  const __nv_bfloat16* x;   // [M, ldx]
  const __nv_bfloat16* w;   // [N, ldw]
  const __nv_bfloat16* bias;   // [N] or null
  void* y;                  // [M, ldy] bf16 or fp32
  int ldx, ldw, ldy, N, K, act, f32, accumulate;
  float act_arg;            // the cap, or of a gated unit the slope
  float limit, shift;       // SK_GLU: rows of w alternate, y [M, N / 2] (clamped_glu)
};
struct SkinnyArgs {
  SkinnyProblem p[2];
  int tiles0;               // CTAs of the first problem
  int M;
};

__device__ __forceinline__ void sk_mma(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                       uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, "
               "{%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 ldg_stream(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// MW 16-row weight tiles per CTA, NT 8-token tiles, WARPS warps splitting K
template <int MW, int NT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) linear_skinny_kernel(const SkinnyArgs args) {
  extern __shared__ float red[];            // [WARPS][NT * 8][MW * 16 + 1]
  const bool second = static_cast<int>(blockIdx.x) >= args.tiles0;
  const SkinnyProblem& p = args.p[second ? 1 : 0];
  const int n0 = (second ? blockIdx.x - args.tiles0 : blockIdx.x) * (MW * 16);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = lane >> 2, t = lane & 3;
  float acc[MW][NT][4];
#pragma unroll
  for (int i = 0; i < MW; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[i][j][k] = 0.f;
  const __nv_bfloat16* wp[MW][2];
#pragma unroll
  for (int i = 0; i < MW; ++i)
#pragma unroll
    for (int h = 0; h < 2; ++h)             // rows past the end repeat the last one
      wp[i][h] = p.w + static_cast<size_t>(min(n0 + i * 16 + h * 8 + r, p.N - 1)) * p.ldw + t * 16;
  const __nv_bfloat16* xp[NT];
#pragma unroll
  for (int j = 0; j < NT; ++j)
    xp[j] = p.x + static_cast<size_t>(min(j * 8 + r, args.M - 1)) * p.ldx + t * 16;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const int chunks = (p.K + 63) / 64;
  constexpr int U = (MW * NT <= 2) ? 4 : (MW * NT <= 4 ? 2 : 1);   // slices in flight
  for (int c0 = warp; c0 < chunks; c0 += WARPS * U) {
    uint4 a[U][MW][2][2];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k0 = (c0 + u * WARPS) * 64;
#pragma unroll
      for (int i = 0; i < MW; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int v = 0; v < 2; ++v)
            a[u][i][h][v] = k0 + t * 16 + v * 8 < p.K ? ldg_stream(wp[i][h] + k0 + v * 8) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k0 = (c0 + u * WARPS) * 64;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        uint4 b[2];
#pragma unroll
        for (int v = 0; v < 2; ++v)
          b[v] = k0 + t * 16 + v * 8 < p.K
                     ? *reinterpret_cast<const uint4*>(xp[j] + k0 + v * 8) : zero;
#pragma unroll
        for (int i = 0; i < MW; ++i)
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            const uint4 lo = a[u][i][0][v], hi = a[u][i][1][v];
            sk_mma(acc[i][j], lo.x, hi.x, lo.y, hi.y, b[v].x, b[v].y);
            sk_mma(acc[i][j], lo.z, hi.z, lo.w, hi.w, b[v].z, b[v].w);
          }
      }
    }
  }
  constexpr int LD = MW * 16 + 1;
  float* mine = red + warp * NT * 8 * LD;
#pragma unroll
  for (int i = 0; i < MW; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k)
        mine[(j * 8 + t * 2 + (k & 1)) * LD + i * 16 + r + (k >> 1) * 8] = acc[i][j][k];
  __syncthreads();
  if (p.act == SK_GLU) {
    for (int i = threadIdx.x; i < args.M * MW * 8; i += WARPS * 32) {
      const int m = i / (MW * 8), c = i % (MW * 8) * 2, n = n0 + c;
      if (n >= p.N) continue;
      float g = 0.f, u = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) {
        g += red[(w * NT * 8 + m) * LD + c];
        u += red[(w * NT * 8 + m) * LD + c + 1];
      }
      if (p.bias != nullptr) {
        g += __bfloat162float(p.bias[n]);
        u += __bfloat162float(p.bias[n + 1]);
      }
      static_cast<__nv_bfloat16*>(p.y)[static_cast<size_t>(m) * p.ldy + n / 2] =
          __float2bfloat16(clamped_glu(g, u, p.act_arg, p.limit, p.shift));
    }
    return;
  }
  for (int i = threadIdx.x; i < args.M * MW * 16; i += WARPS * 32) {
    const int m = i / (MW * 16), c = i % (MW * 16), n = n0 + c;
    if (n >= p.N) continue;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) v += red[(w * NT * 8 + m) * LD + c];
    if (p.bias != nullptr) v += __bfloat162float(p.bias[n]);
    if (p.act == SK_GELU_ERF) {
      v = gelu_erf(v);
    } else if (p.act == SK_RELU2) {
      v = fmaxf(v, 0.f);
      v *= v;
    } else if (p.act == SK_SOFTCAP) {
      v = p.act_arg * tanhf(v / p.act_arg);
    }
    const size_t at = static_cast<size_t>(m) * p.ldy + n;
    if (p.f32) {
      float* y = static_cast<float*>(p.y) + at;
      *y = p.accumulate ? *y + v : v;
    } else {
      static_cast<__nv_bfloat16*>(p.y)[at] = __float2bfloat16(v);
    }
  }
}

template <int MW, int NT, int WARPS>
static int launch_skinny(SkinnyArgs a, int count, cudaStream_t st) {
  constexpr int smem = WARPS * NT * 8 * (MW * 16 + 1) * 4;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(linear_skinny_kernel<MW, NT, WARPS>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -4;
    set = true;
  }
  a.tiles0 = (a.p[0].N + MW * 16 - 1) / (MW * 16);
  const int tiles = a.tiles0 + (count > 1 ? (a.p[1].N + MW * 16 - 1) / (MW * 16) : 0);
  linear_skinny_kernel<MW, NT, WARPS><<<tiles, WARPS * 32, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

using namespace cb;

static int skinny_problem(SkinnyProblem& p, const void* x, int ldx, const void* w, int ldw,
                          const void* bias, void* y, int ldy, int N, int K, int act, float act_arg, int f32, int accumulate) {
  if (N <= 0 || K <= 0 || K % 8 || ldx % 8 || ldw % 8 || (accumulate && !f32)) return -1;
  if ((reinterpret_cast<uintptr_t>(x) & 15u) || (reinterpret_cast<uintptr_t>(w) & 15u)) return -2;
  p.x = static_cast<const __nv_bfloat16*>(x);
  p.w = static_cast<const __nv_bfloat16*>(w);
  p.bias = static_cast<const __nv_bfloat16*>(bias);
  p.y = y; p.ldx = ldx; p.ldw = ldw; p.ldy = ldy; p.N = N; p.K = K; p.act = act; p.f32 = f32;
  p.accumulate = accumulate; p.act_arg = act_arg;
  return 0;
}

static int launch_skinny_m(const SkinnyArgs& a, int count, int K, cudaStream_t st) {
  const bool deep = K >= 4096 && count == 1;
  if (a.M <= 8) return deep ? launch_skinny<1, 1, 16>(a, count, st) : launch_skinny<1, 1, 8>(a, count, st);
  return deep ? launch_skinny<1, 2, 16>(a, count, st) : launch_skinny<1, 2, 8>(a, count, st);
}

// y [M, N / 2]: a gated unit (see clamped_glu) over alternating rows of w, after the bias [N] (null: none).
extern "C" int cb_linear_skinny_glu(const void* x, int ldx, const void* w, int ldw, const void* bias, void* y,
                                    int ldy, int N, int K, float slope, float limit, float shift, int M,
                                    void* stream) {
  if (M <= 0 || M > 16 || N % 2) return -1;
  SkinnyArgs a = {};
  a.M = M;
  const int rc = skinny_problem(a.p[0], x, ldx, w, ldw, bias, y, ldy, N, K, SK_GLU, slope, 0, 0);
  if (rc != 0) return rc;
  a.p[0].limit = limit;
  a.p[0].shift = shift;
  return launch_skinny_m(a, 1, K, static_cast<cudaStream_t>(stream));
}

// The second problem is skipped when x1 is null.
extern "C" int cb_linear_skinny(const void* x0, int ldx0, const void* w0, int ldw0,
                                const void* b0, void* y0, int ldy0, int N0, int K0, int act0, float arg0, int f32_0, int acc0,
                                const void* x1, int ldx1, const void* w1, int ldw1,
                                const void* b1, void* y1, int ldy1, int N1, int K1, int act1, float arg1, int f32_1, int acc1,
                                int M, void* stream) {
  if (M <= 0 || M > 16) return -1;
  SkinnyArgs a = {};
  a.M = M;
  int rc = skinny_problem(a.p[0], x0, ldx0, w0, ldw0, b0, y0, ldy0, N0, K0, act0, arg0, f32_0, acc0);
  if (rc != 0) return rc;
  int count = 1;
  if (x1 != nullptr) {
    rc = skinny_problem(a.p[1], x1, ldx1, w1, ldw1, b1, y1, ldy1, N1, K1, act1, arg1, f32_1, acc1);
    if (rc != 0) return rc;
    count = 2;
  }
  return launch_skinny_m(a, count, K0, static_cast<cudaStream_t>(stream));
}
