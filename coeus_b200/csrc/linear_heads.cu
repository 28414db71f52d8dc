// A small linear layer per head, for a ragged batch's decoded rows:
//   Y[i, h, n] = sum_k X[i, h, k] W[h, n, k]            (optionally times sigmoid(gate[i, h, n]))
// used to bring queries into the latent space of a compressed key/value cache and to bring the
// attention's result back out of it.  bf16: mma m16n8k16 with 16 rows of X against 16 columns per
// warp; every lane reads 32 consecutive bytes per 64-wide slice of k on both sides (the contraction
// index is permuted alike), so the fragments come straight from global memory.  fp32: one output
// column per thread.
#include "ragged.cuh"

namespace cb {

struct HeadsArgs {
  const void* x;           // row i: x + (x_rows ? x_rows[i] : i) * ldx, head h at h * x_head
  const void* w;           // [heads, N, ldw]
  void* y;                 // row i: y + (y_rows ? y_rows[i] : i) * ldy, head h at h * y_head
  const int* x_rows;
  const int* y_rows;
  const void* gate;        // like y, pitch ldg, heads y_head apart; or null
  int ldx, x_head, ldw, ldy, y_head, ldg;
  int M, N, K;
};

constexpr int LH_WARPS = 4;
constexpr int LH_COLS = LH_WARPS * 16;

// SPLIT: the warps of a block share 16 columns and take the slices of k in turn; else 16 columns each
template <bool SPLIT>
__global__ void __launch_bounds__(LH_WARPS * 32) linear_heads_kernel(const HeadsArgs p) {
  using bf16 = __nv_bfloat16;
  __shared__ float red[SPLIT ? LH_WARPS : 1][8][32];
  const int h = blockIdx.y, m0 = blockIdx.z * 16, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = SPLIT ? blockIdx.x * 16 : blockIdx.x * LH_COLS + warp * 16;
  if (!SPLIT && n0 >= p.N) return;
  const int r = lane >> 2, t = lane & 3;
  const bf16* xp[2];
  const bf16* wp[2];
#pragma unroll
  for (int j = 0; j < 2; ++j) {             // rows and columns past the end repeat the last one
    const int i = min(m0 + r + 8 * j, p.M - 1);
    xp[j] = static_cast<const bf16*>(p.x) +
            static_cast<size_t>(p.x_rows != nullptr ? p.x_rows[i] : i) * p.ldx + h * p.x_head + t * 16;
    wp[j] = static_cast<const bf16*>(p.w) +
            (static_cast<size_t>(h) * p.N + min(n0 + 8 * j + r, p.N - 1)) * p.ldw + t * 16;
  }
  float acc[2][4] = {};
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  constexpr int STEP = SPLIT ? 64 * LH_WARPS : 64;
#pragma unroll 2
  for (int k0 = SPLIT ? warp * 64 : 0; k0 < p.K; k0 += STEP) {
    uint4 a[2][2], b[2][2];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const bool in = k0 + t * 16 + v * 8 < p.K;
        a[j][v] = in ? *reinterpret_cast<const uint4*>(xp[j] + k0 + v * 8) : zero;
        b[j][v] = in ? *reinterpret_cast<const uint4*>(wp[j] + k0 + v * 8) : zero;
      }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const uint32_t lo[4] = {a[0][v].x, a[1][v].x, a[0][v].y, a[1][v].y};
        const uint32_t hi[4] = {a[0][v].z, a[1][v].z, a[0][v].w, a[1][v].w};
        mma_bf16(acc[j], lo, b[j][v].x, b[j][v].y);
        mma_bf16(acc[j], hi, b[j][v].z, b[j][v].w);
      }
  }
  if constexpr (SPLIT) {
#pragma unroll
    for (int j = 0; j < 8; ++j) red[warp][j][lane] = acc[j / 4][j % 4];
    __syncthreads();
    if (warp != 0) return;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < LH_WARPS; ++w) v += red[w][j][lane];
      acc[j / 4][j % 4] = v;
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int i = m0 + r + 8 * e;
    if (i >= p.M) continue;
    const int row = p.y_rows != nullptr ? p.y_rows[i] : i;
    bf16* dst = static_cast<bf16*>(p.y) + static_cast<size_t>(row) * p.ldy + h * p.y_head;
    const bf16* g = p.gate == nullptr ? nullptr
        : static_cast<const bf16*>(p.gate) + static_cast<size_t>(row) * p.ldg + h * p.y_head;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int n = n0 + 8 * j + t * 2 + c;
        if (n >= p.N) continue;
        float v = acc[j][e * 2 + c];
        if (g != nullptr) v *= sigmoidf_(__bfloat162float(g[n]));
        dst[n] = __float2bfloat16(v);
      }
  }
}

__global__ void __launch_bounds__(128) linear_heads_f32_kernel(const HeadsArgs p) {
  extern __shared__ float sx[];
  const int h = blockIdx.y, i = blockIdx.z;
  const float* x = static_cast<const float*>(p.x) +
                   static_cast<size_t>(p.x_rows != nullptr ? p.x_rows[i] : i) * p.ldx + h * p.x_head;
  for (int k = threadIdx.x; k < p.K; k += blockDim.x) sx[k] = x[k];
  __syncthreads();
  const int n = blockIdx.x * blockDim.x + threadIdx.x;
  if (n >= p.N) return;
  const float* w = static_cast<const float*>(p.w) + (static_cast<size_t>(h) * p.N + n) * p.ldw;
  float v = 0.f;
  for (int k = 0; k < p.K; k += 4) {        // K is a multiple of 8
    const float4 f = *reinterpret_cast<const float4*>(w + k);
    v += f.x * sx[k] + f.y * sx[k + 1] + f.z * sx[k + 2] + f.w * sx[k + 3];
  }
  const int row = p.y_rows != nullptr ? p.y_rows[i] : i;
  if (p.gate != nullptr)
    v *= sigmoidf_(static_cast<const float*>(p.gate)[static_cast<size_t>(row) * p.ldg + h * p.y_head + n]);
  static_cast<float*>(p.y)[static_cast<size_t>(row) * p.ldy + h * p.y_head + n] = v;
}

}  // namespace cb

using namespace cb;

extern "C" int cb_linear_heads(const void* x, int ldx, int x_head, const int* x_rows, const void* w,
                               int ldw, void* y, int ldy, int y_head, const int* y_rows,
                               const void* gate, int ldg, int heads, int M, int N, int K, int f32,
                               void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || heads <= 0 || heads > 65535) return -1;
  if (K % 8 || ldx % 8 || x_head % 8 || ldw % 8 || ldw < K) return -2;
  if ((reinterpret_cast<uintptr_t>(x) & 15u) || (reinterpret_cast<uintptr_t>(w) & 15u)) return -3;
  HeadsArgs p;
  p.x = x; p.w = w; p.y = y; p.x_rows = x_rows; p.y_rows = y_rows; p.gate = gate;
  p.ldx = ldx; p.x_head = x_head; p.ldw = ldw; p.ldy = ldy; p.y_head = y_head; p.ldg = ldg;
  p.M = M; p.N = N; p.K = K;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) {
    if (K * 4 > 48 * 1024) return -1;
    for (int i0 = 0; i0 < M; i0 += 65535) {
      HeadsArgs q = p;
      q.M = min(M - i0, 65535);
      if (x_rows != nullptr) q.x_rows = x_rows + i0;
      else q.x = static_cast<const float*>(x) + static_cast<size_t>(i0) * ldx;
      if (y_rows != nullptr) q.y_rows = y_rows + i0;
      else {
        q.y = static_cast<float*>(y) + static_cast<size_t>(i0) * ldy;
        if (gate != nullptr) q.gate = static_cast<const float*>(gate) + static_cast<size_t>(i0) * ldg;
      }
      linear_heads_f32_kernel<<<dim3((N + 127) / 128, heads, q.M), 128, K * 4, st>>>(q);
    }
  } else {
    const int tiles = (M + 15) / 16;
    if (tiles > 65535) return -1;
    if (K >= 64 * LH_WARPS)
      linear_heads_kernel<true><<<dim3((N + 15) / 16, heads, tiles), LH_WARPS * 32, 0, st>>>(p);
    else
      linear_heads_kernel<false><<<dim3((N + LH_COLS - 1) / LH_COLS, heads, tiles), LH_WARPS * 32, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
