// fp32 linear layer Y[M, N] = act(X[M, K] . W[N, K]^T + bias[N]) on the FMA units, for serving a model in
// full 32-bit precision: 64 x 64 tiles, 4 x 4 outputs per thread, operands staged in shared memory.
// Grouped: the rows of x come in blocks of which each has a weight of its own (experts).
#include "ragged.cuh"

namespace cb {

constexpr int LT = 64, LK = 16;
enum : int { ACT_NONE = 0, ACT_RELU2 = 4, ACT_SOFTCAP = 5, ACT_GELU_ERF = 6, ACT_GLU = 7 };

__global__ void __launch_bounds__(256)
linear_f32_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, int ldw,
                  const float* __restrict__ bias, float* __restrict__ y, int ldy, int M, int N,
                  int K, int act, float act_arg, float limit, float shift, int accumulate,
                  const int* __restrict__ block_expert, int block_rows) {
  __shared__ float sx[LK][LT + 4], sw[LK][LT + 4];
  const int m0 = blockIdx.y * LT, n0 = blockIdx.x * LT;
  if (block_expert != nullptr) {
    const int e = block_expert[m0 / block_rows];
    if (e < 0) return;
    w += static_cast<size_t>(e) * N * ldw;
  }
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const int lr = threadIdx.x / 4, lc = (threadIdx.x % 4) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += LK) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (k0 + lc < K) {                              // K is a multiple of 4
      if (m0 + lr < M) a = *reinterpret_cast<const float4*>(x + static_cast<size_t>(m0 + lr) * ldx + k0 + lc);
      if (n0 + lr < N) b = *reinterpret_cast<const float4*>(w + static_cast<size_t>(n0 + lr) * ldw + k0 + lc);
    }
    __syncthreads();
    sx[lc][lr] = a.x; sx[lc + 1][lr] = a.y; sx[lc + 2][lr] = a.z; sx[lc + 3][lr] = a.w;
    sw[lc][lr] = b.x; sw[lc + 1][lr] = b.y; sw[lc + 2][lr] = b.z; sw[lc + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < LK; ++k) {
      const float4 u = *reinterpret_cast<const float4*>(&sx[k][ty * 4]);
      const float4 v = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float uu[4] = {u.x, u.y, u.z, u.w}, vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += uu[i] * vv[j];
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
    if (act == ACT_GLU) {                   // columns alternate: one result of every two
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = n0 + tx * 4 + j;
        if (n >= N) continue;
        const float g = fminf(acc[i][j] + (bias != nullptr ? bias[n] : 0.f), limit);
        const float u = fminf(fmaxf(acc[i][j + 1] + (bias != nullptr ? bias[n + 1] : 0.f), -limit), limit);
        y[static_cast<size_t>(m) * ldy + n / 2] = g * (u + shift) / (1.0f + expf(-act_arg * g));
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j];
      if (bias != nullptr) v += bias[n];
      if (act == ACT_GELU_ERF) {
        v = gelu_erf(v);
      } else if (act == ACT_RELU2) {
        v = fmaxf(v, 0.f);
        v *= v;
      } else if (act == ACT_SOFTCAP) {
        v = act_arg * tanhf(v / act_arg);
      }
      float* dst = y + static_cast<size_t>(m) * ldy + n;
      *dst = accumulate ? *dst + v : v;
    }
  }
}

}  // namespace cb

extern "C" int cb_linear_f32(const float* x, int ldx, const float* w, int ldw,
                             const float* bias, float* y, int ldy, int M, int N, int K, int act, float act_arg, int accumulate,
                             void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || K % 4 || ldx % 4 || ldw % 4) return -1;
  dim3 grid((N + cb::LT - 1) / cb::LT, (M + cb::LT - 1) / cb::LT);
  if (grid.y > 65535) return -1;
  cb::linear_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      x, ldx, w, ldw, bias, y, ldy, M, N, K, act, act_arg, 0.f, 0.f, accumulate, nullptr, 0);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

// block_expert[b]: which of the weights [experts, N, K] block b of block_rows (a multiple of 64) rows takes
// (-1: none, they are left alone); null: one weight.  glu: alternating columns g, u make one (clamped_glu).
extern "C" int cb_linear_f32_grouped(const float* x, int ldx, const float* w, int ldw, const float* bias,
                                     const int* block_expert, int block_rows, float* y, int ldy, int M, int N, int K,
                                     int glu, float slope, float limit, float shift, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || K % 4 || ldx % 4 || ldw % 4 || (glu && N % 2)) return -1;
  if (block_expert != nullptr && (block_rows < cb::LT || block_rows % cb::LT || M % block_rows)) return -1;
  dim3 grid((N + cb::LT - 1) / cb::LT, (M + cb::LT - 1) / cb::LT);
  if (grid.y > 65535) return -1;
  cb::linear_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      x, ldx, w, ldw, bias, y, ldy, M, N, K, glu ? cb::ACT_GLU : cb::ACT_NONE, slope, limit, shift, 0, block_expert,
      block_rows);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
