// The state-space recurrence with one decay per head, over a ragged batch.  Per head, with the state
// S [state, vdim] in fp32 carried from token to token (B and C are shared by the heads of a group):
//   dt = softplus(dt_raw + dt_bias);   S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x
//
//   step kernel    token by token on the FMA units: everything in fp32, and short entries
//   chunk kernel   bf16 prompts: 64 tokens at a time as matrix products (ssd_chunk.cu)
//   gated norm     y silu(z), RMS norm in equal parts, weight
#include "ssd.cuh"

namespace cb {

// ------------------------------------------------------------------------------ step kernel
// A block takes one (entry, head) and 64 columns: a thread has four columns and NR = N / 8 rows.
template <typename T, int NR>
__global__ void __launch_bounds__(128) ssd_step_kernel(const Ssd p) {
  __shared__ float red[2][4][64];
  const int e = p.entry[blockIdx.y], h = blockIdx.x % p.heads, col0 = blockIdx.x / p.heads * 64;
  const int row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e], g = h / (p.heads / p.groups);
  const int c = threadIdx.x & 15, n0 = (threadIdx.x >> 4) * NR, warp = threadIdx.x >> 5;
  const int col = col0 + c * 4;
  const bool in = col < p.Pp;
  float* st = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.N * p.Pp + col;
  float S[NR][4];
  const bool has = p.e.pos0[e] > 0 && in;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    if (has && n0 + i < p.N) {
      load_vec<4>(st + static_cast<size_t>(n0 + i) * p.Pp, S[i]);
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) S[i][k] = 0.f;
    }
  }
  const float rate = expf(p.A_log[h]), bias = p.dt_bias[h], D = p.D[h];
  const bool vec = NR % 4 == 0 && p.N == 8 * NR && p.boff % 4 == 0 && p.coff % 4 == 0;
  for (int t = 0; t < len; ++t) {
    const T* u = static_cast<const T*>(p.u) + static_cast<size_t>(row0 + t) * p.ldu;
    const float dt = ssd_dt(to_f32(static_cast<const T*>(p.dt)[static_cast<size_t>(row0 + t) * p.lddt + h]), bias);
    const float a = expf(-rate * dt);
    float x[4], w[4], y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      x[k] = col + k < p.P ? to_f32(u[h * p.P + col + k]) : 0.f;
      w[k] = dt * x[k];
    }
    const T* B = u + p.boff + g * p.N + n0;
    const T* C = u + p.coff + g * p.N + n0;
    float b[4], cc[4];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      if (vec) {
        if (i % 4 == 0) {
          load_vec<4>(B + i, b);
          load_vec<4>(C + i, cc);
        }
      } else {
        const bool ok = n0 + i < p.N;
        b[i % 4] = ok ? to_f32(B[i]) : 0.f;
        cc[i % 4] = ok ? to_f32(C[i]) : 0.f;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        S[i][k] = a * S[i][k] + b[i % 4] * w[k];
        y[k] += cc[i % 4] * S[i][k];
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) y[k] += __shfl_xor_sync(0xffffffffu, y[k], 16);
    float (*r)[64] = red[t & 1];
    if ((threadIdx.x & 16) == 0) {
#pragma unroll
      for (int k = 0; k < 4; ++k) r[warp][c * 4 + k] = y[k];
    }
    __syncthreads();
    if (threadIdx.x < 64 && col0 + static_cast<int>(threadIdx.x) < p.P) {
      const int k = threadIdx.x;
      const float xk = to_f32(u[h * p.P + col0 + k]);
      static_cast<T*>(p.y)[static_cast<size_t>(row0 + t) * p.ldy + h * p.P + col0 + k] =
          from_f32<T>(r[0][k] + r[1][k] + r[2][k] + r[3][k] + D * xk);
    }
  }
  if (!in) return;
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (n0 + i < p.N) store_vec<4>(st + static_cast<size_t>(n0 + i) * p.Pp, S[i]);
}

// One block per (row, part): y silu(z) / rms * weight.
template <typename T, int V>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(const T* __restrict__ y, int ldy, const T* __restrict__ z, int ldz,
                        const float* __restrict__ w, T* __restrict__ out, int ldo, int part, float eps) {
  __shared__ float red[32];
  const int row = blockIdx.x, c0 = blockIdx.y * part;
  const T* yp = y + static_cast<size_t>(row) * ldy + c0;
  const T* zp = z + static_cast<size_t>(row) * ldz + c0;
  auto act = [](float a, float b) {
    if constexpr (sizeof(T) == 2) return a * __fdividef(b, 1.0f + __expf(-b));
    else return a * (b / (1.0f + expf(-b)));
  };
  constexpr int KEEP = 2;
  float keep[KEEP][V], s = 0.f;
  auto value = [&](int c, float* f) {
    float b[V];
    load_vec<V>(yp + c, f);
    load_vec<V>(zp + c, b);
#pragma unroll
    for (int k = 0; k < V; ++k) f[k] = act(f[k], b[k]);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c >= part) continue;
    value(c, keep[i]);
#pragma unroll
    for (int k = 0; k < V; ++k) s += keep[i][k] * keep[i][k];
  }
  for (int c = (threadIdx.x + KEEP * blockDim.x) * V; c < part; c += blockDim.x * V) {
    float f[V];
    value(c, f);
#pragma unroll
    for (int k = 0; k < V; ++k) s += f[k] * f[k];
  }
  s = block_sum(s, red);
  const float rs = 1.0f / sqrtf(s / part + eps);
  T* dst = out + static_cast<size_t>(row) * ldo + c0;
  auto put = [&](int c, float* f) {
    float g[V];
    load_vec<V>(w + c0 + c, g);
#pragma unroll
    for (int k = 0; k < V; ++k) f[k] *= rs * g[k];
    store_vec<V>(dst + c, f);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < part) put(c, keep[i]);
  }
  for (int c = (threadIdx.x + KEEP * blockDim.x) * V; c < part; c += blockDim.x * V) {
    float f[V];
    value(c, f);
    put(c, f);
  }
}

template <typename T>
static int launch_step(const Ssd& p, int n, cudaStream_t st) {
  dim3 grid(p.heads * ((p.P + 63) / 64), n);
  if (p.N <= 32) ssd_step_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else if (p.N <= 64) ssd_step_kernel<T, 8><<<grid, 128, 0, st>>>(p);
  else if (p.N <= 128) ssd_step_kernel<T, 16><<<grid, 128, 0, st>>>(p);
  else ssd_step_kernel<T, 32><<<grid, 128, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
static int launch_norm(const void* y, int ldy, const void* z, int ldz, const float* w, void* out, int ldo,
                       int rows, int inner, int parts, float eps, cudaStream_t st) {
  const int part = inner / parts;
  const bool vec = part % 8 == 0 && ldy % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0;
  const int threads = min(256, ((vec ? part / 8 : part) + 31) / 32 * 32);
  dim3 grid(rows, parts);
  if (vec)
    gated_group_norm_kernel<T, 8><<<grid, threads, 0, st>>>(static_cast<const T*>(y), ldy, static_cast<const T*>(z),
                                                           ldz, w, static_cast<T*>(out), ldo, part, eps);
  else
    gated_group_norm_kernel<T, 1><<<grid, threads, 0, st>>>(static_cast<const T*>(y), ldy, static_cast<const T*>(z),
                                                           ldz, w, static_cast<T*>(out), ldo, part, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

using namespace cb;

extern "C" int cb_ssd_step(const void* u, int ldu, int boff, int coff, const void* dt, int lddt,
                           const float* dt_bias, const float* A_log, const float* D, float* state,
                           void* y, int ldy, int heads, int groups, int N, int P, int Pp,
                           const int* slot, const int* row0, const int* len, const int* pos0,
                           const int* entry, int n, int f32, void* stream) {
  Ssd p;
  const int rc = fill_ssd(p, u, ldu, boff, coff, dt, lddt, dt_bias, A_log, D, state, y, ldy, heads, groups,
                          N, P, Pp, slot, row0, len, pos0, entry);
  if (rc != 0) return rc;
  if (n <= 0 || n > 65535 || ldu % 4) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_step<float>(p, n, st) : launch_step<__nv_bfloat16>(p, n, st);
}

extern "C" int cb_gated_group_norm(const void* y, int ldy, const void* z, int ldz, const float* w,
                                   void* out, int ldo, int rows, int inner, int parts, float eps,
                                   int f32, void* stream) {
  if (rows <= 0 || parts < 1 || parts > 65535 || inner % parts) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_norm<float>(y, ldy, z, ldz, w, out, ldo, rows, inner, parts, eps, st)
             : launch_norm<__nv_bfloat16>(y, ldy, z, ldz, w, out, ldo, rows, inner, parts, eps, st);
}
