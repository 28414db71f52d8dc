// Row-wise kernels of the ragged serving path, whose residual stream is fp32: embedding lookup
// with a norm, RMS norm with one or two weights (the parallel block normalises the same stream
// twice), the per-step table of rotary angles, the gated per-head norm behind a recurrent mixer,
// and the arg-max of fp32 logits.
#include "ragged.cuh"

namespace cb {

constexpr int ROW_THREADS = 256;

// out row r: rms_norm(embed[tokens[r]]) * w * scale (without w: embed[tokens[r]] * scale), fp32; columns width .. ld-1 are zero.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
embed_norm_kernel(const int* __restrict__ tokens, const T* __restrict__ embed, int lde, int vocab,
                  const float* __restrict__ w, float* __restrict__ x, int ld, int width, float eps, float scale,
                  int* status) {
  __shared__ float red[32];
  const int r = blockIdx.x;
  int tok = tokens[r];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0) record_status(status, ST_BOUNDS, r);
    tok = 0;
  }
  const T* src = embed + static_cast<size_t>(tok) * lde;
  float s = 0.f;
  for (int c = threadIdx.x; c < width; c += ROW_THREADS) {
    const float v = to_f32(src[c]);
    s += v * v;
  }
  s = block_sum(s, red);
  float rs = 1.0f / sqrtf(s / width + eps);
  float* dst = x + static_cast<size_t>(r) * ld;
  for (int c = threadIdx.x; c < ld; c += ROW_THREADS) {
    float v = 0.f;
    if (c < width) {
      v = to_f32(src[c]);
      v = (w != nullptr ? v * rs * w[c] : v) * scale;
    }
    dst[c] = v;
  }
}

// y1 = norm(x[rows[r]]) * w1 and, when y2 is given, y2 = norm(..) * w2.  ld is a multiple of 8 and
// x's padding columns are zero.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
rms_rows_kernel(const float* __restrict__ x, int ldx, const int* __restrict__ rows,
                const float* __restrict__ w1, T* __restrict__ y1, const float* __restrict__ w2,
                T* __restrict__ y2, int ldy, int width, float eps) {
  __shared__ float red[32];
  const int r = blockIdx.x;
  const float* src = x + static_cast<size_t>(rows != nullptr ? rows[r] : r) * ldx;
  constexpr int KEEP = 4;                       // vectors of 8 kept in registers per thread
  float keep[KEEP][8];
  const int nv = ldx / 8;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * ROW_THREADS;
    if (v < nv) {
      load_vec<8>(src + v * 8, keep[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) s += keep[i][e] * keep[i][e];
    }
  }
  for (int v = threadIdx.x + KEEP * ROW_THREADS; v < nv; v += ROW_THREADS) {
    float f[8];
    load_vec<8>(src + v * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) s += f[e] * f[e];
  }
  s = block_sum(s, red);
  const float rs = 1.0f / sqrtf(s / width + eps);
  for (int i = 0, v = threadIdx.x; v < nv; ++i, v += ROW_THREADS) {
    float f[8], g[8], o[8];
    if (i < KEEP) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k)
        if (k == i) {
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = keep[k][e];
        }
    } else {
      load_vec<8>(src + v * 8, f);
    }
    load_vec<8>(w1 + v * 8, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = f[e] * rs * g[e];
    store_vec<8>(y1 + static_cast<size_t>(r) * ldy + v * 8, o);
    if (y2 != nullptr) {
      load_vec<8>(w2 + v * 8, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = f[e] * rs * g[e];
      store_vec<8>(y2 + static_cast<size_t>(r) * ldy + v * 8, o);
    }
  }
}

// table[r][i] = (cos, sin) of pos[r] * inv_freq[i]
__global__ void rope_table_kernel(const int* __restrict__ pos, const float* __restrict__ inv_freq,
                                  int n, int half, float2* __restrict__ table) {
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= n * half) return;
  float s, c;
  sincosf(static_cast<float>(pos[idx / half]) * inv_freq[idx % half], &s, &c);
  table[idx] = make_float2(c, s);
}

// One warp per (row, head): y = o / rms(o) * w * sigmoid(gate), o fp32, gate and y in T.
template <typename T>
__global__ void __launch_bounds__(128)
gated_head_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ldg,
                       const float* __restrict__ w, T* __restrict__ y, int ldy, int rows, int heads,
                       int vdim, float eps, bool vec) {
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= rows * heads) return;
  const int r = unit / heads, h = unit % heads;
  const float* src = o + static_cast<size_t>(unit) * vdim;
  const T* gp = gate + static_cast<size_t>(r) * ldg + h * vdim;
  T* dst = y + static_cast<size_t>(r) * ldy + h * vdim;
  float s = 0.f;
  if (vec) {                                  // four channels per lane, at most 256 in all
    float f[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (lane + 32 * i) * 4;
      if (c < vdim) {
        load_vec<4>(src + c, f[i]);
        s += f[i][0] * f[i][0] + f[i][1] * f[i][1] + f[i][2] * f[i][2] + f[i][3] * f[i][3];
      }
    }
    s = warp_sum(s);
    const float rs = 1.0f / sqrtf(s / vdim + eps);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int c = (lane + 32 * i) * 4;
      if (c < vdim) {
        float g[4], k[4];
        load_vec<4>(gp + c, g);
        load_vec<4>(w + c, k);
#pragma unroll
        for (int x = 0; x < 4; ++x) f[i][x] = f[i][x] * rs * k[x] * sigmoidf_(g[x]);
        store_vec<4>(dst + c, f[i]);
      }
    }
    return;
  }
  for (int c = lane; c < vdim; c += 32) s += src[c] * src[c];
  s = warp_sum(s);
  const float rs = 1.0f / sqrtf(s / vdim + eps);
  for (int c = lane; c < vdim; c += 32)
    dst[c] = from_f32<T>(src[c] * rs * w[c] * sigmoidf_(to_f32(gp[c])));
}

// y <- cap * tanh(y / cap)
__global__ void softcap_kernel(float* __restrict__ y, int ld, int cols, float cap) {
  float* row = y + static_cast<size_t>(blockIdx.y) * ld;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c < cols) row[c] = cap * tanhf(row[c] / cap);
}

__global__ void argmax_f32_kernel(const float* __restrict__ logits, int ld, int V,
                                  int64_t* __restrict__ out) {
  __shared__ float s_val[32];
  __shared__ int s_idx[32];
  const float* row = logits + static_cast<size_t>(blockIdx.x) * ld;
  float best = -INFINITY;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    const float v = row[i];
    if (v > best || bi == 0x7fffffff) { best = v; bi = i; }
  }
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) { s_val[warp] = best; s_idx[warp] = bi; }
  __syncthreads();
  if (warp == 0) {
    best = s_val[lane];                     // the block has 32 warps
    bi = s_idx[lane];
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (lane == 0) out[blockIdx.x] = bi;
  }
}

}  // namespace cb

using namespace cb;
#define CB_RC() (cudaGetLastError() == cudaSuccess ? 0 : -3)

extern "C" int cb_embed_norm(const int* tokens, const void* embed, int lde, int vocab,
                             const float* w, float* x, int ld, int rows, int width, float eps, float scale,
                             int f32, int* status, void* stream) {
  if (rows <= 0 || width > ld || width > lde) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    embed_norm_kernel<float><<<rows, ROW_THREADS, 0, st>>>(
        tokens, static_cast<const float*>(embed), lde, vocab, w, x, ld, width, eps, scale, status);
  else
    embed_norm_kernel<__nv_bfloat16><<<rows, ROW_THREADS, 0, st>>>(
        tokens, static_cast<const __nv_bfloat16*>(embed), lde, vocab, w, x, ld, width, eps, scale, status);
  return CB_RC();
}

extern "C" int cb_rms_rows(const float* x, int ldx, const int* rows, const float* w1, void* y1,
                           const float* w2, void* y2, int ldy, int n, int width, float eps, int f32,
                           void* stream) {
  if (n <= 0 || (ldx % 8) != 0 || (ldy % 8) != 0 || ldy < ldx) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    rms_rows_kernel<float><<<n, ROW_THREADS, 0, st>>>(x, ldx, rows, w1, static_cast<float*>(y1), w2,
                                                      static_cast<float*>(y2), ldy, width, eps);
  else
    rms_rows_kernel<__nv_bfloat16><<<n, ROW_THREADS, 0, st>>>(
        x, ldx, rows, w1, static_cast<__nv_bfloat16*>(y1), w2, static_cast<__nv_bfloat16*>(y2), ldy,
        width, eps);
  return CB_RC();
}

extern "C" int cb_rope_table(const int* pos, const float* inv_freq, int n, int half, void* table,
                             void* stream) {
  if (n <= 0 || half <= 0) return -1;
  rope_table_kernel<<<(n * half + 255) / 256, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      pos, inv_freq, n, half, static_cast<float2*>(table));
  return CB_RC();
}

extern "C" int cb_gated_head_norm(const float* o, const void* gate, int ldg, const float* w, void* y,
                                  int ldy, int rows, int heads, int vdim, float eps, int f32,
                                  void* stream) {
  if (rows <= 0) return -1;
  const int blocks = (rows * heads + 3) / 4;
  const bool vec = vdim % 4 == 0 && vdim <= 256 && ldg % 4 == 0 && ldy % 4 == 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    gated_head_norm_kernel<float><<<blocks, 128, 0, st>>>(
        o, static_cast<const float*>(gate), ldg, w, static_cast<float*>(y), ldy, rows, heads, vdim, eps,
        vec);
  else
    gated_head_norm_kernel<__nv_bfloat16><<<blocks, 128, 0, st>>>(
        o, static_cast<const __nv_bfloat16*>(gate), ldg, w, static_cast<__nv_bfloat16*>(y), ldy, rows,
        heads, vdim, eps, vec);
  return CB_RC();
}

extern "C" int cb_argmax_f32(const float* logits, int ld, int B, int V, int64_t* out, void* stream) {
  argmax_f32_kernel<<<B, 1024, 0, static_cast<cudaStream_t>(stream)>>>(logits, ld, V, out);
  return CB_RC();
}

extern "C" int cb_softcap(float* y, int ld, int rows, int cols, float cap, void* stream) {
  if (rows <= 0 || cols <= 0) return -1;
  for (int r = 0; r < rows; r += 65535) {
    dim3 grid((cols + 255) / 256, min(rows - r, 65535));
    softcap_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
        y + static_cast<size_t>(r) * ld, ld, cols, cap);
  }
  return CB_RC();
}
