// One pass over the fp32 residual stream between two sublayers of a decoder that normalises before
// and after each of them:
//   v = y + bias;  v = v / rms(v) * post          (the sublayer's result; each part optional)
//   x = x + v                                     (written to another buffer than it is read from)
//   h = x / rms(x) * gain                         (what the next sublayer reads, in T)
//   h = h + (h_before - h) * shift                (token shift: h_before is the previous token's h)
// y may also be, or get added, a sum of weighted rows of another buffer: the results of the experts a
// token uses.  Gains are one number or a vector.  x can also be written in T to one or two places (operands of a
// product over [x | x0]).
//
// Without a shift a block takes one row.  With it a block takes a tile of consecutive tokens of one
// entry, keeps the h of the token before in registers and starts with the row in front of the tile:
// recomputed from x and y (hence the separate output buffer), or the slot's state, or zeros at a
// sequence's start.  The block of an entry's first tile alone reads the state, and replaces it at
// its end.
#include "ragged.cuh"

namespace cb {

constexpr int SHIFT_TILE = 16;     // tokens per block with a shift (the convolutions' tile)

struct AddNorm {
  const float* x;          // [rows, ld] or null (then x = v)
  const void* y;           // [rows, ldy] or null
  const float* bias;       // [width ..] or null: added to y
  const float* post;       // gain of the norm of v, or null: no norm
  int post_vec;
  float* x_out;            // [rows, ld] or null
  int ld, ldy;
  const float* gain;       // gain of h, or null: no h
  int gain_vec;
  void* h;                 // [blocks or rows, ldh]
  int ldh;
  void* cast[2];           // x in T, pitch ldc; or null
  int ldc;
  const float* shift;      // [ld] or null
  float* before;           // [slots, ld] the previous token's h
  const int* rows;         // without a shift: row of block b (null: b)
  Entries e;
  const int* tile_entry;
  const int* tile_off;
  const void* spread;      // rows in T, pitch lds, or null: y + sum_k weight[row, k] * spread[slot[row, k]]
  int lds, top;
  const int* spread_slot;  // [rows, top]
  const float* spread_weight;
  int width;
  float eps;
};

template <typename T, typename Y, int KEEP>
__global__ void __launch_bounds__(512) add_norm_kernel(const AddNorm p) {
  __shared__ float red[32];
  const int nv = p.ld / 8;
  // x of one row after the sublayer's result is added (f), and its normalised form (f again)
  auto stream = [&](int row, float (*f)[8], bool store) {
    float s = 0.f;
    const bool added = p.y != nullptr || p.spread != nullptr;
    if (added) {
      const Y* yp = static_cast<const Y*>(p.y) + static_cast<size_t>(row) * p.ldy;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= nv) continue;
        if (p.y != nullptr) {
          load_vec<8>(yp + v * 8, f[i]);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) f[i][e] = 0.f;
        }
        if (p.spread != nullptr) {
#pragma unroll 4
          for (int k = 0; k < p.top; ++k) {
            const size_t at = static_cast<size_t>(row) * p.top + k;
            const float w = p.spread_weight[at];
            float g[8];
            load_vec<8>(static_cast<const T*>(p.spread) + static_cast<size_t>(p.spread_slot[at]) * p.lds + v * 8, g);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[i][e] += w * g[e];
          }
        }
        if (p.bias != nullptr) {
          float b[8];
          load_vec<8>(p.bias + v * 8, b);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[i][e] += b[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) s += f[i][e] * f[i][e];
      }
    }
    float xs[KEEP][8];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (p.x != nullptr && v < nv) load_vec<8>(p.x + static_cast<size_t>(row) * p.ld + v * 8, xs[i]);
      else
#pragma unroll
        for (int e = 0; e < 8; ++e) xs[i][e] = 0.f;
    }
    float rs = 1.f;
    if (added && p.post != nullptr) {
      s = block_sum(s, red);
      rs = 1.0f / sqrtf(s / p.width + p.eps);
      if (!p.post_vec) rs *= *p.post;
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= nv) continue;
      if (!added) {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[i][e] = xs[i][e];
      } else {
        float g[8];
        if (p.post != nullptr && p.post_vec) {
          load_vec<8>(p.post + v * 8, g);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) g[e] = 1.f;
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) f[i][e] = xs[i][e] + f[i][e] * rs * g[e];
      }
      if (store) {
        if (p.x_out != nullptr) store_vec<8>(p.x_out + static_cast<size_t>(row) * p.ld + v * 8, f[i]);
#pragma unroll
        for (int k = 0; k < 2; ++k)
          if (p.cast[k] != nullptr)
            store_vec<8>(static_cast<T*>(p.cast[k]) + static_cast<size_t>(row) * p.ldc + v * 8, f[i]);
      }
    }
    if (p.gain == nullptr) return;
    s = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      if (static_cast<int>(threadIdx.x + i * blockDim.x) >= nv) continue;
#pragma unroll
      for (int e = 0; e < 8; ++e) s += f[i][e] * f[i][e];
    }
    s = block_sum(s, red);
    rs = 1.0f / sqrtf(s / p.width + p.eps);
    if (!p.gain_vec) rs *= *p.gain;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= nv) continue;
      float g[8];
      if (p.gain_vec) {
        load_vec<8>(p.gain + v * 8, g);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) g[e] = 1.f;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[i][e] = f[i][e] * rs * g[e];
    }
  };

  float f[KEEP][8];
  if (p.shift == nullptr) {
    const int row = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x;
    stream(row, f, true);
    if (p.gain == nullptr) return;
    T* dst = static_cast<T*>(p.h) + static_cast<size_t>(blockIdx.x) * p.ldh;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nv) store_vec<8>(dst + v * 8, f[i]);
    }
    return;
  }
  const int e = p.tile_entry[blockIdx.x], off = p.tile_off[blockIdx.x];
  const int row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e];
  float* state = p.before + static_cast<size_t>(slot) * p.ld;
  float prev[KEEP][8];
  if (off > 0) {
    stream(row0 + off - 1, prev, false);
  } else {
    const bool has = p.e.pos0[e] > 0;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (has && v < nv) load_vec<8>(state + v * 8, prev[i]);
      else
#pragma unroll
        for (int k = 0; k < 8; ++k) prev[i][k] = 0.f;
    }
  }
  const int t1 = min(off + SHIFT_TILE, len);
  for (int t = off; t < t1; ++t) {
    stream(row0 + t, f, true);
    T* dst = static_cast<T*>(p.h) + static_cast<size_t>(row0 + t) * p.ldh;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= nv) continue;
      float a[8], o[8];
      load_vec<8>(p.shift + v * 8, a);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        o[k] = f[i][k] + (prev[i][k] - f[i][k]) * a[k];
        prev[i][k] = f[i][k];
      }
      store_vec<8>(dst + v * 8, o);
    }
  }
  if (off > 0) return;
  if (t1 < len) stream(row0 + len - 1, prev, false);
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nv) store_vec<8>(state + v * 8, prev[i]);
  }
}

template <typename T, typename Y>
static int launch_add_norm(const AddNorm& p, int blocks, cudaStream_t st) {
  const int nv = p.ld / 8;
  if (nv <= 512) {
    add_norm_kernel<T, Y, 1><<<blocks, (nv + 31) / 32 * 32, 0, st>>>(p);
  } else if (nv <= 1024) {
    add_norm_kernel<T, Y, 2><<<blocks, 512, 0, st>>>(p);
  } else {
    add_norm_kernel<T, Y, 4><<<blocks, 512, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

using namespace cb;

// blocks: rows (without a shift) or tiles (with it).  y_f32: y is fp32 although T is bf16.
extern "C" int cb_add_norm(const float* x, const void* y, const float* bias, const float* post,
                           int post_vec, float* x_out, int ld, int ldy, const float* gain,
                           int gain_vec, void* h, int ldh, void* cast0, void* cast1, int ldc,
                           const float* shift, float* before, const int* rows, const int* slot,
                           const int* row0, const int* len, const int* pos0, const int* tile_entry,
                           const int* tile_off, int blocks, int width, float eps, int f32, int y_f32,
                           const void* spread, int lds, const int* spread_slot,
                           const float* spread_weight, int top, void* stream) {
  if (blocks <= 0 || ld % 8 || width > ld || ld > 16384) return -1;
  if (y != nullptr && (ldy % 8 || ldy < ld)) return -2;
  if (gain != nullptr && (h == nullptr || ldh % 8 || ldh < ld)) return -2;
  if ((cast0 != nullptr || cast1 != nullptr) && (ldc % 8 || ldc < ld)) return -2;
  if (shift != nullptr && (gain == nullptr || before == nullptr || rows != nullptr)) return -2;
  if (shift != nullptr && x != nullptr && x == x_out) return -2;     // the row in front is read late
  if (spread != nullptr && (lds % 8 || lds < ld || top < 1 || spread_slot == nullptr || spread_weight == nullptr))
    return -2;
  AddNorm p;
  p.spread = spread; p.lds = lds; p.spread_slot = spread_slot; p.spread_weight = spread_weight; p.top = top;
  p.x = x; p.y = y; p.bias = bias; p.post = post; p.post_vec = post_vec; p.x_out = x_out;
  p.ld = ld; p.ldy = ldy; p.gain = gain; p.gain_vec = gain_vec; p.h = h; p.ldh = ldh;
  p.cast[0] = cast0; p.cast[1] = cast1; p.ldc = ldc; p.shift = shift; p.before = before;
  p.rows = rows; p.e.slot = slot; p.e.row0 = row0; p.e.len = len; p.e.pos0 = pos0;
  p.tile_entry = tile_entry; p.tile_off = tile_off; p.width = width; p.eps = eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return launch_add_norm<float, float>(p, blocks, st);
  return y_f32 ? launch_add_norm<__nv_bfloat16, float>(p, blocks, st)
               : launch_add_norm<__nv_bfloat16, __nv_bfloat16>(p, blocks, st);
}
