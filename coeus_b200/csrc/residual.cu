// One pass over the fp32 residual stream between two sublayers of a decoder that normalises before
// (and after) each of them:
//   v = y + bias;  v = v / rms(v) * post          (the sublayer's result; each part optional)
//   x = x + v * scale                             (written to another buffer than it is read from)
//   h = x / rms(x) * gain                         (what the next sublayer reads, in T; with a center:
//                                                  (x - mean) / deviation * gain + center)
//   h = h + (h_before - h) * shift                (token shift: h_before is the previous token's h)
//   h = h + conv(h)                               (or: a causal convolution over time on every channel)
// y may have a factor per row, and also be, or get added, a sum of weighted rows of another buffer: the
// results of the experts a token uses.  Gains are one number or a vector.  x can also be written in T to one or two places (operands of a
// product over [x | x0]).
//
// Without a shift a block takes one row.  With it a block takes a tile of consecutive tokens of one
// entry, keeps the h of the token before in registers and starts with the row in front of the tile:
// recomputed from x and y (hence the separate output buffer), or the slot's state, or zeros at a
// sequence's start.  The block of an entry's first tile alone reads the state, and replaces it at
// its end.
//
// With a convolution a block takes such a tile too, in two phases: its warps take the rows, and leave x and
// the rows' statistics; then its threads take the columns, walk along the rows and keep the last h in
// registers.  The rows in front of the tile go through shared memory.
#include "ragged.cuh"

namespace cb {

constexpr int CN_SMEM = 208 * 1024;
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
  const void* own;         // [rows, ldo] in T: stands for a spread row whose slot is negative, or null
  int ldo;
  const float* y_weight;   // [rows] or null
  const float* scale;      // [ld] or null
  const float* center;     // [ld] or null
  const float* taps;       // [n_taps, ld] or null; before is then [slots, n_taps - 1, ld]
  int n_taps;
  int width;
  float eps;
};

// Columns 8 v .. 8 v + 7 of a row of the sublayer's result, before its norm.
template <typename T, typename Y>
__device__ __forceinline__ void sublayer_result(const AddNorm& p, int row, int v, float* f) {
  if (p.y != nullptr) {
    load_vec<8>(static_cast<const Y*>(p.y) + static_cast<size_t>(row) * p.ldy + v * 8, f);
    if (p.y_weight != nullptr) {
      const float w = p.y_weight[row];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = 0.f;
  }
  if (p.spread != nullptr) {
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      const size_t at = static_cast<size_t>(row) * p.top + k;
      const float w = p.spread_weight[at];
      const int slot = p.spread_slot[at];
      const T* src = slot < 0 && p.own != nullptr
                         ? static_cast<const T*>(p.own) + static_cast<size_t>(row) * p.ldo
                         : static_cast<const T*>(p.spread) + static_cast<size_t>(max(slot, 0)) * p.lds;
      float g[8];
      load_vec<8>(src + v * 8, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += w * g[e];
    }
  }
  if (p.bias != nullptr) {
    float b[8];
    load_vec<8>(p.bias + v * 8, b);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] += b[e];
  }
}
// Sum of the squares of eight columns' distances from the mean, of those that the row has.
__device__ __forceinline__ float squares_about(const float* f, float mean, int col, int width) {
  float s = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    const float d = col + e < width ? f[e] - mean : 0.f;
    s += d * d;
  }
  return s;
}

template <typename T, typename Y, int KEEP>
__global__ void __launch_bounds__(512) add_norm_kernel(const AddNorm p) {
  __shared__ float red[32];
  const int nv = p.ld / 8;
  // x of one row after the sublayer's result is added (f), and its normalised form (f again)
  auto stream = [&](int row, float (*f)[8], bool store) {
    float s = 0.f;
    const bool added = p.y != nullptr || p.spread != nullptr;
    if (added) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= nv) continue;
        sublayer_result<T, Y>(p, row, v, f[i]);
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
        if (p.scale != nullptr) {
          float c[8];
          load_vec<8>(p.scale + v * 8, c);
#pragma unroll
          for (int e = 0; e < 8; ++e) g[e] *= c[e];
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
    float mean = 0.f;
    if (p.center != nullptr) {
      s = 0.f;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        if (static_cast<int>(threadIdx.x + i * blockDim.x) >= nv) continue;
#pragma unroll
        for (int e = 0; e < 8; ++e) s += f[i][e];           // zeros behind the width
      }
      mean = block_sum(s, red) / p.width;
    }
    s = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nv) s += squares_about(f[i], mean, v * 8, p.width);
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
      float c[8];
      if (p.center != nullptr) {
        load_vec<8>(p.center + v * 8, c);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) c[e] = 0.f;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[i][e] = (f[i][e] - mean) * rs * g[e] + c[e];
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

// ------------------------------------------------------------------------- with a convolution
constexpr int CN_THREADS = 256;
constexpr int CN_KEEP = 8;         // vectors of eight that a lane keeps of a row

struct RowStats {
  float mean, rs;
};

// One warp, one row: x with the sublayer's result to dst (not when the stream itself is the source and the
// same), and the row's statistics.
template <typename T, typename Y>
__device__ __forceinline__ RowStats conv_row(const AddNorm& p, int row, float* dst) {
  const int lane = threadIdx.x & 31, nv = p.ld / 8;
  const bool added = p.y != nullptr || p.spread != nullptr;
  const float* src = p.x + static_cast<size_t>(row) * p.ld;
  auto make = [&](int v, float* f) {
    if (added) {
      sublayer_result<T, Y>(p, row, v, f);
      if (p.scale != nullptr) {
        float c[8];
        load_vec<8>(p.scale + v * 8, c);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= c[e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = 0.f;
    }
    if (p.x != nullptr) {
      float a[8];
      load_vec<8>(src + v * 8, a);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += a[e];
    }
    if (dst != nullptr) store_vec<8>(dst + v * 8, f);
  };
  float f[CN_KEEP][8], s = 0.f;
#pragma unroll
  for (int i = 0; i < CN_KEEP; ++i) {
    const int v = lane + 32 * i;
    if (v >= nv) continue;
    make(v, f[i]);
#pragma unroll
    for (int e = 0; e < 8; ++e) s += f[i][e];
  }
  for (int v = lane + 32 * CN_KEEP; v < nv; v += 32) {
    float g[8];
    make(v, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) s += g[e];
  }
  RowStats r = {0.f, 0.f};
  if (p.center != nullptr) r.mean = warp_sum(s) / p.width;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < CN_KEEP; ++i) {
    const int v = lane + 32 * i;
    if (v < nv) s += squares_about(f[i], r.mean, v * 8, p.width);
  }
  const float* again = dst != nullptr ? dst : src;      // this lane's own writes
  for (int v = lane + 32 * CN_KEEP; v < nv; v += 32) {
    float g[8];
    load_vec<8>(again + v * 8, g);
    s += squares_about(g, r.mean, v * 8, p.width);
  }
  r.rs = 1.0f / sqrtf(warp_sum(s) / p.width + p.eps);
  return r;
}

// Columns of the norm's gain and center.
__device__ __forceinline__ void norm_vectors(const AddNorm& p, int v, float* g, float* c) {
  if (p.gain_vec) {
    load_vec<8>(p.gain + v * 8, g);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = *p.gain;
  }
  if (p.center != nullptr) {
    load_vec<8>(p.center + v * 8, c);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) c[e] = 0.f;
  }
}

// One warp, one row whose x was just left at f: its h instead.
__device__ __forceinline__ void norm_in_place(const AddNorm& p, float* row, RowStats r) {
  for (int v = threadIdx.x & 31; v < p.ld / 8; v += 32) {
    float f[8], g[8], c[8];
    load_vec<8>(row + v * 8, f);
    norm_vectors(p, v, g, c);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = (f[e] - r.mean) * r.rs * g[e] + c[e];
    store_vec<8>(row + v * 8, f);
  }
}

template <typename T, typename Y, int HIST>     // n_taps - 1 <= HIST
__global__ void __launch_bounds__(CN_THREADS) add_norm_conv_kernel(const AddNorm p) {
  extern __shared__ __align__(16) float halo[];          // [n_taps - 1, ld]: h in front of the tile
  __shared__ RowStats stats[SHIFT_TILE];
  const int back = p.n_taps - 1, nv = p.ld / 8;
  const int e = p.tile_entry[blockIdx.x], off = p.tile_off[blockIdx.x];
  const int row0 = p.e.row0[e], len = p.e.len[e];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = min(SHIFT_TILE, len - off);
  float* state = p.before + static_cast<size_t>(p.e.slot[e]) * back * p.ld;
  if (off == 0) {
    const bool has = p.e.pos0[e] > 0;
    for (int i = threadIdx.x; i < back * p.ld / 4; i += CN_THREADS)
      reinterpret_cast<float4*>(halo)[i] = has ? reinterpret_cast<const float4*>(state)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int i = warp - (off > 0 ? back : 0); i < n; i += CN_THREADS / 32) {
    const int row = row0 + off + i;
    if (i < 0) {
      float* dst = halo + (back + i) * p.ld;
      norm_in_place(p, dst, conv_row<T, Y>(p, row, dst));
    } else {
      const RowStats r = conv_row<T, Y>(p, row, p.x_out != nullptr ? p.x_out + static_cast<size_t>(row) * p.ld : nullptr);
      if (lane == 0) stats[i] = r;
    }
  }
  __syncthreads();
  const float* src = (p.x_out != nullptr ? p.x_out : p.x) + static_cast<size_t>(row0 + off) * p.ld;
  T* dst = static_cast<T*>(p.h) + static_cast<size_t>(row0 + off) * p.ldh;
  const bool all = off == 0 && n == len;                 // the state is what this tile leaves
  for (int v = threadIdx.x; v < nv; v += CN_THREADS) {
    float w[HIST + 1][8], prev[HIST][8], g[8], c[8];     // [d]: d tokens back; prev[d - 1]
    norm_vectors(p, v, g, c);
#pragma unroll
    for (int d = 0; d <= HIST; ++d) {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        w[d][k] = 0.f;
        if (d > 0) prev[d > 0 ? d - 1 : 0][k] = 0.f;
      }
      if (d <= back) {
        load_vec<8>(p.taps + static_cast<size_t>(back - d) * p.ld + v * 8, w[d]);
        if (d > 0) load_vec<8>(halo + (back - d) * p.ld + v * 8, prev[d > 0 ? d - 1 : 0]);
      }
    }
    if (all)                                             // tokens that stay in the state, moved on
      for (int k = 0; k < back - n; ++k) {
        float f[8];
        load_vec<8>(halo + (n + k) * p.ld + v * 8, f);
        store_vec<8>(state + static_cast<size_t>(k) * p.ld + v * 8, f);
      }
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
      float f[8], o[8];
      load_vec<8>(src + static_cast<size_t>(t) * p.ld + v * 8, f);
      const RowStats r = stats[t];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        f[k] = (f[k] - r.mean) * r.rs * g[k] + c[k];
        float a = w[0][k] * f[k];
#pragma unroll
        for (int d = 1; d <= HIST; ++d) a += w[d][k] * prev[d - 1][k];
        o[k] = f[k] + a;
#pragma unroll
        for (int d = HIST - 1; d > 0; --d) prev[d][k] = prev[d - 1][k];
        prev[0][k] = f[k];
      }
      store_vec<8>(dst + static_cast<size_t>(t) * p.ldh + v * 8, o);
      if (all && t >= n - back) store_vec<8>(state + static_cast<size_t>(t - n + back) * p.ld + v * 8, f);
    }
  }
  if (off > 0 || all) return;
  __syncthreads();                                       // the state has been read
  for (int k = warp; k < back; k += CN_THREADS / 32) {   // a longer entry's last tokens
    float* row = state + static_cast<size_t>(k) * p.ld;
    norm_in_place(p, row, conv_row<T, Y>(p, row0 + len - back + k, row));
  }
}

template <typename T, typename Y, int HIST>
static int launch_add_norm_conv(const AddNorm& p, int blocks, cudaStream_t st) {
  const int smem = (p.n_taps - 1) * p.ld * 4;
  static int set = 48 * 1024;
  if (smem > set) {
    if (cudaFuncSetAttribute(add_norm_conv_kernel<T, Y, HIST>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             CN_SMEM) != cudaSuccess)
      return -4;
    set = CN_SMEM;
  }
  add_norm_conv_kernel<T, Y, HIST><<<blocks, CN_THREADS, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, typename Y>
static int launch_add_norm(const AddNorm& p, int blocks, cudaStream_t st) {
  if (p.taps != nullptr)
    return p.n_taps <= 4 ? launch_add_norm_conv<T, Y, 3>(p, blocks, st) : launch_add_norm_conv<T, Y, 16>(p, blocks, st);
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

// blocks: rows (without a shift or a convolution) or tiles.  y_f32: y is fp32 although T is bf16.
extern "C" int cb_add_norm(const float* x, const void* y, const float* bias, const float* post,
                           int post_vec, float* x_out, int ld, int ldy, const float* gain,
                           int gain_vec, void* h, int ldh, void* cast0, void* cast1, int ldc,
                           const float* shift, float* before, const int* rows, const int* slot,
                           const int* row0, const int* len, const int* pos0, const int* tile_entry,
                           const int* tile_off, int blocks, int width, float eps, int f32, int y_f32,
                           const void* spread, int lds, const int* spread_slot,
                           const float* spread_weight, int top, const void* own, int ldo, const float* y_weight,
                           const float* scale, const float* center, const float* taps, int n_taps,
                           void* stream) {
  if (blocks <= 0 || ld % 8 || width > ld || ld > 16384) return -1;
  if (y != nullptr && (ldy % 8 || ldy < ld)) return -2;
  if (gain != nullptr && (h == nullptr || ldh % 8 || ldh < ld)) return -2;
  if ((cast0 != nullptr || cast1 != nullptr) && (ldc % 8 || ldc < ld)) return -2;
  if (shift != nullptr && (gain == nullptr || before == nullptr || rows != nullptr)) return -2;
  if (shift != nullptr && x != nullptr && x == x_out) return -2;     // the row in front is read late
  if (spread != nullptr && (lds % 8 || lds < ld || top < 1 || spread_slot == nullptr || spread_weight == nullptr))
    return -2;
  if (own != nullptr && (ldo % 8 || ldo < ld)) return -2;
  if (taps != nullptr) {
    if (gain == nullptr || shift != nullptr || rows != nullptr || post != nullptr || cast0 != nullptr ||
        cast1 != nullptr || tile_entry == nullptr || tile_off == nullptr)
      return -2;
    if (n_taps < 1 || n_taps > 17 || (n_taps > 1 && before == nullptr) || (n_taps - 1) * ld * 4 > CN_SMEM) return -2;
    if (x_out != nullptr ? x == x_out : (x == nullptr || y != nullptr || spread != nullptr)) return -2;
  }
  AddNorm p;
  p.own = own; p.ldo = ldo; p.y_weight = y_weight; p.scale = scale; p.center = center; p.taps = taps;
  p.n_taps = n_taps;
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
