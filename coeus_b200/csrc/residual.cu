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
// With a convolution a first pass over rows leaves x and the rows' statistics; a second one takes columns of
// such a tile, walks along its rows and keeps the last h in registers.  When every entry is one token, one
// pass does, which finds the earlier h in the state.
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
  const void* own;         // [rows, ldo] in T: stands for a spread row whose slot is negative, or null
  int ldo;
  const float* y_weight;   // [rows] or null
  const float* scale;      // [ld] or null
  const float* center;     // [ld] or null
  const float* taps;       // [n_taps, ld] or null; before is then [slots, n_taps - 1, ld], and without
                           // tile_entry every entry is one token
  int n_taps;
  float2* stats;           // [rows] mean and 1 / deviation, between the two passes of a convolution
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

// A row per block; a tile with a shift; a row, with the convolution of entries of one token; rows whose
// statistics stand for h.
enum : int { AN_ROWS = 0, AN_SHIFT = 1, AN_TOKEN = 2, AN_STATS = 3 };

template <typename T, typename Y, int KEEP, int MODE>
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
    if constexpr (MODE == AN_STATS) {
      if (threadIdx.x == 0) p.stats[row] = make_float2(mean, rs);
      return;
    }
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
  if constexpr (MODE != AN_SHIFT) {
    const int row = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x;
    stream(row, f, true);
    if (MODE == AN_STATS || p.gain == nullptr) return;
    if constexpr (MODE == AN_TOKEN) {
      const int back = p.n_taps - 1;
      const bool has = p.e.pos0[row] > 0;
      float* state = p.before + static_cast<size_t>(p.e.slot[row]) * back * p.ld;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= nv) continue;
        float w[8], o[8], prev[8];
        load_vec<8>(p.taps + static_cast<size_t>(back) * p.ld + v * 8, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = f[i][e] + w[e] * f[i][e];
        for (int k = 0; k < back; ++k) {                 // oldest first; each moves one place
          if (has) {
            load_vec<8>(state + static_cast<size_t>(k) * p.ld + v * 8, prev);
          } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) prev[e] = 0.f;
          }
          load_vec<8>(p.taps + static_cast<size_t>(k) * p.ld + v * 8, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) o[e] += w[e] * prev[e];
          if (k > 0) store_vec<8>(state + static_cast<size_t>(k - 1) * p.ld + v * 8, prev);
        }
        if (back > 0) store_vec<8>(state + static_cast<size_t>(back - 1) * p.ld + v * 8, f[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[i][e] = o[e];
      }
    }
    T* dst = static_cast<T*>(p.h) + static_cast<size_t>(blockIdx.x) * p.ldh;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nv) store_vec<8>(dst + v * 8, f[i]);
    }
  } else {
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
}

// ------------------------------------------------------------------------------- the convolution
constexpr int CN_THREADS = 128;    // columns / 8 of a block
constexpr int CN_AHEAD = 4;        // rows loaded ahead

// One thread: eight columns of a tile of tokens of one entry, from x and the rows' statistics.  HIST > 0: the
// last HIST >= n_taps - 1 tokens' h stay in registers; 0: they are read again.
template <typename T, int HIST>
__global__ void __launch_bounds__(CN_THREADS) conv_pass_kernel(const AddNorm p) {
  const int v = blockIdx.y * CN_THREADS + threadIdx.x;
  if (v >= p.ld / 8) return;
  const int back = p.n_taps - 1;
  const int e = p.tile_entry[blockIdx.x], off = p.tile_off[blockIdx.x];
  const int row0 = p.e.row0[e], len = p.e.len[e], t1 = min(off + SHIFT_TILE, len);
  const bool has = p.e.pos0[e] > 0;
  const float* src = (p.x_out != nullptr ? p.x_out : p.x) + static_cast<size_t>(row0) * p.ld + v * 8;
  const float2* stats = p.stats + row0;
  float* state = p.before + static_cast<size_t>(p.e.slot[e]) * back * p.ld + v * 8;
  T* dst = static_cast<T*>(p.h) + static_cast<size_t>(row0) * p.ldh + v * 8;
  float g[8], c[8];
  if (p.gain_vec) {
    load_vec<8>(p.gain + v * 8, g);
  } else {
#pragma unroll
    for (int k = 0; k < 8; ++k) g[k] = *p.gain;
  }
  if (p.center != nullptr) {
    load_vec<8>(p.center + v * 8, c);
  } else {
#pragma unroll
    for (int k = 0; k < 8; ++k) c[k] = 0.f;
  }
  auto norm = [&](int t, float* f) {
    const float2 r = stats[t];
#pragma unroll
    for (int k = 0; k < 8; ++k) f[k] = (f[k] - r.x) * r.y * g[k] + c[k];
  };
  auto h_of = [&](int t, float* f) {             // of the entry's token t; negative: of the step before
    if (t >= 0) {
      load_vec<8>(src + static_cast<size_t>(t) * p.ld, f);
      norm(t, f);
    } else if (has) {
      load_vec<8>(state + static_cast<size_t>(back + t) * p.ld, f);
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) f[k] = 0.f;
    }
  };
  if constexpr (HIST > 0) {
    float w[HIST + 1][8], prev[HIST][8];         // [d]: d tokens back; prev[d - 1]
#pragma unroll
    for (int d = 0; d <= HIST; ++d) {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        w[d][k] = 0.f;
        if (d > 0) prev[d > 0 ? d - 1 : 0][k] = 0.f;
      }
      if (d <= back) {
        load_vec<8>(p.taps + static_cast<size_t>(back - d) * p.ld + v * 8, w[d]);
        if (d > 0) h_of(off - d, prev[d > 0 ? d - 1 : 0]);
      }
    }
    for (int t0 = off; t0 < t1; t0 += CN_AHEAD) {
      float x[CN_AHEAD][8];
#pragma unroll
      for (int i = 0; i < CN_AHEAD; ++i)
        if (t0 + i < t1) load_vec<8>(src + static_cast<size_t>(t0 + i) * p.ld, x[i]);
#pragma unroll
      for (int i = 0; i < CN_AHEAD; ++i) {
        if (t0 + i >= t1) break;
        norm(t0 + i, x[i]);
        float o[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          float a = w[0][k] * x[i][k];
#pragma unroll
          for (int d = 1; d <= HIST; ++d) a += w[d][k] * prev[d - 1][k];
          o[k] = x[i][k] + a;
#pragma unroll
          for (int d = HIST - 1; d > 0; --d) prev[d][k] = prev[d - 1][k];
          prev[0][k] = x[i][k];
        }
        store_vec<8>(dst + static_cast<size_t>(t0 + i) * p.ldh, o);
      }
    }
  } else {
    for (int t = off; t < t1; ++t) {
      float f[8], o[8], w[8];
      h_of(t, f);
#pragma unroll
      for (int k = 0; k < 8; ++k) o[k] = f[k];
      for (int d = 0; d <= back; ++d) {
        if (d > 0) h_of(t - d, f);
        load_vec<8>(p.taps + static_cast<size_t>(back - d) * p.ld + v * 8, w);
#pragma unroll
        for (int k = 0; k < 8; ++k) o[k] += w[k] * f[k];
      }
      store_vec<8>(dst + static_cast<size_t>(t) * p.ldh, o);
    }
  }
  if (off > 0) return;
  for (int k = 0; k < back; ++k) {               // the entry's last tokens; what is read lies behind k
    float f[8];
    h_of(len - back + k, f);
    store_vec<8>(state + static_cast<size_t>(k) * p.ld, f);
  }
}

template <typename T>
static void launch_conv_pass(const AddNorm& p, int tiles, cudaStream_t st) {
  const dim3 grid(tiles, (p.ld / 8 + CN_THREADS - 1) / CN_THREADS);
  if (p.n_taps <= 4) conv_pass_kernel<T, 3><<<grid, CN_THREADS, 0, st>>>(p);
  else conv_pass_kernel<T, 0><<<grid, CN_THREADS, 0, st>>>(p);
}

template <typename T, typename Y, int MODE>
static int launch_add_norm(const AddNorm& p, int blocks, cudaStream_t st) {
  const int nv = p.ld / 8;
  if (nv <= 512) {
    add_norm_kernel<T, Y, 1, MODE><<<blocks, (nv + 31) / 32 * 32, 0, st>>>(p);
  } else if (nv <= 1024) {
    add_norm_kernel<T, Y, 2, MODE><<<blocks, 512, 0, st>>>(p);
  } else {
    add_norm_kernel<T, Y, 4, MODE><<<blocks, 512, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <typename T, typename Y>
static int launch_add_norm_mode(const AddNorm& p, int blocks, int rows, cudaStream_t st) {
  if (p.shift != nullptr) return launch_add_norm<T, Y, AN_SHIFT>(p, blocks, st);
  if (p.taps == nullptr) return launch_add_norm<T, Y, AN_ROWS>(p, blocks, st);
  if (p.tile_entry == nullptr) return launch_add_norm<T, Y, AN_TOKEN>(p, blocks, st);
  const int rc = launch_add_norm<T, Y, AN_STATS>(p, rows, st);
  if (rc == 0) launch_conv_pass<T>(p, blocks, st);
  return rc == 0 && cudaGetLastError() != cudaSuccess ? -3 : rc;
}

}  // namespace cb

using namespace cb;

// blocks: rows (without a shift or a convolution) or tiles, with rows_all rows in all and a convolution's stats
// [rows_all, 2].  y_f32: y is fp32 although T is bf16.
extern "C" int cb_add_norm(const float* x, const void* y, const float* bias, const float* post,
                           int post_vec, float* x_out, int ld, int ldy, const float* gain,
                           int gain_vec, void* h, int ldh, void* cast0, void* cast1, int ldc,
                           const float* shift, float* before, const int* rows, const int* slot,
                           const int* row0, const int* len, const int* pos0, const int* tile_entry,
                           const int* tile_off, int blocks, int width, float eps, int f32, int y_f32,
                           const void* spread, int lds, const int* spread_slot,
                           const float* spread_weight, int top, const void* own, int ldo, const float* y_weight,
                           const float* scale, const float* center, const float* taps, int n_taps,
                           float* stats, int rows_all, void* stream) {
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
        cast1 != nullptr || (tile_entry == nullptr) != (tile_off == nullptr) || slot == nullptr || pos0 == nullptr)
      return -2;
    if (n_taps < 1 || n_taps > SHIFT_TILE + 1 || (n_taps > 1 && before == nullptr)) return -2;
    if (tile_entry != nullptr && (stats == nullptr || rows_all < 1)) return -2;
    if (x_out != nullptr ? x == x_out : (x == nullptr || y != nullptr || spread != nullptr)) return -2;
  }
  AddNorm p;
  p.own = own; p.ldo = ldo; p.y_weight = y_weight; p.scale = scale; p.center = center; p.taps = taps;
  p.n_taps = n_taps; p.stats = reinterpret_cast<float2*>(stats);
  p.spread = spread; p.lds = lds; p.spread_slot = spread_slot; p.spread_weight = spread_weight; p.top = top;
  p.x = x; p.y = y; p.bias = bias; p.post = post; p.post_vec = post_vec; p.x_out = x_out;
  p.ld = ld; p.ldy = ldy; p.gain = gain; p.gain_vec = gain_vec; p.h = h; p.ldh = ldh;
  p.cast[0] = cast0; p.cast[1] = cast1; p.ldc = ldc; p.shift = shift; p.before = before;
  p.rows = rows; p.e.slot = slot; p.e.row0 = row0; p.e.len = len; p.e.pos0 = pos0;
  p.tile_entry = tile_entry; p.tile_off = tile_off; p.width = width; p.eps = eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return launch_add_norm_mode<float, float>(p, blocks, rows_all, st);
  return y_f32 ? launch_add_norm_mode<__nv_bfloat16, float>(p, blocks, rows_all, st)
               : launch_add_norm_mode<__nv_bfloat16, __nv_bfloat16>(p, blocks, rows_all, st);
}
