// Short causal convolutions over time in front of a mixer, for a ragged batch, together with what
// follows them element by element:
//   shortconv_attn   q, k, v of an attention layer: convolution, rotary embedding of q and k,
//                    value mixing, and the write of k and v into the cache pages
//   shortconv_delta  q, k, v of a gated delta layer: convolution, SiLU, unit norm of q and k,
//                    the decay of every key channel and the step size
//   shortconv_act    any channels: convolution, bias, SiLU (in front of a state-space layer)
// The convolution of a channel with n taps needs the n - 1 projected values before the current
// one.  Inside a step they are earlier rows of the projection; at the start of an entry they come
// from the slot's state, [n - 1, channels] projected values in time order.  The block that owns
// an entry's first tile is the only one that reads the state, so it alone replaces it, after its
// last read.  (A convolution may have at most CONV_TILE + 1 taps, so that no other
// tile reaches back to the state.)
#include "ragged.cuh"

namespace cb {

constexpr int CONV_TILE = 16;      // tokens per block
constexpr int CONV_THREADS = 128;

struct ConvIn {
  const void* raw;        // [rows, ld] projections: q at column 0, k at koff, v at voff
  int ld, koff, voff;
  const float* taps_w;    // [taps, channels], channels = q | k | v without gaps
  int taps;
  void* state;            // [slots, taps - 1, channels] in the activation type
  int heads, kv_heads, dim, vdim;
  Entries e;
  const int* tile_entry;  // [tiles]
  const int* tile_off;    // [tiles] first token of the tile inside its entry
};

// Column of channel c (q | k | v numbering) in the projection buffer.
__device__ __forceinline__ int raw_col(const ConvIn& p, int c) {
  const int qc = p.heads * p.dim, kc = p.kv_heads * p.dim;
  return c < qc ? c : (c < qc + kc ? p.koff + (c - qc) : p.voff + (c - qc - kc));
}
// The delta layer has kv_heads query heads.
__device__ __forceinline__ int raw_col_delta(const ConvIn& p, int c) {
  const int qc = p.kv_heads * p.dim;
  return c < qc ? c : (c < 2 * qc ? p.koff + (c - qc) : p.voff + (c - 2 * qc));
}

// Channel c (column col) of the token at offset t of the entry, any number of taps.
template <typename T>
__device__ __forceinline__ float conv_at(const ConvIn& p, int c, int col, int channels, int row0,
                                         int t, int slot, bool has_state) {
  const T* raw = static_cast<const T*>(p.raw) + static_cast<ptrdiff_t>(row0) * p.ld + col;
  const int n1 = p.taps - 1;
  const T* st = static_cast<const T*>(p.state) + static_cast<ptrdiff_t>(slot) * n1 * channels + c;
  float y = 0.f;
  for (int j = 0; j <= n1; ++j) {
    const int o = t - n1 + j;
    if (o < 0 && !has_state) continue;
    const float u = to_f32(o >= 0 ? raw[static_cast<ptrdiff_t>(o) * p.ld]
                                  : st[static_cast<ptrdiff_t>(n1 + o) * channels]);
    y += u * p.taps_w[static_cast<ptrdiff_t>(j) * channels + c];
  }
  return y;
}

// The state of channel c after the entry's len tokens.
template <typename T>
__device__ __forceinline__ void conv_advance(const ConvIn& p, int c, int col, int channels,
                                             int row0, int len, int slot, bool has_state) {
  const int n1 = p.taps - 1;
  const T* raw = static_cast<const T*>(p.raw);
  T* st = static_cast<T*>(p.state) + static_cast<size_t>(slot) * n1 * channels + c;
  for (int j = 0; j < n1; ++j) {          // ascending: st[j + len] is read before it is replaced
    const int o = len - n1 + j;
    T v;
    if (o >= 0) v = raw[static_cast<size_t>(row0 + o) * p.ld + col];
    else v = has_state ? st[static_cast<size_t>(n1 + o) * channels] : from_f32<T>(0.f);
    st[static_cast<size_t>(j) * channels] = v;
  }
}

struct AttnPre {
  ConvIn c;
  int half;                // rotated pairs per head (0: no rotation)
  const float2* rope;      // [rows, half] (cos, sin)
  void* q;                 // out [rows, heads, q_head]
  int q_head, row_head;    // distance of the heads in q, and in k_rows and v_rows
  void* k_cache;           // [pages, PAGE, kv_heads, dim_p]
  void* v_cache;           // [pages, PAGE, kv_heads, vdim_p]
  int dim_p, vdim_p;
  const int* page_table;   // [slots, max_pages]
  int max_pages, num_pages;
  void* v_first;           // [rows, kv_heads * vdim]: written when mix_mode = 1, read when 2
  const float* lambda;
  int mix_mode;
  void* k_rows;            // out [rows, kv_heads, row_head]: k once more, row by row (or null)
  void* v_rows;            // out [rows, kv_heads, row_head]
  int* status;
};

// grid (tiles, kv_heads): the block's channels are its key/value head and the query heads on it.
// One channel (or rotated pair) at a time, for sizes and taps that the tile kernel does not take.
template <typename T>
__global__ void __launch_bounds__(CONV_THREADS) shortconv_attn_kernel(const AttnPre p) {
  const ConvIn& ci = p.c;
  const int e = ci.tile_entry[blockIdx.x], off = ci.tile_off[blockIdx.x], g = blockIdx.y;
  const int row0 = ci.e.row0[e], len = ci.e.len[e], pos0 = ci.e.pos0[e], slot = ci.e.slot[e];
  const bool has_state = pos0 > 0;
  const int per = ci.heads / ci.kv_heads, dim = ci.dim, vdim = ci.vdim;
  const int qc = ci.heads * dim, kc = ci.kv_heads * dim;
  const int channels = qc + kc + ci.kv_heads * vdim;
  const int nt = min(CONV_TILE, len - off);
  const int head_u = dim - p.half;           // per head: rotated pairs, then single channels
  const int heads_u = (per + 1) * head_u, units = heads_u + vdim;
  const float lam = p.mix_mode == 2 ? *p.lambda : 0.f;
  for (int i = threadIdx.x; i < nt * units; i += CONV_THREADS) {
    const int t = off + i / units, u = i % units, row = row0 + t, pos = pos0 + t;
    const int lp = pos / RAGGED_PAGE;
    const int page = lp < p.max_pages ? p.page_table[static_cast<size_t>(slot) * p.max_pages + lp] : -1;
    if (page < 0 || page >= p.num_pages) {
      record_status(p.status, ST_BOUNDS, row);
      continue;
    }
    const size_t cell = (static_cast<size_t>(page) * RAGGED_PAGE + pos % RAGGED_PAGE) * ci.kv_heads + g;
    const size_t row_cell = (static_cast<size_t>(row) * ci.kv_heads + g) * p.row_head;
    if (u < heads_u) {
      const int hi = u / head_u, k = u % head_u;       // hi < per: query head, else the key head
      const bool is_q = hi < per;
      const int base = is_q ? (g * per + hi) * dim : qc + g * dim;
      const int colb = is_q ? base : ci.koff + g * dim;
      T* dst = is_q ? static_cast<T*>(p.q) + (static_cast<size_t>(row) * ci.heads + g * per + hi) * p.q_head
                    : static_cast<T*>(p.k_cache) + cell * p.dim_p;
      T* kr = !is_q && p.k_rows != nullptr ? static_cast<T*>(p.k_rows) + row_cell : nullptr;
      const int d = k < p.half ? k : k + p.half;
      float a = conv_at<T>(ci, base + d, colb + d, channels, row0, t, slot, has_state);
      if (k < p.half) {
        const float b = conv_at<T>(ci, base + p.half + d, colb + p.half + d, channels, row0, t, slot, has_state);
        const float2 cs = p.rope[static_cast<size_t>(row) * p.half + d];
        const T hi_half = from_f32<T>(b * cs.x + a * cs.y);
        a = a * cs.x - b * cs.y;
        dst[p.half + d] = hi_half;
        if (kr != nullptr) kr[p.half + d] = hi_half;
      }
      dst[d] = from_f32<T>(a);
      if (kr != nullptr) kr[d] = from_f32<T>(a);
    } else {
      const int d = u - heads_u;
      float a = conv_at<T>(ci, qc + kc + g * vdim + d, ci.voff + g * vdim + d, channels, row0, t, slot, has_state);
      if (p.mix_mode != 0) {
        T* vf = static_cast<T*>(p.v_first) + static_cast<size_t>(row) * ci.kv_heads * vdim + g * vdim + d;
        if (p.mix_mode == 1) *vf = from_f32<T>(a);
        else a = (1.f - lam) * a + lam * to_f32(*vf);
      }
      static_cast<T*>(p.v_cache)[cell * p.vdim_p + d] = from_f32<T>(a);
      if (p.v_rows != nullptr) static_cast<T*>(p.v_rows)[row_cell + d] = from_f32<T>(a);
    }
  }
  if (off == 0 && ci.taps > 1) {
    __syncthreads();
    const int mine = (per + 1) * dim + vdim;
    for (int i = threadIdx.x; i < mine; i += CONV_THREADS) {
      const int c = i < per * dim ? g * per * dim + i
                  : (i < (per + 1) * dim ? qc + g * dim + (i - per * dim)
                                         : qc + kc + g * vdim + (i - (per + 1) * dim));
      conv_advance<T>(ci, c, raw_col(ci, c), channels, row0, len, slot, has_state);
    }
  }
}

// The tile kernels do the same with V = 4 consecutive channels per thread for a whole tile of
// tokens.  The projected rows of the tile and the TAPS - 1 before it are staged in shared memory in
// one go, and the taps of a thread's channels stay in registers.  dim, vdim and half are multiples
// of four.
template <typename T>
__device__ __forceinline__ void cp_async_quad(uint32_t dst, const T* src, bool in) {
  if constexpr (sizeof(T) == 2)
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(dst), "l"(src), "r"(in ? 8 : 0)
                 : "memory");
  else
    cp_async16_zfill(dst, src, in ? 16 : 0);
}

// Four channels of one thread: projection column col (state channel c) for the rows off - (TAPS-1)
// .. off + nt - 1 of an entry, to shared memory at dst with a pitch of `pitch` elements.
template <typename T, int TAPS>
__device__ __forceinline__ void stage_quad(const ConvIn& p, int c, int col, int channels, int row0,
                                           int off, int nt, int slot, bool has_state, T* dst,
                                           int pitch) {
  const T* raw = static_cast<const T*>(p.raw) + static_cast<ptrdiff_t>(row0) * p.ld + col;
  const T* st = static_cast<const T*>(p.state) + static_cast<ptrdiff_t>(slot) * (TAPS - 1) * channels + c;
  const uint32_t d = smem_u32(dst);
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int o = off - (TAPS - 1) + j;
    const bool in = o >= 0 || has_state;
    const T* src = o >= 0 ? raw + static_cast<ptrdiff_t>(o) * p.ld
                          : (in ? st + static_cast<ptrdiff_t>(TAPS - 1 + o) * channels : raw);
    cp_async_quad<T>(d + j * pitch * sizeof(T), src, in);
  }
#pragma unroll 4
  for (int j = 0; j < nt; ++j)
    cp_async_quad<T>(d + (TAPS - 1 + j) * pitch * sizeof(T),
                     raw + static_cast<ptrdiff_t>(off + j) * p.ld, true);
}

template <typename T, int TAPS>
struct Window {
  static constexpr int V = 4;
  float w[TAPS][V], u[TAPS][V];
  __device__ __forceinline__ void taps(const ConvIn& p, int c, int channels) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_vec<V>(p.taps_w + static_cast<ptrdiff_t>(j) * channels + c, w[j]);
  }
  // the rows before the first token t: rows t .. t + TAPS - 2 of the staged tile
  __device__ __forceinline__ void start(const T* s, int pitch) {
#pragma unroll
    for (int j = 1; j < TAPS; ++j) load_vec<V>(s + (j - 1) * pitch, u[j]);
  }
  // takes the next staged row in, y = convolution at its token
  __device__ __forceinline__ void next(const T* row, float* y) {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) u[j][i] = u[j + 1][i];
    load_vec<V>(row, u[TAPS - 1]);
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] += u[j][i] * w[j][i];
  }
};

template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 3) shortconv_attn_tile_kernel(const AttnPre p) {
  constexpr int V = 4;
  const ConvIn& ci = p.c;
  const int e = ci.tile_entry[blockIdx.x], off = ci.tile_off[blockIdx.x], g = blockIdx.y;
  const int row0 = ci.e.row0[e], len = ci.e.len[e], pos0 = ci.e.pos0[e], slot = ci.e.slot[e];
  const bool has_state = pos0 > 0;
  const int per = ci.heads / ci.kv_heads, dim = ci.dim, vdim = ci.vdim;
  const int qc = ci.heads * dim, kc = ci.kv_heads * dim;
  const int channels = qc + kc + ci.kv_heads * vdim;
  const int t1 = min(off + CONV_TILE, len);
  // units: the rotated pairs of all heads, then their other vectors, then the values, so that
  // the threads of a warp mostly do the same
  const int pair_u = p.half / V, plain_u = (dim - 2 * p.half) / V;
  const int pairs_u = (per + 1) * pair_u, heads_u = pairs_u + (per + 1) * plain_u;
  const int nt = t1 - off, cols = (per + 1) * dim + vdim;   // staged columns: q heads | k | v
  extern __shared__ __align__(16) unsigned char conv_smem[];
  float2* s_rope = reinterpret_cast<float2*>(conv_smem);     // [CONV_TILE][half]
  T* s_raw = reinterpret_cast<T*>(s_rope + CONV_TILE * p.half);
  __shared__ int s_page[2];
  for (int i = threadIdx.x * V; i < cols; i += blockDim.x * V) {
    const int c = i < per * dim ? g * per * dim + i
                : (i < (per + 1) * dim ? qc + g * dim + (i - per * dim)
                                       : qc + kc + g * vdim + (i - (per + 1) * dim));
    stage_quad<T, TAPS>(ci, c, raw_col(ci, c), channels, row0, off, nt, slot, has_state, s_raw + i, cols);
  }
  cp_async_commit();
  for (int i = threadIdx.x; i < nt * p.half; i += blockDim.x)
    s_rope[i] = p.rope[static_cast<size_t>(row0 + off) * p.half + i];
  const int lp0 = (pos0 + off) / RAGGED_PAGE;
  if (threadIdx.x < 2) {                     // a tile of 16 tokens touches at most two pages
    const int lp = lp0 + threadIdx.x;
    int page = lp < p.max_pages ? p.page_table[static_cast<size_t>(slot) * p.max_pages + lp] : -1;
    const bool used = lp <= (pos0 + t1 - 1) / RAGGED_PAGE;
    if (used && (page < 0 || page >= p.num_pages)) record_status(p.status, ST_BOUNDS, row0 + off);
    s_page[threadIdx.x] = used && page >= 0 && page < p.num_pages ? page : -1;
  }
  cp_async_wait<0>();
  __syncthreads();
  for (int u = threadIdx.x; u < heads_u + vdim / V; u += blockDim.x) {
    const bool is_v = u >= heads_u, pair = u < pairs_u;
    int c, d, i, hi = 0;                     // channel, place in the head, staged column
    if (is_v) {
      d = (u - heads_u) * V;
      c = qc + kc + g * vdim + d;
      i = (per + 1) * dim + d;
    } else {
      hi = pair ? u / pair_u : (u - pairs_u) / plain_u;
      d = pair ? u % pair_u * V : 2 * p.half + (u - pairs_u) % plain_u * V;
      c = (hi < per ? (g * per + hi) * dim : qc + g * dim) + d;
      i = hi * dim + d;
    }
    const bool is_q = !is_v && hi < per;
    const T* src = s_raw + i;
    float wa[TAPS][V], wb[TAPS][V];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float* w = ci.taps_w + static_cast<ptrdiff_t>(j) * channels + c;
      load_vec<V>(w, wa[j]);
      if (pair) load_vec<V>(w + p.half, wb[j]);
    }
    // where the first token goes, and how far apart the tokens of a page are
    T* kr = nullptr;
    T* vf = nullptr;
    T* dst = nullptr;
    int step = 0;
    const int q_step = ci.heads * p.q_head, kr_step = ci.kv_heads * p.row_head, vf_step = ci.kv_heads * vdim;
    if (is_q) {
      dst = static_cast<T*>(p.q) + static_cast<size_t>(row0 + off) * q_step + (g * per + hi) * p.q_head + d;
    } else {
      step = ci.kv_heads * (is_v ? p.vdim_p : p.dim_p);
      if (p.k_rows != nullptr)
        kr = static_cast<T*>(is_v ? p.v_rows : p.k_rows) + static_cast<size_t>(row0 + off) * kr_step +
             g * p.row_head + d;
      if (is_v && p.mix_mode != 0)
        vf = static_cast<T*>(p.v_first) + static_cast<size_t>(row0 + off) * vf_step + g * vdim + d;
    }
    T* cache = static_cast<T*>(is_v ? p.v_cache : p.k_cache);
    const int in_cell = is_v ? g * p.vdim_p + d : g * p.dim_p + d;
    const float lam = is_v && p.mix_mode == 2 ? *p.lambda : 0.f;
    auto conv = [&](const T* at, const float (*w)[V], float* y) {
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        float f[V];
        load_vec<V>(at + j * cols, f);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] += f[k] * w[j][k];
      }
    };
#pragma unroll 2
    for (int t = 0; t < nt; ++t, src += cols) {
      if (!is_q) {
        const int pos = pos0 + off + t;
        const int page = s_page[pos / RAGGED_PAGE - lp0];
        dst = page < 0 ? nullptr
                       : cache + (static_cast<size_t>(page) * RAGGED_PAGE + pos % RAGGED_PAGE) * step + in_cell;
      }
      float a[V];
      conv(src, wa, a);
      if (pair) {
        float b[V], oa[V], ob[V];
        conv(src + p.half, wb, b);
        const float4* cs = reinterpret_cast<const float4*>(s_rope + t * p.half + d);
        const float4 x = cs[0], y = cs[1];
        const float cc[V] = {x.x, x.z, y.x, y.z}, ss[V] = {x.y, x.w, y.y, y.w};
#pragma unroll
        for (int k = 0; k < V; ++k) {
          oa[k] = a[k] * cc[k] - b[k] * ss[k];
          ob[k] = b[k] * cc[k] + a[k] * ss[k];
        }
        if (dst != nullptr) {
          store_vec<V>(dst, oa);
          store_vec<V>(dst + p.half, ob);
        }
        if (kr != nullptr) {
          store_vec<V>(kr, oa);
          store_vec<V>(kr + p.half, ob);
        }
      } else {
        if (vf != nullptr) {
          if (p.mix_mode == 1) {
            store_vec<V>(vf, a);
          } else {
            float f[V];
            load_vec<V>(vf, f);
#pragma unroll
            for (int k = 0; k < V; ++k) a[k] = (1.f - lam) * a[k] + lam * f[k];
          }
          vf += vf_step;
        }
        if (dst != nullptr) store_vec<V>(dst, a);
        if (kr != nullptr) store_vec<V>(kr, a);
      }
      if (is_q) dst += q_step;
      if (kr != nullptr) kr += kr_step;
    }
  }
  if (off == 0) {
    __syncthreads();
    const int mine = (per + 1) * dim + vdim;
    for (int i = threadIdx.x; i < mine; i += blockDim.x) {
      const int c = i < per * dim ? g * per * dim + i
                  : (i < (per + 1) * dim ? qc + g * dim + (i - per * dim)
                                         : qc + kc + g * vdim + (i - (per + 1) * dim));
      conv_advance<T>(ci, c, raw_col(ci, c), channels, row0, len, slot, has_state);
    }
  }
}

struct DeltaPre {
  ConvIn c;                // heads value heads, kv_heads query/key heads
  int boff;                // column of the step-size projection in raw
  const float* a;          // [rows, heads * dim] decay projection, fp32
  int lda;
  const float* A_log;      // [heads]
  const float* dt_bias;    // [heads * dim]
  float* q;                // out [kv_heads, rows, dim_p] unit norm, scaled by dim^-1/2
  float* k;                // out [kv_heads, rows, dim_p] unit norm
  float* kq;               // out [kv_heads, rows] their dot product
  float* v;                // out [rows, heads, vdim]
  float* g;                // out [heads, rows, dim_p] decay factors
  float* beta;             // out [heads, rows]
  int rows, dim_p;         // dim_p: dim rounded up to a multiple of 32; the padding is zero
};

__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_exact(float x) {
  return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
}
// grid (tiles, kv_heads): one query/key head and the value heads on it; one channel at a time.
template <typename T>
__global__ void __launch_bounds__(CONV_THREADS) shortconv_delta_kernel(const DeltaPre p) {
  const ConvIn& ci = p.c;
  const int e = ci.tile_entry[blockIdx.x], off = ci.tile_off[blockIdx.x], g = blockIdx.y;
  const int row0 = ci.e.row0[e], len = ci.e.len[e], slot = ci.e.slot[e];
  const bool has_state = ci.e.pos0[e] > 0;
  const int per = ci.heads / ci.kv_heads, dim = ci.dim, vdim = ci.vdim;
  const int qc = ci.kv_heads * dim;
  const int channels = 2 * qc + ci.heads * vdim;
  const int nt = min(CONV_TILE, len - off);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float qscale = 1.0f / sqrtf(static_cast<float>(dim));
  // q and k: a warp per token
  for (int t = off + warp; t < off + nt; t += CONV_THREADS / 32) {
    constexpr int NI = 8;                        // dim <= 256
    float qv[NI], kv[NI], sq = 0.f, sk = 0.f, dot = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = lane + 32 * i;
      qv[i] = kv[i] = 0.f;
      if (d < dim) {
        qv[i] = silu_exact(conv_at<T>(ci, g * dim + d, g * dim + d, channels, row0, t, slot, has_state));
        kv[i] = silu_exact(conv_at<T>(ci, qc + g * dim + d, ci.koff + g * dim + d, channels, row0, t, slot, has_state));
      }
      sq += qv[i] * qv[i];
      sk += kv[i] * kv[i];
    }
    const float rq = qscale / sqrtf(warp_sum(sq) + 1e-6f), rk = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
    const size_t cell = static_cast<size_t>(g) * p.rows + row0 + t;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = lane + 32 * i;
      qv[i] *= rq;
      kv[i] *= rk;
      dot += qv[i] * kv[i];
      if (d < p.dim_p) {
        p.q[cell * p.dim_p + d] = qv[i];
        p.k[cell * p.dim_p + d] = kv[i];
      }
    }
    dot = warp_sum(dot);
    if (lane == 0) p.kq[cell] = dot;
  }
  const T* raw = static_cast<const T*>(ci.raw);
  for (int i = threadIdx.x; i < nt * per * vdim; i += CONV_THREADS) {
    const int t = off + i / (per * vdim), c = g * per * vdim + i % (per * vdim);
    p.v[static_cast<size_t>(row0 + t) * ci.heads * vdim + c] =
        silu_exact(conv_at<T>(ci, 2 * qc + c, ci.voff + c, channels, row0, t, slot, has_state));
  }
  for (int i = threadIdx.x; i < nt * per * p.dim_p; i += CONV_THREADS) {
    const int h = g * per + (i / p.dim_p) % per, row = row0 + off + i / (p.dim_p * per), d = i % p.dim_p;
    float f = 0.f;
    if (d < dim)
      f = expf(-expf(p.A_log[h]) *
               softplus_exact(p.a[static_cast<size_t>(row) * p.lda + h * dim + d] + p.dt_bias[h * dim + d]));
    p.g[(static_cast<size_t>(h) * p.rows + row) * p.dim_p + d] = f;
  }
  for (int i = threadIdx.x; i < nt * per; i += CONV_THREADS) {
    const int h = g * per + i / nt, row = row0 + off + i % nt;
    p.beta[static_cast<size_t>(h) * p.rows + row] =
        sigmoidf_(to_f32(raw[static_cast<size_t>(row) * ci.ld + p.boff + h]));
  }
  if (off == 0 && ci.taps > 1) {
    __syncthreads();
    const int mine = 2 * dim + per * vdim;
    for (int i = threadIdx.x; i < mine; i += CONV_THREADS) {
      const int c = i < dim ? g * dim + i
                  : (i < 2 * dim ? qc + g * dim + (i - dim) : 2 * qc + g * per * vdim + (i - 2 * dim));
      conv_advance<T>(ci, c, raw_col_delta(ci, c), channels, row0, len, slot, has_state);
    }
  }
}

// SiLU of a convolution's output (an activation: the fast form where activations are bf16).
template <typename T>
__device__ __forceinline__ float silu_act(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(x, 1.0f + __expf(-x));
  else return silu_exact(x);
}

// The same with four channels per thread over a tile of tokens.  Work of a block, dealt to its
// warps: q and k of the two halves of the tile (a token's 128 or 256 channels are one warp's, the
// norms are warp sums), the values and the decays in pieces of 128 channels.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CONV_THREADS, 6) shortconv_delta_tile_kernel(const DeltaPre p) {
  constexpr int V = 4;
  const ConvIn& ci = p.c;
  const int e = ci.tile_entry[blockIdx.x], off = ci.tile_off[blockIdx.x], g = blockIdx.y;
  const int row0 = ci.e.row0[e], len = ci.e.len[e], slot = ci.e.slot[e];
  const bool has_state = ci.e.pos0[e] > 0;
  const int per = ci.heads / ci.kv_heads, dim = ci.dim, vdim = ci.vdim;
  const int qc = ci.kv_heads * dim;
  const int channels = 2 * qc + ci.heads * vdim;
  const int t1 = min(off + CONV_TILE, len);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float qscale = 1.0f / sqrtf(static_cast<float>(dim));
  const T* raw = static_cast<const T*>(ci.raw) + static_cast<ptrdiff_t>(row0) * ci.ld;
  const int nt = t1 - off, cols = 2 * dim + per * vdim;      // staged columns: q | k | values
  extern __shared__ __align__(16) unsigned char conv_smem[];
  T* s_raw = reinterpret_cast<T*>(conv_smem);
  for (int i = threadIdx.x * V; i < cols; i += CONV_THREADS * V) {
    const int c = i < dim ? g * dim + i
                : (i < 2 * dim ? qc + g * dim + (i - dim) : 2 * qc + g * per * vdim + (i - 2 * dim));
    stage_quad<T, TAPS>(ci, c, raw_col_delta(ci, c), channels, row0, off, nt, slot, has_state, s_raw + i, cols);
  }
  cp_async_commit();
  // the decays meanwhile, in pieces of 128 channels
  {
    const int pieces = (p.dim_p + 127) / 128;
    for (int u = warp; u < per * pieces * 4; u += CONV_THREADS / 32) {   // a quarter of the tile each
      const int i = u / 4, ta = (u & 3) * (CONV_TILE / 4), tb = min(ta + CONV_TILE / 4, nt);
      const int h = g * per + i / pieces, d = ((i % pieces) * 32 + lane) * V;
      if (ta >= tb || d >= p.dim_p) continue;
      const bool in = d < dim;
      const float rate = expf(p.A_log[h]);
      float b[V] = {};
      if (in) load_vec<V>(p.dt_bias + h * dim + d, b);
      float4 ra[CONV_TILE / 4];
#pragma unroll
      for (int j = 0; j < CONV_TILE / 4; ++j) {
        ra[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (in)
          ra[j] = *reinterpret_cast<const float4*>(
              p.a + static_cast<size_t>(row0 + off + min(ta + j, tb - 1)) * p.lda + h * dim + d);
      }
#pragma unroll
      for (int j = 0; j < CONV_TILE / 4; ++j) {
        if (ta + j >= tb) break;
        const float a[V] = {ra[j].x, ra[j].y, ra[j].z, ra[j].w};
        float f[V];
#pragma unroll
        for (int x = 0; x < V; ++x) f[x] = in ? expf(-rate * softplus_exact(a[x] + b[x])) : 0.f;
        store_vec<V>(p.g + (static_cast<size_t>(h) * p.rows + row0 + off + ta + j) * p.dim_p + d, f);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // q and k: a quarter of the tile per warp, the norms are warp sums (dim <= 256)
  {
    const int ta = warp * (CONV_TILE / 4), tb = min(ta + CONV_TILE / 4, nt);
    constexpr int NI = 2;
    for (int t = ta; t < tb; ++t) {
      float k[NI][V], sq = 0.f, sk = 0.f, dot = 0.f;
      float qq[NI][V];
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = (lane + 32 * i) * V;
#pragma unroll
        for (int x = 0; x < V; ++x) qq[i][x] = k[i][x] = 0.f;
        if (d >= dim) continue;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          float u[V], w[V];
          load_vec<V>(s_raw + (t + j) * cols + d, u);
          load_vec<V>(ci.taps_w + static_cast<ptrdiff_t>(j) * channels + g * dim + d, w);
#pragma unroll
          for (int x = 0; x < V; ++x) qq[i][x] += u[x] * w[x];
          load_vec<V>(s_raw + (t + j) * cols + dim + d, u);
          load_vec<V>(ci.taps_w + static_cast<ptrdiff_t>(j) * channels + qc + g * dim + d, w);
#pragma unroll
          for (int x = 0; x < V; ++x) k[i][x] += u[x] * w[x];
        }
#pragma unroll
        for (int x = 0; x < V; ++x) {
          qq[i][x] = silu_act<T>(qq[i][x]);
          k[i][x] = silu_act<T>(k[i][x]);
          sq += qq[i][x] * qq[i][x];
          sk += k[i][x] * k[i][x];
          dot += qq[i][x] * k[i][x];
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        dot += __shfl_xor_sync(0xffffffffu, dot, o);
      }
      const float rq = qscale / sqrtf(sq + 1e-6f), rk = 1.0f / sqrtf(sk + 1e-6f);
      const size_t cell = static_cast<size_t>(g) * p.rows + row0 + off + t;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = (lane + 32 * i) * V;
        if (d >= p.dim_p) continue;
#pragma unroll
        for (int x = 0; x < V; ++x) {
          qq[i][x] *= rq;
          k[i][x] *= rk;
        }
        store_vec<V>(p.q + cell * p.dim_p + d, qq[i]);
        store_vec<V>(p.k + cell * p.dim_p + d, k[i]);
      }
      if (lane == 0) p.kq[cell] = dot * rq * rk;
    }
  }
  // values: four channels per thread
  for (int i = threadIdx.x * V; i < per * vdim; i += CONV_THREADS * V) {
    const int c = g * per * vdim + i;
    Window<T, TAPS> w;
    w.taps(ci, 2 * qc + c, channels);
    const T* src = s_raw + 2 * dim + i;
    w.start(src, cols);
    src += (TAPS - 1) * cols;
    float* dst = p.v + static_cast<size_t>(row0 + off) * ci.heads * vdim + c;
#pragma unroll 4
    for (int t = 0; t < nt; ++t, src += cols, dst += ci.heads * vdim) {
      float y[V];
      w.next(src, y);
#pragma unroll
      for (int x = 0; x < V; ++x) y[x] = silu_act<T>(y[x]);
      store_vec<V>(dst, y);
    }
  }
  for (int i = threadIdx.x; i < (t1 - off) * per; i += CONV_THREADS) {
    const int h = g * per + i / (t1 - off), t = off + i % (t1 - off);
    p.beta[static_cast<size_t>(h) * p.rows + row0 + t] =
        sigmoidf_(to_f32(raw[static_cast<ptrdiff_t>(t) * ci.ld + p.boff + h]));
  }
  if (off == 0) {
    __syncthreads();
    const int mine = 2 * dim + per * vdim;
    for (int i = threadIdx.x; i < mine; i += CONV_THREADS) {
      const int c = i < dim ? g * dim + i
                  : (i < 2 * dim ? qc + g * dim + (i - dim) : 2 * qc + g * per * vdim + (i - 2 * dim));
      conv_advance<T>(ci, c, raw_col_delta(ci, c), channels, row0, len, slot, has_state);
    }
  }
}

struct ConvAct {
  const void* raw;         // [rows, ld], the channels from column off on
  int ld, off;
  const float* taps_w;     // [taps, channels], channels a multiple of eight
  const float* bias;       // [channels]
  int taps, channels;
  void* state;             // [slots, taps - 1, channels]
  void* out;               // [rows, channels]
  Entries e;
  const int* tile_entry;
  const int* tile_off;
};

// Eight channels per thread over a tile of tokens, the last TAPS values in registers (TAPS = 0: any
// number of taps, read again for every token).
template <typename T, int TAPS>
__global__ void __launch_bounds__(CONV_THREADS) shortconv_act_kernel(const ConvAct p) {
  constexpr int V = 8, W = TAPS > 0 ? TAPS : 1;
  const int e = p.tile_entry[blockIdx.x], off = p.tile_off[blockIdx.x];
  const int c = (blockIdx.y * CONV_THREADS + threadIdx.x) * V;
  if (c >= p.channels) return;
  const int row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e], n1 = p.taps - 1;
  const bool has_state = p.e.pos0[e] > 0;
  const T* raw = static_cast<const T*>(p.raw) + static_cast<ptrdiff_t>(row0) * p.ld + p.off + c;
  T* st = static_cast<T*>(p.state) + static_cast<ptrdiff_t>(slot) * n1 * p.channels + c;
  T* out = static_cast<T*>(p.out) + static_cast<ptrdiff_t>(row0) * p.channels + c;
  auto at = [&](int o, float* f) {                       // the value at offset o, which may be negative
    if (o >= 0) {
      load_vec<V>(raw + static_cast<ptrdiff_t>(o) * p.ld, f);
    } else if (has_state) {
      load_vec<V>(st + static_cast<ptrdiff_t>(n1 + o) * p.channels, f);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) f[k] = 0.f;
    }
  };
  float w[W][V], u[W][V], b[V];
  load_vec<V>(p.bias + c, b);
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_vec<V>(p.taps_w + static_cast<ptrdiff_t>(j) * p.channels + c, w[j]);
#pragma unroll
    for (int j = 1; j < TAPS; ++j) at(off - TAPS + j, u[j]);
  }
  const int t1 = min(off + CONV_TILE, len);
  auto finish = [&](int t, float* y) {
#pragma unroll
    for (int k = 0; k < V; ++k) y[k] = silu_act<T>(y[k]);
    store_vec<V>(out + static_cast<ptrdiff_t>(t) * p.channels, y);
  };
  if constexpr (TAPS > 0) {
    auto step = [&](int t, const float* f) {
      float y[V];
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) u[j][k] = u[j + 1][k];
#pragma unroll
      for (int k = 0; k < V; ++k) {
        u[W - 1][k] = f[k];
        y[k] = b[k];
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] += u[j][k] * w[j][k];
      finish(t, y);
    };
    int t = off;
    constexpr int AHEAD = 4;               // rows loaded together
    for (; t + AHEAD <= t1; t += AHEAD) {
      float f[AHEAD][V];
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) load_vec<V>(raw + static_cast<ptrdiff_t>(t + i) * p.ld, f[i]);
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) step(t + i, f[i]);
    }
    for (; t < t1; ++t) {
      float f[V];
      load_vec<V>(raw + static_cast<ptrdiff_t>(t) * p.ld, f);
      step(t, f);
    }
  } else {
    for (int t = off; t < t1; ++t) {
      float y[V];
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = b[k];
      for (int j = 0; j <= n1; ++j) {
        at(t - n1 + j, u[0]);
        load_vec<V>(p.taps_w + static_cast<ptrdiff_t>(j) * p.channels + c, w[0]);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] += u[0][k] * w[0][k];
      }
      finish(t, y);
    }
  }
  if (off == 0)
    for (int j = 0; j < n1; ++j) {        // ascending: row j + len is read before it is replaced
      float f[V];
      at(len - n1 + j, f);
      store_vec<V>(st + static_cast<ptrdiff_t>(j) * p.channels, f);
    }
}

template <typename T>
static int launch_conv_act(const ConvAct& p, int tiles, cudaStream_t st) {
  dim3 grid(tiles, (p.channels / 8 + CONV_THREADS - 1) / CONV_THREADS);
  switch (p.taps) {
    case 1: shortconv_act_kernel<T, 1><<<grid, CONV_THREADS, 0, st>>>(p); break;
    case 2: shortconv_act_kernel<T, 2><<<grid, CONV_THREADS, 0, st>>>(p); break;
    case 3: shortconv_act_kernel<T, 3><<<grid, CONV_THREADS, 0, st>>>(p); break;
    case 4: shortconv_act_kernel<T, 4><<<grid, CONV_THREADS, 0, st>>>(p); break;
    default: shortconv_act_kernel<T, 0><<<grid, CONV_THREADS, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

// One block per row, vectors of eight bf16; the padding of a head is zero.  v may be absent.
__global__ void kv_gather_kernel(const uint4* __restrict__ k_cache, const uint4* __restrict__ v_cache,
                                 int k_heads, int v_heads, int kw, int vw, const int* __restrict__ page_table,
                                 int max_pages, int num_pages, const int2* __restrict__ where,
                                 uint4* __restrict__ k_rows, uint4* __restrict__ v_rows, int krow_w,
                                 int vrow_w, int* status) {
  const int2 at = where[blockIdx.x];
  const int lp = at.y / RAGGED_PAGE;
  int page = lp < max_pages ? page_table[static_cast<size_t>(at.x) * max_pages + lp] : -1;
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) record_status(status, ST_BOUNDS, blockIdx.x);
    return;
  }
  const size_t cell = static_cast<size_t>(page) * RAGGED_PAGE + at.y % RAGGED_PAGE;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int i = threadIdx.x; i < k_heads * krow_w; i += blockDim.x) {
    const int g = i / krow_w, c = i % krow_w;
    k_rows[static_cast<size_t>(blockIdx.x) * k_heads * krow_w + i] =
        c < kw ? k_cache[(cell * k_heads + g) * kw + c] : zero;
  }
  if (v_rows == nullptr) return;
  for (int i = threadIdx.x; i < v_heads * vrow_w; i += blockDim.x) {
    const int g = i / vrow_w, c = i % vrow_w;
    v_rows[static_cast<size_t>(blockIdx.x) * v_heads * vrow_w + i] =
        c < vw ? v_cache[(cell * v_heads + g) * vw + c] : zero;
  }
}

constexpr int CONV_SMEM_MAX = 200 * 1024;

template <typename T, int TAPS>
static int launch_attn_tile(const AttnPre& p, dim3 grid, int threads, int smem, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(shortconv_attn_tile_kernel<T, TAPS>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, CONV_SMEM_MAX) != cudaSuccess)
      return -4;
    set = true;
  }
  shortconv_attn_tile_kernel<T, TAPS><<<grid, threads, smem, st>>>(p);
  return 0;
}
template <typename T, int TAPS>
static int launch_delta_tile(const DeltaPre& p, dim3 grid, int smem, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(shortconv_delta_tile_kernel<T, TAPS>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, CONV_SMEM_MAX) != cudaSuccess)
      return -4;
    set = true;
  }
  shortconv_delta_tile_kernel<T, TAPS><<<grid, CONV_THREADS, smem, st>>>(p);
  return 0;
}

template <typename T>
static int launch_conv_attn(const AttnPre& p, dim3 grid, bool vec, cudaStream_t st) {
  const int per = p.c.heads / p.c.kv_heads, cols = (per + 1) * p.c.dim + p.c.vdim;
  const int smem = CONV_TILE * p.half * static_cast<int>(sizeof(float2)) +
                   (CONV_TILE + p.c.taps - 1) * cols * static_cast<int>(sizeof(T));
  int rc = 0;
  if (vec && smem <= CONV_SMEM_MAX) {
    const int units = (per + 1) * ((p.c.dim - p.half) / 4) + p.c.vdim / 4;
    const int threads = min(256, (units + 31) / 32 * 32);
    switch (p.c.taps) {
      case 2: rc = launch_attn_tile<T, 2>(p, grid, threads, smem, st); break;
      case 3: rc = launch_attn_tile<T, 3>(p, grid, threads, smem, st); break;
      default: rc = launch_attn_tile<T, 4>(p, grid, threads, smem, st);
    }
  } else {
    shortconv_attn_kernel<T><<<grid, CONV_THREADS, 0, st>>>(p);
  }
  return rc != 0 ? rc : (cudaGetLastError() == cudaSuccess ? 0 : -3);
}
template <typename T>
static int launch_conv_delta(const DeltaPre& p, dim3 grid, bool vec, cudaStream_t st) {
  const int cols = 2 * p.c.dim + p.c.heads / p.c.kv_heads * p.c.vdim;
  const int smem = (CONV_TILE + p.c.taps - 1) * cols * static_cast<int>(sizeof(T));
  int rc = 0;
  if (vec && smem <= CONV_SMEM_MAX) {
    switch (p.c.taps) {
      case 2: rc = launch_delta_tile<T, 2>(p, grid, smem, st); break;
      case 3: rc = launch_delta_tile<T, 3>(p, grid, smem, st); break;
      default: rc = launch_delta_tile<T, 4>(p, grid, smem, st);
    }
  } else {
    shortconv_delta_kernel<T><<<grid, CONV_THREADS, 0, st>>>(p);
  }
  return rc != 0 ? rc : (cudaGetLastError() == cudaSuccess ? 0 : -3);
}

}  // namespace cb

using namespace cb;

static ConvIn conv_in(const void* raw, int ld, int koff, int voff, const float* taps_w, int taps,
                      void* state, int heads, int kv_heads, int dim, int vdim, const int* slot,
                      const int* row0, const int* len, const int* pos0, const int* tile_entry,
                      const int* tile_off) {
  ConvIn c;
  c.raw = raw; c.ld = ld; c.koff = koff; c.voff = voff; c.taps_w = taps_w; c.taps = taps;
  c.state = state; c.heads = heads; c.kv_heads = kv_heads; c.dim = dim; c.vdim = vdim;
  c.e.slot = slot; c.e.row0 = row0; c.e.len = len; c.e.pos0 = pos0;
  c.tile_entry = tile_entry; c.tile_off = tile_off;
  return c;
}

extern "C" int cb_conv_tile() { return CONV_TILE; }

extern "C" int cb_shortconv_attn(const void* raw, int ld, int koff, int voff, const float* taps_w,
                                 int taps, void* state, int heads, int kv_heads, int dim, int vdim,
                                 const int* slot, const int* row0, const int* len, const int* pos0,
                                 const int* tile_entry, const int* tile_off, int tiles, int half,
                                 const void* rope, void* q, int q_head, void* k_cache, void* v_cache, int dim_p,
                                 int vdim_p, const int* page_table, int max_pages, int num_pages,
                                 void* v_first, const float* lambda, int mix_mode, void* k_rows,
                                 void* v_rows, int row_head, int f32, int* status, void* stream) {
  if (tiles <= 0 || taps < 1 || taps > CONV_TILE + 1 || kv_heads < 1 || heads % kv_heads != 0 || 2 * half > dim) return -1;
  if (mix_mode != 0 && v_first == nullptr) return -2;
  AttnPre p;
  p.c = conv_in(raw, ld, koff, voff, taps_w, taps, state, heads, kv_heads, dim, vdim, slot, row0, len,
                pos0, tile_entry, tile_off);
  p.half = half; p.rope = static_cast<const float2*>(rope); p.q = q; p.k_cache = k_cache;
  p.v_cache = v_cache; p.dim_p = dim_p; p.vdim_p = vdim_p; p.page_table = page_table;
  p.max_pages = max_pages; p.num_pages = num_pages; p.v_first = v_first; p.lambda = lambda;
  p.mix_mode = mix_mode; p.status = status;
  p.k_rows = k_rows; p.v_rows = v_rows; p.q_head = q_head; p.row_head = row_head;
  const bool vec = taps >= 2 && taps <= 4 && dim % 4 == 0 && vdim % 4 == 0 && half % 4 == 0 &&
                   half <= 128 && q_head % 4 == 0 && row_head % 4 == 0 && ld % 8 == 0 && koff % 8 == 0 && voff % 8 == 0;
  dim3 grid(tiles, kv_heads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_conv_attn<float>(p, grid, vec, st)
             : launch_conv_attn<__nv_bfloat16>(p, grid, vec, st);
}

// Rows gathered from the cache pages: row i of k_rows [n, k_heads, kr_head] and v_rows [n, v_heads,
// vr_head] is the token at position where[2 i + 1] of slot where[2 i].
extern "C" int cb_kv_gather(const void* k_cache, const void* v_cache, int k_heads, int v_heads, int dim_p,
                            int vdim_p, const int* page_table, int max_pages, int num_pages,
                            const void* where, int n, void* k_rows, void* v_rows, int kr_head,
                            int vr_head, int* status, void* stream) {
  if (n <= 0 || dim_p % 8 || vdim_p % 8 || kr_head % 8 || vr_head % 8 || dim_p > kr_head || vdim_p > vr_head)
    return -1;
  kv_gather_kernel<<<n, 128, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(k_cache), static_cast<const uint4*>(v_cache), k_heads, v_heads, dim_p / 8,
      vdim_p / 8, page_table, max_pages, num_pages, static_cast<const int2*>(where),
      static_cast<uint4*>(k_rows), static_cast<uint4*>(v_rows), kr_head / 8, vr_head / 8, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int cb_shortconv_delta(const void* raw, int ld, int koff, int voff, int boff,
                                  const float* taps_w, int taps, void* state, int heads,
                                  int kv_heads, int dim, int vdim, const int* slot, const int* row0,
                                  const int* len, const int* pos0, const int* tile_entry,
                                  const int* tile_off, int tiles, const float* a, int lda,
                                  const float* A_log, const float* dt_bias, float* q, float* k,
                                  float* kq, float* v, float* g, float* beta, int rows, int dim_p,
                                  int f32,
                                  void* stream) {
  if (tiles <= 0 || taps < 1 || taps > CONV_TILE + 1 || kv_heads < 1 || heads % kv_heads != 0) return -1;
  if (dim > 256 || dim_p % 32 != 0 || dim_p < dim || dim_p > 256) return -2;
  DeltaPre p;
  p.c = conv_in(raw, ld, koff, voff, taps_w, taps, state, heads, kv_heads, dim, vdim, slot, row0, len,
                pos0, tile_entry, tile_off);
  p.boff = boff; p.a = a; p.lda = lda; p.A_log = A_log; p.dt_bias = dt_bias; p.q = q; p.k = k;
  p.kq = kq; p.v = v; p.g = g; p.beta = beta; p.rows = rows;
  p.dim_p = dim_p;
  dim3 grid(tiles, kv_heads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = taps >= 2 && taps <= 4 && dim % 4 == 0 && vdim % 4 == 0 && lda % 4 == 0 && ld % 8 == 0 && koff % 8 == 0 &&
                   voff % 8 == 0;
  return f32 ? launch_conv_delta<float>(p, grid, vec, st)
             : launch_conv_delta<__nv_bfloat16>(p, grid, vec, st);
}

extern "C" int cb_shortconv_act(const void* raw, int ld, int off, const float* taps_w, const float* bias,
                                int taps, int channels, void* state, void* out, const int* slot,
                                const int* row0, const int* len, const int* pos0,
                                const int* tile_entry, const int* tile_off, int tiles, int f32,
                                void* stream) {
  if (tiles <= 0 || taps < 1 || taps > CONV_TILE + 1 || channels <= 0 || channels % 8 || ld % 8 || off % 8)
    return -1;
  ConvAct p;
  p.raw = raw; p.ld = ld; p.off = off; p.taps_w = taps_w; p.bias = bias; p.taps = taps;
  p.channels = channels; p.state = state; p.out = out;
  p.e.slot = slot; p.e.row0 = row0; p.e.len = len; p.e.pos0 = pos0;
  p.tile_entry = tile_entry; p.tile_off = tile_off;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_conv_act<float>(p, tiles, st) : launch_conv_act<__nv_bfloat16>(p, tiles, st);
}
