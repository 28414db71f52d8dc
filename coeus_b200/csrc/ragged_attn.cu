// Attention of a ragged batch over the paged cache: every query row sits at its own position of
// its own sequence and sees the cached keys of its chunk or its sliding window up to itself (both 0: all
// of them), and with a window the sequence's first `keep` positions.  Scores may be capped (s -> cap tanh(s / cap)), the softmax may have a sink per head (a logit
// in the denominator only) and the head's output a gate (a sigmoid of a projected number, one per head or
// one per number).  Query head h reads key/value head h / (heads / kv_heads); query/key width and value
// width are independent.
//
// With two maps a head has two queries and a key head two keys over the same values, and the head's
// output is (a0 - w a1) / rms * factor of the two results.  A cached key is then the keys of both maps
// side by side; a query of one map is zero at the other's places, so that both maps of a group share
// every load, and two maps are twice as many query heads on a key twice as wide.
//
//   rows kernel    one CTA per (query row, key/value head, split): the query heads of the group
//                  share every key and value that is loaded.  Everything in fp32, and decoding
//                  of heads wider than 128.
//   group kernel   decoding in bf16: the same split of the work, on the tensor cores.
//   tiles kernel   64 query rows of one head on the tensor cores (mma m16n8k16), one cache page
//                  per step through a double-buffered shared-memory ring.  The weights enter the
//                  second product as the sum of two bf16 numbers, so they keep 16 mantissa bits.
#include "ragged.cuh"

namespace cb {

constexpr float LOG2E = 1.4426950408889634f;

struct RaggedSpec {        // as the host gives it
  int heads, kv_heads, dim, vdim, dim_p, vdim_p, chunk, window, keep, maps, gate_wide;
  float scale, softcap, map_factor, eps;
};

struct RaggedAttn {
  const void* q;           // [rows, heads, q_head]
  int q_head;
  const void* k_cache;     // [pages, PAGE, kv_heads, kdim]
  const void* v_cache;     // [pages, PAGE, kv_heads, vdim_p]
  const int* page_table;   // [slots, max_pages]
  int max_pages, num_pages;
  int heads, kv_heads, dim, vdim, dim_p, vdim_p;    // heads: of all maps
  int maps, kdim;          // kdim = maps * dim_p
  int chunk, window, keep;
  float scale;             // products to units of log2, or with a cap to the tanh's argument
  float cap;               // 0, or the cap in units of log2
  const float* sink;       // [heads] or null
  const void* gate;        // [rows, ldg] or null: column h gates head h, or (gate_wide) h * vdim + d
  int ldg, gate_wide;
  const float* map_weight; // two maps: weight of the second
  float map_factor, eps;
  void* out;               // [rows, ldo]
  int ldo;
  int* status;
};

// First position that position pos sees; it does not fall as pos grows.
__device__ __forceinline__ int first_seen(const RaggedAttn& p, int pos) {
  if (p.window > 0) return max(0, pos + 1 - p.window);
  return p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
}
// The keys that position pos sees, counted 0 .. n - 1: the kept positions below its window, then the window.
struct Seen {
  int lo, kept, n;
  __device__ __forceinline__ Seen(const RaggedAttn& p, int pos)
      : lo(first_seen(p, pos)), kept(min(p.keep, lo)), n(pos + 1 - lo + kept) {}
  __device__ __forceinline__ int place(int i) const { return i < kept ? i : i - kept + lo; }
};
template <typename T>
__device__ __forceinline__ float exp2_t(float x) {
  if constexpr (sizeof(T) == 4) return exp2f(x);
  else return fast_exp2(x);
}
// A product of a query and a key (times p.scale) to a score in units of log2.
template <typename T>
__device__ __forceinline__ float score_of(const RaggedAttn& p, float s) {
  if (p.cap == 0.f) return s;
  if constexpr (sizeof(T) == 4) return p.cap * tanhf(s);
  else return p.cap * tanh_exp(s);
}
// Column of the key's row where the query of head h starts.
__device__ __forceinline__ int map_off(const RaggedAttn& p, int h) { return p.maps == 2 ? (h & 1) * p.dim_p : 0; }
template <typename T>
__device__ __forceinline__ float gate_wide_of(const RaggedAttn& p, int row, int col) {
  if (p.gate == nullptr || !p.gate_wide) return 1.f;
  return sigmoidf_(to_f32(static_cast<const T*>(p.gate)[static_cast<size_t>(row) * p.ldg + col]));
}
template <typename T>
__device__ __forceinline__ float gate_of(const RaggedAttn& p, int row, int h) {
  if (p.gate == nullptr || p.gate_wide) return 1.f;
  return sigmoidf_(to_f32(static_cast<const T*>(p.gate)[static_cast<size_t>(row) * p.ldg + h]));
}
// Softmax denominator with the sink, in units of 2^m.
template <typename T>
__device__ __forceinline__ float denom(const RaggedAttn& p, int h, float m, float l) {
  return p.sink != nullptr ? l + exp2_t<T>(p.sink[h] * LOG2E - m) : l;
}

// ------------------------------------------------------------------------------ rows kernel
constexpr int RA_WARPS = 4;

struct RowsArgs {
  RaggedAttn a;
  const int* rows;         // [n] query rows, or null: row i
  const int* row_slot;     // [rows of the batch]
  const int* row_pos;
  int splits;
  float* part_o;           // [n, heads, splits, vdim]
  float* part_ml;          // [n, heads, splits, 2]
};

template <typename T, int KIT, int GM>    // dim <= 64 KIT, GM query heads at a time
__global__ void __launch_bounds__(RA_WARPS * 32) ragged_attn_rows_kernel(const RowsArgs ra) {
  const RaggedAttn& p = ra.a;
  constexpr int DC = 64 * KIT;
  __shared__ __align__(16) float sq[GM][DC];
  __shared__ __align__(16) float sp[RA_WARPS][32][GM];     // scores, then weights, [key][head]
  __shared__ float sm_m[RA_WARPS][GM], sm_l[RA_WARPS][GM];
  __shared__ __align__(16) float red[RA_WARPS * 32 * 8];
  const int i = blockIdx.x, split = blockIdx.z;
  const int per = p.heads / p.kv_heads, subs = (per + GM - 1) / GM;
  const int hk = blockIdx.y / subs, h0 = hk * per + (blockIdx.y % subs) * GM;
  const int ng = min(GM, (hk + 1) * per - h0);
  const int row = ra.rows != nullptr ? ra.rows[i] : i;
  const int slot = ra.row_slot[row], pos = ra.row_pos[row];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* pt = p.page_table + static_cast<size_t>(slot) * p.max_pages;
  const T* qp = static_cast<const T*>(p.q) + static_cast<size_t>(row) * p.heads * p.q_head;
  for (int j = threadIdx.x; j < GM * DC; j += RA_WARPS * 32) {
    const int g = j / DC, d = j % DC;
    const int c = d - map_off(p, h0 + g);
    sq[g][d] = (g < ng && c >= 0 && c < p.dim) ? to_f32(qp[(h0 + g) * p.q_head + c]) * p.scale : 0.f;
  }
  __syncthreads();
  const Seen seen(p, pos);
  const int piece = (seen.n + ra.splits - 1) / ra.splits;
  const int t0 = split * piece, t1 = min(seen.n, t0 + piece);
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);
  const int nchunk = p.vdim_p / 8, ngroups = 32 / nchunk;
  const int kg = lane / nchunk, vch = lane % nchunk;
  float m[GM], l[GM], acc[GM][8];
#pragma unroll
  for (int g = 0; g < GM; ++g) {
    m[g] = -INFINITY;
    l[g] = 0.f;
#pragma unroll
    for (int x = 0; x < 8; ++x) acc[g][x] = 0.f;
  }
  for (int tb = t0 + warp * 32; tb < t1; tb += RA_WARPS * 32) {
    // scores of 32 keys: eight lanes per key, four keys at a time
    const int my_t = tb + lane;
    int my_page = 0;
    if (my_t < t1) {
      const int lp = seen.place(my_t) / RAGGED_PAGE;
      my_page = lp < p.max_pages ? pt[lp] : -1;
      if (my_page < 0 || my_page >= p.num_pages) {
        record_status(p.status, ST_BOUNDS, row);
        my_page = 0;
      }
    }
#pragma unroll 4
    for (int r = 0; r < 8; ++r) {
      const int key = r * 4 + (lane >> 3), t = tb + key;
      const int page = __shfl_sync(0xffffffffu, my_page, key);
      float s[GM];
#pragma unroll
      for (int g = 0; g < GM; ++g) s[g] = 0.f;
      if (t < t1) {
        const T* kp = kc + ((static_cast<size_t>(page) * RAGGED_PAGE + seen.place(t) % RAGGED_PAGE) * p.kv_heads + hk) * p.kdim;
#pragma unroll
        for (int c = 0; c < KIT; ++c) {
          const int d = ((lane & 7) + 8 * c) * 8;
          if (d < p.kdim) {
            float f[8];
            load_vec<8>(kp + d, f);
#pragma unroll
            for (int g = 0; g < GM; ++g) {
              const float4 a = *reinterpret_cast<const float4*>(&sq[g][d]);
              const float4 b = *reinterpret_cast<const float4*>(&sq[g][d + 4]);
              s[g] += f[0] * a.x + f[1] * a.y + f[2] * a.z + f[3] * a.w + f[4] * b.x + f[5] * b.y +
                      f[6] * b.z + f[7] * b.w;
            }
          }
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int g = 0; g < GM; ++g) s[g] += __shfl_xor_sync(0xffffffffu, s[g], o);
#pragma unroll
      for (int g = 0; g < GM; ++g)
        if ((lane & 7) == (g & 7)) sp[warp][key][g] = s[g];
    }
    __syncwarp();
    // weights: one key per lane
#pragma unroll
    for (int g = 0; g < GM; ++g) {
      const float s = my_t < t1 ? score_of<T>(p, sp[warp][lane][g]) : -INFINITY;
      const float mn = fmaxf(m[g], warp_max(s));          // finite: the block has a key
      const float c = exp2_t<T>(m[g] - mn), w = exp2_t<T>(s - mn);
      m[g] = mn;
      l[g] = l[g] * c + warp_sum(w);
#pragma unroll
      for (int x = 0; x < 8; ++x) acc[g][x] *= c;
      sp[warp][lane][g] = w;
    }
    __syncwarp();
    // weighted values: lane (kg, vch) takes every ngroups-th key and eight value channels
    const int nk = min(32, t1 - tb);
#pragma unroll 4
    for (int k0 = 0; k0 < nk; k0 += ngroups) {
      const int key = k0 + kg, t = tb + key;
      const int page = __shfl_sync(0xffffffffu, my_page, key & 31);
      if (kg < ngroups && key < nk) {
        const T* vp = vc + ((static_cast<size_t>(page) * RAGGED_PAGE + seen.place(t) % RAGGED_PAGE) * p.kv_heads + hk) * p.vdim_p;
        float f[8];
        load_vec<8>(vp + vch * 8, f);
#pragma unroll
        for (int g = 0; g < GM; ++g) {
          const float w = sp[warp][key][g];
#pragma unroll
          for (int x = 0; x < 8; ++x) acc[g][x] += w * f[x];
        }
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int g = 0; g < GM; ++g)
    if (lane == 0) {
      sm_m[warp][g] = m[g];
      sm_l[warp][g] = l[g];
    }
  __syncthreads();
  // merge the warps and their key groups, one query head after the other
  const int parts = ngroups * RA_WARPS;
#pragma unroll
  for (int g = 0; g < GM; ++g) {
    if (g >= ng) break;
    float gm = -INFINITY, gl = 0.f;
#pragma unroll
    for (int w = 0; w < RA_WARPS; ++w) gm = fmaxf(gm, sm_m[w][g]);
#pragma unroll
    for (int w = 0; w < RA_WARPS; ++w)
      gl += sm_m[w][g] == -INFINITY ? 0.f : sm_l[w][g] * exp2_t<T>(sm_m[w][g] - gm);
    const float c = m[g] == -INFINITY ? 0.f : exp2_t<T>(m[g] - gm);
    if (kg < ngroups) {
#pragma unroll
      for (int x = 0; x < 8; ++x)
        red[(warp * ngroups + kg) * p.vdim_p + vch * 8 + x] = acc[g][x] * c;
    }
    __syncthreads();
    const int h = h0 + g;
    const bool direct = ra.part_o == nullptr;
    const float dn = direct ? gate_of<T>(p, row, h) / denom<T>(p, h, gm, gl) : 1.f;
    for (int d = threadIdx.x; d < p.vdim; d += RA_WARPS * 32) {
      float o = 0.f;
      for (int w = 0; w < parts; ++w) o += red[w * p.vdim_p + d];
      if (direct)
        static_cast<T*>(p.out)[static_cast<size_t>(row) * p.ldo + h * p.vdim + d] =
            from_f32<T>(o * dn * gate_wide_of<T>(p, row, h * p.vdim + d));
      else
        ra.part_o[((static_cast<size_t>(i) * p.heads + h) * ra.splits + split) * p.vdim + d] = o;
    }
    if (!direct && threadIdx.x == 0) {
      float* ml = ra.part_ml + ((static_cast<size_t>(i) * p.heads + h) * ra.splits + split) * 2;
      ml[0] = gm;
      ml[1] = gl;
    }
    __syncthreads();
  }
}

template <typename T>
__global__ void __launch_bounds__(64) ragged_attn_merge_kernel(const RowsArgs ra) {
  const RaggedAttn& p = ra.a;
  const int i = blockIdx.x, h = blockIdx.y;
  const int row = ra.rows != nullptr ? ra.rows[i] : i;
  const size_t base = (static_cast<size_t>(i) * p.heads + h) * ra.splits;
  float gm = -INFINITY, gl = 0.f;
  for (int s = 0; s < ra.splits; ++s) gm = fmaxf(gm, ra.part_ml[(base + s) * 2]);
  for (int s = 0; s < ra.splits; ++s) {
    const float ms = ra.part_ml[(base + s) * 2];
    gl += ms == -INFINITY ? 0.f : ra.part_ml[(base + s) * 2 + 1] * exp2_t<T>(ms - gm);
  }
  const float dn = gate_of<T>(p, row, h) / denom<T>(p, h, gm, gl);
  for (int d = threadIdx.x; d < p.vdim; d += 64) {
    float o = 0.f;
    for (int s = 0; s < ra.splits; ++s) {
      const float ms = ra.part_ml[(base + s) * 2];
      if (ms != -INFINITY) o += ra.part_o[(base + s) * p.vdim + d] * exp2_t<T>(ms - gm);
    }
    static_cast<T*>(p.out)[static_cast<size_t>(row) * p.ldo + h * p.vdim + d] =
        from_f32<T>(o * dn * gate_wide_of<T>(p, row, h * p.vdim + d));
  }
}

// Two maps: merges the splits of both and takes their difference.  At most 256 columns.
constexpr int RA_SPLITS = 16;
template <typename T>
__global__ void __launch_bounds__(128) ragged_attn_difference_kernel(const RowsArgs ra) {
  const RaggedAttn& p = ra.a;
  __shared__ float red[32];
  __shared__ float part[2 * RA_SPLITS];          // factor of every split's sum
  const int i = blockIdx.x, h = blockIdx.y, n = ra.splits;
  const int row = ra.rows != nullptr ? ra.rows[i] : i;
  const size_t base = (static_cast<size_t>(i) * p.heads + h * 2) * n;      // the second map's follow
  if (threadIdx.x < 32) {
    // lanes 0 .. 15: the first map's splits, 16 .. 31: the second's
    const int m = threadIdx.x / RA_SPLITS, k = threadIdx.x % RA_SPLITS;
    const bool in = k < n;
    const float mk = in ? ra.part_ml[(base + m * n + k) * 2] : -INFINITY;
    const float lk = in ? ra.part_ml[(base + m * n + k) * 2 + 1] : 0.f;
    float gm = mk;
#pragma unroll
    for (int o = RA_SPLITS / 2; o > 0; o >>= 1) gm = fmaxf(gm, __shfl_xor_sync(0xffffffffu, gm, o));
    const float c = mk == -INFINITY ? 0.f : exp2_t<T>(mk - gm);
    float gl = lk * c;
#pragma unroll
    for (int o = RA_SPLITS / 2; o > 0; o >>= 1) gl += __shfl_xor_sync(0xffffffffu, gl, o);
    part[threadIdx.x] = (m == 0 ? c : -*p.map_weight * c) / gl;
  }
  __syncthreads();
  float o[2] = {0.f, 0.f};
#pragma unroll
  for (int m = 0; m < 2; ++m) {
#pragma unroll 8
    for (int k = 0; k < n; ++k) {
      const float c = part[m * RA_SPLITS + k];
      const float* src = ra.part_o + (base + m * n + k) * p.vdim;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int d = threadIdx.x + 128 * x;
        if (d < p.vdim) o[x] += c != 0.f ? src[d] * c : 0.f;     // a split without keys has no sum
      }
    }
  }
  const float ss = block_sum(o[0] * o[0] + o[1] * o[1], red);
  const float rs = p.map_factor / sqrtf(ss / p.vdim + p.eps) * gate_of<T>(p, row, h);
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int d = threadIdx.x + 128 * x;
    if (d < p.vdim)
      static_cast<T*>(p.out)[static_cast<size_t>(row) * p.ldo + h * p.vdim + d] =
          from_f32<T>(o[x] * rs * gate_wide_of<T>(p, row, h * p.vdim + d));
  }
}

template <typename T>
static void launch_merge(const RowsArgs& a, int n, cudaStream_t st) {
  if (a.a.maps == 2) {
    ragged_attn_difference_kernel<T><<<dim3(n, a.a.heads / 2), 128, 0, st>>>(a);
  } else if (a.part_o != nullptr) {
    ragged_attn_merge_kernel<T><<<dim3(n, a.a.heads), 64, 0, st>>>(a);
  }
}

// ------------------------------------------------------------------------------ tiles kernel
constexpr int TA_WARPS = 4;
constexpr int TA_ROWS = 16 * TA_WARPS;

struct TilesArgs {
  RaggedAttn a;
  Entries e;
  const int* tile_entry;   // [tiles]
  const int* tile_off;     // [tiles] first token of the tile inside its entry
  const int* tile_len;     // [tiles] its tokens, at most TA_ROWS
};

// dim <= DC, vdim <= VC, multiples of 32.  With two maps the block has warps for both: they share the
// values, and the second map's results cross to the first map's warps through shared memory.
template <int DC, int VC, int MAPS>
__global__ void __launch_bounds__(MAPS * TA_WARPS * 32) ragged_attn_tiles_kernel(const TilesArgs ta) {
  using bf16 = __nv_bfloat16;
  const RaggedAttn& p = ta.a;
  constexpr int KS = MAPS * DC + 8, VS = VC + 8;       // padded rows (elements): conflict-free ldmatrix
  constexpr int NT = MAPS * TA_WARPS * 32;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* sK = reinterpret_cast<bf16*>(smem);                      // [2][PAGE][KS]
  bf16* sV = sK + 2 * RAGGED_PAGE * KS;                          // [2][PAGE][VS]
  bf16* sQ = sV + 2 * RAGGED_PAGE * VS;                          // [TA_ROWS][KS]
  const int e = ta.tile_entry[blockIdx.x], off = ta.tile_off[blockIdx.x], h = blockIdx.y;
  const int hk = h / (p.heads / MAPS / p.kv_heads);
  const int row0 = ta.e.row0[e] + off, len = min(TA_ROWS, ta.tile_len[blockIdx.x]);
  const int pos0 = ta.e.pos0[e] + off, slot = ta.e.slot[e];
  const int tid = threadIdx.x, lane = tid & 31;
  const int warp = (tid >> 5) % TA_WARPS, map = tid / (TA_WARPS * 32);
  const int* pt = p.page_table + static_cast<size_t>(slot) * p.max_pages;
  const bf16* q = static_cast<const bf16*>(p.q);
  const bf16* kc = static_cast<const bf16*>(p.k_cache);
  const bf16* vc = static_cast<const bf16*>(p.v_cache);
  // padding columns of the rings are zero once and for all
#pragma unroll
  for (int m = 0; m < MAPS; ++m)
    for (int i = tid; i < 2 * RAGGED_PAGE * (DC - p.dim_p); i += NT)
      sK[(i / (DC - p.dim_p)) * KS + m * DC + p.dim_p + i % (DC - p.dim_p)] = __float2bfloat16(0.f);
  for (int i = tid; i < 2 * RAGGED_PAGE * (VS - p.vdim_p); i += NT)
    sV[(i / (VS - p.vdim_p)) * VS + p.vdim_p + i % (VS - p.vdim_p)] = __float2bfloat16(0.f);
  const int last = pos0 + len - 1;
  // pages of kept positions, then those from the first row's window on
  const int pg0 = first_seen(p, pos0) / RAGGED_PAGE, pg1 = last / RAGGED_PAGE;
  const int kp = min(pg0, (p.keep + RAGGED_PAGE - 1) / RAGGED_PAGE), n_pages = kp + pg1 - pg0 + 1;
  auto page_at = [&](int i) { return i < kp ? i : pg0 + i - kp; };
  auto fetch = [&](int pg, int st) {
    int page = pg < p.max_pages ? pt[pg] : -1;
    if (page < 0 || page >= p.num_pages) {
      if (tid == 0) record_status(p.status, ST_BOUNDS, row0);
      page = 0;
    }
    const int base = pg * RAGGED_PAGE;
    const int kch = p.dim_p / 8, vch = p.vdim_p / 8;
    for (int i = tid; i < RAGGED_PAGE * MAPS * kch; i += NT) {
      const int t = i / (MAPS * kch), c = i % (MAPS * kch), m = c / kch;
      const bf16* src = kc + ((static_cast<size_t>(page) * RAGGED_PAGE + t) * p.kv_heads + hk) * p.kdim + c * 8;
      cp_async16_zfill(smem_u32(sK + (st * RAGGED_PAGE + t) * KS + m * DC + (c - m * kch) * 8), src,
                       base + t <= last ? 16 : 0);
    }
    for (int i = tid; i < RAGGED_PAGE * vch; i += NT) {
      const int t = i / vch, c = i % vch;
      const bf16* src = vc + ((static_cast<size_t>(page) * RAGGED_PAGE + t) * p.kv_heads + hk) * p.vdim_p + c * 8;
      cp_async16_zfill(smem_u32(sV + (st * RAGGED_PAGE + t) * VS + c * 8), src, base + t <= last ? 16 : 0);
    }
    cp_async_commit();
  };
  fetch(page_at(0), 0);
  if (p.dim % 8 == 0 && p.q_head % 8 == 0) {
    for (int i = tid; i < TA_ROWS * MAPS * (DC / 8); i += NT) {
      const int t = i / (MAPS * (DC / 8)), x = i % (MAPS * (DC / 8)), m = x / (DC / 8), c = x % (DC / 8) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (t < len && c < p.dim)
        v = *reinterpret_cast<const uint4*>(q + (static_cast<size_t>(row0 + t) * p.heads + h * MAPS + m) * p.q_head + c);
      *reinterpret_cast<uint4*>(sQ + t * KS + m * DC + c) = v;
    }
  } else {
    for (int i = tid; i < TA_ROWS * MAPS * DC; i += NT) {
      const int t = i / (MAPS * DC), x = i % (MAPS * DC), m = x / DC, c = x % DC;
      sQ[t * KS + x] = (t < len && c < p.dim)
                           ? q[(static_cast<size_t>(row0 + t) * p.heads + h * MAPS + m) * p.q_head + c]
                           : __float2bfloat16(0.f);
    }
  }
  __syncthreads();
  uint32_t qf[DC / 16][4];
#pragma unroll
  for (int k = 0; k < DC / 16; ++k)
    ldsm4(qf[k], smem_u32(sQ + (warp * 16 + (lane & 15)) * KS + map * DC + k * 16 + (lane >> 4) * 8));
  float o[VC / 8][4];
#pragma unroll
  for (int i = 0; i < VC / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int r0 = warp * 16 + (lane >> 2);
  const int qpos[2] = {pos0 + r0, pos0 + r0 + 8};
  const int qlo[2] = {first_seen(p, qpos[0]), first_seen(p, qpos[1])};
  const int w_first = pos0 + warp * 16, w_last = min(w_first + 15, last);
  for (int i_pg = 0; i_pg < n_pages; ++i_pg) {
    const int st = i_pg & 1, base = page_at(i_pg) * RAGGED_PAGE;
    if (i_pg + 1 < n_pages) {
      fetch(page_at(i_pg + 1), st ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    // skip pages that no row of this warp sees
    if (w_first <= last && base <= w_last &&
        (base + RAGGED_PAGE > first_seen(p, w_first) || base < p.keep)) {
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
      const bf16* kb = sK + st * RAGGED_PAGE * KS;
#pragma unroll
      for (int k = 0; k < DC / 16; ++k) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {       // 16 keys: two n-tiles
          uint32_t b[4];
          ldsm4(b, smem_u32(kb + (i * 16 + (lane & 7) + (lane >> 4) * 8) * KS + map * DC + k * 16 + ((lane >> 3) & 1) * 8));
          mma_bf16(s[2 * i], qf[k], b[0], b[1]);
          mma_bf16(s[2 * i + 1], qf[k], b[2], b[3]);
        }
      }
      const bool full = (base >= first_seen(p, w_last) || base + RAGGED_PAGE <= p.keep) &&
                        base + RAGGED_PAGE - 1 <= w_first;
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = j >> 1, t = base + i * 8 + (lane & 3) * 2 + (j & 1);
          s[i][j] = (full || (t <= qpos[r] && (t >= qlo[r] || t < p.keep))) ? score_of<bf16>(p, s[i][j] * p.scale) : -INFINITY;
          mx[r] = fmaxf(mx[r], s[i][j]);
        }
      float c[2], sum[2] = {0.f, 0.f};
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float mn = fmaxf(m[r], mx[r]);
        c[r] = m[r] == -INFINITY ? 0.f : fast_exp2(m[r] - mn);
        m[r] = mn;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = j >> 1;
          s[i][j] = s[i][j] == -INFINITY ? 0.f : fast_exp2(s[i][j] - m[r]);
          sum[r] += s[i][j];
        }
      l[0] = l[0] * c[0] + sum[0];          // this lane's keys; the lanes are added at the end
      l[1] = l[1] * c[1] + sum[1];
#pragma unroll
      for (int i = 0; i < VC / 8; ++i) {
        o[i][0] *= c[0];
        o[i][1] *= c[0];
        o[i][2] *= c[1];
        o[i][3] *= c[1];
      }
      const bf16* vb = sV + st * RAGGED_PAGE * VS;
#pragma unroll
      for (int k = 0; k < 4; ++k) {         // 16 keys
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float u = s[2 * k + (x >> 1)][(x & 1) * 2], w = s[2 * k + (x >> 1)][(x & 1) * 2 + 1];
          ph[x] = pack_bf16x2(u, w);
          const float2 b = unpack_bf16x2(ph[x]);
          pl[x] = pack_bf16x2(u - b.x, w - b.y);
        }
#pragma unroll
        for (int i = 0; i < VC / 16; ++i) {
          uint32_t b[4];
          ldsm4_t(b, smem_u32(vb + (k * 16 + (lane & 15)) * VS + i * 16 + (lane >> 4) * 8));
          mma_bf16(o[2 * i], ph, b[0], b[1]);
          mma_bf16(o[2 * i + 1], ph, b[2], b[3]);
          mma_bf16(o[2 * i], pl, b[0], b[1]);
          mma_bf16(o[2 * i + 1], pl, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int t = r0 + r * 8;
    const float dn = t < len ? 1.f / denom<bf16>(p, h * MAPS + map, m[r], l[r]) : 0.f;
#pragma unroll
    for (int i = 0; i < VC / 8; ++i) {
      o[i][2 * r] *= dn;
      o[i][2 * r + 1] *= dn;
    }
  }
  if constexpr (MAPS == 2) {
    float* other = reinterpret_cast<float*>(smem);         // [TA_ROWS][VC + 8]: the rings are free
    constexpr int OS = VC + 8;
    if (map == 1) {
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int i = 0; i < VC / 8; ++i)
          *reinterpret_cast<float2*>(other + (r0 + r * 8) * OS + i * 8 + (lane & 3) * 2) =
              make_float2(o[i][2 * r], o[i][2 * r + 1]);
    }
    __syncthreads();
    if (map == 1) return;
    const float w = *p.map_weight;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VC / 8; ++i) {
        const float2 b = *reinterpret_cast<const float2*>(other + (r0 + r * 8) * OS + i * 8 + (lane & 3) * 2);
        o[i][2 * r] -= w * b.x;
        o[i][2 * r + 1] -= w * b.y;
        ss += o[i][2 * r] * o[i][2 * r] + o[i][2 * r + 1] * o[i][2 * r + 1];
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      const float f = p.map_factor / sqrtf(ss / p.vdim + p.eps);
#pragma unroll
      for (int i = 0; i < VC / 8; ++i) {
        o[i][2 * r] *= f;
        o[i][2 * r + 1] *= f;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = r0 + r * 8;
    if (t >= len) continue;
    const int row = row0 + t;
    const float dn = gate_of<bf16>(p, row, h);
    bf16* dst = static_cast<bf16*>(p.out) + static_cast<size_t>(row) * p.ldo + h * p.vdim;
    const bool pairs = (p.vdim & 1) == 0 && (p.ldo & 1) == 0;
#pragma unroll
    for (int i = 0; i < VC / 8; ++i) {
      const int d = i * 8 + (lane & 3) * 2;
      float u = o[i][r * 2] * dn, w = o[i][r * 2 + 1] * dn;
      if (p.gate_wide) {
        if (d < p.vdim) u *= gate_wide_of<bf16>(p, row, h * p.vdim + d);
        if (d + 1 < p.vdim) w *= gate_wide_of<bf16>(p, row, h * p.vdim + d + 1);
      }
      if (pairs) {
        if (d < p.vdim) *reinterpret_cast<__nv_bfloat162*>(dst + d) = __floats2bfloat162_rn(u, w);
      } else {
        if (d < p.vdim) dst[d] = __float2bfloat16(u);
        if (d + 1 < p.vdim) dst[d + 1] = __float2bfloat16(w);
      }
    }
  }
}

// ------------------------------------------------------------------------------ group kernel
// Decoding in bf16: one query row, the (up to 16) query heads of one key/value head as the rows
// of the tensor-core tile.  The warps of a CTA take blocks of 32 keys in turn, each through its
// own double-buffered ring, and their partial softmaxes are merged at the end.
constexpr int GA_WARPS = 4;
constexpr int GA_KEYS = 32;

template <int DC, int VC>
__global__ void __launch_bounds__(GA_WARPS * 32) ragged_attn_group_kernel(const RowsArgs ra) {
  using bf16 = __nv_bfloat16;
  const RaggedAttn& p = ra.a;
  constexpr int KS = DC + 8, VS = VC + 8;
  constexpr int STAGE = GA_KEYS * (KS + VS);            // elements of one stage of one warp
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* ring = reinterpret_cast<bf16*>(smem);           // [GA_WARPS][2][STAGE]
  bf16* sQ = ring + GA_WARPS * 2 * STAGE;               // [16][KS]
  __shared__ float sm_m[GA_WARPS][16], sm_l[GA_WARPS][16];
  const int i = blockIdx.x, split = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int per = p.heads / p.kv_heads, subs = (per + 15) / 16;
  const int hk = blockIdx.y / subs, h0 = hk * per + (blockIdx.y % subs) * 16;
  const int ng = min(16, (hk + 1) * per - h0);
  const int row = ra.rows != nullptr ? ra.rows[i] : i;
  const int slot = ra.row_slot[row], pos = ra.row_pos[row];
  const int* pt = p.page_table + static_cast<size_t>(slot) * p.max_pages;
  const bf16* kc = static_cast<const bf16*>(p.k_cache) + hk * p.kdim;
  const bf16* vc = static_cast<const bf16*>(p.v_cache) + hk * p.vdim_p;
  const Seen seen(p, pos);
  const int piece = (seen.n + ra.splits - 1) / ra.splits;
  const int t0 = split * piece, t1 = min(seen.n, t0 + piece);
  bf16* mine = ring + warp * 2 * STAGE;
  const int kch = p.kdim / 8, vch = p.vdim_p / 8;
  // rows of nch vectors of eight, one per key (cell), to shared memory
  auto copy = [&](const bf16* src, size_t stride, int nch, uint32_t dst, int pitch, int cell, int left) {
    if ((nch & (nch - 1)) == 0 && nch <= 32) {          // a lane keeps its column
      const int sh = __ffs(nch) - 1, c = lane & (nch - 1);
      src += c * 8;
      dst += c * 16;
#pragma unroll 4
      for (int key = lane >> sh; key < GA_KEYS; key += 32 >> sh)
        cp_async16_zfill(dst + key * pitch * 2, src + __shfl_sync(0xffffffffu, cell, key) * stride,
                         key < left ? 16 : 0);
      return;
    }
    for (int x = lane; x < GA_KEYS * nch; x += 32) {
      const int key = x / nch, c = x % nch;
      cp_async16_zfill(dst + (key * pitch + c * 8) * 2, src + __shfl_sync(0xffffffffu, cell, key) * stride + c * 8,
                       key < left ? 16 : 0);
    }
  };
  auto fetch = [&](int tb, int st) {                    // keys tb .. tb + 31 into a stage
    int cell = 0;
    if (tb + lane < t1) {
      const int t = seen.place(tb + lane), lp = t / RAGGED_PAGE;
      int page = lp < p.max_pages ? pt[lp] : -1;
      if (page < 0 || page >= p.num_pages) {
        record_status(p.status, ST_BOUNDS, row);
        page = 0;
      }
      cell = page * RAGGED_PAGE + t % RAGGED_PAGE;
    }
    const uint32_t kd = smem_u32(mine + st * STAGE);
    copy(kc, static_cast<size_t>(p.kv_heads) * p.kdim, kch, kd, KS, cell, t1 - tb);
    copy(vc, static_cast<size_t>(p.kv_heads) * p.vdim_p, vch, kd + GA_KEYS * KS * 2, VS, cell, t1 - tb);
    cp_async_commit();
  };
  // zero the padding columns of this warp's ring, then start loading
  for (int x = lane; x < 2 * GA_KEYS * (DC - p.kdim); x += 32) {
    const int r = x / (DC - p.kdim), c = p.kdim + x % (DC - p.kdim);
    mine[(r / GA_KEYS) * STAGE + (r % GA_KEYS) * KS + c] = __float2bfloat16(0.f);
  }
  for (int x = lane; x < 2 * GA_KEYS * (VC - p.vdim_p); x += 32) {
    const int r = x / (VC - p.vdim_p), c = p.vdim_p + x % (VC - p.vdim_p);
    mine[(r / GA_KEYS) * STAGE + GA_KEYS * KS + (r % GA_KEYS) * VS + c] = __float2bfloat16(0.f);
  }
  int tb = t0 + warp * GA_KEYS;
  if (tb < t1) fetch(tb, 0);
  const bf16* q = static_cast<const bf16*>(p.q) + (static_cast<size_t>(row) * p.heads + h0) * p.q_head;
  for (int x = tid; x < 16 * DC; x += GA_WARPS * 32) {
    const int g = x / DC, d = x % DC;
    const int c = d - map_off(p, h0 + g);
    sQ[g * KS + d] = g < ng && c >= 0 && c < p.dim ? q[g * p.q_head + c] : __float2bfloat16(0.f);
  }
  __syncthreads();
  uint32_t qf[DC / 16][4];
#pragma unroll
  for (int k = 0; k < DC / 16; ++k)
    ldsm4(qf[k], smem_u32(sQ + (lane & 15) * KS + k * 16 + (lane >> 4) * 8));
  float o[VC / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int x = 0; x < VC / 8; ++x)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[x][j] = 0.f;
  for (int st = 0; tb < t1; tb += GA_WARPS * GA_KEYS, st ^= 1) {
    if (tb + GA_WARPS * GA_KEYS < t1) {
      fetch(tb + GA_WARPS * GA_KEYS, st ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncwarp();
    const bf16* kb = mine + st * STAGE;
    const bf16* vb = kb + GA_KEYS * KS;
    float s[4][4];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[x][j] = 0.f;
#pragma unroll
    for (int k = 0; k < DC / 16; ++k)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        uint32_t b[4];
        ldsm4(b, smem_u32(kb + (x * 16 + (lane & 7) + (lane >> 4) * 8) * KS + k * 16 + ((lane >> 3) & 1) * 8));
        mma_bf16(s[2 * x], qf[k], b[0], b[1]);
        mma_bf16(s[2 * x + 1], qf[k], b[2], b[3]);
      }
    float mx[2] = {-INFINITY, -INFINITY}, c[2];
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = tb + x * 8 + (lane & 3) * 2 + (j & 1);
        s[x][j] = t < t1 ? score_of<bf16>(p, s[x][j] * p.scale) : -INFINITY;
        mx[j >> 1] = fmaxf(mx[j >> 1], s[x][j]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float mn = fmaxf(m[r], mx[r]);              // finite: the block has a key
      c[r] = fast_exp2(m[r] - mn);
      m[r] = mn;
      l[r] *= c[r];
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[x][j] = fast_exp2(s[x][j] - m[j >> 1]);
        l[j >> 1] += s[x][j];
      }
#pragma unroll
    for (int x = 0; x < VC / 8; ++x)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[x][j] *= c[j >> 1];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float u = s[2 * k + (x >> 1)][(x & 1) * 2], w = s[2 * k + (x >> 1)][(x & 1) * 2 + 1];
        ph[x] = pack_bf16x2(u, w);
        const float2 f = unpack_bf16x2(ph[x]);
        pl[x] = pack_bf16x2(u - f.x, w - f.y);
      }
#pragma unroll
      for (int x = 0; x < VC / 16; ++x) {
        uint32_t b[4];
        ldsm4_t(b, smem_u32(vb + (k * 16 + (lane & 15)) * VS + x * 16 + (lane >> 4) * 8));
        mma_bf16(o[2 * x], ph, b[0], b[1]);
        mma_bf16(o[2 * x + 1], ph, b[2], b[3]);
        mma_bf16(o[2 * x], pl, b[0], b[1]);
        mma_bf16(o[2 * x + 1], pl, b[2], b[3]);
      }
    }
    __syncwarp();                                       // before the stage is filled again
  }
  // merge the warps through shared memory (the rings are free): [GA_WARPS][16][VC]
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if ((lane & 3) == 0) {
      sm_m[warp][(lane >> 2) + 8 * r] = m[r];
      sm_l[warp][(lane >> 2) + 8 * r] = l[r];
    }
  }
  __syncthreads();
  float* red = reinterpret_cast<float*>(smem);
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int g = (lane >> 2) + 8 * r;
    float gm = -INFINITY;
#pragma unroll
    for (int w = 0; w < GA_WARPS; ++w) gm = fmaxf(gm, sm_m[w][g]);
    const float c = m[r] == -INFINITY ? 0.f : fast_exp2(m[r] - gm);
#pragma unroll
    for (int x = 0; x < VC / 8; ++x)
      *reinterpret_cast<float2*>(red + (warp * 16 + g) * VC + x * 8 + (lane & 3) * 2) =
          make_float2(o[x][2 * r] * c, o[x][2 * r + 1] * c);
  }
  __syncthreads();
  for (int g = warp; g < ng; g += GA_WARPS) {
    const int h = h0 + g;
    float gm = -INFINITY, gl = 0.f;
#pragma unroll
    for (int w = 0; w < GA_WARPS; ++w) gm = fmaxf(gm, sm_m[w][g]);
#pragma unroll
    for (int w = 0; w < GA_WARPS; ++w)
      gl += sm_m[w][g] == -INFINITY ? 0.f : sm_l[w][g] * fast_exp2(sm_m[w][g] - gm);
    const size_t part = (static_cast<size_t>(i) * p.heads + h) * ra.splits + split;
    const bool direct = ra.part_o == nullptr;
    const float dn = direct ? gate_of<bf16>(p, row, h) / denom<bf16>(p, h, gm, gl) : 1.f;
    for (int d = lane; d < p.vdim; d += 32) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < GA_WARPS; ++w) v += red[(w * 16 + g) * VC + d];
      if (direct)
        static_cast<bf16*>(p.out)[static_cast<size_t>(row) * p.ldo + h * p.vdim + d] =
            __float2bfloat16(v * dn * gate_wide_of<bf16>(p, row, h * p.vdim + d));
      else
        ra.part_o[part * p.vdim + d] = v;
    }
    if (!direct && lane == 0) {
      ra.part_ml[part * 2] = gm;
      ra.part_ml[part * 2 + 1] = gl;
    }
  }
}

template <int DC, int VC>
static int launch_group(const RowsArgs& a, int n, cudaStream_t st) {
  constexpr int ring = GA_WARPS * 2 * GA_KEYS * (DC + 8 + VC + 8) * 2 + 16 * (DC + 8) * 2;
  constexpr int merge = GA_WARPS * 16 * VC * 4;
  constexpr int smem = ring > merge ? ring : merge;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ragged_attn_group_kernel<DC, VC>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -4;
    set = true;
  }
  const int per = a.a.heads / a.a.kv_heads;
  dim3 grid(n, a.a.kv_heads * ((per + 15) / 16), a.splits);
  ragged_attn_group_kernel<DC, VC><<<grid, GA_WARPS * 32, smem, st>>>(a);
  launch_merge<__nv_bfloat16>(a, n, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int DC>
static int launch_group_v(const RowsArgs& a, int n, cudaStream_t st) {
  if (a.a.vdim <= 64) return launch_group<DC, 64>(a, n, st);
  return launch_group<DC, 128>(a, n, st);
}

template <int DC, int VC, int MAPS>
static int launch_tiles(const TilesArgs& a, int tiles, cudaStream_t st) {
  const int ring = (2 * RAGGED_PAGE * (MAPS * DC + 8) + 2 * RAGGED_PAGE * (VC + 8) + TA_ROWS * (MAPS * DC + 8)) * 2;
  const int other = MAPS == 2 ? TA_ROWS * (VC + 8) * 4 : 0;
  const int smem = ring > other ? ring : other;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ragged_attn_tiles_kernel<DC, VC, MAPS>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return -4;
    set = true;
  }
  dim3 grid(tiles, a.a.heads / MAPS);
  ragged_attn_tiles_kernel<DC, VC, MAPS><<<grid, MAPS * TA_WARPS * 32, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int DC, int MAPS>
static int launch_tiles_v(const TilesArgs& a, int tiles, cudaStream_t st) {
  if (a.a.vdim <= 64) return launch_tiles<DC, 64, MAPS>(a, tiles, st);
  if (a.a.vdim <= 128) return launch_tiles<DC, 128, MAPS>(a, tiles, st);
  return launch_tiles<DC, 256, MAPS>(a, tiles, st);
}

template <typename T, int KIT>
static int launch_rows(const RowsArgs& a, int n, cudaStream_t st) {
  const int per = a.a.heads / a.a.kv_heads;
#define CB_ROWS(GM_)                                                                         \
  do {                                                                                       \
    dim3 grid(n, a.a.kv_heads * ((per + GM_ - 1) / GM_), a.splits);                          \
    ragged_attn_rows_kernel<T, KIT, GM_><<<grid, RA_WARPS * 32, 0, st>>>(a);                 \
  } while (0)
  if (per == 1) CB_ROWS(1);
  else if (per == 2) CB_ROWS(2);
  else if (per <= 4) CB_ROWS(4);
  else CB_ROWS(8);
#undef CB_ROWS
  launch_merge<T>(a, n, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <typename T>
static int launch_rows_d(const RowsArgs& a, int n, cudaStream_t st) {
  if (a.a.kdim <= 64) return launch_rows<T, 1>(a, n, st);
  if (a.a.kdim <= 128) return launch_rows<T, 2>(a, n, st);
  if (a.a.kdim <= 256) return launch_rows<T, 4>(a, n, st);
  return launch_rows<T, 8>(a, n, st);
}

}  // namespace cb

using namespace cb;

static int fill_attn(RaggedAttn& p, const void* q, int q_head, const void* k_cache, const void* v_cache,
                     const int* page_table, int max_pages, int num_pages, const RaggedSpec& c,
                     const float* sink, const void* gate, int ldg, const float* map_weight, void* out,
                     int ldo, int* status) {
  if (c.kv_heads < 1 || c.heads % c.kv_heads != 0 || c.dim < 1 || c.vdim < 1 || c.dim > 256 || c.vdim > 256)
    return -1;
  if (c.dim_p % 8 != 0 || c.vdim_p % 8 != 0 || c.dim_p < c.dim || c.vdim_p < c.vdim || c.dim_p > 256 ||
      c.vdim_p > 256)
    return -2;
  if (c.maps == 2 && sink != nullptr) return -2;
  if ((c.maps != 1 && c.maps != 2) || (c.maps == 2 && map_weight == nullptr) || c.window < 0 || c.chunk < 0 || c.keep < 0 ||
      (c.window > 0 && c.chunk > 0) || c.softcap < 0.f)
    return -2;
  p.q = q; p.q_head = q_head; p.k_cache = k_cache; p.v_cache = v_cache; p.page_table = page_table;
  p.max_pages = max_pages; p.num_pages = num_pages; p.heads = c.heads * c.maps; p.kv_heads = c.kv_heads;
  p.dim = c.dim; p.vdim = c.vdim; p.dim_p = c.dim_p; p.vdim_p = c.vdim_p; p.maps = c.maps;
  p.kdim = c.maps * c.dim_p; p.chunk = c.chunk; p.window = c.window; p.keep = c.window > 0 ? c.keep : 0;
  p.scale = c.softcap > 0.f ? c.scale / c.softcap : c.scale * LOG2E;
  p.cap = c.softcap * LOG2E;
  p.sink = sink; p.gate = gate; p.ldg = ldg; p.gate_wide = c.gate_wide; p.map_weight = map_weight;
  p.map_factor = c.map_factor; p.eps = c.eps; p.out = out; p.ldo = ldo; p.status = status;
  return 0;
}

extern "C" int cb_ragged_attn_tile() { return TA_ROWS; }

extern "C" int cb_ragged_attn_rows(const void* q, int q_head, const void* k_cache, const void* v_cache,
                                   const int* page_table, int max_pages, int num_pages,
                                   const RaggedSpec* spec, const float* sink, const void* gate, int ldg,
                                   const float* map_weight, void* out, int ldo, const int* rows,
                                   const int* row_slot, const int* row_pos, int n, int splits,
                                   float* part_o, float* part_ml, int f32, int* status, void* stream) {
  RowsArgs a;
  const int rc = fill_attn(a.a, q, q_head, k_cache, v_cache, page_table, max_pages, num_pages, *spec, sink,
                           gate, ldg, map_weight, out, ldo, status);
  if (rc != 0) return rc;
  if (n <= 0 || splits < 1 || (spec->maps == 2 && splits > RA_SPLITS) || ((splits > 1 || spec->maps == 2) && (part_o == nullptr || part_ml == nullptr)))
    return -5;
  a.rows = rows; a.row_slot = row_slot; a.row_pos = row_pos; a.splits = splits;
  a.part_o = part_o; a.part_ml = part_ml;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return launch_rows_d<float>(a, n, st);
  if (a.a.kdim > 256) return launch_rows<__nv_bfloat16, 8>(a, n, st);
  if (a.a.kdim > 128 || a.a.vdim > 128) return launch_rows<__nv_bfloat16, 4>(a, n, st);
  return a.a.kdim <= 64 ? launch_group_v<64>(a, n, st) : launch_group_v<128>(a, n, st);
}

extern "C" int cb_ragged_attn_tiles(const void* q, int q_head, const void* k_cache, const void* v_cache,
                                    const int* page_table, int max_pages, int num_pages,
                                    const RaggedSpec* spec, const float* sink, const void* gate, int ldg,
                                    const float* map_weight, void* out, int ldo, const int* slot,
                                    const int* row0, const int* len, const int* pos0,
                                    const int* tile_entry, const int* tile_off, const int* tile_len,
                                    int tiles, int* status, void* stream) {
  TilesArgs a;
  const int rc = fill_attn(a.a, q, q_head, k_cache, v_cache, page_table, max_pages, num_pages, *spec, sink,
                           gate, ldg, map_weight, out, ldo, status);
  if (rc != 0) return rc;
  if (tiles <= 0) return -5;
  a.e.slot = slot; a.e.row0 = row0; a.e.len = len; a.e.pos0 = pos0;
  a.tile_entry = tile_entry; a.tile_off = tile_off; a.tile_len = tile_len;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int dim = a.a.dim;
  if (spec->maps == 2) {
    if (dim <= 64) return launch_tiles_v<64, 2>(a, tiles, st);
    if (dim <= 128) return launch_tiles_v<128, 2>(a, tiles, st);
    return -6;
  }
  if (dim <= 64) return launch_tiles_v<64, 1>(a, tiles, st);
  if (dim <= 128) return launch_tiles_v<128, 1>(a, tiles, st);
  return launch_tiles_v<256, 1>(a, tiles, st);
}
