// Attention over a compressed cache: one row of `rank` latent numbers and `rot` rotated key numbers
// per token, shared by all heads.
//
//   latent_prep   behind the projections: RMS norm of the latent, rotation of the shared key part
//                 and of every query head's rotated part (pairs of neighbours), the write of the
//                 token's row into the cache pages (and, when given, row by row into a buffer)
//   rows / group  attention with the queries brought into the latent space ([rank | rot] numbers per
//                 head): score = q . row, value = the row's first `rank` numbers.  A position sees
//                 itself and the window - 1 positions before it (window = 0: all of them).
//                 group (bf16): up to 16 query heads of one row are the rows of an mma tile, 64
//                 cached rows at a time through a double-buffered ring in shared memory, the eight
//                 warps splitting the keys for the scores and the latent columns for the values.
//                 rows (fp32): a CTA per query row and head.
#include "ragged.cuh"

namespace cb {

constexpr float LA_LOG2E = 1.4426950408889634f;

struct LatentPrep {
  const void* raw;         // [rows, ld]: queries at qoff, latent and shared key part at doff
  int ld, qoff, doff;
  int heads, dim, rot, rank;
  const float* norm;       // [rank]
  float eps;
  const float2* rope;      // [rows, rot / 2] (cos, sin)
  void* q;                 // out [rows, heads, q_head], zeros behind dim + rot
  int q_head;
  void* cache;             // [pages, PAGE, lat_p]
  int lat_p;
  void* rows_out;          // out [rows, lat_p] or null
  const int* page_table;
  int max_pages, num_pages;
  const int* row_slot;
  const int* row_pos;
  int* status;
};

// V = 8: dim, rot, rank, q_head and the row sizes are multiples of eight, rank at most 2048; V = 1:
// any sizes
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrep p) {
  __shared__ float red[32];
  const int row = blockIdx.x;
  const T* raw = static_cast<const T*>(p.raw) + static_cast<size_t>(row) * p.ld;
  const T* lat = raw + p.doff;
  const float2* rope = p.rope + static_cast<size_t>(row) * (p.rot / 2);
  const int pos = p.row_pos[row], lp = pos / RAGGED_PAGE;
  int page = lp < p.max_pages ? p.page_table[static_cast<size_t>(p.row_slot[row]) * p.max_pages + lp] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0) record_status(p.status, ST_BOUNDS, row);
    page = -1;
  }
  T* cell = page < 0 ? nullptr
                     : static_cast<T*>(p.cache) + (static_cast<size_t>(page) * RAGGED_PAGE + pos % RAGGED_PAGE) * p.lat_p;
  T* keep = p.rows_out != nullptr ? static_cast<T*>(p.rows_out) + static_cast<size_t>(row) * p.lat_p : nullptr;
  float s = 0.f, own[V];                     // V = 8: a thread has eight numbers of the row
  const int c8 = threadIdx.x * 8;
  if constexpr (V == 8) {
    if (c8 < p.rank + p.rot) load_vec<V>(lat + c8, own);
    if (c8 < p.rank)
#pragma unroll
      for (int k = 0; k < V; ++k) s += own[k] * own[k];
  } else {
    for (int c = threadIdx.x; c < p.rank; c += blockDim.x) s += to_f32(lat[c]) * to_f32(lat[c]);
  }
  const int units = p.q_head / V, full = p.dim + p.rot;
  T* q = static_cast<T*>(p.q) + static_cast<size_t>(row) * p.heads * p.q_head;
  for (int i = threadIdx.x; i < p.heads * units; i += blockDim.x) {
    const int h = i / units, d = (i % units) * V;
    const T* src = raw + p.qoff + h * full;
    float o[V];
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = 0.f;
    if (d < p.dim) {
      load_vec<V>(src + d, o);
    } else if (d < full) {
      if constexpr (V == 1) {
        const int k = (d - p.dim) / 2, odd = (d - p.dim) & 1;
        const float a = to_f32(src[p.dim + 2 * k]), b = to_f32(src[p.dim + 2 * k + 1]);
        const float2 cs = rope[k];
        o[0] = odd ? b * cs.x + a * cs.y : a * cs.x - b * cs.y;
      } else {
        float f[V];
        load_vec<V>(src + d, f);
#pragma unroll
        for (int k = 0; k < V; k += 2) {
          const float2 cs = rope[(d - p.dim + k) / 2];
          o[k] = f[k] * cs.x - f[k + 1] * cs.y;
          o[k + 1] = f[k + 1] * cs.x + f[k] * cs.y;
        }
      }
    }
    store_vec<V>(q + h * p.q_head + d, o);
  }
  s = block_sum(s, red);
  const float rs = 1.0f / sqrtf(s / p.rank + p.eps);
  if constexpr (V == 8) {
    if (c8 >= p.lat_p) return;
    float o[V];
    if (c8 < p.rank) {
      float g[V];
      load_vec<V>(p.norm + c8, g);
#pragma unroll
      for (int k = 0; k < V; ++k) o[k] = own[k] * rs * g[k];
    } else {
#pragma unroll
      for (int k = 0; k < V; k += 2) {
        const float2 cs = rope[(c8 - p.rank + k) / 2];
        o[k] = own[k] * cs.x - own[k + 1] * cs.y;
        o[k + 1] = own[k + 1] * cs.x + own[k] * cs.y;
      }
    }
    if (cell != nullptr) store_vec<V>(cell + c8, o);
    if (keep != nullptr) store_vec<V>(keep + c8, o);
  } else {
    for (int c = threadIdx.x; c < p.lat_p; c += blockDim.x) {
      float v = 0.f;
      if (c < p.rank) {
        v = to_f32(lat[c]) * rs * p.norm[c];
      } else if (c < p.rank + p.rot) {
        const int i = (c - p.rank) / 2, odd = (c - p.rank) & 1;
        const float a = to_f32(lat[p.rank + 2 * i]), b = to_f32(lat[p.rank + 2 * i + 1]);
        const float2 cs = rope[i];
        v = odd ? b * cs.x + a * cs.y : a * cs.x - b * cs.y;
      }
      const T o = from_f32<T>(v);
      if (cell != nullptr) cell[c] = o;
      if (keep != nullptr) keep[c] = o;
    }
  }
}

struct LatentAttn {
  const void* q;           // [n, heads, lat_p]
  const void* cache;       // [pages, PAGE, lat_p]
  const int* page_table;
  int max_pages, num_pages;
  int heads, lat, lat_p, rank, rank_p;
  int window;
  float scale;
  void* out;               // [n, heads, rank_p]
  const int* rows;         // [n] row of the batch
  const int* row_slot;
  const int* row_pos;
  int splits;
  float* part_o;           // [n, heads, splits, rank]
  float* part_ml;          // [n, heads, splits, 2]
  int* status;
};

// keys of split s of query row i: t0 .. t1 - 1
__device__ __forceinline__ void latent_range(const LatentAttn& p, int pos, int split, int& t0, int& t1) {
  const int lo = p.window > 0 ? max(0, pos + 1 - p.window) : 0, n = pos + 1 - lo;
  const int piece = (n + p.splits - 1) / p.splits;
  t0 = lo + split * piece;
  t1 = min(pos + 1, t0 + piece);
}
__device__ __forceinline__ int latent_page(const LatentAttn& p, const int* pt, int t, int row) {
  const int lp = t / RAGGED_PAGE;
  const int page = lp < p.max_pages ? pt[lp] : -1;
  if (page >= 0 && page < p.num_pages) return page;
  record_status(p.status, ST_BOUNDS, row);
  return 0;
}

constexpr int LA_WARPS = 8;
constexpr int LA_KEYS = 8 * LA_WARPS;
constexpr int LA_PS = LA_KEYS + 8;        // pitch of the weights (bf16)
constexpr int LA_SS = LA_KEYS + 2;        // pitch of the scores (fp32)

__host__ __device__ constexpr int latent_pitch(int lat) { return (lat + 31) / 32 * 32 + 8; }
static int latent_smem(int lat) {
  const int LS = latent_pitch(lat);
  return (2 * LA_KEYS * LS + 16 * LS + 2 * 16 * LA_PS) * 2 + (16 * LA_SS + 3 * 16) * 4;
}

template <int NV>          // 16-wide column groups per warp: rank <= 128 NV
__global__ void __launch_bounds__(LA_WARPS * 32) latent_group_kernel(const LatentAttn p) {
  using bf16 = __nv_bfloat16;
  extern __shared__ __align__(16) unsigned char la_smem[];
  const int LS = latent_pitch(p.lat);
  bf16* sK = reinterpret_cast<bf16*>(la_smem);          // [2][LA_KEYS][LS]
  bf16* sQ = sK + 2 * LA_KEYS * LS;                     // [16][LS]
  bf16* sP = sQ + 16 * LS;                              // [2][16][LA_PS] weights, high and low part
  float* sS = reinterpret_cast<float*>(sP + 2 * 16 * LA_PS);   // [16][LA_SS]
  float* sC = sS + 16 * LA_SS;                          // [16] correction, then m and l at the end
  const int i = blockIdx.x, h0 = blockIdx.y * 16, split = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ng = min(16, p.heads - h0);
  const int row = p.rows[i], pos = p.row_pos[row];
  const int* pt = p.page_table + static_cast<size_t>(p.row_slot[row]) * p.max_pages;
  int t0, t1;
  latent_range(p, pos, split, t0, t1);
  const bf16* cache = static_cast<const bf16*>(p.cache);
  const int chunks = p.lat_p / 8;
  auto fetch = [&](int tb, int st) {                    // rows tb .. tb + 63: at most two pages
    const int pa = latent_page(p, pt, tb, row);
    const int tl = min(tb + LA_KEYS, t1) - 1, pb = latent_page(p, pt, tl, row);
    for (int x = tid; x < LA_KEYS * chunks; x += LA_WARPS * 32) {
      const int key = x / chunks, c = x % chunks, t = tb + key;
      const int page = t / RAGGED_PAGE == tb / RAGGED_PAGE ? pa : pb;
      cp_async16_zfill(smem_u32(sK + (st * LA_KEYS + key) * LS + c * 8),
                       cache + (static_cast<size_t>(page) * RAGGED_PAGE + t % RAGGED_PAGE) * p.lat_p + c * 8,
                       t < t1 ? 16 : 0);
    }
    cp_async_commit();
  };
  if (t0 < t1) fetch(t0, 0);
  const int lat32 = LS - 8, tail = LS - p.lat_p;        // columns behind lat_p are zero
  for (int x = tid; x < 2 * LA_KEYS * tail; x += LA_WARPS * 32)
    sK[(x / tail) * LS + p.lat_p + x % tail] = __float2bfloat16(0.f);
  const bf16* q = static_cast<const bf16*>(p.q) + (static_cast<size_t>(i) * p.heads + h0) * p.lat_p;
  for (int x = tid; x < 16 * (LS / 8); x += LA_WARPS * 32) {
    const int g = x / (LS / 8), c = (x % (LS / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (g < ng && c < p.lat_p) v = *reinterpret_cast<const uint4*>(q + static_cast<size_t>(g) * p.lat_p + c);
    *reinterpret_cast<uint4*>(sQ + g * LS + c) = v;
  }
  float o[NV][2][4];
#pragma unroll
  for (int a = 0; a < NV; ++a)
#pragma unroll
    for (int b = 0; b < 2; ++b)
#pragma unroll
      for (int c = 0; c < 4; ++c) o[a][b][c] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};   // of heads 2 warp and 2 warp + 1
  const float sl2 = p.scale * LA_LOG2E;
  for (int tb = t0, st = 0; tb < t1; tb += LA_KEYS, st ^= 1) {
    if (tb + LA_KEYS < t1) {
      fetch(tb + LA_KEYS, st ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* kb = sK + st * LA_KEYS * LS;
    {                                                   // scores of this warp's eight keys
      float s[4] = {0.f, 0.f, 0.f, 0.f}, u[4] = {0.f, 0.f, 0.f, 0.f};
      const bf16* mine = kb + (warp * 8 + (lane & 7)) * LS + (lane >> 3) * 8;
      const bf16* qa = sQ + (lane & 15) * LS + (lane >> 4) * 8;
#pragma unroll 4
      for (int k = 0; k < lat32; k += 32) {
        uint32_t b[4], a[4], c[4];
        ldsm4(b, smem_u32(mine + k));
        ldsm4(a, smem_u32(qa + k));
        ldsm4(c, smem_u32(qa + k + 16));
        mma_bf16(s, a, b[0], b[1]);
        mma_bf16(u, c, b[2], b[3]);
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int key = warp * 8 + (lane & 3) * 2 + (x & 1);
        sS[((lane >> 2) + 8 * (x >> 1)) * LA_SS + key] = tb + key < t1 ? (s[x] + u[x]) * sl2 : -INFINITY;
      }
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < 2; ++x) {                       // softmax of two heads
      const int g = warp * 2 + x;
      const float a = sS[g * LA_SS + lane], b = sS[g * LA_SS + 32 + lane];
      const float mn = fmaxf(m[x], warp_max(fmaxf(a, b)));     // finite: the block has a key
      const float c = fast_exp2(m[x] - mn), wa = fast_exp2(a - mn), wb = fast_exp2(b - mn);
      m[x] = mn;
      l[x] = l[x] * c + warp_sum(wa + wb);
      const bf16 ha = __float2bfloat16(wa), hb = __float2bfloat16(wb);
      sP[g * LA_PS + lane] = ha;
      sP[g * LA_PS + 32 + lane] = hb;
      sP[(16 + g) * LA_PS + lane] = __float2bfloat16(wa - __bfloat162float(ha));
      sP[(16 + g) * LA_PS + 32 + lane] = __float2bfloat16(wb - __bfloat162float(hb));
      if (lane == 0) sC[g] = c;
    }
    __syncthreads();
    const float c0 = sC[lane >> 2], c1 = sC[(lane >> 2) + 8];
#pragma unroll
    for (int a = 0; a < NV; ++a)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        o[a][b][0] *= c0;
        o[a][b][1] *= c0;
        o[a][b][2] *= c1;
        o[a][b][3] *= c1;
      }
#pragma unroll
    for (int k = 0; k < LA_KEYS / 16; ++k) {
      uint32_t ph[4], pl[4];
      ldsm4(ph, smem_u32(sP + (lane & 15) * LA_PS + k * 16 + (lane >> 4) * 8));
      ldsm4(pl, smem_u32(sP + (16 + (lane & 15)) * LA_PS + k * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int a = 0; a < NV; ++a) {
        const int col = (warp * NV + a) * 16;
        if (col < p.rank) {
          uint32_t b[4];
          ldsm4_t(b, smem_u32(kb + (k * 16 + (lane & 15)) * LS + col + (lane >> 4) * 8));
          mma_bf16(o[a][0], ph, b[0], b[1]);
          mma_bf16(o[a][1], ph, b[2], b[3]);
          mma_bf16(o[a][0], pl, b[0], b[1]);
          mma_bf16(o[a][1], pl, b[2], b[3]);
        }
      }
    }
    __syncthreads();                                    // before the stage is filled again
  }
  if (lane < 2) {
    sC[16 + warp * 2 + lane] = lane ? m[1] : m[0];
    sC[32 + warp * 2 + lane] = lane ? l[1] : l[0];
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int g = (lane >> 2) + 8 * e;
    if (g >= ng) continue;
    const size_t at = static_cast<size_t>(i) * p.heads + h0 + g;
    const float dn = p.splits == 1 ? 1.0f / sC[32 + g] : 1.f;
#pragma unroll
    for (int a = 0; a < NV; ++a)
#pragma unroll
      for (int b = 0; b < 2; ++b)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int col = (warp * NV + a) * 16 + b * 8 + (lane & 3) * 2 + c;
          if (col >= p.rank) continue;
          const float v = o[a][b][e * 2 + c] * dn;
          if (p.splits == 1) static_cast<bf16*>(p.out)[at * p.rank_p + col] = __float2bfloat16(v);
          else p.part_o[(at * p.splits + split) * p.rank + col] = v;
        }
  }
  if (p.splits > 1 && tid < ng) {
    const size_t at = static_cast<size_t>(i) * p.heads + h0 + tid;
    p.part_ml[(at * p.splits + split) * 2] = sC[16 + tid];
    p.part_ml[(at * p.splits + split) * 2 + 1] = sC[32 + tid];
  }
}

__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentAttn p) {
  const size_t at = static_cast<size_t>(blockIdx.x) * p.heads + blockIdx.y;
  const float* ml = p.part_ml + at * p.splits * 2;
  float gm = -INFINITY, gl = 0.f;
  for (int s = 0; s < p.splits; ++s) gm = fmaxf(gm, ml[2 * s]);
  for (int s = 0; s < p.splits; ++s)
    gl += ml[2 * s] == -INFINITY ? 0.f : ml[2 * s + 1] * fast_exp2(ml[2 * s] - gm);
  const float dn = 1.0f / gl;
  for (int d = threadIdx.x; d < p.rank; d += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < p.splits; ++s)
      if (ml[2 * s] != -INFINITY)
        o += p.part_o[(at * p.splits + s) * p.rank + d] * fast_exp2(ml[2 * s] - gm);
    static_cast<__nv_bfloat16*>(p.out)[at * p.rank_p + d] = __float2bfloat16(o * dn);
  }
}

// fp32: the warps of a CTA take the keys in turn; a lane holds every 32nd number of the query and of
// the weighted sum.
constexpr int LR_WARPS = 4;
constexpr int LR_MAX = 20;                 // lat <= 640

__global__ void __launch_bounds__(LR_WARPS * 32) latent_rows_f32_kernel(const LatentAttn p) {
  __shared__ float red[LR_WARPS][LR_MAX * 32];
  __shared__ float sm[LR_WARPS], sl[LR_WARPS];
  const int i = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = p.rows[i], pos = p.row_pos[row];
  const int* pt = p.page_table + static_cast<size_t>(p.row_slot[row]) * p.max_pages;
  const size_t at = static_cast<size_t>(i) * p.heads + h;
  const float* qp = static_cast<const float*>(p.q) + at * p.lat_p;
  float q[LR_MAX], acc[LR_MAX], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int k = 0; k < LR_MAX; ++k) {
    q[k] = lane + 32 * k < p.lat ? qp[lane + 32 * k] * (p.scale * LA_LOG2E) : 0.f;
    acc[k] = 0.f;
  }
  int t0, t1;
  latent_range(p, pos, 0, t0, t1);
  for (int t = t0 + warp; t < t1; t += LR_WARPS) {
    const int page = latent_page(p, pt, t, row);
    const float* kp = static_cast<const float*>(p.cache) +
                      (static_cast<size_t>(page) * RAGGED_PAGE + t % RAGGED_PAGE) * p.lat_p;
    float f[LR_MAX], s = 0.f;
#pragma unroll
    for (int k = 0; k < LR_MAX; ++k) {
      f[k] = lane + 32 * k < p.lat ? kp[lane + 32 * k] : 0.f;
      s += q[k] * f[k];
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s), c = exp2f(m - mn), w = exp2f(s - mn);
    m = mn;
    l = l * c + w;
#pragma unroll
    for (int k = 0; k < LR_MAX; ++k) acc[k] = acc[k] * c + w * f[k];
  }
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
  for (int k = 0; k < LR_MAX; ++k) red[warp][lane + 32 * k] = acc[k];
  __syncthreads();
  float gm = -INFINITY, gl = 0.f, c[LR_WARPS];
#pragma unroll
  for (int w = 0; w < LR_WARPS; ++w) gm = fmaxf(gm, sm[w]);
#pragma unroll
  for (int w = 0; w < LR_WARPS; ++w) {
    c[w] = sm[w] == -INFINITY ? 0.f : exp2f(sm[w] - gm);
    gl += sl[w] * c[w];
  }
  for (int d = threadIdx.x; d < p.rank; d += LR_WARPS * 32) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < LR_WARPS; ++w) o += red[w][d] * c[w];
    static_cast<float*>(p.out)[at * p.rank_p + d] = o / gl;
  }
}

template <int NV>
static int launch_latent_group(const LatentAttn& p, int n, cudaStream_t st) {
  const int smem = latent_smem(p.lat);
  static int set = 0;
  if (smem > set) {
    if (cudaFuncSetAttribute(latent_group_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             smem) != cudaSuccess)
      return -4;
    set = smem;
  }
  latent_group_kernel<NV><<<dim3(n, (p.heads + 15) / 16, p.splits), LA_WARPS * 32, smem, st>>>(p);
  if (p.splits > 1) latent_merge_kernel<<<dim3(n, p.heads), 128, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

using namespace cb;

extern "C" int cb_latent_prep(const void* raw, int ld, int qoff, int doff, int heads, int dim, int rot,
                              int rank, const float* norm, float eps, const void* rope, void* q,
                              int q_head, void* cache, int lat_p, void* rows_out,
                              const int* page_table, int max_pages, int num_pages,
                              const int* row_slot, const int* row_pos, int rows, int f32, int* status,
                              void* stream) {
  if (rows <= 0 || heads < 1 || rot % 2 || q_head < dim + rot || lat_p < rank + rot) return -1;
  LatentPrep p;
  p.raw = raw; p.ld = ld; p.qoff = qoff; p.doff = doff; p.heads = heads; p.dim = dim; p.rot = rot;
  p.rank = rank; p.norm = norm; p.eps = eps; p.rope = static_cast<const float2*>(rope); p.q = q;
  p.q_head = q_head; p.cache = cache; p.lat_p = lat_p; p.rows_out = rows_out;
  p.page_table = page_table; p.max_pages = max_pages; p.num_pages = num_pages;
  p.row_slot = row_slot; p.row_pos = row_pos; p.status = status;
  const bool vec = dim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && lat_p == rank + rot && lat_p <= 2048 &&
                   q_head % 8 == 0 && ld % 8 == 0 && qoff % 8 == 0 && doff % 8 == 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) {
    if (vec) latent_prep_kernel<float, 8><<<rows, 256, 0, st>>>(p);
    else latent_prep_kernel<float, 1><<<rows, 256, 0, st>>>(p);
  } else {
    if (vec) latent_prep_kernel<__nv_bfloat16, 8><<<rows, 256, 0, st>>>(p);
    else latent_prep_kernel<__nv_bfloat16, 1><<<rows, 256, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int cb_latent_attn(const void* q, const void* cache, const int* page_table, int max_pages,
                              int num_pages, int heads, int lat, int lat_p, int rank, int rank_p,
                              int window, float scale, void* out, const int* rows,
                              const int* row_slot, const int* row_pos, int n, int splits,
                              float* part_o, float* part_ml, int f32, int* status, void* stream) {
  if (n <= 0 || heads < 1 || lat < rank || lat > 32 * LR_MAX || rank < 1 || lat_p % 8 || lat_p < lat ||
      rank_p < rank || splits < 1)
    return -1;
  if (splits > 1 && (f32 || part_o == nullptr || part_ml == nullptr)) return -2;
  LatentAttn p;
  p.q = q; p.cache = cache; p.page_table = page_table; p.max_pages = max_pages;
  p.num_pages = num_pages; p.heads = heads; p.lat = lat; p.lat_p = lat_p; p.rank = rank;
  p.rank_p = rank_p; p.window = window; p.scale = scale; p.out = out; p.rows = rows;
  p.row_slot = row_slot; p.row_pos = row_pos; p.splits = splits; p.part_o = part_o;
  p.part_ml = part_ml; p.status = status;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) {
    latent_rows_f32_kernel<<<dim3(n, heads), LR_WARPS * 32, 0, st>>>(p);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  if (rank <= 128) return launch_latent_group<1>(p, n, st);
  if (rank <= 256) return launch_latent_group<2>(p, n, st);
  if (rank <= 512) return launch_latent_group<4>(p, n, st);
  return launch_latent_group<5>(p, n, st);
}
