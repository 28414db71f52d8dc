// Between the projections and the scores of an attention layer without a convolution, for a ragged
// batch: RMS norms of q and of k over all heads at once, rotary embedding of q and k (pairs half a rotation
// apart, or neighbours), division of the heads of q and k, or of v, by their root mean square, a factor per
// query head, and the write of k and v into the cache pages and, for the kernel that
// works on pieces of prompts, row by row.
//
// One block per row; a group of L lanes takes one head of q or k, eight consecutive numbers per lane, or
// as many of a head of v.  Without key/value heads only q is made.
#include "ragged.cuh"

namespace cb {

constexpr int HP_THREADS = 128;

struct HeadPrep {
  const void* raw;         // [rows, ld]: q at column 0, k at koff, v at voff
  int ld, koff, voff;
  int heads, kv_heads, v_heads, dim, vdim;
  int half;                // rotated pairs per head (0: none)
  const float2* rope;      // [rows, half] (cos, sin)
  int interleaved, unit, unit_v;
  float eps;
  const float* q_norm;     // [heads * dim] or null
  const float* k_norm;
  const float* q_factor;   // [heads] or null
  void* q;                 // [rows, heads, q_head]
  int q_head;
  void* k_cache;           // [pages, PAGE, kv_heads, dim_p]
  void* v_cache;           // [pages, PAGE, v_heads, vdim_p]
  int dim_p, vdim_p;
  void* k_rows;            // [rows, kv_heads, kr_head] or null
  void* v_rows;            // [rows, v_heads, vr_head]
  int kr_head, vr_head;
  const int* page_table;   // [slots, max_pages]
  int max_pages, num_pages;
  const int* row_slot;
  const int* row_pos;
  int* status;
};

// Entries d .. d + 7 of a head, zeros behind its n entries.
template <typename T, bool VEC>
__device__ __forceinline__ void head_load(const T* src, int d, int n, float* f) {
  if constexpr (VEC) {
    if (d < n) {
      load_vec<8>(src + d, f);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = 0.f;
    }
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = d + i < n ? to_f32(src[d + i]) : 0.f;
  }
}

// Sum of squares of n numbers, this thread's share.
template <typename T, bool VEC>
__device__ __forceinline__ float row_squares(const T* src, int n) {
  float s = 0.f;
#pragma unroll 2
  for (int c = threadIdx.x * 8; c < n; c += HP_THREADS * 8) {
    float f[8];
    head_load<T, VEC>(src + c, 0, n - c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) s += f[i] * f[i];
  }
  return s;
}

// VEC: head sizes (and, for pairs half a rotation apart, half) are multiples of eight.
template <typename T, int L, bool VEC>
__global__ void __launch_bounds__(HP_THREADS) head_prep_kernel(const HeadPrep p) {
  const int row = blockIdx.x, d0 = (threadIdx.x % L) * 8;
  const int pos = p.row_pos[row], lp = pos / RAGGED_PAGE;
  int page = lp < p.max_pages ? p.page_table[static_cast<size_t>(p.row_slot[row]) * p.max_pages + lp] : -1;
  if (page < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0) record_status(p.status, ST_BOUNDS, row);
    return;
  }
  const size_t cell = static_cast<size_t>(page) * RAGGED_PAGE + pos % RAGGED_PAGE;
  const T* raw = static_cast<const T*>(p.raw) + static_cast<size_t>(row) * p.ld;
  const float2* rope = p.rope + static_cast<size_t>(row) * p.half;
  float q_rs = 1.f, k_rs = 1.f;
  if (p.q_norm != nullptr) {
    __shared__ float red[2][HP_THREADS / 32];
    const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim;
    float sq = row_squares<T, VEC>(raw, nq), sk = row_squares<T, VEC>(raw + p.koff, nk);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
      red[0][threadIdx.x >> 5] = sq;
      red[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < HP_THREADS / 32; ++i) {
      sq += red[0][i];
      sk += red[1][i];
    }
    q_rs = 1.0f / sqrtf(sq / nq + p.eps);
    if (nk > 0) k_rs = 1.0f / sqrtf(sk / nk + p.eps);
  }
  const int v_units = (max(p.vdim_p, p.vr_head) + 8 * L - 1) / (8 * L);     // per head
  const int units = p.heads + p.kv_heads + p.v_heads * v_units;
  for (int u = threadIdx.x / L; u < (units + HP_THREADS / L - 1) / (HP_THREADS / L) * (HP_THREADS / L);
       u += HP_THREADS / L) {                     // whole groups: the lanes of a warp stay together
    const bool live = u < units, is_q = u < p.heads, is_v = u >= p.heads + p.kv_heads;
    const int n = is_v ? p.vdim : p.dim;
    const int uv = u - p.heads - p.kv_heads;
    const int h = is_q ? u : (is_v ? uv / v_units : u - p.heads);
    const int d = is_v ? d0 + uv % v_units * 8 * L : d0;
    const T* src = raw + (is_q ? 0 : (is_v ? p.voff : p.koff)) + static_cast<size_t>(h) * n;
    float f[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = 0.f;
    if (live) head_load<T, VEC>(src, d, n, f);
    const float* gain = is_v || p.q_norm == nullptr ? nullptr : (is_q ? p.q_norm : p.k_norm) + static_cast<size_t>(h) * n;
    const float row_rs = is_q ? q_rs : k_rs;
    if (live && gain != nullptr) {
      float g[8];
      head_load<float, VEC>(gain, d, n, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= row_rs * g[i];
    }
    if (live && !is_v && d < 2 * p.half) {
      if (p.interleaved) {                        // both numbers of a pair are this lane's
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
          if (d + i < 2 * p.half) {
            const float2 cs = rope[(d + i) >> 1];
            const float a = f[i], b = f[i + 1];
            f[i] = a * cs.x - b * cs.y;
            f[i + 1] = b * cs.x + a * cs.y;
          }
        }
      } else if constexpr (VEC) {                 // the other numbers lie half further or half before
        const bool low = d < p.half;
        const int first = low ? d : d - p.half;
        float o[8];
        load_vec<8>(src + (low ? d + p.half : first), o);
        if (gain != nullptr) {
          float g[8];
          load_vec<8>(gain + (low ? d + p.half : first), g);
#pragma unroll
          for (int i = 0; i < 8; ++i) o[i] *= row_rs * g[i];
        }
        const float sign = low ? -1.f : 1.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float2 cs = rope[first + i];
          f[i] = f[i] * cs.x + sign * o[i] * cs.y;
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int c = d + i;
          if (c < 2 * p.half) {
            const bool low = c < p.half;
            const float2 cs = rope[low ? c : c - p.half];
            const int other = low ? c + p.half : c - p.half;
            const float o = to_f32(src[other]) * (gain != nullptr ? row_rs * gain[other] : 1.f);
            f[i] = f[i] * cs.x + (low ? -o : o) * cs.y;
          }
        }
      }
    }
    if (p.unit || p.unit_v) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) s += f[i] * f[i];
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (is_v ? p.unit_v : p.unit) {
        const float r = 1.0f / sqrtf(s / n + p.eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= r;
      }
    }
    if (!live) continue;
    if (is_q) {
      if (p.q_factor != nullptr) {
        const float c = p.q_factor[h];
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= c;
      }
      if (d < p.q_head)
        store_vec<8>(static_cast<T*>(p.q) + (static_cast<size_t>(row) * p.heads + h) * p.q_head + d, f);
      continue;
    }
    const int hs = is_v ? p.v_heads : p.kv_heads, w = is_v ? p.vdim_p : p.dim_p;
    if (d < w) store_vec<8>(static_cast<T*>(is_v ? p.v_cache : p.k_cache) + (cell * hs + h) * w + d, f);
    const int rw = is_v ? p.vr_head : p.kr_head;
    T* rows = static_cast<T*>(is_v ? p.v_rows : p.k_rows);
    if (rows != nullptr && d < rw)
      store_vec<8>(rows + (static_cast<size_t>(row) * hs + h) * rw + d, f);
  }
}

template <typename T, int L>
static void launch_head_prep(const HeadPrep& p, int rows, bool vec, cudaStream_t st) {
  if (vec) head_prep_kernel<T, L, true><<<rows, HP_THREADS, 0, st>>>(p);
  else head_prep_kernel<T, L, false><<<rows, HP_THREADS, 0, st>>>(p);
}
template <typename T>
static int head_prep(const HeadPrep& p, int rows, int widest, cudaStream_t st) {
  const bool vec = p.dim % 8 == 0 && p.vdim % 8 == 0 && p.ld % 8 == 0 && p.koff % 8 == 0 &&
                   p.voff % 8 == 0 && (p.interleaved || p.half % 8 == 0);
  if (widest <= 32) launch_head_prep<T, 4>(p, rows, vec, st);
  else if (widest <= 64) launch_head_prep<T, 8>(p, rows, vec, st);
  else if (widest <= 128) launch_head_prep<T, 16>(p, rows, vec, st);
  else launch_head_prep<T, 32>(p, rows, vec, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

extern "C" int cb_head_prep(const void* raw, int ld, int koff, int voff, int heads, int kv_heads,
                            int v_heads, int dim, int vdim, int half, const void* rope,
                            int interleaved, int unit, float eps, const float* q_norm, const float* k_norm,
                            int unit_v, const float* q_factor, void* q, int q_head, void* k_cache,
                            void* v_cache, int dim_p, int vdim_p, void* k_rows, void* v_rows,
                            int kr_head, int vr_head, const int* page_table, int max_pages,
                            int num_pages, const int* row_slot, const int* row_pos, int rows, int f32,
                            int* status, void* stream) {
  using namespace cb;
  if (rows <= 0 || heads < 1 || kv_heads < 0 || (v_heads < 1) != (kv_heads < 1) || dim < 1 || vdim < 1 || half < 0 || 2 * half > dim)
    return -1;
  if (half > 0 && rope == nullptr) return -1;
  if (q_head % 8 || dim_p % 8 || vdim_p % 8 || q_head < dim || dim_p < dim || vdim_p < vdim) return -2;
  if (k_rows != nullptr && (v_rows == nullptr || kr_head % 8 || vr_head % 8 || kr_head < dim || vr_head < vdim))
    return -2;
  int widest = q_head;
  for (int w : {dim_p, kr_head}) widest = w > widest ? w : widest;
  if (widest > 256 || vdim_p > 256 || vr_head > 256) return -2;
  if (q_norm != nullptr && kv_heads > 0 && k_norm == nullptr) return -2;
  if (kv_heads > 0 && unit_v)              // a head of v by one group of lanes
    for (int w : {vdim_p, vr_head}) widest = w > widest ? w : widest;
  HeadPrep p;
  p.raw = raw; p.ld = ld; p.koff = koff; p.voff = voff; p.heads = heads; p.kv_heads = kv_heads;
  p.v_heads = v_heads; p.dim = dim; p.vdim = vdim; p.half = half; p.rope = static_cast<const float2*>(rope);
  p.interleaved = interleaved; p.unit = unit; p.eps = eps; p.q_norm = q_norm; p.k_norm = k_norm;
  p.unit_v = kv_heads > 0 && unit_v; p.q_factor = q_factor; p.q = q; p.q_head = q_head; p.k_cache = k_cache;
  p.v_cache = v_cache; p.dim_p = dim_p; p.vdim_p = vdim_p; p.k_rows = k_rows; p.v_rows = v_rows;
  p.kr_head = kr_head; p.vr_head = vr_head; p.page_table = page_table; p.max_pages = max_pages;
  p.num_pages = num_pages; p.row_slot = row_slot; p.row_pos = row_pos; p.status = status;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? head_prep<float>(p, rows, widest, st) : head_prep<__nv_bfloat16>(p, rows, widest, st);
}
