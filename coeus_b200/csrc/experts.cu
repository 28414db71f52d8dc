// Mixture of experts of the serving step: no capacity, every chosen expert runs.
//   moe_choose   sigmoid or softmax scores, the best groups (by the sum of a group's largest scores, two or
//                one), the top experts in them, weights = scores (over their sum) * scale.  A correction per
//                expert can be added to the scores for the choice.  Few tokens: one block per token
//                computes the router's product as well.  More: the logits are given, a block takes
//                CHOOSE_TOKENS tokens and counts its pairs per expert.  One more logit can be the gate of the
//                shared expert.  The last experts can be identities: they get no rows and no weights.
//   moe_place    one block: where every block's pairs of an expert go in a buffer sorted by expert, whose
//                experts start at multiples of a block of rows, and the expert of every block
//   moe_gather   rows into that buffer
//   moe_few_in / moe_few_down   up to 16 rows: the weights of the chosen experts and of the shared one are
//                streamed straight into mma fragments.  The activations of all live experts lie side by
//                side (zeros where a token does not use the expert, else times the token's weight), so
//                that the second product is one long contraction whose result is complete.
#include "ragged.cuh"

namespace cb {

constexpr int CHOOSE_TOKENS = 32;
constexpr int CHOOSE_WARPS = 8;
constexpr int MOE_E = 256, MOE_K = 16;
constexpr unsigned FULL = 0xffffffffu;

struct Choose {
  const float* logits;     // [T, ldl], or null: h . router^T
  int ldl;
  const void* h;           // [T, ldh]
  const void* router;      // [E, ldr]
  int ldh, ldr, W;
  int T, E, top, groups, keep;
  float scale;
  int softmax, group_best, normalise;
  const float* correction; // [E] or null
  float* shared;           // [T] or null: sigmoid of logit E
  int* expert;             // [T, top]
  float* weight;           // [T, top]
  int* rank;               // [T, top] among the block's earlier pairs of the same expert
  int* counts;             // [E, blocks]
  int blocks;
};

// (value, index) of the largest of v over the warp, the lowest index among equals.
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(FULL, v, o);
    const int oi = __shfl_xor_sync(FULL, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
}

// One warp, one token: s[E] holds the logits and becomes the scores that are compared; gv is scratch for the
// groups.  NI: experts per lane.
template <int NI>
__device__ __forceinline__ void choose_token(const Choose& p, int t, float* s, float* gv) {
  const int lane = threadIdx.x & 31, n = p.E / p.groups;
  float score[NI];                       // of this lane's experts lane, lane + 32, ...
  float total = 1.f, top = 0.f;
  if (p.softmax) {
    top = -INFINITY;
    for (int e = lane; e < p.E; e += 32) top = fmaxf(top, s[e]);
    top = warp_max(top);
    total = 0.f;
    for (int e = lane; e < p.E; e += 32) total += expf(s[e] - top);
    total = warp_sum(total);
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e = lane + 32 * i;
    score[i] = 0.f;
    if (e < p.E) {
      score[i] = p.softmax ? expf(s[e] - top) / total : sigmoidf_(s[e]);
      s[e] = p.correction != nullptr ? score[i] + p.correction[e] : score[i];
    }
  }
  __syncwarp();
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;
      for (int i = 0; i < n; ++i) {
        const float v = s[g * n + i];
        b = fmaxf(b, fminf(a, v));
        a = fmaxf(a, v);
      }
      gv[g] = p.group_best == 2 && n > 1 ? a + b : a;
    }
    __syncwarp();
    for (int k = 0; k < p.keep; ++k) {
      float v = -INFINITY;
      int at = p.groups - 1;                     // of scores that are no numbers, any
      for (int g = lane; g < p.groups; g += 32)
        if (gv[g] > v) { v = gv[g]; at = g; }
      warp_best(v, at);
      __syncwarp();
      if (lane == 0) gv[at] = -INFINITY;         // kept
      __syncwarp();
    }
  }
  float left[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e = lane + 32 * i;
    left[i] = e < p.E && (p.keep == p.groups || gv[e / n] == -INFINITY) ? s[e] : -INFINITY;
    if (e < p.E) s[e] = score[i];
  }
  __syncwarp();
  float mine = 0.f, sum = 0.f;
  int chosen = 0;
  for (int k = 0; k < p.top; ++k) {
    float v = -INFINITY;
    int at = p.E - 1;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (left[i] > v) { v = left[i]; at = lane + 32 * i; }
    warp_best(v, at);
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (at == lane + 32 * i) left[i] = -INFINITY;
    const float w = s[at];
    sum += w;
    if (lane == k) { mine = w; chosen = at; }
  }
  if (lane < p.top) {
    p.expert[static_cast<size_t>(t) * p.top + lane] = chosen;
    p.weight[static_cast<size_t>(t) * p.top + lane] = (p.normalise ? mine / (sum + 1e-20f) : mine) * p.scale;
  }
  __syncwarp();
}

template <int NI>
__global__ void __launch_bounds__(CHOOSE_WARPS * 32) moe_choose_kernel(const Choose p) {
  __shared__ float s[CHOOSE_WARPS][MOE_E], gv[CHOOSE_WARPS][MOE_E];
  __shared__ int pair[CHOOSE_TOKENS * MOE_K], hist[MOE_E];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * CHOOSE_TOKENS, nt = min(CHOOSE_TOKENS, p.T - t0);
  for (int t = warp; t < nt; t += CHOOSE_WARPS) {
    for (int e = lane; e < p.E; e += 32) s[warp][e] = p.logits[static_cast<size_t>(t0 + t) * p.ldl + e];
    __syncwarp();
    if (p.shared != nullptr && lane == 0)
      p.shared[t0 + t] = sigmoidf_(p.logits[static_cast<size_t>(t0 + t) * p.ldl + p.E]);
    choose_token<NI>(p, t0 + t, s[warp], gv[warp]);
  }
  for (int e = threadIdx.x; e < p.E; e += CHOOSE_WARPS * 32) hist[e] = 0;
  __syncthreads();
  const int n = nt * p.top;
  for (int i = threadIdx.x; i < n; i += CHOOSE_WARPS * 32) {
    pair[i] = p.expert[static_cast<size_t>(t0) * p.top + i];
    atomicAdd(&hist[pair[i]], 1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += CHOOSE_WARPS * 32) {
    int r = 0;
    for (int j = 0; j < i; ++j) r += pair[j] == pair[i];
    p.rank[static_cast<size_t>(t0) * p.top + i] = r;
  }
  for (int e = threadIdx.x; e < p.E; e += CHOOSE_WARPS * 32)
    p.counts[static_cast<size_t>(e) * p.blocks + blockIdx.x] = hist[e];
}

// One token per block, with the router's product: two experts per warp at a time.
template <typename T, int NI>
__global__ void __launch_bounds__(512) moe_choose_few_kernel(const Choose p) {
  __shared__ float s[MOE_E + 4], gv[MOE_E];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x, nw = blockDim.x >> 5;
  const T* h = static_cast<const T*>(p.h) + static_cast<size_t>(t) * p.ldh;
  const T* r = static_cast<const T*>(p.router);
  const int outputs = p.E + (p.shared != nullptr);
  for (int e0 = warp * 2; e0 < outputs; e0 += nw * 2) {
    const T* r0 = r + static_cast<size_t>(e0) * p.ldr;
    const T* r1 = r + static_cast<size_t>(min(e0 + 1, outputs - 1)) * p.ldr;
    float a = 0.f, b = 0.f;
#pragma unroll 4
    for (int c = lane * 8; c < p.W; c += 256) {
      float x[8], u[8], v[8];
      load_vec<8>(h + c, x);
      load_vec<8>(r0 + c, u);
      load_vec<8>(r1 + c, v);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        a += x[k] * u[k];
        b += x[k] * v[k];
      }
    }
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) {
      s[e0] = a;
      s[e0 + 1] = b;
    }
  }
  __syncthreads();
  if (warp != 0) return;
  if (p.shared != nullptr && lane == 0) p.shared[t] = sigmoidf_(s[p.E]);
  choose_token<NI>(p, t, s, gv);
  for (int e = lane; e < p.E; e += 32) p.counts[static_cast<size_t>(e) * p.blocks + t] = 0;
  __syncwarp();
  if (lane < p.top) {
    const size_t at = static_cast<size_t>(t) * p.top + lane;
    p.rank[at] = 0;
    p.counts[static_cast<size_t>(p.expert[at]) * p.blocks + t] = 1;
  }
}

__global__ void __launch_bounds__(1024)
moe_place_kernel(const int* __restrict__ counts, int blocks, int E, int* __restrict__ base,
                 int* __restrict__ block_expert, int n_tiles, int tile_rows) {
  __shared__ int total[MOE_E], start[MOE_E + 1];        // start: in tiles
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = warp; e < E; e += 32) {
    int n = 0;
#pragma unroll 8
    for (int b = lane; b < blocks; b += 32) n += counts[static_cast<size_t>(e) * blocks + b];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(FULL, n, o);
    if (lane == 0) total[e] = n;
  }
  __syncthreads();
  if (warp == 0) {
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int n = e0 + lane < E ? (total[e0 + lane] + tile_rows - 1) / tile_rows : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(FULL, incl, o);
        if (lane >= o) incl += v;
      }
      if (e0 + lane < E) start[e0 + lane] = run + incl - n;
      run += __shfl_sync(FULL, incl, 31);
    }
    if (lane == 0) start[E] = run;
  }
  __syncthreads();
  for (int i = start[E] + threadIdx.x; i < n_tiles; i += blockDim.x) block_expert[i] = -1;
  for (int e = warp; e < E; e += 32) {
    for (int i = start[e] + lane; i < start[e + 1]; i += 32)
      if (i < n_tiles) block_expert[i] = e;
    int run = start[e] * tile_rows;
    const size_t at = static_cast<size_t>(e) * blocks;
    for (int b0 = 0; b0 < blocks; b0 += 256) {       // a lane sums up eight blocks
      int n[8], sum = 0;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int b = b0 + lane * 8 + i;
        n[i] = b < blocks ? counts[at + b] : 0;
        sum += n[i];
      }
      int incl = sum;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(FULL, incl, o);
        if (lane >= o) incl += v;
      }
      int before = run + incl - sum;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int b = b0 + lane * 8 + i;
        if (b < blocks) base[at + b] = before;
        before += n[i];
      }
      run += __shfl_sync(FULL, incl, 31);
    }
  }
}

// One block per token: its row (nv vectors of 16 bytes) once per expert.
__global__ void __launch_bounds__(256)
moe_gather_kernel(const uint4* __restrict__ h, int ldh, const int* __restrict__ expert,
                  const int* __restrict__ rank, const int* __restrict__ base, int blocks, int top,
                  int per_block, int* __restrict__ slot, uint4* __restrict__ rows, int nv, int n_rows, int E,
                  int* status) {
  __shared__ int to[MOE_K];
  const int t = blockIdx.x;
  if (threadIdx.x < top) {
    const size_t i = static_cast<size_t>(t) * top + threadIdx.x;
    int at = -1;                                 // an identity expert
    if (expert[i] < E) {
      at = base[static_cast<size_t>(expert[i]) * blocks + t / per_block] + rank[i];
      if (at < 0 || at >= n_rows) {
        record_status(status, ST_BOUNDS, t);
        at = 0;
      }
    }
    to[threadIdx.x] = at;
    slot[i] = at;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < nv; c += blockDim.x) {
    const uint4 v = h[static_cast<size_t>(t) * ldh + c];
    for (int k = 0; k < top; ++k)
      if (to[k] >= 0) rows[static_cast<size_t>(to[k]) * nv + c] = v;
  }
}

// ------------------------------------------------------------------------------- few rows
constexpr int FEW_WARPS = 8, DOWN_WARPS = 16;    // the second product has few blocks and long sums

struct Few {
  const __nv_bfloat16* h;        // [M, ldh]
  int ldh, M, W, E, top;         // W: multiple of 8; experts from E on are identities
  const int* expert;             // [M, top]
  const float* weight;
  const float* s_weight;         // [M] of the shared expert, or null: 1
  const __nv_bfloat16* w_in;     // [E, 2 n, W], gate and up rows alternate
  const __nv_bfloat16* w_down;   // [E, W, n]
  const __nv_bfloat16* s_in;     // [2 ns, W] or null
  const __nv_bfloat16* s_down;   // [W, ns]
  int n, ns, live;               // live: most experts that can be in use
  float limit, s_limit, slope, shift;
  __nv_bfloat16* act;            // [M, lda]: live * n columns of experts, then ns
  int lda;
  float* y;                      // [M, ldy]
  int ldy;
};

// The experts in use, in ascending order, by all threads of the block.  Returns how many.
__device__ __forceinline__ int live_experts(const Few& p, int* list, uint32_t* bits, int* count) {
  if (threadIdx.x < MOE_E / 32) bits[threadIdx.x] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < p.M * p.top; i += blockDim.x)
    if (p.expert[i] < p.E) atomicOr(&bits[p.expert[i] >> 5], 1u << (p.expert[i] & 31));
  __syncthreads();
  if (threadIdx.x < 32) {
    const uint32_t b = threadIdx.x < MOE_E / 32 ? bits[threadIdx.x] : 0u;
    int incl = __popc(b);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(FULL, incl, o);
      if (static_cast<int>(threadIdx.x) >= o) incl += v;
    }
    int at = incl - __popc(b);
    for (uint32_t r = b; r != 0; r &= r - 1) list[at++] = threadIdx.x * 32 + __ffs(r) - 1;
    if (threadIdx.x == 31) *count = incl;
  }
  __syncthreads();
  return *count;
}

__device__ __forceinline__ uint4 few_ldg(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// 16 weight rows against NT * 8 tokens over 64 numbers of the contraction, of which this lane reads
// 16 + 16 of two weight rows (their order is permuted alike on both sides).
template <int NT>
__device__ __forceinline__ void few_mma(float (*acc)[4], const uint4 (*a)[2], const uint4 (*b)[2]) {
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int v = 0; v < 2; ++v) {
      const uint32_t f0[4] = {a[0][v].x, a[1][v].x, a[0][v].y, a[1][v].y};
      const uint32_t f1[4] = {a[0][v].z, a[1][v].z, a[0][v].w, a[1][v].w};
      mma_bf16(acc[j], f0, b[j][v].x, b[j][v].y);
      mma_bf16(acc[j], f1, b[j][v].z, b[j][v].w);
    }
}

// Adds the warps' 16 x (NT * 8) results; the sum of row c, token m is red[m * 17 + c] of warp 0's part.
template <int NT, int WARPS>
__device__ __forceinline__ float few_sum(const float* red, int m, int c) {
  float v = 0.f;
#pragma unroll
  for (int w = 0; w < WARPS; ++w) v += red[(w * NT * 8 + m) * 17 + c];
  return v;
}
template <int NT>
__device__ __forceinline__ void few_store(float* red, int warp, int lane, const float (*acc)[4]) {
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int k = 0; k < 4; ++k)
      red[(warp * NT * 8 + j * 8 + (lane & 3) * 2 + (k & 1)) * 17 + (lane >> 2) + (k >> 1) * 8] = acc[j][k];
}

// blocks: live * tiles of the experts, then the tiles of the shared one
template <int NT>
__global__ void __launch_bounds__(FEW_WARPS * 32) moe_few_in_kernel(const Few p) {
  __shared__ float red[FEW_WARPS * NT * 8 * 17];
  __shared__ int list[MOE_E], count;
  __shared__ uint32_t bits[MOE_E / 32];
  __shared__ float wt[16];
  const int tiles = (2 * p.n + 15) / 16, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool shared = static_cast<int>(blockIdx.x) >= p.live * tiles;
  const int a = shared ? 0 : blockIdx.x / tiles, tile = shared ? blockIdx.x - p.live * tiles : blockIdx.x % tiles;
  const __nv_bfloat16* w = p.s_in;
  int rows = 2 * p.ns, col0 = p.live * p.n;
  if (!shared) {
    if (a >= live_experts(p, list, bits, &count)) return;
    const int e = list[a];
    w = p.w_in + static_cast<size_t>(e) * 2 * p.n * p.W;
    rows = 2 * p.n;
    col0 = a * p.n;
    if (threadIdx.x < 16) {
      float v = 0.f;
      if (threadIdx.x < p.M)
        for (int k = 0; k < p.top; ++k)
          if (p.expert[threadIdx.x * p.top + k] == e) v = p.weight[threadIdx.x * p.top + k];
      wt[threadIdx.x] = v;
    }
  } else if (threadIdx.x < 16) {
    wt[threadIdx.x] = p.s_weight != nullptr && static_cast<int>(threadIdx.x) < p.M ? p.s_weight[threadIdx.x] : 1.f;
  }
  const int r = lane >> 2, q = (lane & 3) * 16;
  const __nv_bfloat16* wp[2];
#pragma unroll
  for (int i = 0; i < 2; ++i)                  // rows past the end repeat the last one
    wp[i] = w + static_cast<size_t>(min(tile * 16 + i * 8 + r, rows - 1)) * p.W + q;
  const __nv_bfloat16* xp[NT];
#pragma unroll
  for (int j = 0; j < NT; ++j) xp[j] = p.h + static_cast<size_t>(min(j * 8 + r, p.M - 1)) * p.ldh + q;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[j][k] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const int chunks = (p.W + 63) / 64;
  constexpr int U = NT == 1 ? 4 : 2;
  for (int c0 = warp; c0 < chunks; c0 += FEW_WARPS * U) {
    uint4 x[U][2][2];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k0 = (c0 + u * FEW_WARPS) * 64;
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int v = 0; v < 2; ++v) x[u][i][v] = k0 + q + v * 8 < p.W ? few_ldg(wp[i] + k0 + v * 8) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k0 = (c0 + u * FEW_WARPS) * 64;
      uint4 b[NT][2];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int v = 0; v < 2; ++v)
          b[j][v] = k0 + q + v * 8 < p.W ? *reinterpret_cast<const uint4*>(xp[j] + k0 + v * 8) : zero;
      few_mma<NT>(acc, x[u], b);
    }
  }
  few_store<NT>(red, warp, lane, acc);
  __syncthreads();
  const float limit = shared ? p.s_limit : p.limit;
  for (int i = threadIdx.x; i < p.M * 8; i += FEW_WARPS * 32) {
    const int m = i >> 3, c = i & 7, ch = tile * 8 + c;
    if (2 * ch >= rows) continue;
    float v = 0.f;
    if (wt[m] != 0.f)
      v = wt[m] * clamped_glu(few_sum<NT, FEW_WARPS>(red, m, 2 * c), few_sum<NT, FEW_WARPS>(red, m, 2 * c + 1), p.slope, limit,
                              p.shift);
    p.act[static_cast<size_t>(m) * p.lda + col0 + ch] = __float2bfloat16(v);
  }
}

template <int NT>
__global__ void __launch_bounds__(DOWN_WARPS * 32) moe_few_down_kernel(const Few p) {
  __shared__ float red[DOWN_WARPS * NT * 8 * 17];
  __shared__ int list[MOE_E], count;
  __shared__ uint32_t bits[MOE_E / 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = blockIdx.x * 16;
  const int live = live_experts(p, list, bits, &count);
  const int r = lane >> 2, q = (lane & 3) * 16;
  const int row[2] = {min(n0 + r, p.W - 1), min(n0 + 8 + r, p.W - 1)};
  const __nv_bfloat16* xp[NT];
#pragma unroll
  for (int j = 0; j < NT; ++j) xp[j] = p.act + static_cast<size_t>(min(j * 8 + r, p.M - 1)) * p.lda;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[j][k] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const int per = (p.n + 63) / 64, chunks = live * per + (p.ns + 63) / 64;
  constexpr int U = NT == 1 ? 4 : 2;
  for (int c0 = warp; c0 < chunks; c0 += DOWN_WARPS * U) {
    uint4 x[U][2][2], b[U][NT][2];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * DOWN_WARPS;
      const bool in = c < chunks, sh = c >= live * per;
      const int a = sh ? 0 : c / per, k0 = (sh ? c - live * per : c % per) * 64 + q;
      const int n = sh ? p.ns : p.n;
      const __nv_bfloat16* w = sh ? p.s_down : p.w_down + static_cast<size_t>(in ? list[a] : 0) * p.W * p.n;
      const int col = sh ? p.live * p.n : a * p.n;
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const bool ok = in && k0 + v * 8 < n;
#pragma unroll
        for (int i = 0; i < 2; ++i)
          x[u][i][v] = ok ? few_ldg(w + static_cast<size_t>(row[i]) * n + k0 + v * 8) : zero;
#pragma unroll
        for (int j = 0; j < NT; ++j)
          b[u][j][v] = ok ? *reinterpret_cast<const uint4*>(xp[j] + col + k0 + v * 8) : zero;
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) few_mma<NT>(acc, x[u], b[u]);
  }
  few_store<NT>(red, warp, lane, acc);
  __syncthreads();
  for (int i = threadIdx.x; i < p.M * 16; i += DOWN_WARPS * 32) {
    const int m = i >> 4, c = i & 15;
    if (n0 + c >= p.W) continue;
    float v = few_sum<NT, DOWN_WARPS>(red, m, c);
    for (int k = 0; k < p.top; ++k)
      if (p.expert[m * p.top + k] >= p.E)
        v += p.weight[m * p.top + k] * __bfloat162float(p.h[static_cast<size_t>(m) * p.ldh + n0 + c]);
    p.y[static_cast<size_t>(m) * p.ldy + n0 + c] = v;
  }
}

}  // namespace cb

using namespace cb;
#define CB_RC() (cudaGetLastError() == cudaSuccess ? 0 : -3)

template <int NI>
static void launch_choose(const Choose& p, int f32, cudaStream_t st) {
  if (p.logits != nullptr) moe_choose_kernel<NI><<<p.blocks, CHOOSE_WARPS * 32, 0, st>>>(p);
  else if (f32) moe_choose_few_kernel<float, NI><<<p.T, 512, 0, st>>>(p);
  else moe_choose_few_kernel<__nv_bfloat16, NI><<<p.T, 512, 0, st>>>(p);
}

// logits null: computed here, one block (of the counts) per token; else blocks of CHOOSE_TOKENS tokens.  E
// counts the identity experts too; shared (or null) gets the sigmoid of logit E.
extern "C" int cb_moe_choose(const float* logits, int ldl, const void* h, int ldh, const void* router,
                             int ldr, int W, int T, int E, int top, int groups, int keep, float scale,
                             int softmax, int group_best, int normalise, const float* correction, float* shared,
                             int* expert, float* weight, int* rank, int* counts, int f32, void* stream) {
  if (T <= 0 || E < 1 || E > MOE_E || top < 1 || top > MOE_K || groups < 1 || E % groups || keep < 1 ||
      keep > groups || top > keep * (E / groups) || group_best < 1 || group_best > 2)
    return -1;
  if (logits != nullptr && ldl < E + (shared != nullptr)) return -2;
  if (logits == nullptr && (h == nullptr || W % 8 || ldh % 8 || ldr % 8 || ldh < W || ldr < W)) return -2;
  Choose p;
  p.logits = logits; p.ldl = ldl; p.h = h; p.ldh = ldh; p.router = router; p.ldr = ldr; p.W = W;
  p.softmax = softmax; p.group_best = group_best; p.normalise = normalise; p.correction = correction;
  p.shared = shared;
  p.T = T; p.E = E; p.top = top; p.groups = groups; p.keep = keep; p.scale = scale; p.expert = expert;
  p.weight = weight; p.rank = rank; p.counts = counts;
  p.blocks = logits != nullptr ? (T + CHOOSE_TOKENS - 1) / CHOOSE_TOKENS : T;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (E <= 32) launch_choose<1>(p, f32, st);
  else launch_choose<MOE_E / 32>(p, f32, st);
  return CB_RC();
}

// rows [n_tiles * tile_rows, W]; base has the shape of counts [E, blocks].  Pairs of experts from E on have no
// row, their slot is -1.
extern "C" int cb_moe_sort(const void* h, int ldh, const int* expert, const int* rank, const int* counts,
                           int T, int E, int top, int per_block, int blocks, int* base, int* slot,
                           int* block_expert, int n_tiles, int tile_rows, void* rows, int W, int f32, int* status,
                           void* stream) {
  const int v = f32 ? 4 : 8;
  if (T <= 0 || E < 1 || E > MOE_E || top < 1 || top > MOE_K || W % v || ldh % v || per_block < 1) return -1;
  if (blocks != (T + per_block - 1) / per_block || tile_rows < 1) return -1;
  if (static_cast<long long>(n_tiles) < static_cast<long long>(T) * top / tile_rows + (T * top < E ? T * top : E))
    return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  moe_place_kernel<<<1, 1024, 0, st>>>(counts, blocks, E, base, block_expert, n_tiles, tile_rows);
  const int nv = W / v, threads = nv >= 256 ? 256 : (nv + 31) / 32 * 32;
  moe_gather_kernel<<<T, threads, 0, st>>>(static_cast<const uint4*>(h), ldh / v, expert, rank, base, blocks, top,
                                           per_block, slot, static_cast<uint4*>(rows), nv,
                                           n_tiles * tile_rows, E, status);
  return CB_RC();
}

// All experts of up to 16 bf16 rows and the shared one (s_in null: none), complete in y (fp32).
extern "C" int cb_moe_few(const void* h, int ldh, int M, int W, int E, int top, const int* expert,
                          const float* weight, const float* s_weight, const void* w_in, const void* w_down, int n, float limit,
                          const void* s_in, const void* s_down, int ns, float s_limit, float slope,
                          float shift, void* act, int lda, float* y, int ldy, void* stream) {
  if (M < 1 || M > 16 || E < 1 || E > MOE_E || top < 1 || top > MOE_K || W % 8 || ldh % 8 || n % 8 || n < 1 ||
      ns % 8 || (s_in == nullptr) != (ns == 0) || ldh < W || ldy < W)
    return -1;
  Few p;
  p.live = E < M * top ? E : M * top;
  if (lda % 8 || lda < p.live * n + ns) return -2;
  p.h = static_cast<const __nv_bfloat16*>(h); p.ldh = ldh; p.M = M; p.W = W; p.E = E; p.top = top;
  p.expert = expert; p.weight = weight; p.w_in = static_cast<const __nv_bfloat16*>(w_in);
  p.w_down = static_cast<const __nv_bfloat16*>(w_down); p.s_in = static_cast<const __nv_bfloat16*>(s_in);
  p.s_down = static_cast<const __nv_bfloat16*>(s_down); p.n = n; p.ns = ns; p.limit = limit;
  p.s_limit = s_limit; p.slope = slope; p.shift = shift; p.s_weight = s_weight; p.act = static_cast<__nv_bfloat16*>(act); p.lda = lda; p.y = y;
  p.ldy = ldy;
  const int in_blocks = p.live * ((2 * n + 15) / 16) + (2 * ns + 15) / 16, down_blocks = (W + 15) / 16;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (M <= 8) {
    moe_few_in_kernel<1><<<in_blocks, FEW_WARPS * 32, 0, st>>>(p);
    moe_few_down_kernel<1><<<down_blocks, DOWN_WARPS * 32, 0, st>>>(p);
  } else {
    moe_few_in_kernel<2><<<in_blocks, FEW_WARPS * 32, 0, st>>>(p);
    moe_few_down_kernel<2><<<down_blocks, DOWN_WARPS * 32, 0, st>>>(p);
  }
  return CB_RC();
}
