// The state-space recurrence over bf16 prompts, 64 tokens at a time on the tensor cores (mma
// m16n8k16).  With c_i the sum of the log-decays of a chunk's tokens up to and including i:
//   y_i = exp(c_i) C_i . S  +  sum_{j <= i} (C_i . B_j) exp(c_i - c_j) dt_j x_j  +  D x_i
//   S  <- exp(c_last) S  +  sum_j exp(c_last - c_j) dt_j B_j x_j^T
// x, B and C enter as the bf16 numbers they are.  The state stays in fp32 registers from an entry's
// first token to its last, and what is added to it (the weighted B) enters its product as the sum of
// two bf16 numbers; only for reading y, which is rounded to bf16 itself, are the state and the
// weighted scores rounded to bf16 operands.
//
// A block of four warps takes one head (and 64 of its columns) of one segment of an entry; a warp
// owns 16 of the chunk's rows for y and every fourth 16-row tile of S.  Where entries and heads do
// not fill the GPU, entries are cut into segments: a first launch finds what each segment adds to an
// empty state, a second one carries the states through, a third one runs all segments at once.
#include <type_traits>

#include "ssd.cuh"

namespace cb {

constexpr int SC_TOK = 64, SC_COLS = 64, SC_WARPS = 4, SC_THREADS = SC_WARPS * 32;
constexpr int SC_XP = SC_COLS + 8;
constexpr float SC_LOG2E = 1.4426950408889634f;

// (u, v) as the sum of two packed bf16 pairs
__device__ __forceinline__ void split2(float u, float v, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(u, v);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(u - f.x, v - f.y);
}

template <int NP>
constexpr int sc_smem() {
  return (2 * SC_TOK * (NP + 8) + SC_TOK * SC_XP + NP * SC_XP) * 2 + 4 * SC_TOK * 4;
}

enum : int { SC_WHOLE = 0, SC_STATE = 1, SC_FROM = 2 };

template <int NP, int MODE>
__global__ void __launch_bounds__(SC_THREADS, 3) ssd_chunk_kernel(const Ssd p) {
  using bf16 = __nv_bfloat16;
  constexpr int LD = NP + 8, RT = NP / 64;                 // RT 16-row tiles of S per warp
  extern __shared__ __align__(16) unsigned char sc_raw[];
  bf16* sB = reinterpret_cast<bf16*>(sc_raw);              // [SC_TOK][LD]
  bf16* sC = sB + SC_TOK * LD;                             // [SC_TOK][LD]
  bf16* sX = sC + SC_TOK * LD;                             // [SC_TOK][SC_XP]
  bf16* sS = sX + SC_TOK * SC_XP;                          // [NP][SC_XP] state in front of the chunk
  float* sCum = reinterpret_cast<float*>(sS + NP * SC_XP); // [SC_TOK] c_i, in units of log 2
  float* sDt = sCum + SC_TOK;
  float* sE = sDt + SC_TOK;                                // exp(c_i)
  float* sW = sE + SC_TOK;                                 // exp(c_last - c_i) dt_i
  const int4 seg = p.segs[blockIdx.y];
  const int e = seg.x, len = seg.z;
  const int h = blockIdx.x % p.heads, col0 = blockIdx.x / p.heads * SC_COLS;
  const int slot = p.e.slot[e], g = h / (p.heads / p.groups);
  const size_t row0 = static_cast<size_t>(p.e.row0[e]) + seg.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, t = lane & 3;
  const int cols = min(SC_COLS, p.P - col0);
  const bf16* u = static_cast<const bf16*>(p.u) + row0 * p.ldu;
  const bf16* gx = u + h * p.P + col0;
  const bf16* gB = u + p.boff + g * p.N;
  const bf16* gC = u + p.coff + g * p.N;
  const bool vec = p.ldu % 8 == 0 && p.P % 8 == 0 && p.N % 8 == 0 && p.boff % 8 == 0 && p.coff % 8 == 0;
  // everything behind N and P stays zero
  for (int i = tid; i < (2 * SC_TOK * LD + SC_TOK * SC_XP) / 2; i += SC_THREADS)
    reinterpret_cast<uint32_t*>(sB)[i] = 0u;
  const size_t cell = (static_cast<size_t>(slot) * p.heads + h) * p.N * p.Pp;
  const size_t seg_cell = (static_cast<size_t>(blockIdx.y) * p.heads + h) * p.N * p.Pp;
  const float* from = nullptr;
  if (MODE == SC_FROM) from = p.seg_state + seg_cell;
  else if (MODE == SC_WHOLE && p.e.pos0[e] > 0) from = p.state + cell;
  float S[RT][8][4];
#pragma unroll
  for (int a = 0; a < RT; ++a)
#pragma unroll
    for (int b = 0; b < 8; ++b)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int n = (warp + 4 * a) * 16 + r + (c >> 1) * 8, q = b * 8 + t * 2 + (c & 1);
        S[a][b][c] = from != nullptr && n < p.N && q < cols ? from[static_cast<size_t>(n) * p.Pp + col0 + q] : 0.f;
      }
  const float rate = expf(p.A_log[h]) * SC_LOG2E, bias = p.dt_bias[h], D = p.D[h];
  float total = 0.f;                                       // of the log-decays
  __syncthreads();
  for (int c0 = 0; c0 < len; c0 += SC_TOK) {
    const int n_tok = min(SC_TOK, len - c0);
    // ---- the chunk into shared memory; rows behind the segment's end are zero
    if (vec) {
      auto rows_in = [&](bf16* dst, int pitch, const bf16* src, auto width, int n) {   // n of width columns
        constexpr int C8 = decltype(width)::value / 8;
        const int k = tid % C8;
        if (k * 8 >= n) return;
        const uint32_t to = smem_u32(dst + k * 8);
#pragma unroll
        for (int i = 0; i < SC_TOK * C8 / SC_THREADS; ++i) {
          const int tok = tid / C8 + i * (SC_THREADS / C8);
          cp_async16_zfill(to + tok * pitch * 2, src + static_cast<size_t>(c0 + min(tok, n_tok - 1)) * p.ldu + k * 8,
                           tok < n_tok ? 16 : 0);
        }
      };
      rows_in(sB, LD, gB, std::integral_constant<int, NP>(), p.N);
      if (MODE != SC_STATE) rows_in(sC, LD, gC, std::integral_constant<int, NP>(), p.N);
      rows_in(sX, SC_XP, gx, std::integral_constant<int, SC_COLS>(), cols);
      cp_async_commit();
    } else {
      const int per = 2 * p.N + cols;
      for (int i = tid; i < SC_TOK * per; i += SC_THREADS) {
        const int tok = i / per, k = i % per;
        const size_t at = static_cast<size_t>(c0 + tok) * p.ldu;
        const bool in = tok < n_tok;
        const bf16 zero = __float2bfloat16(0.f);
        if (k < p.N) sB[tok * LD + k] = in ? gB[at + k] : zero;
        else if (k < 2 * p.N) sC[tok * LD + k - p.N] = in ? gC[at + k - p.N] : zero;
        else sX[tok * SC_XP + k - 2 * p.N] = in ? gx[at + k - 2 * p.N] : zero;
      }
    }
    if (warp == 0) {                                       // decays: two tokens per lane
      float d[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int tok = 2 * lane + k;
        d[k] = tok < n_tok ? ssd_dt(__bfloat162float(static_cast<const bf16*>(p.dt)[(row0 + c0 + tok) * p.lddt + h]), bias)
                           : 0.f;
      }
      const float a0 = -rate * d[0], a1 = a0 - rate * d[1];
      float run = a1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += v;
      }
      const float last = __shfl_sync(0xffffffffu, run, 31), c1 = run, cb = run - a1 + a0;
      sCum[2 * lane] = cb;
      sCum[2 * lane + 1] = c1;
      sDt[2 * lane] = d[0];
      sDt[2 * lane + 1] = d[1];
      sE[2 * lane] = exp2f(cb);
      sE[2 * lane + 1] = exp2f(c1);
      sW[2 * lane] = exp2f(last - cb) * d[0];
      sW[2 * lane + 1] = exp2f(last - c1) * d[1];
    }
    if (MODE != SC_STATE) {
#pragma unroll
      for (int a = 0; a < RT; ++a)
#pragma unroll
        for (int b = 0; b < 8; ++b)
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const int at = ((warp + 4 * a) * 16 + r + c * 8) * SC_XP + b * 8 + t * 2;
            *reinterpret_cast<uint32_t*>(sS + at) = pack_bf16x2(S[a][b][2 * c], S[a][b][2 * c + 1]);
          }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (MODE != SC_STATE) {
      // ---- scores C_i . B_j of this warp's rows, columns up to its own
      const int i0 = warp * 16 + r;
      const bf16* rowsC = sC + (warp * 16 + (lane & 15)) * LD + (lane >> 4) * 8;
      uint32_t m[4][4];                                    // weighted, as operands of the product with x
      {
        float G[8][4];
#pragma unroll
        for (int b = 0; b < 8; ++b)
#pragma unroll
          for (int c = 0; c < 4; ++c) G[b][c] = 0.f;
#pragma unroll
        for (int k = 0; k < NP / 16; ++k) {
          uint32_t a[4];
          ldsm4(a, smem_u32(rowsC + k * 16));
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (j <= warp) {
              uint32_t b[4];
              ldsm4(b, smem_u32(sB + (j * 16 + (lane & 7) + (lane >> 4) * 8) * LD + k * 16 + ((lane >> 3) & 1) * 8));
              mma_bf16(G[2 * j], a, b[0], b[1]);
              mma_bf16(G[2 * j + 1], a, b[2], b[3]);
            }
          }
        }
        const float ci[2] = {sCum[i0], sCum[i0 + 8]};
#pragma unroll
        for (int b = 0; b < 8; ++b) {
          const float2 cj = *reinterpret_cast<const float2*>(sCum + b * 8 + t * 2);
          const float2 dj = *reinterpret_cast<const float2*>(sDt + b * 8 + t * 2);
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const int i = i0 + c * 8, j = b * 8 + t * 2;
            const float u = j <= i ? G[b][2 * c] * fast_exp2(ci[c] - cj.x) * dj.x : 0.f;
            const float v = j < i ? G[b][2 * c + 1] * fast_exp2(ci[c] - cj.y) * dj.y : 0.f;
            m[b / 2][(b & 1) * 2 + c] = pack_bf16x2(u, v);
          }
        }
      }
      float y[8][4];
#pragma unroll
      for (int b = 0; b < 8; ++b)
#pragma unroll
        for (int c = 0; c < 4; ++c) y[b][c] = 0.f;
#pragma unroll
      for (int k = 0; k < NP / 16; ++k) {                  // C . S
        uint32_t a[4];
        ldsm4(a, smem_u32(rowsC + k * 16));
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t b[4];
          ldsm4_t(b, smem_u32(sS + (k * 16 + (lane & 15)) * SC_XP + j * 16 + (lane >> 4) * 8));
          mma_bf16(y[2 * j], a, b[0], b[1]);
          mma_bf16(y[2 * j + 1], a, b[2], b[3]);
        }
      }
      const float ei[2] = {sE[i0], sE[i0 + 8]};
#pragma unroll
      for (int b = 0; b < 8; ++b)
#pragma unroll
        for (int c = 0; c < 4; ++c) y[b][c] *= ei[c >> 1];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (k <= warp) {
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t b[4];
            ldsm4_t(b, smem_u32(sX + (k * 16 + (lane & 15)) * SC_XP + j * 16 + (lane >> 4) * 8));
            mma_bf16(y[2 * j], m[k], b[0], b[1]);
            mma_bf16(y[2 * j + 1], m[k], b[2], b[3]);
          }
        }
      }
      const bool pairs = p.P % 2 == 0 && p.ldy % 2 == 0;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int i = i0 + c * 8;
        if (i >= n_tok) continue;
        bf16* dst = static_cast<bf16*>(p.y) + (row0 + c0 + i) * p.ldy + h * p.P + col0;
#pragma unroll
        for (int b = 0; b < 8; ++b) {
          const int q = b * 8 + t * 2;
          const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sX + i * SC_XP + q));
          const float v0 = y[b][2 * c] + D * x.x, v1 = y[b][2 * c + 1] + D * x.y;
          if (pairs) {
            if (q < cols) *reinterpret_cast<uint32_t*>(dst + q) = pack_bf16x2(v0, v1);
          } else {
            if (q < cols) dst[q] = __float2bfloat16(v0);
            if (q + 1 < cols) dst[q + 1] = __float2bfloat16(v1);
          }
        }
      }
    }
    // ---- the state after the chunk
    const float last = sCum[SC_TOK - 1], decay = sE[SC_TOK - 1];
    total += last;
#pragma unroll
    for (int a = 0; a < RT; ++a)
#pragma unroll
      for (int b = 0; b < 8; ++b)
#pragma unroll
        for (int c = 0; c < 4; ++c) S[a][b][c] *= decay;
#pragma unroll
    for (int k = 0; k < SC_TOK / 16; ++k) {
      const float2 w0 = *reinterpret_cast<const float2*>(sW + k * 16 + t * 2);
      const float2 w1 = *reinterpret_cast<const float2*>(sW + k * 16 + 8 + t * 2);
      uint32_t hi[RT][4], lo[RT][4];
#pragma unroll
      for (int a = 0; a < RT; ++a) {
        uint32_t m[4];
        ldsm4_t(m, smem_u32(sB + (k * 16 + (lane >> 4) * 8 + (lane & 7)) * LD + (warp + 4 * a) * 16 +
                               ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 f = unpack_bf16x2(m[x]), w = x < 2 ? w0 : w1;
          split2(f.x * w.x, f.y * w.y, hi[a][x], lo[a][x]);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t b[4];
        ldsm4_t(b, smem_u32(sX + (k * 16 + (lane & 15)) * SC_XP + j * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int a = 0; a < RT; ++a) {
          mma_bf16(S[a][2 * j], hi[a], b[0], b[1]);
          mma_bf16(S[a][2 * j + 1], hi[a], b[2], b[3]);
          mma_bf16(S[a][2 * j], lo[a], b[0], b[1]);
          mma_bf16(S[a][2 * j + 1], lo[a], b[2], b[3]);
        }
      }
    }
    __syncthreads();                                       // before the chunk is replaced
  }
  if (MODE == SC_FROM) return;
  float* to = MODE == SC_STATE ? p.seg_state + seg_cell : p.state + cell;
#pragma unroll
  for (int a = 0; a < RT; ++a)
#pragma unroll
    for (int b = 0; b < 8; ++b)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int n = (warp + 4 * a) * 16 + r + (c >> 1) * 8, q = b * 8 + t * 2 + (c & 1);
        if (n < p.N && q < cols) to[static_cast<size_t>(n) * p.Pp + col0 + q] = S[a][b][c];
      }
  if (MODE == SC_STATE && tid == 0 && col0 == 0)
    p.seg_decay[static_cast<size_t>(blockIdx.y) * p.heads + h] = exp2f(total);
}

// Turns what the segments of an entry add to an empty state into the state in front of each, and
// leaves the state behind the last one in the slot.
__global__ void __launch_bounds__(256) ssd_carry_kernel(const Ssd p) {
  const int4 run = p.seg_runs[blockIdx.z];
  const int e = run.x, h = blockIdx.y, i = blockIdx.x * 256 + threadIdx.x, size = p.N * p.Pp;
  if (i >= size || i % p.Pp >= p.P) return;
  float* st = p.state + (static_cast<size_t>(p.e.slot[e]) * p.heads + h) * size + i;
  float s = p.e.pos0[e] > 0 ? *st : 0.f;
  for (int k = run.y; k < run.y + run.z; ++k) {
    float* at = p.seg_state + (static_cast<size_t>(k) * p.heads + h) * size + i;
    const float add = *at;
    *at = s;
    s = p.seg_decay[static_cast<size_t>(k) * p.heads + h] * s + add;
  }
  *st = s;
}

template <int NP, int MODE>
static int launch_chunk(const Ssd& p, int n, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ssd_chunk_kernel<NP, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             sc_smem<NP>()) != cudaSuccess)
      return -4;
    set = true;
  }
  dim3 grid(p.heads * ((p.P + SC_COLS - 1) / SC_COLS), n);
  ssd_chunk_kernel<NP, MODE><<<grid, SC_THREADS, sc_smem<NP>(), st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int NP>
static int launch_chunks(const Ssd& p, int n, int runs, cudaStream_t st) {
  if (p.seg_state == nullptr) return launch_chunk<NP, SC_WHOLE>(p, n, st);
  const int rc = launch_chunk<NP, SC_STATE>(p, n, st);
  if (rc != 0) return rc;
  ssd_carry_kernel<<<dim3((p.N * p.Pp + 255) / 256, p.heads, runs), 256, 0, st>>>(p);
  return launch_chunk<NP, SC_FROM>(p, n, st);
}

}  // namespace cb

using namespace cb;

extern "C" int cb_ssd_chunk(const void* u, int ldu, int boff, int coff, const void* dt, int lddt,
                            const float* dt_bias, const float* A_log, const float* D, float* state,
                            void* y, int ldy, int heads, int groups, int N, int P, int Pp,
                            const int* slot, const int* row0, const int* len, const int* pos0,
                            const void* segs, int n, const void* seg_runs, int runs, float* seg_state,
                            float* seg_decay, void* stream) {
  Ssd p;
  const int rc = fill_ssd(p, u, ldu, boff, coff, dt, lddt, dt_bias, A_log, D, state, y, ldy, heads, groups,
                          N, P, Pp, slot, row0, len, pos0, nullptr);
  if (rc != 0) return rc;
  if (n <= 0 || n > 65535 || runs <= 0 || runs > 65535 || N > 128) return -2;
  if ((seg_state == nullptr) != (seg_decay == nullptr)) return -2;
  if ((reinterpret_cast<uintptr_t>(segs) & 15u) || (reinterpret_cast<uintptr_t>(seg_runs) & 15u)) return -5;
  p.segs = static_cast<const int4*>(segs); p.seg_runs = static_cast<const int4*>(seg_runs);
  p.seg_state = seg_state; p.seg_decay = seg_decay;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return N <= 64 ? launch_chunks<64>(p, n, runs, st) : launch_chunks<128>(p, n, runs, st);
}
