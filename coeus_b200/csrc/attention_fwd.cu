// Flash-style attention forward on tcgen05 with the probabilities kept in tensor memory.
//
// Every CTA works on TWO 128-row query tiles of one (batch, head) at a time.  The work of an item
// is a stream of steps (query tile t, key tile j); step g uses score buffer g % NBUF of tensor
// memory, and the scores of step g + NBUF are issued as soon as P.V of step g has completed, so
// that (with three buffers) a softmax warpgroup finds its next scores computed when it finishes:
//   S  = Q_t . K_j^T      tcgen05.mma, operands in 128-byte-swizzled shared memory, S in TMEM
//   P  = exp2(S - m)      one thread per query row; P overwrites S in TMEM as packed bf16
//   O_t += P . V_j        tcgen05.mma with the A operand read from TMEM (no shared-memory trip)
// The S x S score matrix of the reference (plugins/model-transformer/src/lib.rs:237-277) is never
// materialised; causal masking is implicit (lib.rs:746-756) and fully-masked key tiles are skipped.
//
// Roles (384 threads, one CTA per SM, persistent over a heavy-first list of work items):
//   warp 0        TMA producer: Q_A, Q_B once per item, K_j / V_j through two rings
//   warp 1        MMA issue of O_t += P . V (warp-uniform control flow, one elected lane issues)
//   warp 2        MMA issue of the scores, NBUF steps ahead (same form)
//   warps 4..7    softmax of tile A (row r = 32 * (warp % 4) + lane, the TMEM lane it may read)
//   warps 8..11   softmax of tile B
// Online softmax in the exp2 domain with lazy rescaling of O (only when the running maximum grew
// by more than 2^8); optionally a quarter of the exponentials is evaluated as a cubic polynomial
// on the FMA pipe, because the exponential unit (16 results per clock per SM) bounds dh = 64.
// Grouped-query attention: query head h reads K/V head h / (nh / nkv).
//
// Two variants serve prompts of unequal length (PIECES) only.  CAP: scores s become cap * tanh(s / cap),
// from the exponential unit (1) or, where the argument is known not to leave [-1, 1] or [-1/2, 1/2], as
// an odd polynomial on the FMA pipe (2, 3).  DIFF: a head has two maps, each with queries and keys of its own over the same values; an item is ONE
// query tile of a head, tiles A and B of the step are its two maps, every step has its own key tile and
// every pair of steps its value tile.  At the end each warpgroup takes half of the columns of
// o = a0 - w a1, and the two meet at two barriers: one when both results are complete, one for the sum of
// squares of o, which is divided by its root mean square.  KEPT (with a window): the first positions of the
// sequence stay visible behind the window; their keys are tiles of their own.  They come right before the
// first key tile of B: from there on A and B take turns, so that no tile sits out while a buffer that its
// last step used goes round (the wait before rescaling O counts on that).
// Every wait is bounded; a wait that runs out records a status code and the CTA leaves.
#include <cmath>

#include "common.cuh"
#include "ptx.cuh"

namespace cb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, uint64_t inner, uint64_t outer,
                      uint64_t ld, uint32_t box_inner, uint32_t box_outer);
int sm_count();

constexpr int AF_BM = 128;        // rows of one query tile
constexpr int AF_THREADS = 384;

struct AttnFwdArgs {
  int B, S, nh, nkv;
  __nv_bfloat16* O;
  int ldo;
  float* lse;          // [B, nh, S] natural-log LSE of the scaled scores
  float scale_log2;    // softmax scale * log2(e)
  int causal;
  int* status;
  // dropout on the probabilities (training only; drop_thr = 0: none): P is dropped before P.V,
  // the row sums and the LSE are those of the full softmax.  The mask is the one of
  // dropout_bits() over the [B*nh*S, S] probability matrix in row-major order (S % 4 == 0).
  int drop_thr;
  uint32_t drop_key;
  float drop_scale;
  // Pieces of unequal length instead of B sequences of S rows.  Piece b has y = pieces[b].y query
  // rows (at most S) from row pieces[b].x on and w + y keys from row pieces[b].z of K and V on; its
  // query i sees the first w + i + 1 of them (causal), or of those the last `window`.  Two quadruples per
  // piece: with KEPT the second one says that positions 0 .. y - 1 of the sequence, keys from row x on,
  // stay visible, and that z positions lie before the piece's first key.  null: none
  const int4* pieces;
  int vdim;                    // columns of a head that are stored, vdim apart in O
  const float* sink;           // [nh] logits that enter the denominator only, or null
  const __nv_bfloat16* gate;   // [rows, ldg] or null: the output times its sigmoid, column h for all
  int ldg;                     // of head h, or (gate_wide) column h * vdim + d for its column d
  int gate_wide;
  int window;                  // 0: no window
  float cap_log2, cap_in;      // CAP: the cap in units of log2, and what takes a product to the tanh
  float cap_poly[7];           // CAP 2, 3: score / product as a polynomial in the product's square, of
                               // degree 6 or 3
  const float* map_weight;     // DIFF: weight of the second map, factor and eps of the norm
  float map_factor, map_eps;
};

// Optional device timeline of CTA 0 (clock64 stamps; see cb_attn_fwd_set_trace): softmax warp 0
// of tile t writes five stamps per step at [t * 1024 + n * 8 + 0..4] (scores ready, scores in
// registers, maximum known, exponentials done, P handed over), the MMA warp two per step at
// [2048 + n * 8 + 0..1] (P ready, P.V issued and committed), the score warp at [.. + 2..3].
__device__ long long* g_attn_fwd_trace = nullptr;
__device__ int g_attn_fwd_trace_cta = 0;   // which CTA writes the step timeline

template <int DQ, int DV, bool DIFF = false>
struct AFCfg {
  // Keys per step, and score buffers in tensor memory.  Next to two results of 128 columns there is room
  // for 256 columns of scores: two buffers of 128 keys, or four of 64, of which a tile's next scores are
  // computed during its softmax (DIFF: 6 % faster; 1 % slower without, as the steps double).
  static constexpr int BKV = (DIFF && DV == 128) ? 64 : 128;
  static constexpr int NBUF = (DV == 64) ? 3 : 256 / BKV;
  static constexpr int Q_BYTES = AF_BM * DQ * 2;        // one query tile
  static constexpr int K_BYTES = BKV * DQ * 2;          // one K tile
  static constexpr int V_BYTES = BKV * DV * 2;          // one V tile
  static constexpr int KST = DIFF ? (DV == 64 ? 4 : (DQ == 64 ? 8 : 4)) : (DQ == 64 ? 3 : 2);   // ring depth of K
  static constexpr int VST = (DV == 64) ? 3 : 256 / BKV;                                        // and of V
  static constexpr int OFF_Q = 0;
  static constexpr int OFF_K = 2 * Q_BYTES;
  static constexpr int OFF_V = OFF_K + KST * K_BYTES;
  static constexpr int OFF_BAR = OFF_V + VST * V_BYTES;
  static constexpr int OFF_X = OFF_BAR + 512;           // DIFF: two numbers per row and warpgroup
  static constexpr int SMEM_BYTES = OFF_X + (DIFF ? 4 * AF_BM * 4 : 0);
  static constexpr int TMEM_COLS = 512;
  static constexpr int O_COL0 = 0;            // O_t (fp32, DV columns each)
  static constexpr int S_COL0 = 2 * DV;       // NBUF score buffers of BKV fp32 columns; P (bf16)
                                              // takes the first BKV / 2 columns of its buffer
  static_assert(S_COL0 + NBUF * BKV <= TMEM_COLS, "tensor memory budget");
  static_assert(SMEM_BYTES <= 227 * 1024, "shared memory budget");
  // barrier indices
  static constexpr int B_QF = 0, B_QE = 2, B_SF = 4, B_PR = B_SF + NBUF, B_BF = B_PR + NBUF,
                       B_KF = B_BF + NBUF, B_KE = B_KF + KST, B_VF = B_KE + KST,
                       B_VE = B_VF + VST, B_X = B_VE + VST, N_BARS = B_X + 2;
  static_assert(N_BARS * 8 + 16 <= 512, "barrier area");
};

// 2^x for x <= ~8 without the special-function unit and without conversion instructions (which
// share that unit): adding 1.5 * 2^23 rounded down leaves floor(x) in the low mantissa bits, so
// n = floor(x) and f = x - n come from three additions; 2^f is a cubic (relative error 8.6e-5,
// below bf16 resolution) and 2^n is added to the exponent field with a shift and an integer add.
__device__ __forceinline__ float exp2_poly(float x) {
  x = fmaxf(x, -120.0f);
  const float magic = 12582912.0f;
  const float fi = __fadd_rd(x, magic);
  const float f = x - (fi - magic);
  float p = 0.07710139f;
  p = fmaf(p, f, 0.22760755f);
  p = fmaf(p, f, 0.69512522f);
  p = fmaf(p, f, 1.0f);
  return __int_as_float(__float_as_int(p) + (__float_as_int(fi) << 23));
}

// The steps of one CTA in the order every role walks them: items wave by wave (CTA c takes one
// item of every wave of gridDim.x items, counted from the front of even waves and from the back
// of odd ones, so that the heavy and the light ends of the sorted list meet in one CTA), within
// an item key tile by key tile, tile A before tile B.
template <bool PIECES, bool DIFF = false, bool KEPT = false>
struct AFWalk {
  // problem
  int n_items, n_bh, n_pairs, n_q_tiles, n_kv_tiles, nh, causal, bkv, n_waves;
  // position
  int wave, j, t;
  int b, h, qa;          // batch, head, first query tile of the pair
  int4 piece;            // PIECES: the entry of AttnFwdArgs::pieces
  const int4* pieces;
  int n0, n1, nmax;      // key tiles of tile A / B (0: the tile does not exist)
  int lo0, lo1, window;  // first key tile of A / B that a row's window reaches
  int kv_seq;            // how many (item, j) groups came before this one: the K/V ring position
  bool valid;
  int4 kept;             // KEPT: the piece's second quadruple; its kt tiles are j = -kt .. -1, between
                         // lo1 - 1 and lo1
  int kt;

  __device__ int first_row(const AttnFwdArgs& p) const { return PIECES ? piece.x : b * p.S; }
  __device__ int first_key(const AttnFwdArgs& p) const { return PIECES ? piece.z : b * p.S; }
  __device__ int rows(const AttnFwdArgs& p) const { return PIECES ? piece.y : p.S; }
  __device__ int tile() const { return DIFF ? qa : qa + t; }           // query tile of this step
  __device__ int keys_ahead() const { return PIECES ? piece.w : 0; }   // keys before query 0's own
  // KEPT: first position in the window of query q
  __device__ int low_position(int q) const { return kept.z + max(0, piece.w + q + 1 - window); }
  __device__ int first_tile() const { return KEPT && kt > 0 && lo0 >= lo1 ? -kt : lo0; }
  __device__ int next_tile(int i) const {
    if (KEPT && i == -1) return lo1;
    return KEPT && kt > 0 && i + 1 == lo1 && i >= 0 ? -kt : i + 1;
  }
  __device__ int tile_row(const AttnFwdArgs& p, int i) const {
    return KEPT && i < 0 ? kept.x + (i + kt) * bkv : first_key(p) + i * bkv;
  }
  __device__ bool b_has(int i) const { return KEPT && i < 0 ? n1 > 0 : i < n1 && i >= lo1; }
  __device__ void init(const AttnFwdArgs& p, int bkv_) {
    bkv = bkv_;
    n_q_tiles = (p.S + AF_BM - 1) / AF_BM;
    n_kv_tiles = (p.S + bkv - 1) / bkv;
    n_pairs = DIFF ? n_q_tiles : (n_q_tiles + 1) / 2;
    nh = p.nh;
    n_bh = p.B * p.nh;
    n_items = n_pairs * n_bh;
    causal = p.causal;
    window = p.window;
    pieces = p.pieces;
    n_waves = (n_items + gridDim.x - 1) / gridDim.x;
    wave = -1;
    kv_seq = -1;
    valid = true;
    next_item();
  }
  __device__ void next_item() {
    while (true) {
      ++wave;
      if (wave >= n_waves) { valid = false; return; }
      const int c = (wave & 1) ? static_cast<int>(gridDim.x - 1 - blockIdx.x)
                               : static_cast<int>(blockIdx.x);
      const int i = wave * static_cast<int>(gridDim.x) + c;
      if (i >= n_items) continue;
      const int bh = i % n_bh;
      const int pair = n_pairs - 1 - i / n_bh;     // pairs with the most key tiles first
      b = bh / nh;
      h = bh % nh;
      qa = DIFF ? pair : 2 * pair;
      if constexpr (PIECES) {
        piece = pieces[2 * b];
        if constexpr (KEPT) kept = pieces[2 * b + 1];
        n_q_tiles = (piece.y + AF_BM - 1) / AF_BM;
        n_kv_tiles = (piece.w + piece.y + bkv - 1) / bkv;
        if (qa >= n_q_tiles) continue;             // a shorter piece ends before this pair
      }
      const int ahead = keys_ahead();
      n0 = causal ? min(n_kv_tiles, (ahead + (qa + 1) * AF_BM + bkv - 1) / bkv) : n_kv_tiles;
      n1 = DIFF ? n0
           : qa + 1 >= n_q_tiles ? 0
           : (causal ? min(n_kv_tiles, (ahead + (qa + 2) * AF_BM + bkv - 1) / bkv) : n_kv_tiles);
      nmax = max(n0, n1);
      lo0 = lo1 = 0;
      if constexpr (PIECES) {
        if (window > 0) {
          const int low = ahead + qa * AF_BM + 1 - window;     // first key of the tile's first row
          lo0 = max(0, low) / bkv;
          lo1 = DIFF ? lo0 : max(0, low + AF_BM) / bkv;
        }
      }
      if constexpr (KEPT) {
        const int low = low_position(min(piece.y, (qa + 2) * AF_BM) - 1);
        kt = (min(kept.y, low) + bkv - 1) / bkv;
      }
      j = first_tile();
      t = 0;
      ++kv_seq;
      return;
    }
  }
  __device__ void advance() {
    if (t == 0 && b_has(j)) { t = 1; return; }
    j = next_tile(j);
    if (j < nmax) {
      ++kv_seq;
      t = j < n0 ? 0 : 1;
      return;
    }
    next_item();
  }
  __device__ bool last_of_kv() const { return t == 1 || !b_has(j); }   // last tile using K_j / V_j
  __device__ bool first_of_tile() const { return j == (t == 0 ? first_tile() : KEPT && kt > 0 ? -kt : lo1); }
  __device__ bool last_of_tile() const {
    return j == (t ? n1 : KEPT && kt > 0 && n0 <= lo1 ? 0 : n0) - 1;     // tile A may end with kept keys
  }
};

template <int DQ, int DV, bool POLY, bool DROP, bool PIECES, int CAP, bool DIFF, bool KEPT>
__global__ void __launch_bounds__(AF_THREADS, 1)
attn_fwd_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, const AttnFwdArgs p) {
  static_assert(PIECES || (!CAP && !DIFF && !KEPT), "the variants of pieces");
  static_assert(!CAP || !DIFF, "no kernel has both");
  using Cfg = AFCfg<DQ, DV, DIFF>;
  using Walk = AFWalk<PIECES, DIFF, KEPT>;
  constexpr int KST = Cfg::KST, VST = Cfg::VST, NBUF = Cfg::NBUF, BKV = Cfg::BKV;
  constexpr int MAPS = DIFF ? 2 : 1;
  extern __shared__ __align__(1024) uint8_t smem[];
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Cfg::OFF_BAR);
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bars + Cfg::N_BARS);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  volatile uint32_t* seen = tmem_slot + 2;   // [t]: 1 + the last step whose scores tile t's warps saw
  auto bar = [&](int i) { return smem_u32(bars + i); };

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((sbase & 1023u) != 0u) {  // swizzled tiles need a 1024-byte aligned base
    if (threadIdx.x == 0) record_status(p.status, ST_BAD_ARG, 950);
    return;
  }
  const int group = p.nh / p.nkv;

  if (threadIdx.x == 0) {
    for (int t = 0; t < 2; ++t) {
      mbar_init(bar(Cfg::B_QF + t), 1);
      mbar_init(bar(Cfg::B_QE + t), 1);
    }
    for (int s = 0; s < NBUF; ++s) {
      mbar_init(bar(Cfg::B_BF + s), 1);
      mbar_init(bar(Cfg::B_SF + s), 1);
      mbar_init(bar(Cfg::B_PR + s), 4);      // one arrival per softmax warp
    }
    for (int s = 0; s < KST; ++s) {
      mbar_init(bar(Cfg::B_KF + s), 1);
      mbar_init(bar(Cfg::B_KE + s), 1);
    }
    for (int s = 0; s < VST; ++s) {
      mbar_init(bar(Cfg::B_VF + s), 1);
      mbar_init(bar(Cfg::B_VE + s), 1);
    }
    for (int s = 0; s < 2; ++s) mbar_init(bar(Cfg::B_X + s), 8);   // one arrival per softmax warp
    *abort_flag = 0;
    seen[0] = 0;
    seen[1] = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 0) {
    tmem_alloc(smem_u32(const_cast<uint32_t*>(tmem_slot)), Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  auto sQ = [&](int t) { return sbase + Cfg::OFF_Q + t * Cfg::Q_BYTES; };
  auto sK = [&](int s) { return sbase + Cfg::OFF_K + s * Cfg::K_BYTES; };
  auto sV = [&](int s) { return sbase + Cfg::OFF_V + s * Cfg::V_BYTES; };

  // The kernel starts with 168 registers per thread (384 threads); the first warpgroup (producer
  // and MMA issue: little state) hands registers to the two softmax warpgroups, whose step keeps a
  // whole score row plus the walk state in registers: 128 * (88 + 208 + 208) = 64512.
  if (threadIdx.x == 0 && g_attn_fwd_trace != nullptr)
    g_attn_fwd_trace[3072 + 2 * blockIdx.x] = static_cast<long long>(globaltimer_ns());
  if (warp < 4) {
  asm volatile("setmaxnreg.dec.sync.aligned.u32 88;" ::: "memory");
  if (warp == 0) {
    // ---------------------------------------------------------------- producer
    if (lane == 0) {
      uint32_t qcnt[2] = {0u, 0u};     // uses of each query buffer so far
      uint32_t kcnt = 0, vcnt = 0;     // K / V tiles loaded so far
      bool ok = true;
      Walk w;
      w.init(p, BKV);
      while (w.valid && ok) {
        const int row0 = w.first_row(p);
        const int h = w.h, hk = w.h / group, qa = w.qa;
        const int n0 = w.n0, n1 = w.n1, nmax = w.nmax, lo = w.first_tile();
        auto load_q = [&](int t) {
          if ((t == 0 ? n0 : n1) == 0) return;
          if (!mbar_wait(bar(Cfg::B_QE + t), (qcnt[t] & 1u) ^ 1u, abort_flag)) {
            record_status(p.status, ST_WAIT_TIMEOUT, 951);
            ok = false;
            return;
          }
          mbar_arrive_expect_tx(bar(Cfg::B_QF + t), Cfg::Q_BYTES);
#pragma unroll
          for (int c = 0; c < DQ / 64; ++c)
            tma_load_2d(sQ(t) + c * (AF_BM * 128), &tmQ, bar(Cfg::B_QF + t),
                        (h * MAPS + (DIFF ? t : 0)) * DQ + c * 64,
                        row0 + (DIFF ? qa : qa + t) * AF_BM);
          ++qcnt[t];
        };
        auto load_k = [&](int j, int map) {
          const int s = kcnt % KST;
          if (!mbar_wait(bar(Cfg::B_KE + s), ((kcnt / KST) & 1u) ^ 1u, abort_flag)) {
            record_status(p.status, ST_WAIT_TIMEOUT, 952);
            ok = false;
            return;
          }
          mbar_arrive_expect_tx(bar(Cfg::B_KF + s), Cfg::K_BYTES);
#pragma unroll
          for (int c = 0; c < DQ / 64; ++c)
            tma_load_2d(sK(s) + c * (BKV * 128), &tmK, bar(Cfg::B_KF + s), (hk * MAPS + map) * DQ + c * 64,
                        w.tile_row(p, j));
          ++kcnt;
        };
        auto load_v = [&](int j) {
          const int s = vcnt % VST;
          if (!mbar_wait(bar(Cfg::B_VE + s), ((vcnt / VST) & 1u) ^ 1u, abort_flag)) {
            record_status(p.status, ST_WAIT_TIMEOUT, 953);
            ok = false;
            return;
          }
          mbar_arrive_expect_tx(bar(Cfg::B_VF + s), Cfg::V_BYTES);
#pragma unroll
          for (int c = 0; c < DV / 64; ++c)
            tma_load_2d(sV(s) + c * (BKV * 128), &tmV, bar(Cfg::B_VF + s), hk * DV + c * 64,
                        w.tile_row(p, j));
          ++vcnt;
        };
        load_q(0);
        if (ok) load_k(lo, 0);
        if (ok) load_q(1);
        if (DIFF && ok) load_k(lo, 1);
        if (ok) load_v(lo);
        for (int j = w.next_tile(lo); j < nmax && ok; j = w.next_tile(j)) {
          load_k(j, 0);
          if (DIFF && ok) load_k(j, 1);
          if (ok) load_v(j);
        }
        w.next_item();
      }
      if (*abort_flag) {
        // let the copies already in flight land before shared memory is released
        const uint64_t t0 = globaltimer_ns();
        auto drain = [&](int full0, uint32_t cnt, int depth) {
          const uint32_t first = cnt > static_cast<uint32_t>(depth) ? cnt - depth : 0u;
          for (uint32_t u = first; u < cnt; ++u) {
            while (!mbar_try_wait(bar(full0 + u % depth), (u / depth) & 1u)) {
              if (globaltimer_ns() - t0 > 200000000ull) return;
            }
          }
        };
        drain(Cfg::B_KF, kcnt, KST);
        drain(Cfg::B_VF, vcnt, VST);
        for (int t = 0; t < 2; ++t)
          if (qcnt[t] > 0) drain(Cfg::B_QF + t, qcnt[t], 1);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issue: P.V
    // Two warps issue the tensor-core work because the issue cost of an MMA is of the order of
    // its run time at these tile sizes: this warp issues O_t += P.V for every step in order, warp
    // 2 the scores NBUF steps ahead.  Both run warp-uniform control flow with one elected lane
    // issuing (measured ~35 clocks per MMA against ~60-100 from a divergent single lane), and
    // build their descriptors once; a step only adds constants to the address field.
    {
      constexpr uint32_t idesc_o = umma_idesc_bf16(AF_BM, DV, 0, 1);
      const uint64_t dV0 = umma_desc_sw128(sV(0), BKV * 128, 1024);
      const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem_base, 0);
      bool ok = true;
      int v_waited = -1;
      Walk wp;
      wp.init(p, BKV);
      for (uint32_t gp = 0; wp.valid && ok; wp.advance(), ++gp) {
        const uint32_t buf = gp % NBUF;
        const int t = wp.t;
        const int vs = wp.kv_seq % VST;
        if (v_waited != wp.kv_seq) {
          if (!mbar_wait(bar(Cfg::B_VF + vs), (wp.kv_seq / VST) & 1u, abort_flag)) {
            record_status(p.status, ST_WAIT_TIMEOUT, 962);
            break;
          }
          v_waited = wp.kv_seq;
        }
        if (!mbar_wait(bar(Cfg::B_PR + buf), (gp / NBUF) & 1u, abort_flag)) {
          record_status(p.status, ST_WAIT_TIMEOUT, 964);
          break;
        }
        long long* tr = (blockIdx.x == g_attn_fwd_trace_cta && gp < 120 && lane == 0) ? g_attn_fwd_trace : nullptr;
        if (tr) tr[2048 + gp * 8] = clock64();
        tc_fence_after();
        const uint64_t bd0 = dV0 + static_cast<uint64_t>((vs * Cfg::V_BYTES) >> 4);
        const uint32_t d_addr = tmem_u + Cfg::O_COL0 + t * DV;
        const uint32_t a_addr = tmem_u + Cfg::S_COL0 + buf * BKV;
        const uint32_t acc0 = wp.first_of_tile() ? 0u : 1u;
        const bool last_kv = wp.last_of_kv();
        if (elect_one()) {
#pragma unroll
          for (int kk = 0; kk < BKV / 16; ++kk)
            umma_bf16_ts(d_addr, a_addr + kk * 8, bd0 + static_cast<uint64_t>((kk * 2048) >> 4),
                         idesc_o, kk > 0 ? 1u : acc0);
          umma_commit(bar(Cfg::B_BF + buf));     // P consumed, O_t updated
          if (last_kv) umma_commit(bar(Cfg::B_VE + vs));
        }
        __syncwarp();
        if (tr) tr[2048 + gp * 8 + 1] = clock64();
      }
    }
    __syncwarp();
  } else if (warp == 2) {
    // ---------------------------------------------------------------- MMA issue: scores
    {
      constexpr uint32_t idesc_s = umma_idesc_bf16(AF_BM, BKV, 0, 0);
      const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem_base, 0);
      const uint64_t dQ0 = umma_desc_sw128(sQ(0), 16, 1024);
      const uint64_t dK0 = umma_desc_sw128(sK(0), 16, 1024);
      uint32_t qc0 = 0u, qc1 = 0u;
      int k_waited = -1;
      bool ok = true;
      auto wait1 = [&](int b_idx, uint32_t parity, int where) {
        if (!mbar_wait(bar(b_idx), parity, abort_flag)) {
          record_status(p.status, ST_WAIT_TIMEOUT, where);
          ok = false;
        }
        return ok;
      };
      Walk ws;
      ws.init(p, BKV);
      for (uint32_t gs = 0; ws.valid && ok; ws.advance(), ++gs) {
        const int t = ws.t;
        const uint32_t buf = gs % NBUF;
        // the buffer is free once P.V of the step that used it last has completed
        if (gs >= NBUF && !wait1(Cfg::B_BF + buf, ((gs / NBUF) - 1u) & 1u, 963)) break;
        if (ws.first_of_tile()) {
          if (!wait1(Cfg::B_QF + t, (t ? qc1 : qc0) & 1u, 960)) break;
          if (t) ++qc1; else ++qc0;
        }
        const int k_seq = DIFF ? static_cast<int>(gs) : ws.kv_seq;    // K tiles that came before
        const int ks = k_seq % KST;
        if (k_waited != k_seq) {
          if (!wait1(Cfg::B_KF + ks, (k_seq / KST) & 1u, 961)) break;
          k_waited = k_seq;
        }
        long long* tr = (blockIdx.x == g_attn_fwd_trace_cta && gs < 120 && lane == 0) ? g_attn_fwd_trace : nullptr;
        if (tr) tr[2048 + gs * 8 + 2] = clock64();
        tc_fence_after();
        const uint64_t ad0 = dQ0 + static_cast<uint64_t>((t * Cfg::Q_BYTES) >> 4);
        const uint64_t bd0 = dK0 + static_cast<uint64_t>((ks * Cfg::K_BYTES) >> 4);
        const uint32_t d_addr = tmem_u + Cfg::S_COL0 + buf * BKV;
        const bool last_tile = ws.last_of_tile(), last_kv = DIFF || ws.last_of_kv();
        if (elect_one()) {
#pragma unroll
          for (int kk = 0; kk < DQ / 16; ++kk) {
            const uint64_t a_off = static_cast<uint64_t>(((kk / 4) * (AF_BM * 128) + (kk % 4) * 32) >> 4);
            const uint64_t b_off = static_cast<uint64_t>(((kk / 4) * (BKV * 128) + (kk % 4) * 32) >> 4);
            umma_bf16_ss(d_addr, ad0 + a_off, bd0 + b_off, idesc_s, kk > 0 ? 1u : 0u);
          }
          umma_commit(bar(Cfg::B_SF + buf));
          if (last_tile) umma_commit(bar(Cfg::B_QE + t));   // Q_t's buffer may be refilled
          if (last_kv) umma_commit(bar(Cfg::B_KE + ks));
        }
        __syncwarp();
        if (tr) tr[2048 + gs * 8 + 3] = clock64();
      }
    }
    __syncwarp();
  }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 208;" ::: "memory");
    // ---------------------------------------------------------------- softmax + epilogue
    const int t = (warp - 4) >> 2;             // which query tile of the pair
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;         // query row within the tile = TMEM lane
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    const uint32_t o_addr = lane_addr + Cfg::O_COL0 + t * DV;
    uint32_t items = 0;                          // DIFF: items finished
    uint32_t g = 0, g_prev = 0, mine = 0, own_seen = 0;
    bool ok = true;
    float m_used = -INFINITY;
    float l[4] = {0.f, 0.f, 0.f, 0.f};           // the row sum is kept as four partial sums
    Walk w;
    w.init(p, BKV);
    for (; w.valid && ok; w.advance(), ++g) {
      if (w.t != t) continue;
      const int j = w.j;
      const int q0 = w.tile() * AF_BM;
      const int q_idx = q0 + r;
      const bool first = w.first_of_tile();
      if (first) {
        m_used = -INFINITY;
        l[0] = l[1] = l[2] = l[3] = 0.f;
      }
      const uint32_t buf = g % NBUF;
      const uint32_t s_addr = lane_addr + Cfg::S_COL0 + buf * BKV;
      // The parity wait below is only meaningful once the scores of step g - NBUF (the previous
      // use of this barrier) are known to be complete: with that phase still open, the wait for
      // the opposite parity would return at once.  A warpgroup's own recent steps imply it; after
      // sitting out several steps (an item with a single query tile; key tiles that only tile B
      // sees under a causal mask) the other warpgroup's published progress does: it owned all the
      // steps in between, none of which depends on this warpgroup.
      {
        const uint32_t need = g >= NBUF ? g - NBUF + 1u : 0u;
        if (own_seen < need) {
          bool got = true;
          if (seen[1 - t] < need) {
            const uint64_t t0 = globaltimer_ns();
            uint32_t n = 0;
            while (seen[1 - t] < need) {
              if ((++n & 63u) == 0u) {
                if (*abort_flag) { got = false; break; }
                if (globaltimer_ns() - t0 > CB_WAIT_LIMIT_NS) {
                  *abort_flag = 1u;
                  got = false;
                  break;
                }
              }
            }
          }
          if (!__all_sync(0xffffffffu, got)) {
            if (lane == 0) record_status(p.status, ST_WAIT_TIMEOUT, 973);
            ok = false;
            break;
          }
        }
      }
      {
        const bool got = mbar_wait(bar(Cfg::B_SF + buf), (g / NBUF) & 1u, abort_flag);
        if (!__all_sync(0xffffffffu, got)) {
          if (lane == 0) record_status(p.status, ST_WAIT_TIMEOUT, 970);
          ok = false;
          break;
        }
      }
      own_seen = g + 1u;
      if (quarter == 0 && lane == 0) seen[t] = g + 1u;   // one writer per tile: monotonic
      long long* tr = (blockIdx.x == g_attn_fwd_trace_cta && mine < 120 && quarter == 0 && lane == 0)
                          ? g_attn_fwd_trace : nullptr;
      const uint32_t tri = t * 1024 + mine * 8;
      ++mine;
      if (tr) tr[tri] = clock64();
      tc_fence_after();
      int kv0 = j * BKV;
      const bool below = PIECES && p.window > 0;
      bool need_mask = (p.causal && kv0 + BKV - 1 > q0 + w.keys_ahead()) ||
                             (kv0 + BKV > w.keys_ahead() + w.rows(p)) ||
                             (below && kv0 < q0 + AF_BM + w.keys_ahead() - p.window);
      int kv_limit = w.keys_ahead() + (p.causal ? min(q_idx, w.rows(p) - 1) : (w.rows(p) - 1));  // last visible key
      int kv_low = below ? kv_limit - p.window : -1;                                             // last one hidden below
      if constexpr (KEPT) {
        if (j < 0) {          // kept positions that lie below the row's window
          kv0 = (j + w.kt) * BKV;
          kv_limit = min(w.kept.y, w.low_position(min(q_idx, w.rows(p) - 1))) - 1;
          kv_low = -1;
          need_mask = true;
        }
      }
      uint32_t v[BKV];
#pragma unroll
      for (int c = 0; c < BKV / 32; ++c) tmem_ld_32x32b_x32(s_addr + c * 32, v + c * 32);
      tmem_ld_wait();
      if (tr) tr[tri + 1] = clock64();
      if constexpr (CAP >= 2) {
        constexpr int DEG = CAP == 2 ? 6 : 3;
#pragma unroll
        for (int e = 0; e < BKV; e += 2) {
          const float a = __uint_as_float(v[e]), b = __uint_as_float(v[e + 1]);
          float wa, wb, ra = p.cap_poly[DEG], rb = ra;
          fma2(wa, wb, a, b, a, b, 0.f, 0.f);
#pragma unroll
          for (int i = DEG - 1; i >= 0; --i) fma2(ra, rb, ra, rb, wa, wb, p.cap_poly[i], p.cap_poly[i]);
          fma2(ra, rb, ra, rb, a, b, 0.f, 0.f);
          v[e] = __float_as_uint(ra);
          v[e + 1] = __float_as_uint(rb);
        }
      } else if constexpr (CAP == 1) {
#pragma unroll
        for (int e = 0; e < BKV; ++e)
          v[e] = __float_as_uint(p.cap_log2 * tanh_exp(__uint_as_float(v[e]) * p.cap_in));
      }
      if (need_mask) {
        // hidden keys get a score of -inf, after which the step takes the common path (their
        // exponential is an exact zero); with causal masking every row sees at least key 0, with
        // a window at least its own key
#pragma unroll
        for (int e = 0; e < BKV; ++e)
          if (kv0 + e > kv_limit || (PIECES && kv0 + e <= kv_low)) v[e] = 0xff800000u;
      }
      float mx;
      {
        float m0 = -INFINITY, m1 = -INFINITY, m2 = -INFINITY, m3 = -INFINITY;
#pragma unroll
        for (int e = 0; e < BKV; e += 8) {     // four chains of three-input maxima
          m0 = max3(m0, __uint_as_float(v[e]), __uint_as_float(v[e + 1]));
          m1 = max3(m1, __uint_as_float(v[e + 2]), __uint_as_float(v[e + 3]));
          m2 = max3(m2, __uint_as_float(v[e + 4]), __uint_as_float(v[e + 5]));
          m3 = max3(m3, __uint_as_float(v[e + 6]), __uint_as_float(v[e + 7]));
        }
        mx = fmaxf(fmaxf(m0, m1), fmaxf(m2, m3));
      }
      if constexpr (!CAP) mx *= p.scale_log2;  // scale > 0, so max commutes with it
      const float m_new = fmaxf(m_used, mx);
      const bool grow = (m_new - m_used) > 8.0f;  // also true for the first step (m_used = -inf)
      if (!first && __any_sync(0xffffffffu, grow)) {
        // O_t may be rescaled once P.V of the previous step of this tile has completed.  (The
        // wait is skipped when no row needs rescaling: the barrier of that buffer cannot advance
        // a second time before this step hands over its P, so no phase is missed.)
        const bool got = mbar_wait(bar(Cfg::B_BF + g_prev % NBUF), (g_prev / NBUF) & 1u, abort_flag);
        if (!__all_sync(0xffffffffu, got)) {
          if (lane == 0) record_status(p.status, ST_WAIT_TIMEOUT, 972);
          ok = false;
          break;
        }
        tc_fence_after();
        const float f = grow ? fast_exp2(m_used - m_new) : 1.0f;
#pragma unroll 1
        for (int c = 0; c < DV / 16; ++c) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(o_addr + c * 16, o);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
          tmem_st_32x32b_x16(o_addr + c * 16, o);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a) l[a] *= f;
      }
      g_prev = g;
      // a row that has seen no key yet (below its window) keeps a maximum under every score
      if (grow) m_used = (m_new == -INFINITY) ? 0.f : m_new;
      else if (PIECES && m_used == -INFINITY) m_used = -1e30f;
      // P = exp2(s * scale - m) as packed bf16 over the first half of the score buffer; row sum
      const float sc = CAP ? 1.0f : p.scale_log2, nm = -m_used;
      if (tr) tr[tri + 2] = clock64();
      if constexpr (DROP) {
        // four consecutive keys share one hash; the index of this row's first key of the tile is
        // a multiple of four (S and the tile width are)
        const unsigned long long g0 =
            ((static_cast<unsigned long long>(w.b) * p.nh + w.h) * p.S + q_idx) *
                static_cast<unsigned long long>(p.S >> 2) + static_cast<unsigned long long>(kv0 >> 2);
#pragma unroll
        for (int c = 0; c < BKV / 32; ++c) {
          uint32_t pk[16];
#pragma unroll
          for (int e = 0; e < 32; e += 4) {
            const uint32_t bits = dropout_bits(g0 + (c * 32 + e) / 4, p.drop_key);
            float pe[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              pe[j] = fast_exp2(fmaf(__uint_as_float(v[c * 32 + e + j]), sc, nm));
              l[j] += pe[j];
              pe[j] *= dropout_factor(bits, j, p.drop_thr, p.drop_scale);
            }
            pk[e >> 1] = pack_bf16x2(pe[0], pe[1]);
            pk[(e >> 1) + 1] = pack_bf16x2(pe[2], pe[3]);
          }
          tmem_st_32x32b_x16(s_addr + c * 16, pk);
        }
      } else {
#pragma unroll
      for (int c = 0; c < BKV / 32; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          const float t0 = fmaf(__uint_as_float(v[c * 32 + e]), sc, nm);
          const float t1 = fmaf(__uint_as_float(v[c * 32 + e + 1]), sc, nm);
          float p0, p1;
          if (POLY && (e & 6) == 6) {       // columns 6, 7 of every 8: a quarter of the row
            p0 = exp2_poly(t0);
            p1 = exp2_poly(t1);
          } else {
            p0 = fast_exp2(t0);
            p1 = fast_exp2(t1);
          }
          l[(e >> 1) & 3] += p0 + p1;
          pk[e >> 1] = pack_bf16x2(p0, p1);
        }
        tmem_st_32x32b_x16(s_addr + c * 16, pk);
      }
      }
      if (tr) tr[tri + 3] = clock64();
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(Cfg::B_PR + buf));
      if (tr) tr[tri + 4] = clock64();
      if (!w.last_of_tile()) continue;
      // ---- last step of this tile: O_t / l and the LSE leave once its P.V has completed
      {
        const bool got = mbar_wait(bar(Cfg::B_BF + buf), (g / NBUF) & 1u, abort_flag);
        if (!__all_sync(0xffffffffu, got)) {
          if (lane == 0) record_status(p.status, ST_WAIT_TIMEOUT, 971);
          ok = false;
          break;
        }
      }
      tc_fence_after();
      const float lsum = (l[0] + l[1]) + (l[2] + l[3]);
      float inv_l = lsum > 0.f ? 1.0f / lsum : 0.f;
      const bool row_ok = q_idx < w.rows(p);
      const size_t out_row = static_cast<size_t>(w.first_row(p)) + q_idx;
      if constexpr (DIFF) {
        float* x_norm = reinterpret_cast<float*>(smem + Cfg::OFF_X);      // [2][AF_BM] 1 / row sums
        float* x_sum = x_norm + 2 * AF_BM;                                // [2][AF_BM] sums of squares
        auto meet = [&](int which) {
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(bar(Cfg::B_X + which));
          const bool got = mbar_wait(bar(Cfg::B_X + which), items & 1u, abort_flag);
          if (!__all_sync(0xffffffffu, got)) {
            if (lane == 0) record_status(p.status, ST_WAIT_TIMEOUT, 974 + which);
            return false;
          }
          tc_fence_after();
          return true;
        };
        x_norm[t * AF_BM + r] = inv_l;
        ok = meet(0);
        if (!ok) break;
        const float n0 = x_norm[r], n1 = -*p.map_weight * x_norm[AF_BM + r];
        constexpr int HALF = DV / 2;
        const uint32_t half_addr = lane_addr + Cfg::O_COL0 + t * HALF;
        float y[HALF], ss = 0.f;
#pragma unroll
        for (int c = 0; c < HALF / 16; ++c) {
          uint32_t a[16], b[16];
          tmem_ld_32x32b_x16(half_addr + c * 16, a);
          tmem_ld_32x32b_x16(half_addr + DV + c * 16, b);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const float o = __uint_as_float(a[e]) * n0 + __uint_as_float(b[e]) * n1;
            y[c * 16 + e] = o;
            ss += o * o;
          }
        }
        x_sum[t * AF_BM + r] = ss;
        ok = meet(1);           // both have read both results: the next item may overwrite them
        if (!ok) break;
        ++items;
        if (!row_ok) continue;
        const float f = p.map_factor / sqrtf((x_sum[r] + x_sum[AF_BM + r]) / p.vdim + p.map_eps);
        __nv_bfloat16* dst = p.O + out_row * p.ldo + static_cast<size_t>(w.h) * p.vdim + t * HALF;
        const int left = p.vdim - t * HALF;
        const bool vec = (p.vdim & 7) == 0;
#pragma unroll
        for (int gq = 0; gq < HALF / 8; ++gq) {
          if (vec) {
            if (gq * 8 < left) {
              uint4 wv;
              wv.x = pack_bf16x2(y[8 * gq + 0] * f, y[8 * gq + 1] * f);
              wv.y = pack_bf16x2(y[8 * gq + 2] * f, y[8 * gq + 3] * f);
              wv.z = pack_bf16x2(y[8 * gq + 4] * f, y[8 * gq + 5] * f);
              wv.w = pack_bf16x2(y[8 * gq + 6] * f, y[8 * gq + 7] * f);
              *reinterpret_cast<uint4*>(dst + gq * 8) = wv;
            }
          } else {
#pragma unroll
            for (int x = 0; x < 8; ++x)
              if (gq * 8 + x < left) dst[gq * 8 + x] = __float2bfloat16(y[8 * gq + x] * f);
          }
        }
        continue;
      }
      if constexpr (PIECES) {
        if (p.sink != nullptr)
          inv_l = 1.0f / (lsum + exp2f(p.sink[w.h] * 1.4426950408889634f - m_used));
        if (p.gate != nullptr && row_ok && !p.gate_wide)
          inv_l /= 1.0f + expf(-__bfloat162float(p.gate[out_row * p.ldg + w.h]));
      }
      __nv_bfloat16* orow = p.O + out_row * p.ldo + static_cast<size_t>(w.h) * (PIECES ? p.vdim : DV);
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32b_x32(o_addr + c * 32, o);
        tmem_ld_wait();
        if (row_ok) {
          if constexpr (PIECES) {
            if (p.gate != nullptr && p.gate_wide) {
              const __nv_bfloat16* gp = p.gate + out_row * p.ldg + static_cast<size_t>(w.h) * p.vdim + c * 32;
              const bool vec = (p.vdim & 7) == 0;
#pragma unroll
              for (int gq = 0; gq < 4; ++gq) {
                float f[8];
                if (vec && c * 32 + gq * 8 < p.vdim) {
                  load8(gp + gq * 8, f);
                } else {
#pragma unroll
                  for (int x = 0; x < 8; ++x)
                    f[x] = c * 32 + gq * 8 + x < p.vdim ? __bfloat162float(gp[gq * 8 + x]) : 0.f;
                }
#pragma unroll
                for (int x = 0; x < 8; ++x)
                  o[8 * gq + x] = __float_as_uint(__fdividef(__uint_as_float(o[8 * gq + x]), 1.0f + __expf(-f[x])));
              }
            }
          }
#pragma unroll
          for (int gq = 0; gq < 4; ++gq) {
            uint4 wv;
            wv.x = pack_bf16x2(__uint_as_float(o[8 * gq + 0]) * inv_l, __uint_as_float(o[8 * gq + 1]) * inv_l);
            wv.y = pack_bf16x2(__uint_as_float(o[8 * gq + 2]) * inv_l, __uint_as_float(o[8 * gq + 3]) * inv_l);
            wv.z = pack_bf16x2(__uint_as_float(o[8 * gq + 4]) * inv_l, __uint_as_float(o[8 * gq + 5]) * inv_l);
            wv.w = pack_bf16x2(__uint_as_float(o[8 * gq + 6]) * inv_l, __uint_as_float(o[8 * gq + 7]) * inv_l);
            const int d0 = c * 32 + gq * 8;
            if (!PIECES || (d0 + 8 <= p.vdim && (p.vdim & 7) == 0)) {
              *reinterpret_cast<uint4*>(orow + d0) = wv;
            } else {
#pragma unroll
              for (int x = 0; x < 8; ++x)
                if (d0 + x < p.vdim)
                  orow[d0 + x] = __float2bfloat16(__uint_as_float(o[8 * gq + x]) * inv_l);
            }
          }
        }
      }
      if (row_ok && p.lse != nullptr)
        p.lse[(static_cast<size_t>(w.b) * p.nh + w.h) * p.S + q_idx] =
            (m_used + log2f(lsum)) * 0.6931471805599453f;
      tc_fence_before();   // these reads of O_t precede the next item's first P.V (ordered by B_PR)
    }
  }

  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && g_attn_fwd_trace != nullptr)
    g_attn_fwd_trace[3072 + 2 * blockIdx.x + 1] = static_cast<long long>(globaltimer_ns());
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
  }
}

template <int DQ, int DV, bool POLY, bool DROP = false, bool PIECES = false, int CAP = 0, bool DIFF = false,
          bool KEPT = false>
static int launch_attn_fwd(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv,
                              const AttnFwdArgs& a, int max_ctas, cudaStream_t st) {
  using Cfg = AFCfg<DQ, DV, DIFF>;
  static bool configured = false;
  auto kern = attn_fwd_kernel<DQ, DV, POLY, DROP, PIECES, CAP, DIFF, KEPT>;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES) != cudaSuccess)
      return -10;
    configured = true;
  }
  const int n_q_tiles = (a.S + AF_BM - 1) / AF_BM;
  const int items = (DIFF ? n_q_tiles : (n_q_tiles + 1) / 2) * a.B * a.nh;
  int grid = sm_count();
  if (max_ctas > 0 && max_ctas < grid) grid = max_ctas;
  if (items < grid) grid = items;
  kern<<<grid, AF_THREADS, Cfg::SMEM_BYTES, st>>>(tq, tk, tv, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

}  // namespace cb

// Device buffer of at least 3072 + 2 * (number of CTAs) int64 for the timeline of CTA `cta` and
// the start / end times (globaltimer) of every CTA at [3072 + 2 * c]; nullptr switches it off.
extern "C" int cb_attn_fwd_set_trace(long long* device_buffer, int cta) {
  if (cudaMemcpyToSymbol(cb::g_attn_fwd_trace_cta, &cta, sizeof(cta)) != cudaSuccess) return -1;
  return cudaMemcpyToSymbol(cb::g_attn_fwd_trace, &device_buffer, sizeof(device_buffer)) == cudaSuccess ? 0 : -1;
}

// q: bf16 [B*S, nh*dh] view (row pitch ldq); k, v: bf16 [B*S, nkv*dh] views (pitches ldk, ldv;
// nkv divides nh, query head h reads K/V head h / (nh / nkv)); they may be column slices of one
// fused projection output.  o: [B*S, nh*dh] pitch ldo.  lse: fp32 [B, nh, S].
// poly != 0 evaluates a quarter of the exponentials as a polynomial on the FMA pipe.
// drop_thr in [0, 255] (0: no dropout; needs S % 4 == 0 otherwise), drop_key: see AttnFwdArgs.
extern "C" int cb_attn_fwd_dropout(const void* q, const void* k, const void* v, void* o, float* lse,
                                   int B, int S, int nh, int nkv, int dh, int ldq, int ldk,
                                   int ldv, int ldo, float scale, int causal, int poly,
                                   int drop_thr, unsigned int drop_key, int* status, int max_ctas,
                                   void* stream) {
  using namespace cb;
  if (dh != 64 && dh != 128) return -1;
  if (B <= 0 || S <= 0 || nh <= 0 || nkv <= 0 || (nh % nkv) != 0 || (ldo % 8) != 0) return -2;
  if (drop_thr < 0 || drop_thr > 255 || (drop_thr > 0 && (S % 4) != 0)) return -6;
  CUtensorMap tq, tk, tv;
  const uint64_t rows = static_cast<uint64_t>(B) * S;
  const uint32_t bkv = AFCfg<128, 128>::BKV;
  if (make_tmap_bf16_2d(&tq, q, static_cast<uint64_t>(nh) * dh, rows, ldq, 64, AF_BM) != 0) return -3;
  if (make_tmap_bf16_2d(&tk, k, static_cast<uint64_t>(nkv) * dh, rows, ldk, 64, bkv) != 0) return -4;
  if (make_tmap_bf16_2d(&tv, v, static_cast<uint64_t>(nkv) * dh, rows, ldv, 64, bkv) != 0) return -5;
  AttnFwdArgs a;
  a.B = B; a.S = S; a.nh = nh; a.nkv = nkv;
  a.O = static_cast<__nv_bfloat16*>(o);
  a.ldo = ldo;
  a.lse = lse;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.causal = causal;
  a.status = status;
  a.pieces = nullptr;
  a.vdim = dh;
  a.sink = nullptr;
  a.gate = nullptr;
  a.ldg = 0;
  a.gate_wide = 0;
  a.window = 0;
  a.drop_thr = drop_thr;
  a.drop_key = drop_key;
  a.drop_scale = 256.0f / static_cast<float>(256 - drop_thr);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (drop_thr > 0)
    return dh == 64 ? launch_attn_fwd<64, 64, false, true>(tq, tk, tv, a, max_ctas, st)
                    : launch_attn_fwd<128, 128, false, true>(tq, tk, tv, a, max_ctas, st);
  if (poly)
    return dh == 64 ? launch_attn_fwd<64, 64, true>(tq, tk, tv, a, max_ctas, st)
                    : launch_attn_fwd<128, 128, true>(tq, tk, tv, a, max_ctas, st);
  return dh == 64 ? launch_attn_fwd<64, 64, false>(tq, tk, tv, a, max_ctas, st)
                  : launch_attn_fwd<128, 128, false>(tq, tk, tv, a, max_ctas, st);
}

extern "C" int cb_attn_fwd(const void* q, const void* k, const void* v, void* o, float* lse,
                           int B, int S, int nh, int nkv, int dh, int ldq, int ldk, int ldv,
                           int ldo, float scale, int causal, int poly, int* status, int max_ctas,
                           void* stream) {
  return cb_attn_fwd_dropout(q, k, v, o, lse, B, S, nh, nkv, dh, ldq, ldk, ldv, ldo, scale, causal,
                             poly, 0, 0u, status, max_ctas, stream);
}

// Coefficients c[0 .. n] of the polynomial in u = x * x that meets tanh(x) / x at the n + 1 Chebyshev nodes
// of u in [0, bound^2] (Newton's divided differences, multiplied out).  x times it is within 3e-7 of
// tanh(x) for n = 6, bound = 1 and for n = 3, bound = 1/2.
static void tanh_ratio(double bound, int n, double* c) {
  double u[8], d[8];
  for (int i = 0; i <= n; ++i) {
    u[i] = 0.5 * bound * bound * (1.0 + std::cos(3.14159265358979323846 * (i + 0.5) / (n + 1)));
    d[i] = std::tanh(std::sqrt(u[i])) / std::sqrt(u[i]);
  }
  for (int k = 1; k <= n; ++k)
    for (int i = n; i >= k; --i) d[i] = (d[i] - d[i - 1]) / (u[i] - u[i - k]);
  for (int i = 0; i <= n; ++i) c[i] = 0.0;
  for (int k = n; k >= 0; --k) {                 // c <- c * (x - u[k]) + d[k]
    for (int i = n; i > 0; --i) c[i] = c[i - 1] - u[k] * c[i];
    c[0] = d[k] - u[k] * c[0];
  }
}

// Causal attention of a ragged batch in pieces (see AttnFwdArgs): n_pieces pairs of quadruples over `rows`
// query rows and `kv_rows` key rows, none with more than max_len queries.  Heads of q and k are dq
// apart, heads of v dv (64 or 128, padded with zeros), heads of o vdim <= dv.  sink (fp32 [nh]) is a logit
// per head that enters the softmax denominator only; gate (bf16, column h of a pitch-ldg view, or with
// gate_wide column h * vdim + d) multiplies head h's output by its sigmoid; both may be null.  A
// query sees the last `window` of its keys (0: all), with keep > 0 also the first positions that the pieces
// name.  scale > 0.  Scores are capped by softcap (0: not).
// score_max bounds |q . k| * scale where the caller knows it (0: not known).
// With two maps q and k have two heads per head (map 0 first), and the output is the weighted difference
// divided by its root mean square, times map_factor; it has neither sink, gate nor cap.
extern "C" int cb_attn_fwd_pieces(const void* q, const void* k, const void* v, void* o, int rows,
                                  int kv_rows, const void* pieces, int n_pieces, int max_len, int nh,
                                  int nkv, int dq, int dv, int vdim, int ldq, int ldk, int ldv, int ldo,
                                  float scale, const float* sink, const void* gate, int ldg,
                                  int gate_wide, int window, int keep, float softcap, float score_max, int maps,
                                  const float* map_weight, float map_factor, float map_eps, int* status,
                                  void* stream) {
  using namespace cb;
  if (!(dq == 64 && dv == 64) && !(dq == 128 && dv == 128) && !(dq == 64 && dv == 128 && maps == 2)) return -1;
  if (gate_wide && vdim % 8 == 0 && ((reinterpret_cast<uintptr_t>(gate) & 15u) || ldg % 8)) return -6;
  if (window < 0 || keep < 0 || softcap < 0.f || (maps != 1 && maps != 2)) return -2;
  if (keep > 0 && (window == 0 || maps == 2 || softcap > 0.f)) return -7;
  if (maps == 2 && (sink != nullptr || gate != nullptr || softcap > 0.f || map_weight == nullptr)) return -7;
  if (softcap > 0.f && sink != nullptr) return -7;
  if (rows <= 0 || kv_rows <= 0 || n_pieces <= 0 || max_len <= 0 || nh <= 0 || nkv <= 0 ||
      (nh % nkv) != 0 || (ldo % 8) != 0 || vdim < 1 || vdim > dv || !(scale > 0.f))
    return -2;
  CUtensorMap tq, tk, tv;
  const uint32_t bkv = maps == 2 && dv == 128 ? AFCfg<128, 128, true>::BKV : AFCfg<128, 128>::BKV;
  if (make_tmap_bf16_2d(&tq, q, static_cast<uint64_t>(nh) * maps * dq, rows, ldq, 64, AF_BM) != 0) return -3;
  if (make_tmap_bf16_2d(&tk, k, static_cast<uint64_t>(nkv) * maps * dq, kv_rows, ldk, 64, bkv) != 0) return -4;
  if (make_tmap_bf16_2d(&tv, v, static_cast<uint64_t>(nkv) * dv, kv_rows, ldv, 64, bkv) != 0) return -5;
  AttnFwdArgs a = {};
  a.B = n_pieces; a.S = max_len; a.nh = nh; a.nkv = nkv;
  a.O = static_cast<__nv_bfloat16*>(o);
  a.ldo = ldo;
  a.vdim = vdim;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.causal = 1;
  a.status = status;
  a.drop_scale = 1.0f;
  a.pieces = static_cast<const int4*>(pieces);
  a.sink = sink;
  a.gate = static_cast<const __nv_bfloat16*>(gate);
  a.ldg = ldg;
  a.gate_wide = gate_wide;
  a.window = window;
  a.map_weight = map_weight;
  a.map_factor = map_factor;
  a.map_eps = map_eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (maps == 2) {
    if (dv == 64) return launch_attn_fwd<64, 64, false, false, true, 0, true>(tq, tk, tv, a, 0, st);
    return dq == 64 ? launch_attn_fwd<64, 128, false, false, true, 0, true>(tq, tk, tv, a, 0, st)
                    : launch_attn_fwd<128, 128, false, false, true, 0, true>(tq, tk, tv, a, 0, st);
  }
  if (softcap > 0.f) {
    a.cap_log2 = softcap * 1.4426950408889634f;
    a.cap_in = scale / softcap;
    if (score_max > 0.f && score_max <= softcap) {
      const bool narrow = score_max <= 0.5f * softcap;
      double t[7];
      tanh_ratio(narrow ? 0.5 : 1.0, narrow ? 3 : 6, t);
      double f = static_cast<double>(a.cap_log2) * a.cap_in;
      for (int i = 0; i <= (narrow ? 3 : 6); ++i, f *= static_cast<double>(a.cap_in) * a.cap_in)
        a.cap_poly[i] = static_cast<float>(t[i] * f);
      if (narrow)
        return dv == 64 ? launch_attn_fwd<64, 64, false, false, true, 3>(tq, tk, tv, a, 0, st)
                        : launch_attn_fwd<128, 128, false, false, true, 3>(tq, tk, tv, a, 0, st);
      return dv == 64 ? launch_attn_fwd<64, 64, false, false, true, 2>(tq, tk, tv, a, 0, st)
                      : launch_attn_fwd<128, 128, false, false, true, 2>(tq, tk, tv, a, 0, st);
    }
    return dv == 64 ? launch_attn_fwd<64, 64, false, false, true, 1>(tq, tk, tv, a, 0, st)
                    : launch_attn_fwd<128, 128, false, false, true, 1>(tq, tk, tv, a, 0, st);
  }
  if (keep > 0)
    return dv == 64 ? launch_attn_fwd<64, 64, false, false, true, 0, false, true>(tq, tk, tv, a, 0, st)
                    : launch_attn_fwd<128, 128, false, false, true, 0, false, true>(tq, tk, tv, a, 0, st);
  return dv == 64 ? launch_attn_fwd<64, 64, false, false, true>(tq, tk, tv, a, 0, st)
                  : launch_attn_fwd<128, 128, false, false, true>(tq, tk, tv, a, 0, st);
}
