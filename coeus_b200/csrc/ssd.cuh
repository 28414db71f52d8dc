// The state-space recurrence with one decay per head (see ssd.cu): what its kernels share.
#pragma once
#include "ragged.cuh"

namespace cb {

struct Ssd {
  const void* u;           // [rows, ldu]: x at 0, B at boff, C at coff (behind the convolution)
  int ldu, boff, coff;
  const void* dt;          // [rows, lddt], column h: head h
  int lddt;
  const float* dt_bias;    // [heads]
  const float* A_log;
  const float* D;
  float* state;            // [slots, heads, N, Pp]
  void* y;                 // out [rows, ldy], head h at h * P
  int ldy;
  int heads, groups, N, P, Pp;
  Entries e;
  const int* entry;        // [n] entries this launch works on (step kernel)
  // segments of long entries (chunk kernel)
  const int4* segs;        // [n] (entry, first token inside it, tokens, 0)
  const int4* seg_runs;    // [entries with segments] (entry, first segment, segments, 0)
  float* seg_state;        // [n, heads, N, Pp], or null: one segment per entry, straight from the slot
  float* seg_decay;        // [n, heads]
};

__device__ __forceinline__ float ssd_dt(float raw, float bias) {
  const float x = raw + bias;
  return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
}

inline int fill_ssd(Ssd& p, const void* u, int ldu, int boff, int coff, const void* dt, int lddt,
                    const float* dt_bias, const float* A_log, const float* D, float* state, void* y,
                    int ldy, int heads, int groups, int N, int P, int Pp, const int* slot, const int* row0,
                    const int* len, const int* pos0, const int* entry) {
  if (heads < 1 || groups < 1 || heads % groups || N < 1 || N > 256 || P < 1 || Pp < P || Pp % 4) return -1;
  p.u = u; p.ldu = ldu; p.boff = boff; p.coff = coff; p.dt = dt; p.lddt = lddt; p.dt_bias = dt_bias;
  p.A_log = A_log; p.D = D; p.state = state; p.y = y; p.ldy = ldy; p.heads = heads; p.groups = groups;
  p.N = N; p.P = P; p.Pp = Pp; p.e.slot = slot; p.e.row0 = row0; p.e.len = len; p.e.pos0 = pos0;
  p.entry = entry; p.segs = p.seg_runs = nullptr; p.seg_state = p.seg_decay = nullptr;
  return 0;
}

}  // namespace cb
