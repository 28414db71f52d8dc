// The minGRU recurrence over a ragged batch, element by element in fp32:
//   z = sigmoid(zl);  c = u >= 0 ? u + 1/2 : sigmoid(u);  S <- (1 - z) S + z c;  out = S silu(g)
// with zl, u and g the projections.  A step is S <- a S + b, which composes: (a1, b1) then (a2, b2)
// is (a1 a2, a2 b1 + b2).  A block owns 32 channels of one entry and goes through its tokens 64 at
// a time: 16 threads side by side hold two channels each, 16 groups of them take four tokens each,
// compose them, and learn the state in front of their tokens from the groups before them.
#include "ragged.cuh"

namespace cb {

constexpr int MG_CH = 32, MG_SEG = 16, MG_TOK = 4, MG_BLOCK = MG_SEG * MG_TOK;

struct MinGru {
  const void* raw;        // [rows, ld]: zl at zoff, u at uoff, g at goff
  int ld, zoff, uoff, goff;
  float* state;           // [slots, width]
  void* out;              // [rows, ldo]
  int ldo, width;         // width: even
  Entries e;
};

// two neighbouring numbers as they are stored, and as fp32
template <typename T> struct Pair;
template <> struct Pair<__nv_bfloat16> { using type = uint32_t; };
template <> struct Pair<float> { using type = float2; };
template <typename T>
__device__ __forceinline__ typename Pair<T>::type load_pair(const T* p) {
  return *reinterpret_cast<const typename Pair<T>::type*>(p);
}
__device__ __forceinline__ float2 pair_f32(uint32_t v) { return unpack_bf16x2(v); }
__device__ __forceinline__ float2 pair_f32(float2 v) { return v; }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b);
}
__device__ __forceinline__ void store_pair(float* p, float a, float b) {
  *reinterpret_cast<float2*>(p) = make_float2(a, b);
}
// a and b of one step, and silu(g).  With e_v = exp(-|v|), every sigmoid here is 1 / (1 + e_v) or
// e_v / (1 + e_v), so one reciprocal of the product of the three denominators (in 1..8) serves all.
// bf16 projections take the fast exponential and reciprocal (a few units in the last place of fp32).
template <typename T>
__device__ __forceinline__ void mg_step(float zl, float u, float g, float& a, float& b, float& act) {
  float ez, eu, eg;
  if constexpr (sizeof(T) == 2) {
    constexpr float L2E = -1.4426950408889634f;
    ez = fast_exp2(fabsf(zl) * L2E); eu = fast_exp2(fabsf(u) * L2E); eg = fast_exp2(fabsf(g) * L2E);
  } else {
    ez = expf(-fabsf(zl)); eu = expf(-fabsf(u)); eg = expf(-fabsf(g));
  }
  const float pz = 1.f + ez, pu = 1.f + eu, pg = 1.f + eg, zu = pz * pu;
  float r;
  if constexpr (sizeof(T) == 2) asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(zu * pg));
  else r = 1.0f / (zu * pg);
  const float rz = pu * pg * r;                          // 1 / (1 + ez)
  const float z = zl >= 0.f ? rz : ez * rz;
  a = zl >= 0.f ? ez * rz : rz;                          // 1 - z without cancellation
  b = z * (u >= 0.f ? u + 0.5f : eu * (pz * pg * r));
  act = (g >= 0.f ? g : g * eg) * (zu * r);
}

template <typename T>
__global__ void __launch_bounds__(MG_CH / 2 * MG_SEG, 4) mingru_kernel(const MinGru p) {
  __shared__ float2 sa[MG_SEG / 2][MG_CH / 2], sb[MG_SEG / 2][MG_CH / 2];    // of two groups together
  __shared__ float2 carry[2][MG_CH / 2];
  const int e = blockIdx.y, row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e];
  const int cp = threadIdx.x % (MG_CH / 2), seg = threadIdx.x / (MG_CH / 2);
  const int ch = blockIdx.x * MG_CH + cp * 2;
  const bool in = ch < p.width;
  float* st = p.state + static_cast<size_t>(slot) * p.width + ch;
  const T* raw = static_cast<const T*>(p.raw) + (static_cast<size_t>(row0) + seg * MG_TOK) * p.ld + (in ? ch : 0);
  T* out = static_cast<T*>(p.out) + (static_cast<size_t>(row0) + seg * MG_TOK) * p.ldo + ch;
  const ptrdiff_t ahead = static_cast<ptrdiff_t>(MG_BLOCK) * p.ld, out_ahead = static_cast<ptrdiff_t>(MG_BLOCK) * p.ldo;
  if (seg == 0)
    carry[0][cp] = in && p.e.pos0[e] > 0 ? *reinterpret_cast<const float2*>(st) : make_float2(0.f, 0.f);
  typename Pair<T>::type z[MG_TOK], u[MG_TOK], g[MG_TOK];
  auto fetch = [&](int n) {
    const T* r = raw;
#pragma unroll
    for (int i = 0; i < MG_TOK; ++i, r += p.ld) {
      if (i >= n) continue;
      z[i] = load_pair(r + p.zoff);
      u[i] = load_pair(r + p.uoff);
      g[i] = load_pair(r + p.goff);
    }
  };
  fetch(len - seg * MG_TOK);
  int turn = 0;
  for (int t0 = 0; t0 < len; t0 += MG_BLOCK, turn ^= 1) {
    const int n = len - t0 - seg * MG_TOK;               // of these four; may be <= 0
    float2 a[MG_TOK], b[MG_TOK], act[MG_TOK], ta = make_float2(1.f, 1.f), tb = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < MG_TOK; ++i) {
      a[i] = make_float2(1.f, 1.f);
      b[i] = act[i] = make_float2(0.f, 0.f);
      if (i < n) {
        const float2 fz = pair_f32(z[i]), fu = pair_f32(u[i]), fg = pair_f32(g[i]);
        mg_step<T>(fz.x, fu.x, fg.x, a[i].x, b[i].x, act[i].x);
        mg_step<T>(fz.y, fu.y, fg.y, a[i].y, b[i].y, act[i].y);
      }
      tb = make_float2(a[i].x * tb.x + b[i].x, a[i].y * tb.y + b[i].y);
      ta = make_float2(ta.x * a[i].x, ta.y * a[i].y);
    }
    raw += ahead;
    fetch(n - MG_BLOCK);
    // the even group of the warp's two, seen from the odd one
    const float2 ea = make_float2(__shfl_xor_sync(0xffffffffu, ta.x, 16), __shfl_xor_sync(0xffffffffu, ta.y, 16));
    const float2 eb = make_float2(__shfl_xor_sync(0xffffffffu, tb.x, 16), __shfl_xor_sync(0xffffffffu, tb.y, 16));
    const bool odd = seg & 1;
    if (odd) {
      sa[seg / 2][cp] = make_float2(ta.x * ea.x, ta.y * ea.y);
      sb[seg / 2][cp] = make_float2(ta.x * eb.x + tb.x, ta.y * eb.y + tb.y);
    }
    __syncthreads();
    float2 s = carry[turn][cp];
    for (int k = 0; k < seg / 2; ++k) {
      const float2 ka = sa[k][cp], kb = sb[k][cp];
      s = make_float2(ka.x * s.x + kb.x, ka.y * s.y + kb.y);
    }
    if (odd) s = make_float2(ea.x * s.x + eb.x, ea.y * s.y + eb.y);
    T* o = out;
#pragma unroll
    for (int i = 0; i < MG_TOK; ++i, o += p.ldo) {
      s = make_float2(a[i].x * s.x + b[i].x, a[i].y * s.y + b[i].y);
      if (i < n && in) store_pair(o, s.x * act[i].x, s.y * act[i].y);
    }
    out += out_ahead;
    if (seg == MG_SEG - 1) carry[turn ^ 1][cp] = s;      // identity steps behind the entry's end
    __syncthreads();
  }
  if (seg == 0 && in) *reinterpret_cast<float2*>(st) = carry[turn][cp];
}

// Entries of a few tokens: a thread per channel pair.
template <typename T>
__global__ void __launch_bounds__(128) mingru_short_kernel(const MinGru p) {
  const int e = blockIdx.y, row0 = p.e.row0[e], len = p.e.len[e], slot = p.e.slot[e];
  const int ch = (blockIdx.x * 128 + threadIdx.x) * 2;
  if (ch >= p.width) return;
  float2* st = reinterpret_cast<float2*>(p.state + static_cast<size_t>(slot) * p.width + ch);
  float2 s = p.e.pos0[e] > 0 ? *st : make_float2(0.f, 0.f);
  for (int t = 0; t < len; ++t) {
    const T* r = static_cast<const T*>(p.raw) + static_cast<size_t>(row0 + t) * p.ld + ch;
    const float2 z = pair_f32(load_pair(r + p.zoff)), u = pair_f32(load_pair(r + p.uoff)),
                 g = pair_f32(load_pair(r + p.goff));
    float2 a, b, act;
    mg_step<T>(z.x, u.x, g.x, a.x, b.x, act.x);
    mg_step<T>(z.y, u.y, g.y, a.y, b.y, act.y);
    s = make_float2(a.x * s.x + b.x, a.y * s.y + b.y);
    store_pair(static_cast<T*>(p.out) + static_cast<size_t>(row0 + t) * p.ldo + ch, s.x * act.x,
               s.y * act.y);
  }
  *st = s;
}

template <typename T>
static int launch_mingru(const MinGru& p, int entries, int longest, cudaStream_t st) {
  if (longest <= MG_TOK)
    mingru_short_kernel<T><<<dim3((p.width + 255) / 256, entries), 128, 0, st>>>(p);
  else
    mingru_kernel<T><<<dim3((p.width + MG_CH - 1) / MG_CH, entries), MG_CH / 2 * MG_SEG, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cb

using namespace cb;

extern "C" int cb_mingru(const void* raw, int ld, int zoff, int uoff, int goff, float* state, void* out,
                         int ldo, int width, const int* slot, const int* row0, const int* len,
                         const int* pos0, int entries, int longest, int f32, void* stream) {
  if (entries <= 0 || entries > 65535 || width <= 0 || width % 2) return -1;
  if (ld % 2 || zoff % 2 || uoff % 2 || goff % 2 || ldo % 2) return -2;
  MinGru p;
  p.raw = raw; p.ld = ld; p.zoff = zoff; p.uoff = uoff; p.goff = goff; p.state = state; p.out = out;
  p.ldo = ldo; p.width = width;
  p.e.slot = slot; p.e.row0 = row0; p.e.len = len; p.e.pos0 = pos0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_mingru<float>(p, entries, longest, st)
             : launch_mingru<__nv_bfloat16>(p, entries, longest, st);
}
