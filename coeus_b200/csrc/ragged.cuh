// Shared pieces of the kernels that run a ragged batch: every step brings a number of sequences
// ("entries"), each with its own count of new tokens, laid out one after the other in the rows
// of the activations.  Activations are bf16 or fp32 (template parameter); arithmetic is fp32.
#pragma once
#include "common.cuh"
#include "ptx.cuh"

namespace cb {

int sm_count();

// The entries of one step.  Entry e owns rows row0[e] .. row0[e] + len[e] - 1, its first row is
// the token at position pos0[e] of its sequence, and its cache pages and recurrent state are
// those of slot[e].  A sequence whose pos0 is 0 starts from an empty state whatever its slot
// holds, so slots need no clearing between requests.
struct Entries {
  const int* slot;
  const int* row0;
  const int* len;
  const int* pos0;
};

constexpr int RAGGED_PAGE = 64;   // tokens per cache page

template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// V (1, 4 or 8) consecutive values, aligned to the vector (fp32: to 16 bytes).
template <int V>
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float* f) {
  if constexpr (V == 8) {
    load8(p, f);
  } else if constexpr (V == 4) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(x.x), b = unpack_bf16x2(x.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else f[0] = __bfloat162float(*p);
}
template <int V>
__device__ __forceinline__ void load_vec(const float* p, float* f) {
  if constexpr (V == 8) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  } else if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    f[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float* f) {
  if constexpr (V == 8) store8(p, f);
  else if constexpr (V == 4)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  else *p = __float2bfloat16(f[0]);
}
template <int V>
__device__ __forceinline__ void store_vec(float* p, const float* f) {
  if constexpr (V == 8) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    *p = f[0];
  }
}

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
// copies `bytes` (0 or 16) and zero-fills the rest of the 16 bytes
__device__ __forceinline__ void cp_async16_zfill(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Warp-level tiles: four 8 x 8 matrices from shared memory (plain, transposed), and m16n8k16.
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, "
               "{%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

}  // namespace cb
