// Helpers shared by the sequence-mixer kernel files: element conversion, the per-token row of the step table,
// 1- or 4-element vector loads / stores of float32 and bfloat16 rows, asynchronous copies, ring rows and activations.
#pragma once
#include "common.cuh"

namespace qspec {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

struct TokMeta {
  int slot, pos, seg_begin, seg_end, phase;
};
__device__ __forceinline__ TokMeta load_meta(const int* meta, int ntok, int i) {
  TokMeta m;
  m.slot = meta[i];
  m.pos = meta[ntok + i];
  m.seg_begin = meta[2 * ntok + i];
  m.seg_end = meta[3 * ntok + i];
  m.phase = meta[4 * ntok + i];
  return m;
}

template <int VEC> struct VecF { float v[VEC]; };
template <int VEC> __device__ __forceinline__ VecF<VEC> ldv(const float* p) {
  VecF<VEC> r;
  if (VEC == 4) { const float4 t = *reinterpret_cast<const float4*>(p); r.v[0] = t.x; r.v[1 % VEC] = t.y; r.v[2 % VEC] = t.z; r.v[3 % VEC] = t.w; }
  else r.v[0] = *p;
  return r;
}
template <int VEC> __device__ __forceinline__ VecF<VEC> ldv(const __nv_bfloat16* p) {
  VecF<VEC> r;
  if (VEC == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    r.v[0] = a.x; r.v[1 % VEC] = a.y; r.v[2 % VEC] = b.x; r.v[3 % VEC] = b.y;
  } else r.v[0] = __bfloat162float(*p);
  return r;
}
template <int VEC> __device__ __forceinline__ void stv(float* p, const VecF<VEC>& r) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
  else *p = r.v[0];
}
template <int VEC> __device__ __forceinline__ void stv(__nv_bfloat16* p, const VecF<VEC>& r) {
  if (VEC == 4) {
    uint2 t;
    *reinterpret_cast<__nv_bfloat162*>(&t.x) = __floats2bfloat162_rn(r.v[0], r.v[1 % VEC]);
    *reinterpret_cast<__nv_bfloat162*>(&t.y) = __floats2bfloat162_rn(r.v[2 % VEC], r.v[3 % VEC]);
    *reinterpret_cast<uint2*>(p) = t;
  } else *p = __float2bfloat16_rn(r.v[0]);
}


// Row of a position in a per-slot ring of `cap` rows whose first `keep` rows are never reused: positions below `keep` stay where
// they are, the others go round the remaining rows. keep = 0: position % cap.
__device__ __forceinline__ int ring_row(int pos, int keep, int cap) { return pos < cap ? pos : keep + (pos - keep) % (cap - keep); }

// 4-byte asynchronous copies into shared memory (both addresses on 4-byte boundaries)
__device__ __forceinline__ void cp_async_4(float* smem_dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// 16-byte asynchronous copy into shared memory; `valid` false writes zeros and reads nothing
__device__ __forceinline__ void cp_async_16z(void* smem_dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(src),
               "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

}  // namespace qspec
