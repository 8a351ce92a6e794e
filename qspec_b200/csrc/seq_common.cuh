// Helpers shared by the sequence-mixer kernel files: element conversion, the per-token row of the step table,
// 1- or 4-element vector loads / stores of float32 and bfloat16 rows, asynchronous copies, tensor-core fragments, ring rows and activations.
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
// tensor-core fragments: 8 x 8 matrices of bfloat16 from shared memory (as stored, transposed), products with float32 accumulators
__device__ __forceinline__ void tk_ldmatrix_x4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void tk_ldmatrix_x4_trans(uint32_t (&r)[4], const __nv_bfloat16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
// (hi, lo) split of two float32 weights: hi = bf16(w), lo = bf16(w - hi); hi + lo carries 16 mantissa bits
__device__ __forceinline__ void tk_split_bf2(float w0, float w1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat16 h0 = __float2bfloat16_rn(w0), h1 = __float2bfloat16_rn(w1);
  __nv_bfloat162 hv, lv;
  hv.x = h0; hv.y = h1;
  lv = __floats2bfloat162_rn(w0 - __bfloat162float(h0), w1 - __bfloat162float(h1));
  hi = *reinterpret_cast<uint32_t*>(&hv);
  lo = *reinterpret_cast<uint32_t*>(&lv);
}
__device__ __forceinline__ void tk_mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// silu of a convolution's result: in bfloat16 mode (the inputs are bfloat16 roundings, relative 4e-3) the exponential and the
// division run on the special-function unit
template <typename T> __device__ __forceinline__ float silu_act(float z) { return silu_f(z); }
template <> __device__ __forceinline__ float silu_act<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ---- inputs of a short causal convolution -------------------------------------------------------------------------------------
// The input of channel c at position sp: a row of the step, a row of the slot's tail (the last K1 inputs before the step), or zero
// before the sequence's start.
template <typename T> struct ConvRows {
  const T* in;            // channel 0 of batch row seg_begin
  int ld, first_pos, K1, C;
  const float* told;      // [K1][C] of the slot, as it was before the step
  __device__ __forceinline__ float get(int sp, int c) const {
    if (sp >= first_pos) return to_f(in[(size_t)(sp - first_pos) * ld + c]);
    return sp >= 0 ? told[(size_t)(sp - first_pos + K1) * C + c] : 0.f;
  }
  // the slot's new tail for channel c once the segment's last position is `last`
  __device__ __forceinline__ void write_tail(float* tnew, int last, int c) const {
    for (int r = 0; r < K1; ++r) tnew[(size_t)r * C + c] = get(last + 1 - K1 + r, c);
  }
};

}  // namespace qspec
