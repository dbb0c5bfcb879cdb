// Element and vector access of the layer-stack kernels: bf16 or fp32 storage, fp32 registers; rows that are either
// finished values or split-K partial sums.
#pragma once
#include "common.cuh"
#include "stack.h"

namespace cb {

template <typename T> struct Elem;
template <> struct Elem<float> {
  static __device__ __forceinline__ float get(const float* p) { return *p; }
  static __device__ __forceinline__ void put(float* p, float v) { *p = v; }
};
template <> struct Elem<bf16> {
  static __device__ __forceinline__ float get(const bf16* p) { return __bfloat162float(*p); }
  static __device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
};
template <typename T, int VEC> struct Vec {
  static __device__ __forceinline__ void load(const T* p, float (&v)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = Elem<T>::get(p + e);
  }
  static __device__ __forceinline__ void store(T* p, const float (&v)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) Elem<T>::put(p + e, v[e]);
  }
};
template <> struct Vec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct Vec<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16lo(x.x); v[1] = bf16hi(x.x); v[2] = bf16lo(x.y); v[3] = bf16hi(x.y);
  }
  static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
    uint2 o;
    o.x = pack_bf16(v[0], v[1]); o.y = pack_bf16(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = o;
  }
};

template <> struct Vec<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[8]) {
    const float4 x = reinterpret_cast<const float4*>(p)[0], y = reinterpret_cast<const float4*>(p)[1];
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  }
};
template <> struct Vec<bf16, 8> {
  static __device__ __forceinline__ void load(const bf16* p, float (&v)[8]) {
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    v[0] = bf16lo(x.x); v[1] = bf16hi(x.x); v[2] = bf16lo(x.y); v[3] = bf16hi(x.y);
    v[4] = bf16lo(x.z); v[5] = bf16hi(x.z); v[6] = bf16lo(x.w); v[7] = bf16hi(x.w);
  }
  static __device__ __forceinline__ void store(bf16* p, const float (&v)[8]) {
    uint4 o;
    o.x = pack_bf16(v[0], v[1]); o.y = pack_bf16(v[2], v[3]); o.z = pack_bf16(v[4], v[5]); o.w = pack_bf16(v[6], v[7]);
    *reinterpret_cast<uint4*>(p) = o;
  }
};

// Values still in their storage form: a load whose conversion comes later does not hold up the loads behind it.
template <typename T, int VEC> struct Raw;
template <> struct Raw<bf16, 4> {
  uint2 v;
  __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void get(float (&o)[4]) const { o[0] = bf16lo(v.x); o[1] = bf16hi(v.x); o[2] = bf16lo(v.y); o[3] = bf16hi(v.y); }
};
template <> struct Raw<float, 4> {
  float4 v;
  __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&o)[4]) const { o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w; }
};
template <> struct Raw<bf16, 8> {
  uint4 v;
  __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&o)[8]) const {
    o[0] = bf16lo(v.x); o[1] = bf16hi(v.x); o[2] = bf16lo(v.y); o[3] = bf16hi(v.y);
    o[4] = bf16lo(v.z); o[5] = bf16hi(v.z); o[6] = bf16lo(v.w); o[7] = bf16hi(v.w);
  }
};
template <> struct Raw<float, 8> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
  __device__ __forceinline__ void get(float (&o)[8]) const {
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
  }
};

__device__ __forceinline__ float warp_add(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float fast_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float silu_f32(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.f / (1.f + expf(-z)); }

// VEC consecutive values of a RowSource (stack.h): the row itself, or the sum of its split-K parts.
// PART false: known to be finished values.
template <typename T, int VEC, bool PART = true>
__device__ __forceinline__ void load_source(const cosmos::RowSource& s, long long row, int col, float (&v)[VEC]) {
  if (!PART || s.k_splits == 0) {
    Vec<T, VEC>::load(reinterpret_cast<const T*>(s.p) + row * s.ld + col, v);
    return;
  }
  const float* p = reinterpret_cast<const float*>(s.p) + row * s.ld + col;
  Vec<float, VEC>::load(p, v);
  for (int k = 1; k < s.k_splits; ++k) {
    float t[VEC];
    Vec<float, VEC>::load(p + k * s.split_stride, t);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] += t[e];
  }
}
template <typename T>
__device__ __forceinline__ float load_source1(const cosmos::RowSource& s, long long row, int col) {
  float v[1];
  load_source<T, 1>(s, row, col, v);
  return v[0];
}

// Which tokens a CTA works on: entry `i` of a step's portions, or the one new token of decode slot i.
struct Portion {
  int seq, row0, rows, pos0;
};
__device__ __forceinline__ Portion get_portion(const cosmos::StepRows& s, int i) {
  if (s.portions) {
    const int4 t = reinterpret_cast<const int4*>(s.portions)[i];
    return {t.x, t.y, t.z, t.w};
  }
  return {i, i, 1, s.lens[i] - 1};
}
// State slot of a sequence; negative = none (a bad slot is reported and skipped).
__device__ __forceinline__ long long get_state_slot(const cosmos::StepRows& s, int seq, int* status) {
  const int slot = s.state_slots[seq];
  return index_ok(slot, s.n_state_slots, status, SITE_STATE_SLOT) ? slot : -1;
}

// Sum of two values over the CTA (every thread gets both).
__device__ __forceinline__ float2 block_add2(float a, float b, float2* buf) {
  a = warp_add(a);
  b = warp_add(b);
  const int warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) buf[warp] = make_float2(a, b);
  __syncthreads();
  float2 r = make_float2(0.f, 0.f);
  for (int w = 0; w < warps; ++w) {
    r.x += buf[w].x;
    r.y += buf[w].y;
  }
  return r;
}

}  // namespace cb
