// A sublayer's output that nobody has added up yet: a weighted sum of terms, each a 32-bit tensor or the K slices that a
// contraction over few tokens left unadded, and the packed accesses of the kernels that read one.
#pragma once
#include "common.cuh"

#define CUCA_MAX_TERMS 8
struct CucaTerms {  // (passed from Python by address: keep in step with kernels/ops.py)
  int n;
  const float* data[CUCA_MAX_TERMS];
  int slices[CUCA_MAX_TERMS];
  size_t stride[CUCA_MAX_TERMS];  // between slices, in values
  float scale[CUCA_MAX_TERMS];
};

namespace {

template <int V> struct Pack;
template <> struct Pack<1> { float v[1]; };
template <> struct alignas(16) Pack<4> { float v[4]; };
template <int V> __device__ __forceinline__ Pack<V> ld(const float* p) { return *reinterpret_cast<const Pack<V>*>(p); }
template <int V> __device__ __forceinline__ void st(float* p, const Pack<V>& x) { *reinterpret_cast<Pack<V>*>(p) = x; }
template <int V> __device__ __forceinline__ void st(__nv_bfloat16* p, const Pack<V>& x) {
  if (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(x.v[0], x.v[V > 1 ? 1 : 0]);
    const __nv_bfloat162 hi = __floats2bfloat162_rn(x.v[V > 2 ? 2 : 0], x.v[V > 3 ? 3 : 0]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
    p[0] = __float2bfloat16_rn(x.v[0]);
  }
}
// (slices come from the kernel before this one: past L1, which a dependent launch does not find invalidated)
template <int V> __device__ __forceinline__ Pack<V> ld_cg(const float* p) {
  Pack<V> r;
  if (V == 4) {
    const float4 f = __ldcg(reinterpret_cast<const float4*>(p));
    r.v[0] = f.x;
    if (V > 1) r.v[V > 1 ? 1 : 0] = f.y;
    if (V > 2) r.v[V > 2 ? 2 : 0] = f.z;
    if (V > 3) r.v[V > 3 ? 3 : 0] = f.w;
  } else {
    r.v[0] = __ldcg(p);
  }
  return r;
}

// y[at .. at + V) of the weighted sum of the terms
// (AHEAD slices' loads in flight at once, added in slice order)
template <int V, int AHEAD = 4>
__device__ __forceinline__ Pack<V> term_sum(const CucaTerms& t, size_t at) {
  Pack<V> y;
#pragma unroll
  for (int k = 0; k < V; ++k) y.v[k] = 0.f;
  for (int i = 0; i < t.n; ++i) {
    const float* p = t.data[i] + at;
    Pack<V> s;
#pragma unroll
    for (int k = 0; k < V; ++k) s.v[k] = 0.f;
    for (int k0 = 0; k0 < t.slices[i]; k0 += AHEAD) {
      Pack<V> q[AHEAD];
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        if (k0 + u < t.slices[i]) q[u] = ld_cg<V>(p + (k0 + u) * t.stride[i]);
        else {
#pragma unroll
          for (int k = 0; k < V; ++k) q[u].v[k] = 0.f;
        }
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u)
#pragma unroll
        for (int k = 0; k < V; ++k) s.v[k] += q[u].v[k];
    }
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = fmaf(t.scale[i], s.v[k], y.v[k]);
  }
  return y;
}

inline bool aligned_to(const void* p, size_t a) { return ((uintptr_t)p & (a - 1)) == 0; }

inline bool terms_wide(const CucaTerms& t) {
  for (int i = 0; i < t.n; ++i)
    if (!aligned_to(t.data[i], 16) || t.stride[i] % 4 != 0) return false;
  return true;
}

}  // namespace
