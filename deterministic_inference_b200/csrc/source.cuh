// A kernel input that is either a stored matrix (float32 or bfloat16) or the float32
// partial products of a matrix product whose k was split ([splits][n], `stride` elements
// apart), which the reader adds in split order while it loads.  kind: 0 float32 (one or
// several splits), 1 bfloat16.
#pragma once

#include "common.cuh"

struct Source {
  const void* p;
  int kind;
  int splits;
  long long stride;
};

static inline Source make_source(const void* p, int kind, int splits, long long stride) {
  Source s;
  s.p = p;
  s.kind = kind;
  s.splits = splits < 1 ? 1 : splits;
  s.stride = stride;
  return s;
}

__device__ __forceinline__ float source_load(const Source& s, long long i) {
  if (s.kind == 1) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(s.p)[i]);
  const float* f = reinterpret_cast<const float*>(s.p);
  float v = f[i];
  for (int k = 1; k < s.splits; ++k) v = __fadd_rn(v, f[(long long)k * s.stride + i]);
  return v;
}

// The elements base + t, base + t + step, ... (N of them, those at or beyond base + width are 0) of a
// source, the loads of AHEAD splits issued before the first is used; the splits are added in order (AHEAD 0:
// the source is not split).
template <int N, int AHEAD>
__device__ __forceinline__ void source_load_strided(const Source& s, long long base, int t, int step, int width,
                                                    float (&v)[N]) {
  if (s.kind == 1) {
    const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(s.p) + base;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = t + i * step < width ? __bfloat162float(p[t + i * step]) : 0.f;
    return;
  }
  const float* f = reinterpret_cast<const float*>(s.p) + base;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = t + i * step < width ? f[t + i * step] : 0.f;
  if (AHEAD == 0) return;
  constexpr int U = AHEAD > 0 ? AHEAD : 1;
  int k = 1;
  for (; k + U <= s.splits; k += U) {
    float a[U][N];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int i = 0; i < N; ++i) a[u][i] = t + i * step < width ? f[(long long)(k + u) * s.stride + t + i * step] : 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int i = 0; i < N; ++i) v[i] = __fadd_rn(v[i], a[u][i]);
  }
  for (; k < s.splits; ++k) {
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (t + i * step < width) v[i] = __fadd_rn(v[i], f[(long long)k * s.stride + t + i * step]);
  }
}

// Store a float32 value as the dtype code says (0 float32, 1 bfloat16).
__device__ __forceinline__ void store_as(void* p, int dtype, long long i, float v) {
  if (dtype == 1) reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v);
  else reinterpret_cast<float*>(p)[i] = v;
}
__device__ __forceinline__ float load_as(const void* p, int dtype, long long i) {
  if (dtype == 1) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
  return reinterpret_cast<const float*>(p)[i];
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
