// What the chunked forms of the linear recurrences share (retention, gated linear attention): a prompt
// portion cut into chunks of CH tokens, the place of a chunk in memory, float32 operands as pairs of
// bfloat16 numbers.
#pragma once

#include "sigmoid_attention_mma.cuh"      // ldmatrix / mma.sync / cp.async helpers

namespace chunks {

using sa_mma::pack_bf16;

constexpr int CH = 64;                    // tokens of a chunk
constexpr int PAD = 8;                    // bfloat16 elements of padding per shared-memory row
constexpr int MOST_SMEM = 224 * 1024;

// Chunk c of sequence b (of the B whose boundaries `cu` gives) has the place (cu[b] - cu[0]) / CH + b + c:
// no two chunks share one, and no list is needed.  Returns false for a place without a chunk.
__device__ __forceinline__ int first_place(const int* cu, int b) { return (cu[b] - cu[0]) / CH + b; }
__device__ __forceinline__ bool chunk_at(const int* cu, int B, int place, int& b, int& first, int& count) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {             // the last sequence whose first place is not behind this one
    const int mid = (lo + hi + 1) >> 1;
    if (first_place(cu, mid) <= place) lo = mid;
    else hi = mid - 1;
  }
  b = lo;
  const int len = cu[b + 1] - cu[b];
  first = (place - first_place(cu, b)) * CH;
  count = len - first < CH ? len - first : CH;
  return count > 0;
}

// two float32 values as bfloat16 pairs hi + lo (the value up to 2^-17 of it)
__device__ __forceinline__ void split2(float x, float y, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const unsigned*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack_bf16(__fsub_rn(x, f.x), __fsub_rn(y, f.y));
}
__device__ __forceinline__ float2 join2(unsigned hi, unsigned lo) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&lo));
  return make_float2(__fadd_rn(a.x, b.x), __fadd_rn(a.y, b.y));
}

// A token-by-token kernel's columns of a state row: four a thread where the row's length allows it.
template <int VEC> struct Cols;
template <> struct Cols<4> { using T = float4; };
template <> struct Cols<1> { using T = float; };
// s <- d s + k v; o <- o + s q
__device__ __forceinline__ void col_step(float4& s, float4& o, float d, float k, float q, const float4& v) {
  s.x = __fmaf_rn(k, v.x, __fmul_rn(d, s.x)); o.x = __fmaf_rn(s.x, q, o.x);
  s.y = __fmaf_rn(k, v.y, __fmul_rn(d, s.y)); o.y = __fmaf_rn(s.y, q, o.y);
  s.z = __fmaf_rn(k, v.z, __fmul_rn(d, s.z)); o.z = __fmaf_rn(s.z, q, o.z);
  s.w = __fmaf_rn(k, v.w, __fmul_rn(d, s.w)); o.w = __fmaf_rn(s.w, q, o.w);
}
__device__ __forceinline__ void col_step(float& s, float& o, float d, float k, float q, const float& v) {
  s = __fmaf_rn(k, v, __fmul_rn(d, s));
  o = __fmaf_rn(s, q, o);
}

}  // namespace chunks
