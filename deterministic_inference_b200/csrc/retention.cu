// Retention: a matrix state per head that shrinks by one constant a token, read without a softmax.
//
// proj row (row_width elements): [q: H N | k: H N | v: H P | g: H P].  The first `rot` elements of
// every q and k head turn in halves (element i with i + rot/2, angle = position * freq[i]); k is
// multiplied by N^(-1/2) behind the rotation.  Per head h, with a state S [N][P] from zero:
//     S <- decay[h] S + k v^T;     o = S^T q;     out = o / sqrt(mean(o^2) + eps) * silu(g).
// A request's state slot holds the heads' states [H][N][P], float32; slot 0 is no request's: a
// sequence on it starts from zeros and stores nothing.
//
// Two forms.
//
// retention_step_kernel: a block per (sequence, head) walks the sequence's tokens one by one:
// rotation, state, read-out, norm and gate in one kernel, everything float32.  It serves decoded
// tokens (the state is read and written once, which is all the memory they move), and prompt
// portions of the float32 engine and of sizes the other form does not take.
//
// The chunked form for prompt portions of the bfloat16 engine (N and P multiples of 16, up to 256).
// A portion is cut into chunks of 64 tokens; with d = decay, i and j counting a chunk's tokens from 0,
// c its number of tokens and S the state in front of it,
//     o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j,
//     S  <- d^c S + sum_j d^(c-1-j) k_j v_j^T,
// so all chunks' sums over their own tokens are products that run side by side, and only the states
// are chained:
//   retention_rotate_kernel   q and k rotated, as bfloat16 pairs (hi, lo) with hi + lo the float32
//                             value up to 2^-17 of it
//   retention_chunk_kernel    sum_j d^(c-1-j) k_j v_j^T of every chunk
//   retention_chain_kernel    the states in front of the chunks, as (hi, lo) pairs, and the slot's
//   retention_output_kernel   o, its norm and the gate
// The products run on the tensor cores (mma.sync m16n8k16, bfloat16 operands, float32 accumulators)
// with every float32 operand as its (hi, lo) pair (hi hi + hi lo + lo hi; v is a bfloat16 projection,
// one term), so nothing that enters the recurrence is rounded below 2^-16; decays are applied to
// float32 values.
#include "linear_chunks.cuh"

namespace {

using sa_mma::copy16;
using sa_mma::ldsm_x4;
using sa_mma::ldsm_x4_trans;
using sa_mma::mma_bf16;
using sa_mma::pack_bf16;
using namespace chunks;

// one element of a q or k head behind the rotation; `get(d)` gives the head's projected elements
template <typename Get>
__device__ __forceinline__ float turned(Get get, int d, int rot, float pos, const float* __restrict__ freq) {
  const float v = get(d);
  if (d >= rot) return v;
  const int half = rot >> 1;
  const bool first = d < half;
  const float a = __fmul_rn(pos, freq[first ? d : d - half]);
  const float c = cosf(a), s = sinf(a), o = get(first ? d + half : d - half);
  return first ? __fmaf_rn(v, c, -__fmul_rn(o, s)) : __fmaf_rn(v, c, __fmul_rn(o, s));
}

// ---- token by token --------------------------------------------------------------------------------
// VEC columns a thread (4 where P is a multiple of 4).  Thread (rg, cg) has the rows rg, rg + RG, ...
// of column group cg; a column's read-out adds a thread's rows in ascending order and then the RG
// shares in order: the order depends on N and P alone.  in_smem: the state lives in shared memory
// while the sequence's tokens are walked (else in the slot; a sequence on slot 0 then forgets
// each token).
constexpr int ST = 256;

template <int VEC>
__global__ void __launch_bounds__(ST)
retention_step_kernel(Source proj, long long row_width, const float* __restrict__ decay, const float* __restrict__ freq,
                      int rot, const int* __restrict__ positions, float* state, long long slot_stride,
                      const int* __restrict__ cu_q_lens, const int* __restrict__ state_slots, void* out, int out_dtype,
                      int H, int N, int P, float k_scale, float eps, int in_smem) {
  using V = typename Cols<VEC>::T;
  extern __shared__ __align__(16) float rs_smem[];   // q [N], k [N], v [P], o [P], shares [RG][P], state [N][P] (in_smem)
  __shared__ float scratch[32];
  pdl_prologue(proj.p, state);
  const int b = blockIdx.x, h = blockIdx.y;
  const int t0 = cu_q_lens[b], n_tok = cu_q_lens[b + 1] - t0;
  if (n_tok <= 0) return;
  const long long slot = state_slots[b];
  const int np = (N + 3) / 4 * 4, pp = (P + 3) / 4 * 4;
  float* qs = rs_smem;
  float* ks = qs + np;
  float* vs = ks + np;
  float* os = vs + pp;
  float* part = os + pp;
  const int cols = P / VEC;
  const int CG = cols < ST ? cols : ST, RG = ST / CG;
  const int cg = threadIdx.x % CG, rg = threadIdx.x / CG;
  float* sm_state = part + RG * pp;
  float* srow = state + slot * slot_stride + (long long)h * N * P;
  const float d = decay[h];
  const bool bf = out_dtype == 1;
  const long long qc = (long long)h * N, kc = (long long)(H + h) * N, vc = 2ll * H * N + (long long)h * P,
                  gc = vc + (long long)H * P;
  auto load = [&](long long at) {
    const float x = source_load(proj, at);
    return bf ? round_to<__nv_bfloat16>(x) : x;
  };
  if (in_smem) {
    for (int i = threadIdx.x; i < N * P; i += ST) sm_state[i] = slot != 0 ? srow[i] : 0.f;
    __syncthreads();
  }
  V* S = reinterpret_cast<V*>(in_smem ? sm_state : srow);
  const bool keeps = in_smem || slot != 0;
  for (int k = 0; k < n_tok; ++k) {
    const int t = t0 + k;
    const long long row = (long long)t * row_width;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < 2 * N; i += ST) {
      const bool is_k = i >= N;
      const int e = is_k ? i - N : i;
      const long long at = row + (is_k ? kc : qc);
      const float x = turned([&](int j) { return load(at + j); }, e, rot, pos, freq);
      if (is_k) ks[e] = __fmul_rn(x, k_scale);
      else qs[e] = x;
    }
    for (int i = threadIdx.x; i < P; i += ST) vs[i] = load(row + vc + i);
    __syncthreads();
    if (rg < RG)
      for (int c = cg; c < cols; c += CG) {
        const V v = reinterpret_cast<const V*>(vs)[c];
        V acc = {};
        constexpr int AHEAD = 8;         // rows whose loads are issued before the first is used
        for (int r0 = rg; r0 < N; r0 += AHEAD * RG) {
          V s[AHEAD];
#pragma unroll
          for (int u = 0; u < AHEAD; ++u) {
            const int r = r0 + u * RG;
            if (r < N && keeps) s[u] = S[(long long)r * cols + c];
            else s[u] = V{};
          }
#pragma unroll
          for (int u = 0; u < AHEAD; ++u) {
            const int r = r0 + u * RG;
            if (r < N) {
              col_step(s[u], acc, d, ks[r], qs[r], v);
              if (keeps) S[(long long)r * cols + c] = s[u];
            }
          }
        }
        reinterpret_cast<V*>(part + rg * pp)[c] = acc;
      }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < P; c += ST) {
      float o = part[c];
      for (int r = 1; r < RG; ++r) o = __fadd_rn(o, part[r * pp + c]);
      os[c] = o;
      ss = __fmaf_rn(o, o, ss);
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)P + eps);
    for (int c = threadIdx.x; c < P; c += ST) {
      const float g = load(row + gc + c);
      store_as(out, out_dtype, (long long)t * H * P + (long long)h * P + c, os[c] * rstd * (g * sigmoid_f32(g)));
    }
    __syncthreads();
  }
  if (in_smem && slot != 0)
    for (int i = threadIdx.x; i < N * P; i += ST) srow[i] = sm_state[i];
}

// ---- chunks ----------------------------------------------------------------------------------------
// planes: qh, ql, kh, kl, each [tokens][H N] (plane elements apart)
__global__ void __launch_bounds__(256)
retention_rotate_kernel(const __nv_bfloat16* proj, long long row_width, const float* __restrict__ freq, int rot,
                        const int* __restrict__ positions, int t_first, __nv_bfloat16* planes, long long plane,
                        int H, int N, float k_scale) {
  extern __shared__ __align__(16) float cs[];            // cosines [rot / 2], sines [rot / 2]
  pdl_prologue(proj);
  const int tl = blockIdx.x, t = t_first + tl, half = rot >> 1;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += 256) {
    const float a = __fmul_rn(pos, freq[i]);
    cs[i] = cosf(a);
    cs[half + i] = sinf(a);
  }
  __syncthreads();
  const int HN = H * N;
  const __nv_bfloat16* x = proj + (long long)t * row_width;
  if (rot == N && (half & 1) == 0) {
    // the whole head turns: a thread takes two neighbouring pairs
    const int per = half >> 1;
    for (int i = threadIdx.x; i < 2 * H * per; i += 256) {
      const int head = i / per, d = (i - head * per) * 2;           // heads of q, then of k
      const __nv_bfloat16* src = x + (long long)head * N + d;
      const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src));
      const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + half));
      const float2 c = *reinterpret_cast<const float2*>(cs + d), s = *reinterpret_cast<const float2*>(cs + half + d);
      float a0 = __fmaf_rn(u.x, c.x, -__fmul_rn(w.x, s.x)), a1 = __fmaf_rn(u.y, c.y, -__fmul_rn(w.y, s.y));
      float b0 = __fmaf_rn(w.x, c.x, __fmul_rn(u.x, s.x)), b1 = __fmaf_rn(w.y, c.y, __fmul_rn(u.y, s.y));
      const bool is_k = head >= H;
      if (is_k) {
        a0 = __fmul_rn(a0, k_scale); a1 = __fmul_rn(a1, k_scale);
        b0 = __fmul_rn(b0, k_scale); b1 = __fmul_rn(b1, k_scale);
      }
      __nv_bfloat16* dst = planes + (is_k ? 2 * plane : 0) + (long long)tl * HN + (long long)(is_k ? head - H : head) * N + d;
      unsigned hi, lo;
      split2(a0, a1, hi, lo);
      *reinterpret_cast<unsigned*>(dst) = hi;
      *reinterpret_cast<unsigned*>(dst + plane) = lo;
      split2(b0, b1, hi, lo);
      *reinterpret_cast<unsigned*>(dst + half) = hi;
      *reinterpret_cast<unsigned*>(dst + plane + half) = lo;
    }
    return;
  }
  for (int i = threadIdx.x * 2; i < 2 * HN; i += 512) {       // two neighbouring elements of one head
    const bool is_k = i >= HN;
    const int d = i % N;
    float y[2];
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x + i));
    y[0] = v.x;
    y[1] = v.y;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int dd = d + e;
      if (dd < rot) {
        const bool first = dd < half;
        const int f = first ? dd : dd - half;
        const float o = __bfloat162float(x[i + e + (first ? half : -half)]);
        y[e] = first ? __fmaf_rn(y[e], cs[f], -__fmul_rn(o, cs[half + f])) : __fmaf_rn(y[e], cs[f], __fmul_rn(o, cs[half + f]));
      }
      if (is_k) y[e] = __fmul_rn(y[e], k_scale);
    }
    unsigned hi, lo;
    split2(y[0], y[1], hi, lo);
    __nv_bfloat16* dst = planes + (is_k ? 2 * plane : 0) + (long long)tl * HN + (is_k ? i - HN : i);
    *reinterpret_cast<unsigned*>(dst) = hi;
    *reinterpret_cast<unsigned*>(dst + plane) = lo;
  }
}

// grid (places, H, ceil(N / 64)), four warps of 16 rows of the state each, all P columns.
// add [places][H][N][P] float32.
template <int NPT>
__global__ void __launch_bounds__(128)
retention_chunk_kernel(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                       const float* __restrict__ decay, const int* __restrict__ cu, int B, int t_first, float* add,
                       int H, int N, int P) {
  extern __shared__ __align__(16) unsigned char rc_smem[];
  __shared__ float pw[CH];
  pdl_prologue(planes, proj);
  int b, first, count;
  if (!chunk_at(cu, B, blockIdx.x, b, first, count)) return;
  const int h = blockIdx.y, n0 = blockIdx.z * 64;
  constexpr int KS = 64 + PAD;
  const int vs = P + PAD;
  __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(rc_smem);      // [CH][KS]
  __nv_bfloat16* Kl = Kh + CH * KS;
  __nv_bfloat16* Vs = Kl + CH * KS;                                   // [CH][vs]
  const int t0 = cu[b] + first;
  const int pv = P / 8;
  for (int idx = threadIdx.x; idx < CH * pv; idx += 128) {
    const int j = idx / pv, c = idx - j * pv;
    const bool ok = j < count;
    copy16(Vs + j * vs + c * 8, proj + (long long)(ok ? t0 + j : t0) * row_width + 2ll * H * N + (long long)h * P + c * 8, ok);
  }
  __pipeline_commit();
  if (threadIdx.x < CH) pw[threadIdx.x] = (int)threadIdx.x < count ? powf(decay[h], (float)(count - 1 - (int)threadIdx.x)) : 0.f;
  __syncthreads();
  const __nv_bfloat16* kh = planes + 2 * plane;
  for (int idx = threadIdx.x; idx < CH * 8; idx += 128) {
    const int j = idx >> 3, c = (idx & 7) * 8;
    uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
    if (j < count && n0 + c < N) {
      const long long at = (long long)(t0 - t_first + j) * H * N + (long long)h * N + n0 + c;
      const uint4 a = *reinterpret_cast<const uint4*>(kh + at), r = *reinterpret_cast<const uint4*>(kh + plane + at);
      const unsigned* pa = reinterpret_cast<const unsigned*>(&a);
      const unsigned* pr = reinterpret_cast<const unsigned*>(&r);
      unsigned* ph = reinterpret_cast<unsigned*>(&hi);
      unsigned* pl = reinterpret_cast<unsigned*>(&lo);
      const float f = pw[j];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(pa + e));
        const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(pr + e));
        split2(__fmul_rn(__fadd_rn(x.x, y.x), f), __fmul_rn(__fadd_rn(x.y, y.y), f), ph[e], pl[e]);
      }
    }
    *reinterpret_cast<uint4*>(Kh + j * KS + c) = hi;
    *reinterpret_cast<uint4*>(Kl + j * KS + c) = lo;
  }
  __pipeline_wait_prior(0);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int m0 = warp * 16;
  if (n0 + m0 >= N) return;
  float acc[NPT * 8][4];
#pragma unroll
  for (int n = 0; n < NPT * 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < CH / 16; ++kk) {
    // the rows of the product are the state's: the fragments come transposed out of [token][row]
    const int at = (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * KS + m0 + ((lane >> 3) & 1) * 8;
    unsigned h0, h1, h2, h3, l0, l1, l2, l3;
    ldsm_x4_trans(h0, h1, h2, h3, Kh + at);
    ldsm_x4_trans(l0, l1, l2, l3, Kl + at);
#pragma unroll
    for (int np = 0; np < NPT * 4; ++np)
      if (np * 16 < P) {
        unsigned b0, b1, b2, b3;
        ldsm_x4_trans(b0, b1, b2, b3, Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + np * 16 + (lane >> 4) * 8);
        mma_bf16(acc[2 * np], h0, h1, h2, h3, b0, b1);
        mma_bf16(acc[2 * np + 1], h0, h1, h2, h3, b2, b3);
        mma_bf16(acc[2 * np], l0, l1, l2, l3, b0, b1);
        mma_bf16(acc[2 * np + 1], l0, l1, l2, l3, b2, b3);
      }
  }
  float* dst = add + (((long long)blockIdx.x * H + h) * N + n0 + m0) * P;
#pragma unroll
  for (int n = 0; n < NPT * 8; ++n) {
    const int col = n * 8 + tig * 2;
    if (col < P) {
      *reinterpret_cast<float2*>(dst + (long long)gid * P + col) = make_float2(acc[n][0], acc[n][1]);
      *reinterpret_cast<float2*>(dst + (long long)(gid + 8) * P + col) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

// grid (N P / 256, H, B), a thread per 2 elements of a state.  In place: where a chunk's sum lay, the state
// in front of the chunk, four elements as four hi (8 bytes) and four lo (8 bytes); a warp has read its
// groups of four before it writes them.
__global__ void __launch_bounds__(128)
retention_chain_kernel(float2* chunks, const float* __restrict__ decay, float* state, long long slot_stride,
                       const int* __restrict__ cu, const int* __restrict__ state_slots, int H, int NP2) {
  pdl_prologue(chunks, state);
  const int i = blockIdx.x * 128 + threadIdx.x, h = blockIdx.y, b = blockIdx.z;      // (NP2 is a multiple of 128)
  const int len = cu[b + 1] - cu[b];
  if (len <= 0) return;
  const long long slot = state_slots[b];
  float2* srow = reinterpret_cast<float2*>(state + slot * slot_stride) + (long long)h * NP2;
  float2 S = slot != 0 ? srow[i] : make_float2(0.f, 0.f);
  const float d = decay[h], d_chunk = powf(d, (float)CH);
  const int n_chunks = (len + CH - 1) / CH, place = first_place(cu, b);
  const int hi_at = (i >> 1) * 4 + (i & 1);             // in 4-byte words of a state
  constexpr int AHEAD = 16;          // chunks whose loads are issued before the first is used
  for (int c0 = 0; c0 < n_chunks; c0 += AHEAD) {
    float2 add[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < n_chunks) add[u] = chunks[((long long)(place + c0 + u) * H + h) * NP2 + i];
    __syncwarp();
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < n_chunks) {
        unsigned hi, lo;
        split2(S.x, S.y, hi, lo);
        unsigned* dst = reinterpret_cast<unsigned*>(chunks + ((long long)(place + c0 + u) * H + h) * NP2);
        dst[hi_at] = hi;
        dst[hi_at + 2] = lo;
        const int left = len - (c0 + u) * CH;
        const float f = left >= CH ? d_chunk : powf(d, (float)left);
        S.x = __fmaf_rn(f, S.x, add[u].x);
        S.y = __fmaf_rn(f, S.y, add[u].y);
      }
  }
  if (slot != 0) srow[i] = S;
}

// grid (places, H), HALVES times four warps: a warp has 16 tokens and NPT * 64 of the columns (wide heads
// are cut in two, which keeps more warps on an SM; both halves' warps make the same token weights).
template <int NPT, int HALVES>
__global__ void __launch_bounds__(128 * HALVES, 2)
retention_output_kernel(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                        const unsigned char* chunks, const float* __restrict__ decay, const int* __restrict__ cu, int B,
                        int t_first, __nv_bfloat16* out, int H, int N, int P, float eps) {
  extern __shared__ __align__(16) unsigned char ro_smem[];
  __shared__ float pw[CH + 1];
  __shared__ float squares[2][CH];
  constexpr int OT = 128 * HALVES;
  pdl_prologue(planes, proj, chunks);
  int b, first, count;
  if (!chunk_at(cu, B, blockIdx.x, b, first, count)) return;
  const int h = blockIdx.y;
  const int qs = N + PAD, vs = P + PAD;
  constexpr int SR = 16;                                             // state rows of a stage
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(ro_smem);    // [CH][qs]
  __nv_bfloat16* Ql = Qh + CH * qs;
  __nv_bfloat16* Vs = Ql + CH * qs;                                  // [CH][vs]
  __nv_bfloat16* Kh = Vs + CH * vs;                                  // [CH][qs], then the state's stages
  __nv_bfloat16* Kl = Kh + CH * qs;
  __nv_bfloat16* Ss = Kh;                                            // [2][hi, lo][SR][vs]
  const int t0 = cu[b] + first;
  const int nv = N / 8, pv = P / 8;
  for (int idx = threadIdx.x; idx < CH * nv; idx += OT) {
    const int j = idx / nv, c = (idx - j * nv) * 8;
    const bool ok = j < count;
    const __nv_bfloat16* src = planes + (long long)(t0 - t_first + (ok ? j : 0)) * H * N + (long long)h * N + c;
    copy16(Qh + j * qs + c, src, ok);
    copy16(Ql + j * qs + c, src + plane, ok);
    copy16(Kh + j * qs + c, src + 2 * plane, ok);
    copy16(Kl + j * qs + c, src + 3 * plane, ok);
  }
  for (int idx = threadIdx.x; idx < CH * pv; idx += OT) {
    const int j = idx / pv, c = (idx - j * pv) * 8;
    const bool ok = j < count;
    copy16(Vs + j * vs + c, proj + (long long)(ok ? t0 + j : t0) * row_width + 2ll * H * N + (long long)h * P + c, ok);
  }
  __pipeline_commit();
  if (threadIdx.x <= CH) pw[threadIdx.x] = powf(decay[h], (float)threadIdx.x);
  __pipeline_wait_prior(0);
  __syncthreads();
  const int warp = (threadIdx.x >> 5) & 3, half = threadIdx.x >> 7;
  const int lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int m0 = warp * 16, p0 = half * NPT * 64;          // the warp's first token and column
  const bool active = m0 < count && p0 < P;

  // q_i . k_j of the warp's 16 tokens and the chunk's tokens up to them
  float s[CH / 8][4];
#pragma unroll
  for (int n = 0; n < CH / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
  const int q_at = (m0 + (lane & 15)) * qs + (lane >> 4) * 8;
  if (active)
    for (int kk = 0; kk < N / 16; ++kk) {
      unsigned h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4(h0, h1, h2, h3, Qh + q_at + kk * 16);
      ldsm_x4(l0, l1, l2, l3, Ql + q_at + kk * 16);
#pragma unroll
      for (int np = 0; np < CH / 16; ++np)
        if (np <= warp) {
          const int at = (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * qs + kk * 16 + ((lane >> 3) & 1) * 8;
          unsigned b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4(b0, b1, b2, b3, Kh + at);
          ldsm_x4(c0, c1, c2, c3, Kl + at);
          mma_bf16(s[2 * np], h0, h1, h2, h3, b0, b1);
          mma_bf16(s[2 * np + 1], h0, h1, h2, h3, b2, b3);
          mma_bf16(s[2 * np], h0, h1, h2, h3, c0, c1);
          mma_bf16(s[2 * np + 1], h0, h1, h2, h3, c2, c3);
          mma_bf16(s[2 * np], l0, l1, l2, l3, b0, b1);
          mma_bf16(s[2 * np + 1], l0, l1, l2, l3, b2, b3);
        }
    }
  // times d^(i-j), the later tokens masked, as (hi, lo) operands of the product with v
  unsigned wh[CH / 8][2], wl[CH / 8][2];
#pragma unroll
  for (int n = 0; n < CH / 8; ++n)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = m0 + gid + 8 * r, j = n * 8 + tig * 2;
      const float x = j <= i ? s[n][2 * r] * pw[i - j] : 0.f;
      const float y = j + 1 <= i ? s[n][2 * r + 1] * pw[i - j - 1] : 0.f;
      split2(x, y, wh[n][r], wl[n][r]);
    }
  __syncthreads();            // the keys are read; their place takes the state's stages

  const unsigned char* src = chunks + ((long long)blockIdx.x * H + h) * N * P * 4;
  auto stage = [&](int kk, int buf) {
    __nv_bfloat16* hi = Ss + (size_t)buf * 2 * SR * vs;
    for (int idx = threadIdx.x; idx < SR * (P / 4); idx += OT) {
      const int r = idx / (P / 4), c = idx - r * (P / 4);
      const unsigned char* p = src + ((long long)(kk * SR + r) * P + c * 4) * 4;
      __pipeline_memcpy_async(hi + r * vs + c * 4, p, 8);
      __pipeline_memcpy_async(hi + (SR + r) * vs + c * 4, p + 8, 8);
    }
    __pipeline_commit();
  };
  float o[NPT * 8][4];
#pragma unroll
  for (int n = 0; n < NPT * 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  stage(0, 0);
  for (int kk = 0; kk < N / SR; ++kk) {
    if (kk + 1 < N / SR) {
      stage(kk + 1, (kk + 1) & 1);
      __pipeline_wait_prior(1);
    } else {
      __pipeline_wait_prior(0);
    }
    __syncthreads();
    if (active) {
      const __nv_bfloat16* sh = Ss + (size_t)(kk & 1) * 2 * SR * vs;
      unsigned h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4(h0, h1, h2, h3, Qh + q_at + kk * 16);
      ldsm_x4(l0, l1, l2, l3, Ql + q_at + kk * 16);
#pragma unroll
      for (int np = 0; np < NPT * 4; ++np)
        if (p0 + np * 16 < P) {
          const int at = ((lane & 7) + ((lane >> 3) & 1) * 8) * vs + p0 + np * 16 + (lane >> 4) * 8;
          unsigned b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4_trans(b0, b1, b2, b3, sh + at);
          ldsm_x4_trans(c0, c1, c2, c3, sh + SR * vs + at);
          mma_bf16(o[2 * np], h0, h1, h2, h3, b0, b1);
          mma_bf16(o[2 * np + 1], h0, h1, h2, h3, b2, b3);
          mma_bf16(o[2 * np], h0, h1, h2, h3, c0, c1);
          mma_bf16(o[2 * np + 1], h0, h1, h2, h3, c2, c3);
          mma_bf16(o[2 * np], l0, l1, l2, l3, b0, b1);
          mma_bf16(o[2 * np + 1], l0, l1, l2, l3, b2, b3);
        }
    }
    __syncthreads();         // the stage is written again two steps on
  }
  const float f0 = pw[m0 + gid + 1], f1 = pw[m0 + gid + 9];
#pragma unroll
  for (int n = 0; n < NPT * 8; ++n) {
    o[n][0] *= f0; o[n][1] *= f0;
    o[n][2] *= f1; o[n][3] *= f1;
  }
#pragma unroll
  for (int kk = 0; kk < CH / 16; ++kk)
    if (active && kk <= warp) {
#pragma unroll
      for (int np = 0; np < NPT * 4; ++np)
        if (p0 + np * 16 < P) {
          unsigned b0, b1, b2, b3;
          ldsm_x4_trans(b0, b1, b2, b3, Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + p0 + np * 16 + (lane >> 4) * 8);
          mma_bf16(o[2 * np], wh[2 * kk][0], wh[2 * kk][1], wh[2 * kk + 1][0], wh[2 * kk + 1][1], b0, b1);
          mma_bf16(o[2 * np + 1], wh[2 * kk][0], wh[2 * kk][1], wh[2 * kk + 1][0], wh[2 * kk + 1][1], b2, b3);
          mma_bf16(o[2 * np], wl[2 * kk][0], wl[2 * kk][1], wl[2 * kk + 1][0], wl[2 * kk + 1][1], b0, b1);
          mma_bf16(o[2 * np + 1], wl[2 * kk][0], wl[2 * kk][1], wl[2 * kk + 1][0], wl[2 * kk + 1][1], b2, b3);
        }
    }
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NPT * 8; ++n)
    if (p0 + n * 8 < P)
#pragma unroll
      for (int r = 0; r < 2; ++r) ss[r] = __fmaf_rn(o[n][2 * r + 1], o[n][2 * r + 1], __fmaf_rn(o[n][2 * r], o[n][2 * r], ss[r]));
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
    ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
    if (HALVES == 2 && tig == 0) squares[half][m0 + gid + 8 * r] = ss[r];
  }
  if (HALVES == 2) __syncthreads();       // a token's squares: the first half's columns, then the second's
  if (!active) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = m0 + gid + 8 * r;
    if (i >= count) continue;
    const float total = HALVES == 2 ? __fadd_rn(squares[0][i], squares[1][i]) : ss[r];
    const float rstd = 1.0f / sqrtf(total / (float)P + eps);
    const long long row = (long long)(t0 + i) * row_width + 2ll * H * N + (long long)H * P + (long long)h * P;
    __nv_bfloat16* dst = out + (long long)(t0 + i) * H * P + (long long)h * P;
#pragma unroll
    for (int n = 0; n < NPT * 8; ++n) {
      const int col = p0 + n * 8 + tig * 2;
      if (col < P) {
        const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(proj + row + col));
        *reinterpret_cast<unsigned*>(dst + col) = pack_bf16(o[n][2 * r] * rstd * (g.x * sigmoid_f32(g.x)),
                                                            o[n][2 * r + 1] * rstd * (g.y * sigmoid_f32(g.y)));
      }
    }
  }
}

template <int NPT, int OUT_NPT, int HALVES>
int launch_chunks(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                  const float* decay, float* chunks, float* state, long long slot_stride, const int* cu,
                  const int* state_slots, int B, int t_first, int places, __nv_bfloat16* out, int H, int N, int P,
                  float eps, cudaStream_t st) {
  const size_t smem_c = sizeof(__nv_bfloat16) * (2 * (size_t)CH * (64 + PAD) + (size_t)CH * (P + PAD));
  const size_t keys = 2 * (size_t)CH * (N + PAD), stages = 4 * (size_t)16 * (P + PAD);
  const size_t smem_o = sizeof(__nv_bfloat16) * (2 * (size_t)CH * (N + PAD) + (size_t)CH * (P + PAD) + (keys > stages ? keys : stages));
  if (smem_c > MOST_SMEM || smem_o > MOST_SMEM) return DIB_BAD_SIZE;
  static DeviceOnce once;
  if (!once.done()) {
    if (cudaFuncSetAttribute(retention_chunk_kernel<NPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(retention_output_kernel<OUT_NPT, HALVES>, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return DIB_LAUNCH_FAILED;
    // (as much of an SM's memory as shared memory as there is, so that two blocks of wide heads fit)
    cudaFuncSetAttribute(retention_chunk_kernel<NPT>, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    cudaFuncSetAttribute(retention_output_kernel<OUT_NPT, HALVES>, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    once.mark();
  }
  dib_launch(retention_chunk_kernel<NPT>, dim3(places, H, (N + 63) / 64), dim3(128), smem_c, st, planes, plane, proj,
             row_width, decay, cu, B, t_first, chunks, H, N, P);
  DIB_CHECK_LAUNCH();
  dib_launch(retention_chain_kernel, dim3(N * P / 256, H, B), dim3(128), 0, st, (float2*)chunks, decay, state,
             slot_stride, cu, state_slots, H, N * P / 2);
  DIB_CHECK_LAUNCH();
  dib_launch(retention_output_kernel<OUT_NPT, HALVES>, dim3(places, H), dim3(128 * HALVES), smem_o, st, planes, plane, proj, row_width,
             (const unsigned char*)chunks, decay, cu, B, t_first, out, H, N, P, eps);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

}  // namespace

extern "C" {

// Tokens one by one: B sequences, whose boundaries and slots cu_q_lens and state_slots give (pointers to
// the first of them).  in_smem 1: the state in shared memory while a sequence is walked (DIB_BAD_SIZE
// when it does not fit); 0: in the slot.
int dib_retention_step(const void* proj, int kind, int splits, long long stride, long long row_width, const float* decay,
                       const float* freq, int rot, const int* positions, float* state, long long slot_stride,
                       const int* cu_q_lens, const int* state_slots, void* out, int out_dtype, int B, int H, int N, int P,
                       float k_scale, float eps, int in_smem, cudaStream_t st) {
  if (B == 0) return DIB_OK;
  if (H < 1 || H > 65535 || N < 1 || N > 2048 || P < 1 || P > 4096 || rot < 0 || rot > N || rot % 2 ||
      (rot > 0 && freq == nullptr) || row_width < 2ll * H * (N + P) || slot_stride < (long long)H * N * P)
    return DIB_BAD_SIZE;
  if (out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  const bool v4 = P % 4 == 0 && slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
  const int cols = v4 ? P / 4 : P, CG = cols < ST ? cols : ST, RG = ST / CG;
  const int np = (N + 3) / 4 * 4, pp = (P + 3) / 4 * 4;
  const size_t smem = sizeof(float) * (2 * (size_t)np + 2 * (size_t)pp + (size_t)RG * pp + (in_smem ? (size_t)N * P : 0));
  if (smem > MOST_SMEM) return DIB_BAD_SIZE;
  const Source src = make_source(proj, kind, splits, stride);
  static DeviceOnce once4, once1;
  DeviceOnce& once = v4 ? once4 : once1;
  auto kern = v4 ? retention_step_kernel<4> : retention_step_kernel<1>;
  if (!once.done()) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return DIB_LAUNCH_FAILED;
    once.mark();
  }
  dib_launch(kern, dim3(B, H), dim3(ST), smem, st, src, row_width, decay, freq, rot, positions, state, slot_stride,
             cu_q_lens, state_slots, out, out_dtype, H, N, P, k_scale, eps, in_smem);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// Whether a head's state fits in shared memory (dib_retention_step with in_smem 1), whatever the alignment.
int dib_retention_state_fits(int N, int P) {
  const size_t pp = (P + 3) / 4 * 4, np = (N + 3) / 4 * 4;
  const int cols = P % 4 == 0 ? P / 4 : P;             // (the wider of the two forms' shares)
  const size_t shares = cols < ST ? ST / cols : 1;
  return sizeof(float) * (2 * np + (2 + shares) * pp + (size_t)N * P) <= MOST_SMEM ? 1 : 0;
}

// The chunked form: B sequences (cu and state_slots point at the first of them; its first token is
// t_first of the step), `tokens` tokens.  proj bfloat16.  planes: 4 * tokens * H * N bfloat16; chunks:
// places * H * N * P floats with places = tokens / 64 + B.
int dib_retention_chunked(const void* proj, long long row_width, const float* decay, const float* freq, int rot,
                          const int* positions, float* state, long long slot_stride, const int* cu,
                          const int* state_slots, void* planes, float* chunks, void* out, int B, int t_first, int tokens,
                          int H, int N, int P, float k_scale, float eps, cudaStream_t st) {
  if (B == 0 || tokens == 0) return DIB_OK;
  if (H < 1 || H > 65535 || B > 65535 || N < 16 || N > 256 || N % 16 || P < 16 || P > 256 || P % 16 || rot < 0 || rot > N ||
      rot % 2 || (rot > 0 && freq == nullptr) || row_width < 2ll * H * (N + P) || row_width % 8 || slot_stride % 4)
    return DIB_BAD_SIZE;
  if ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(planes) |
       reinterpret_cast<uintptr_t>(chunks) | reinterpret_cast<uintptr_t>(out)) % 16 != 0)
    return DIB_BAD_ALIGN;
  const long long plane = (long long)tokens * H * N;
  const int places = tokens / CH + B;
  dib_launch(retention_rotate_kernel, dim3(tokens), dim3(256), sizeof(float) * (rot > 0 ? rot : 1), st,
             (const __nv_bfloat16*)proj, row_width, freq, rot, positions, t_first, (__nv_bfloat16*)planes, plane, H, N,
             k_scale);
  DIB_CHECK_LAUNCH();
#define DIB_RC(NPT, OUT_NPT, HALVES)                                                                                  \
  return launch_chunks<NPT, OUT_NPT, HALVES>((const __nv_bfloat16*)planes, plane, (const __nv_bfloat16*)proj, row_width, decay, chunks, state, \
                            slot_stride, cu, state_slots, B, t_first, places, (__nv_bfloat16*)out, H, N, P, eps, st)
  if (P <= 64) DIB_RC(1, 1, 1);
  if (P <= 128) DIB_RC(2, 1, 2);
  if (P <= 192) DIB_RC(3, 2, 2);
  DIB_RC(4, 2, 2);
#undef DIB_RC
}

}  // extern "C"
