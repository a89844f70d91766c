// Gated linear attention: a matrix state per head whose rows decay by a number of their own every token.
//
// proj row (row_width elements): [q: H N | k: H N | v: H P | g: H P | anything].  Per head, with a state S
// [N][P] from zero and a decay alpha per (token, row of S):
//     S <- diag(alpha) S + k v^T;     o = S^T (q q_scale);     out = o / sqrt(mean(o^2) + eps) * w * silu(g),
// w [P] shared by the heads, log alpha = log(sigmoid(z)) / tau with z = hidden A2^T + b, `hidden` R float32
// numbers a token; both forms make the decays they need from it.  A request's state slot holds the heads' states [H][N][P], float32; slot 0 is no
// request's: a sequence on it starts from zeros and stores nothing.
//
// Two forms.
//
// gla_step_kernel: a block per (sequence, head) walks the sequence's tokens one by one: decays, state,
// read-out, norm and gate in one kernel, everything float32.  It serves decoded tokens (the state is read
// and written once, which is all the memory they move), and prompt portions of the float32 engine and of
// sizes the other form does not take.
//
// The chunked form for prompt portions of the bfloat16 engine (N and P multiples of 16, up to 256).  A
// portion is cut into chunks of 64 tokens and a chunk into four runs of 16; L_t is the sum of the log decays
// from the chunk's start up to and including token t, M_i the L of run i's eighth token, E_i that of its
// last one (all per row of the state).  With S the state in front of the chunk,
//     o_t = (q_t e^{L_t})^T S + sum_{s <= t} (sum_n q_tn k_sn e^{L_tn - L_sn}) v_s,
//     S  <- diag(e^{E_3}) S + sum_s (k_s e^{E_3 - L_s}) v_s^T,
// so all chunks' sums over their own tokens are products that run side by side, and only the states are
// chained.  A run's tokens are stored as q e^{L - M_i} and k e^{M_i - L}; what a product needs beyond that is
// a factor per state row (e^{M_i} in front of the state, e^{M_i - E_j} against the keys of an earlier run j,
// which are taken to k e^{E_j - L}, and e^{E_3 - M_j} in the chunk's own sum), never above 1, so nothing
// overflows however fast a row forgets.  Inside a run the exponents reach eight tokens' decays in both
// directions; a log decay below LEAST counts as LEAST there (a factor of 1.2e-4 where the true one is
// smaller), which keeps them within e^72.
//   gla_prepare_kernel   the runs' q and k as bfloat16 pairs (hi, lo) with hi + lo the float32 value up to
//                        2^-17 of it, and M, E of every chunk
//   gla_chunk_kernel     sum_s (k_s e^{E_3 - L_s}) v_s^T of every chunk
//   gla_chain_kernel     the states in front of the chunks, as (hi, lo) pairs, and the slot's
//   gla_output_kernel    o, its norm and the gate
// The products run on the tensor cores (mma.sync m16n8k16, bfloat16 operands, float32 accumulators) with
// every float32 operand as its (hi, lo) pair (hi hi + hi lo + lo hi; v is a bfloat16 projection, one term),
// so nothing that enters the recurrence is rounded below 2^-16.
#include "linear_chunks.cuh"

namespace {

using sa_mma::copy16;
using sa_mma::ldsm_x4;
using sa_mma::ldsm_x4_trans;
using sa_mma::mma_bf16;
using sa_mma::pack_bf16;
using namespace chunks;

constexpr float LEAST = -9.0f;         // the smallest log decay of the chunked form
constexpr int RUN = 16;                // tokens of a run
constexpr int RUNS = CH / RUN;

// What the decays are made of: R numbers a token at column `at` of rows row_width apart, the map a2_t [R][H N]
// (dtype 0 float32, 1 bfloat16) and its bias.
struct Decays {
  Source hidden;
  long long row_width, at;
  const void* a2_t;
  int dtype;
  const float* bias;
  float tau;
  int R;
};
__device__ __forceinline__ float log_decay(float sum, float bias, float tau) {
  const float z = __fadd_rn(sum, bias);
  return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) / tau;
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
gla_step_kernel(Source proj, long long row_width, Decays dec, float* state, long long slot_stride,
                const int* __restrict__ cu_q_lens, const int* __restrict__ state_slots, const float* __restrict__ norm_w,
                void* out, int out_dtype, int H, int N, int P, float q_scale, float eps, int in_smem) {
  using V = typename Cols<VEC>::T;
  extern __shared__ __align__(16) float gs_smem[];   // q [N], k [N], alpha [N], v [P], o [P], hidden [R], shares [RG][P], state [N][P] (in_smem)
  __shared__ float scratch[32];
  pdl_prologue(proj.p, dec.hidden.p, state);
  const int b = blockIdx.x, h = blockIdx.y;
  const int t0 = cu_q_lens[b], n_tok = cu_q_lens[b + 1] - t0;
  if (n_tok <= 0) return;
  const long long slot = state_slots[b];
  const int np = (N + 3) / 4 * 4, pp = (P + 3) / 4 * 4;
  float* qs = gs_smem;
  float* ks = qs + np;
  float* as = ks + np;
  float* vs = as + np;
  float* os = vs + pp;
  float* hs = os + pp;
  float* part = hs + (dec.R + 3) / 4 * 4;
  const int cols = P / VEC;
  const int CG = cols < ST ? cols : ST, RG = ST / CG;
  const int cg = threadIdx.x % CG, rg = threadIdx.x / CG;
  float* sm_state = part + RG * pp;
  float* srow = state + slot * slot_stride + (long long)h * N * P;
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
    for (int i = threadIdx.x; i < dec.R; i += ST) hs[i] = source_load(dec.hidden, (long long)t * dec.row_width + dec.at + i);
    for (int i = threadIdx.x; i < 2 * N; i += ST) {
      if (i < N) qs[i] = __fmul_rn(load(row + qc + i), q_scale);
      else ks[i - N] = load(row + kc + i - N);
    }
    for (int i = threadIdx.x; i < P; i += ST) vs[i] = load(row + vc + i);
    __syncthreads();
    for (int i = threadIdx.x; i < N; i += ST) {
      float z = 0.f;
#pragma unroll 8
      for (int r = 0; r < dec.R; ++r)
        z = __fmaf_rn(hs[r], load_as(dec.a2_t, dec.dtype, (long long)r * H * N + (long long)h * N + i), z);
      as[i] = expf(log_decay(z, dec.bias[h * N + i], dec.tau));
    }
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
              col_step(s[u], acc, as[r], ks[r], qs[r], v);
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
      store_as(out, out_dtype, (long long)t * H * P + (long long)h * P + c, os[c] * rstd * norm_w[c] * (g * sigmoid_f32(g)));
    }
    __syncthreads();
  }
  if (in_smem && slot != 0)
    for (int i = threadIdx.x; i < N * P; i += ST) srow[i] = sm_state[i];
}

// ---- chunks ----------------------------------------------------------------------------------------
// grid (places, H), RUNS groups of N / 2 threads: a group a run, a thread two neighbouring rows of the state.
// planes: q hi, q lo, k hi, k lo, each [tokens][H N] (plane elements apart).  edges [places][H][2 RUNS][N]: M_0 ..
// M_3, E_0 .. E_3.
__global__ void __launch_bounds__(512)
gla_prepare_kernel(const __nv_bfloat16* proj, long long row_width, Decays dec, const int* __restrict__ cu, int B,
                   int t_first, __nv_bfloat16* planes, long long plane, float* edges, int H, int N, float q_scale) {
  extern __shared__ __align__(16) float gp_smem[];      // hidden [R][CH], then the runs' own M and E [2][RUNS][N]
  pdl_prologue(proj, dec.hidden.p);
  int b, first, count;
  if (!chunk_at(cu, B, blockIdx.x, b, first, count)) return;
  const int h = blockIdx.y, half = N / 2;
  const int run = threadIdx.x / half, d = (threadIdx.x - run * half) * 2;
  const int j0 = run * RUN, t0 = cu[b] + first;
  float2 g[RUN];
  unsigned q[RUN], k[RUN];
#pragma unroll
  for (int j = 0; j < RUN; ++j) {
    g[j] = make_float2(0.f, 0.f);
    q[j] = k[j] = 0u;
    if (j0 + j < count) {
      const long long t = t0 + j0 + j;
      const __nv_bfloat16* src = proj + t * row_width + (long long)h * N + d;
      q[j] = *reinterpret_cast<const unsigned*>(src);
      k[j] = *reinterpret_cast<const unsigned*>(src + (long long)H * N);
    }
  }
  for (int i = threadIdx.x; i < CH * dec.R; i += blockDim.x) {
    const int j = i / dec.R, r = i - j * dec.R;
    gp_smem[r * CH + j] = j < count ? source_load(dec.hidden, (long long)(t0 + j) * dec.row_width + dec.at + r) : 0.f;
  }
  __syncthreads();
  const __nv_bfloat16* a2 = reinterpret_cast<const __nv_bfloat16*>(dec.a2_t) + (long long)h * N + d;
#pragma unroll 2
  for (int r = 0; r < dec.R; ++r) {
    const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(a2 + (long long)r * H * N));
    const float4* hr = reinterpret_cast<const float4*>(gp_smem + r * CH + j0);
#pragma unroll
    for (int j4 = 0; j4 < RUN / 4; ++j4) {
      const float4 x = hr[j4];
      const float v[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        g[j4 * 4 + e].x = __fmaf_rn(v[e], w.x, g[j4 * 4 + e].x);
        g[j4 * 4 + e].y = __fmaf_rn(v[e], w.y, g[j4 * 4 + e].y);
      }
    }
  }
  const float2 a2_bias = *reinterpret_cast<const float2*>(dec.bias + h * N + d);
#pragma unroll
  for (int j = 0; j < RUN; ++j) {                       // from the map's sums to log decays and their sums inside the run
    g[j].x = j0 + j < count ? fmaxf(log_decay(g[j].x, a2_bias.x, dec.tau), LEAST) : 0.f;
    g[j].y = j0 + j < count ? fmaxf(log_decay(g[j].y, a2_bias.y, dec.tau), LEAST) : 0.f;
    if (j > 0) {
      g[j].x = __fadd_rn(g[j].x, g[j - 1].x);
      g[j].y = __fadd_rn(g[j].y, g[j - 1].y);
    }
  }
  const float2 mid = g[RUN / 2 - 1];
#pragma unroll
  for (int j = 0; j < RUN; ++j) {
    if (j0 + j >= count) continue;
    const float ux = __fsub_rn(g[j].x, mid.x), uy = __fsub_rn(g[j].y, mid.y);
    const float2 qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j]));
    const float2 kv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&k[j]));
    __nv_bfloat16* dst = planes + (long long)(t0 - t_first + j0 + j) * H * N + (long long)h * N + d;
    unsigned hi, lo;
    split2(__fmul_rn(__fmul_rn(qv.x, q_scale), expf(ux)), __fmul_rn(__fmul_rn(qv.y, q_scale), expf(uy)), hi, lo);
    *reinterpret_cast<unsigned*>(dst) = hi;
    *reinterpret_cast<unsigned*>(dst + plane) = lo;
    split2(__fmul_rn(kv.x, expf(-ux)), __fmul_rn(kv.y, expf(-uy)), hi, lo);
    *reinterpret_cast<unsigned*>(dst + 2 * plane) = hi;
    *reinterpret_cast<unsigned*>(dst + 3 * plane) = lo;
  }
  float2* mids = reinterpret_cast<float2*>(gp_smem + CH * dec.R);
  float2* ends = mids + RUNS * half;
  mids[run * half + d / 2] = mid;
  ends[run * half + d / 2] = g[RUN - 1];
  __syncthreads();
  float2 before = make_float2(0.f, 0.f);                // the sum in front of this run, runs in order
  for (int r = 0; r < run; ++r) {
    const float2 e = ends[r * half + d / 2];
    before.x = __fadd_rn(before.x, e.x);
    before.y = __fadd_rn(before.y, e.y);
  }
  float* dst = edges + ((long long)blockIdx.x * H + h) * 2 * RUNS * N;
  *reinterpret_cast<float2*>(dst + run * N + d) = make_float2(__fadd_rn(before.x, mid.x), __fadd_rn(before.y, mid.y));
  *reinterpret_cast<float2*>(dst + (RUNS + run) * N + d) =
      make_float2(__fadd_rn(before.x, g[RUN - 1].x), __fadd_rn(before.y, g[RUN - 1].y));
}

// grid (places, H, ceil(N / 64)), four warps of 16 rows of the state each, all P columns.
// add [places][H][N][P] float32.
template <int NPT>
__global__ void __launch_bounds__(128)
gla_chunk_kernel(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                 const float* edges, const int* __restrict__ cu, int B, int t_first, float* add, int H, int N, int P) {
  extern __shared__ __align__(16) unsigned char gc_smem[];
  __shared__ float factor[RUNS][64];                                  // e^{E_3 - M_j} of the block's rows
  pdl_prologue(planes, proj, edges);
  int b, first, count;
  if (!chunk_at(cu, B, blockIdx.x, b, first, count)) return;
  const int h = blockIdx.y, n0 = blockIdx.z * 64;
  constexpr int KS = 64 + PAD;
  const int vs = P + PAD;
  __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(gc_smem);      // [CH][KS]
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
  const float* edge = edges + ((long long)blockIdx.x * H + h) * 2 * RUNS * N;
  for (int i = threadIdx.x; i < RUNS * 64; i += 128) {
    const int j = i >> 6, r = n0 + (i & 63);
    factor[j][i & 63] = r < N ? expf(__fsub_rn(edge[(2 * RUNS - 1) * N + r], edge[j * N + r])) : 0.f;
  }
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
      const float* f = factor[j / RUN] + c;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 x = join2(pa[e], pr[e]);
        split2(__fmul_rn(x.x, f[2 * e]), __fmul_rn(x.y, f[2 * e + 1]), ph[e], pl[e]);
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

// grid (N P / 256, H, B), a thread per 2 elements of a state row.  In place: where a chunk's sum lay, the
// state in front of the chunk, four elements as four hi (8 bytes) and four lo (8 bytes); a warp has read
// its groups of four before it writes them.
__global__ void __launch_bounds__(128)
gla_chain_kernel(float2* places, const float* edges, float* state, long long slot_stride, const int* __restrict__ cu,
                 const int* __restrict__ state_slots, int H, int N, int P) {
  pdl_prologue(places, edges, state);
  const int NP2 = N * P / 2;
  const int i = blockIdx.x * 128 + threadIdx.x, h = blockIdx.y, b = blockIdx.z;      // (NP2 is a multiple of 128)
  const int len = cu[b + 1] - cu[b];
  if (len <= 0) return;
  const long long slot = state_slots[b];
  float2* srow = reinterpret_cast<float2*>(state + slot * slot_stride) + (long long)h * NP2;
  float2 S = slot != 0 ? srow[i] : make_float2(0.f, 0.f);
  const int n_chunks = (len + CH - 1) / CH, place = first_place(cu, b), row = 2 * i / P;
  const int hi_at = (i >> 1) * 4 + (i & 1);             // in 4-byte words of a state
  constexpr int AHEAD = 16;          // chunks whose loads are issued before the first is used
  for (int c0 = 0; c0 < n_chunks; c0 += AHEAD) {
    float2 add[AHEAD];
    float total[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < n_chunks) {
        const long long at = (long long)(place + c0 + u) * H + h;
        add[u] = places[at * NP2 + i];
        total[u] = edges[(at * 2 * RUNS + 2 * RUNS - 1) * N + row];
      }
    __syncwarp();
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < n_chunks) {
        unsigned hi, lo;
        split2(S.x, S.y, hi, lo);
        unsigned* dst = reinterpret_cast<unsigned*>(places + ((long long)(place + c0 + u) * H + h) * NP2);
        dst[hi_at] = hi;
        dst[hi_at + 2] = lo;
        const float f = expf(total[u]);
        S.x = __fmaf_rn(f, S.x, add[u].x);
        S.y = __fmaf_rn(f, S.y, add[u].y);
      }
  }
  if (slot != 0) srow[i] = S;
}

// a fragment of 16 rows and 16 columns times a factor per column (this thread's columns f[0], f[1], f[8], f[9])
__device__ __forceinline__ void scale_fragment(const unsigned (&h)[4], const unsigned (&l)[4], const float* f,
                                               unsigned (&oh)[4], unsigned (&ol)[4]) {
  const float2 a = *reinterpret_cast<const float2*>(f), c = *reinterpret_cast<const float2*>(f + 8);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 x = join2(h[e], l[e]), y = e < 2 ? a : c;
    split2(__fmul_rn(x.x, y.x), __fmul_rn(x.y, y.y), oh[e], ol[e]);
  }
}

// grid (places, H), HALVES times four warps: a warp has a run's 16 tokens and NPT * 64 of the columns (wide heads
// are cut in two, which keeps more warps on an SM; both halves' warps make the same token weights).
template <int NPT, int HALVES>
__global__ void __launch_bounds__(128 * HALVES, 2)
gla_output_kernel(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                  const unsigned char* places, const float* edges, const float* __restrict__ norm_w,
                  const int* __restrict__ cu, int B, int t_first, __nv_bfloat16* out, int H, int N, int P, float eps) {
  extern __shared__ __align__(16) unsigned char go_smem[];
  __shared__ float squares[2][CH];
  constexpr int OT = 128 * HALVES;
  pdl_prologue(planes, proj, places, edges);
  int b, first, count;
  if (!chunk_at(cu, B, blockIdx.x, b, first, count)) return;
  const int h = blockIdx.y;
  const int qs = N + PAD, vs = P + PAD;
  constexpr int SR = 16;                                             // state rows of a stage
  constexpr int TABLES = 13;
  float* F = reinterpret_cast<float*>(go_smem);                      // factors [TABLES][N]: see below
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(F + TABLES * N);    // [CH][qs]
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
  // tables 0..3: e^{M_i} (in front of the state); 4 + i (i - 1) / 2 + j: e^{M_i - E_j} (run i's queries, run j's
  // keys, j < i); 10 + j: e^{E_j - M_j}, which takes run j's keys to k e^{E_j - L}
  const float* edge = edges + ((long long)blockIdx.x * H + h) * 2 * RUNS * N;
  for (int r = threadIdx.x; r < N; r += OT) {
    float M[RUNS], E[RUNS];
#pragma unroll
    for (int i = 0; i < RUNS; ++i) {
      M[i] = edge[i * N + r];
      E[i] = edge[(RUNS + i) * N + r];
    }
#pragma unroll
    for (int i = 0; i < RUNS; ++i) {
      F[i * N + r] = expf(M[i]);
#pragma unroll
      for (int j = 0; j < i; ++j) F[(RUNS + i * (i - 1) / 2 + j) * N + r] = expf(__fsub_rn(M[i], E[j]));
      if (i + 1 < RUNS) F[(10 + i) * N + r] = expf(__fsub_rn(E[i], M[i]));
    }
  }
  __pipeline_wait_prior(0);
  __syncthreads();
  const int warp = (threadIdx.x >> 5) & 3, half = threadIdx.x >> 7;
  const int lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int m0 = warp * 16, p0 = half * NPT * 64;          // the warp's first token and column
  const bool active = m0 < count && p0 < P;

  // the products of the warp's 16 tokens and the chunk's tokens up to them: its own run first
  float s[CH / 8][4];
#pragma unroll
  for (int n = 0; n < CH / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
  const int q_at = (m0 + (lane & 15)) * qs + (lane >> 4) * 8;
  const int k_at = ((lane & 7) + ((lane >> 4) << 3)) * qs + ((lane >> 3) & 1) * 8;
  auto products = [&](float (&x)[4], float (&y)[4], const unsigned (&qh)[4], const unsigned (&ql)[4], int at) {
    unsigned b0, b1, b2, b3, c0, c1, c2, c3;
    ldsm_x4(b0, b1, b2, b3, Kh + at);
    ldsm_x4(c0, c1, c2, c3, Kl + at);
    mma_bf16(x, qh[0], qh[1], qh[2], qh[3], b0, b1);
    mma_bf16(y, qh[0], qh[1], qh[2], qh[3], b2, b3);
    mma_bf16(x, qh[0], qh[1], qh[2], qh[3], c0, c1);
    mma_bf16(y, qh[0], qh[1], qh[2], qh[3], c2, c3);
    mma_bf16(x, ql[0], ql[1], ql[2], ql[3], b0, b1);
    mma_bf16(y, ql[0], ql[1], ql[2], ql[3], b2, b3);
  };
  if (active)
    for (int kk = 0; kk < N / 16; ++kk) {
      unsigned qh[4], ql[4];
      ldsm_x4(qh[0], qh[1], qh[2], qh[3], Qh + q_at + kk * 16);
      ldsm_x4(ql[0], ql[1], ql[2], ql[3], Ql + q_at + kk * 16);
#pragma unroll
      for (int np = 0; np < RUNS; ++np)
        if (np == warp) products(s[2 * np], s[2 * np + 1], qh, ql, np * 16 * qs + k_at + kk * 16);
    }
  __syncthreads();
  // the keys of the first three runs, relative to their run's end
  const int n2 = N / 2;
  for (int idx = threadIdx.x; idx < 3 * RUN * n2; idx += OT) {
    const int j = idx / n2, c = (idx - j * n2) * 2;
    unsigned* ph = reinterpret_cast<unsigned*>(Kh + j * qs + c);
    unsigned* pl = reinterpret_cast<unsigned*>(Kl + j * qs + c);
    const float2 x = join2(*ph, *pl), f = *reinterpret_cast<const float2*>(F + (10 + j / RUN) * N + c);
    split2(__fmul_rn(x.x, f.x), __fmul_rn(x.y, f.y), *ph, *pl);
  }
  __syncthreads();
  if (active && warp > 0)
    for (int kk = 0; kk < N / 16; ++kk) {
      unsigned qh[4], ql[4];
      ldsm_x4(qh[0], qh[1], qh[2], qh[3], Qh + q_at + kk * 16);
      ldsm_x4(ql[0], ql[1], ql[2], ql[3], Ql + q_at + kk * 16);
#pragma unroll
      for (int np = 0; np < RUNS - 1; ++np)
        if (np < warp) {
          unsigned fh[4], fl[4];
          scale_fragment(qh, ql, F + (RUNS + warp * (warp - 1) / 2 + np) * N + kk * 16 + tig * 2, fh, fl);
          products(s[2 * np], s[2 * np + 1], fh, fl, np * 16 * qs + k_at + kk * 16);
        }
    }
  // the later tokens masked, as (hi, lo) operands of the product with v
  unsigned wh[CH / 8][2], wl[CH / 8][2];
#pragma unroll
  for (int n = 0; n < CH / 8; ++n)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = m0 + gid + 8 * r, j = n * 8 + tig * 2;
      split2(j <= i ? s[n][2 * r] : 0.f, j + 1 <= i ? s[n][2 * r + 1] : 0.f, wh[n][r], wl[n][r]);
    }
  __syncthreads();            // the keys are read; their place takes the state's stages

  const unsigned char* src = places + ((long long)blockIdx.x * H + h) * N * P * 4;
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
      unsigned qh[4], ql[4], fh[4], fl[4];
      ldsm_x4(qh[0], qh[1], qh[2], qh[3], Qh + q_at + kk * 16);
      ldsm_x4(ql[0], ql[1], ql[2], ql[3], Ql + q_at + kk * 16);
      scale_fragment(qh, ql, F + warp * N + kk * 16 + tig * 2, fh, fl);
#pragma unroll
      for (int np = 0; np < NPT * 4; ++np)
        if (p0 + np * 16 < P) {
          const int at = ((lane & 7) + ((lane >> 3) & 1) * 8) * vs + p0 + np * 16 + (lane >> 4) * 8;
          unsigned b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4_trans(b0, b1, b2, b3, sh + at);
          ldsm_x4_trans(c0, c1, c2, c3, sh + SR * vs + at);
          mma_bf16(o[2 * np], fh[0], fh[1], fh[2], fh[3], b0, b1);
          mma_bf16(o[2 * np + 1], fh[0], fh[1], fh[2], fh[3], b2, b3);
          mma_bf16(o[2 * np], fh[0], fh[1], fh[2], fh[3], c0, c1);
          mma_bf16(o[2 * np + 1], fh[0], fh[1], fh[2], fh[3], c2, c3);
          mma_bf16(o[2 * np], fl[0], fl[1], fl[2], fl[3], b0, b1);
          mma_bf16(o[2 * np + 1], fl[0], fl[1], fl[2], fl[3], b2, b3);
        }
    }
    __syncthreads();         // the stage is written again two steps on
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
        const float2 w = *reinterpret_cast<const float2*>(norm_w + col);
        *reinterpret_cast<unsigned*>(dst + col) = pack_bf16(o[n][2 * r] * rstd * w.x * (g.x * sigmoid_f32(g.x)),
                                                            o[n][2 * r + 1] * rstd * w.y * (g.y * sigmoid_f32(g.y)));
      }
    }
  }
}

template <int NPT, int OUT_NPT, int HALVES>
int launch_chunks(const __nv_bfloat16* planes, long long plane, const __nv_bfloat16* proj, long long row_width,
                  const float* edges, const float* norm_w, float* sums, float* state, long long slot_stride, const int* cu,
                  const int* state_slots, int B, int t_first, int places, __nv_bfloat16* out, int H, int N, int P,
                  float eps, cudaStream_t st) {
  const size_t smem_c = sizeof(__nv_bfloat16) * (2 * (size_t)CH * (64 + PAD) + (size_t)CH * (P + PAD));
  const size_t keys = 2 * (size_t)CH * (N + PAD), stages = 4 * (size_t)16 * (P + PAD);
  const size_t smem_o = sizeof(float) * 13 * (size_t)N +
                        sizeof(__nv_bfloat16) * (2 * (size_t)CH * (N + PAD) + (size_t)CH * (P + PAD) + (keys > stages ? keys : stages));
  if (smem_c > MOST_SMEM || smem_o > MOST_SMEM) return DIB_BAD_SIZE;
  static DeviceOnce once;
  if (!once.done()) {
    if (cudaFuncSetAttribute(gla_chunk_kernel<NPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(gla_output_kernel<OUT_NPT, HALVES>, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return DIB_LAUNCH_FAILED;
    // (as much of an SM's memory as shared memory as there is, so that two blocks of wide heads fit)
    cudaFuncSetAttribute(gla_chunk_kernel<NPT>, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    cudaFuncSetAttribute(gla_output_kernel<OUT_NPT, HALVES>, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    once.mark();
  }
  dib_launch(gla_chunk_kernel<NPT>, dim3(places, H, (N + 63) / 64), dim3(128), smem_c, st, planes, plane, proj, row_width,
             edges, cu, B, t_first, sums, H, N, P);
  DIB_CHECK_LAUNCH();
  dib_launch(gla_chain_kernel, dim3(N * P / 256, H, B), dim3(128), 0, st, (float2*)sums, edges, state, slot_stride, cu,
             state_slots, H, N, P);
  DIB_CHECK_LAUNCH();
  dib_launch(gla_output_kernel<OUT_NPT, HALVES>, dim3(places, H), dim3(128 * HALVES), smem_o, st, planes, plane, proj, row_width,
             (const unsigned char*)sums, edges, norm_w, cu, B, t_first, out, H, N, P, eps);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

constexpr int MOST_CHUNKED_RANK = 512;          // (the tokens' numbers lie in shared memory)
bool decays_fit(int R, long long h_row, long long h_at, float tau) {
  return R >= 1 && R <= 1024 && h_at >= 0 && h_at + R <= h_row && tau > 0.f;
}

}  // namespace

extern "C" {

// What the decays are made of: hidden holds R numbers a token at column h_at of rows h_row apart; a2_t [R][H N] of
// a2_dtype (0 float32, 1 bfloat16; the chunked form: bfloat16), a2_bias [H N].

// Tokens one by one: B sequences, whose boundaries and slots cu_q_lens and state_slots give (pointers to
// the first of them).  in_smem 1: the state in shared memory while a sequence is walked (DIB_BAD_SIZE
// when it does not fit); 0: in the slot.
int dib_gla_step(const void* proj, int kind, int splits, long long stride, long long row_width, const void* hidden,
                 int h_kind, int h_splits, long long h_stride, long long h_row, long long h_at, const void* a2_t, int a2_dtype,
                 const float* a2_bias, float tau, int R, float* state, long long slot_stride, const int* cu_q_lens, const int* state_slots, const float* norm_w,
                 void* out, int out_dtype, int B, int H, int N, int P, float q_scale, float eps, int in_smem,
                 cudaStream_t st) {
  if (B == 0) return DIB_OK;
  if (H < 1 || H > 65535 || N < 1 || N > 2048 || P < 1 || P > 4096 || row_width < 2ll * H * (N + P) ||
      slot_stride < (long long)H * N * P || !decays_fit(R, h_row, h_at, tau))
    return DIB_BAD_SIZE;
  if (a2_dtype != 0 && a2_dtype != 1) return DIB_BAD_DTYPE;
  if (out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  const bool v4 = P % 4 == 0 && slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
  const int cols = v4 ? P / 4 : P, CG = cols < ST ? cols : ST, RG = ST / CG;
  const int np = (N + 3) / 4 * 4, pp = (P + 3) / 4 * 4;
  const size_t smem = sizeof(float) * (3 * (size_t)np + 2 * (size_t)pp + (size_t)((R + 3) / 4 * 4) + (size_t)RG * pp + (in_smem ? (size_t)N * P : 0));
  if (smem > MOST_SMEM) return DIB_BAD_SIZE;
  const Source src = make_source(proj, kind, splits, stride);
  static DeviceOnce once4, once1;
  DeviceOnce& once = v4 ? once4 : once1;
  auto kern = v4 ? gla_step_kernel<4> : gla_step_kernel<1>;
  if (!once.done()) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return DIB_LAUNCH_FAILED;
    once.mark();
  }
  const Decays dec = {make_source(hidden, h_kind, h_splits, h_stride), h_row, h_at, a2_t, a2_dtype, a2_bias, tau, R};
  dib_launch(kern, dim3(B, H), dim3(ST), smem, st, src, row_width, dec, state, slot_stride, cu_q_lens, state_slots,
             norm_w, out, out_dtype, H, N, P, q_scale, eps, in_smem);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// Whether a head's state fits in shared memory (dib_gla_step with in_smem 1), whatever the alignment.
int dib_gla_state_fits(int N, int P, int R) {
  const size_t pp = (P + 3) / 4 * 4, np = (N + 3) / 4 * 4;
  const int cols = P % 4 == 0 ? P / 4 : P;             // (the wider of the two forms' shares)
  const size_t shares = cols < ST ? ST / cols : 1;
  return sizeof(float) * (3 * np + (2 + shares) * pp + (size_t)((R + 3) / 4 * 4) + (size_t)N * P) <= MOST_SMEM ? 1 : 0;
}

// The chunked form: B sequences (cu and state_slots point at the first of them; its first token is
// t_first of the step), `tokens` tokens.  proj bfloat16.  With places = tokens / 64 + B: planes 4 * tokens *
// H * N bfloat16; edges places * H * 8 * N floats; sums places * H * N * P floats.
int dib_gla_chunked(const void* proj, long long row_width, const void* hidden, int h_kind, int h_splits, long long h_stride,
                    long long h_row, long long h_at, const void* a2_t, const float* a2_bias, float tau, int R, float* state,
                    long long slot_stride,
                    const int* cu, const int* state_slots, const float* norm_w, void* planes, float* edges, float* sums,
                    void* out, int B, int t_first, int tokens, int H, int N, int P, float q_scale, float eps,
                    cudaStream_t st) {
  if (B == 0 || tokens == 0) return DIB_OK;
  if (H < 1 || H > 65535 || B > 65535 || N < 16 || N > 256 || N % 16 || P < 16 || P > 256 || P % 16 ||
      row_width < 2ll * H * (N + P) || row_width % 8 || slot_stride % 4 || !decays_fit(R, h_row, h_at, tau) ||
      R > MOST_CHUNKED_RANK)
    return DIB_BAD_SIZE;
  if ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(a2_t) | reinterpret_cast<uintptr_t>(a2_bias) | reinterpret_cast<uintptr_t>(state) |
       reinterpret_cast<uintptr_t>(planes) | reinterpret_cast<uintptr_t>(edges) | reinterpret_cast<uintptr_t>(sums) |
       reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(norm_w)) % 16 != 0)
    return DIB_BAD_ALIGN;
  const long long plane = (long long)tokens * H * N;
  const int places = tokens / CH + B;
  static DeviceOnce once;
  if (!once.done()) {
    if (cudaFuncSetAttribute(gla_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return DIB_LAUNCH_FAILED;
    once.mark();
  }
  const Decays dec = {make_source(hidden, h_kind, h_splits, h_stride), h_row, h_at, a2_t, 1, a2_bias, tau, R};
  dib_launch(gla_prepare_kernel, dim3(places, H), dim3(RUNS * N / 2), sizeof(float) * (2 * RUNS * (size_t)N + (size_t)CH * R), st,
             (const __nv_bfloat16*)proj, row_width, dec, cu, B, t_first, (__nv_bfloat16*)planes, plane, edges, H, N, q_scale);
  DIB_CHECK_LAUNCH();
#define DIB_GC(NPT, OUT_NPT, HALVES)                                                                                     \
  return launch_chunks<NPT, OUT_NPT, HALVES>((const __nv_bfloat16*)planes, plane, (const __nv_bfloat16*)proj, row_width, edges, norm_w, \
                            sums, state, slot_stride, cu, state_slots, B, t_first, places, (__nv_bfloat16*)out, H, N, P, eps, st)
  if (P <= 64) DIB_GC(1, 1, 1);
  if (P <= 128) DIB_GC(2, 1, 2);
  if (P <= 192) DIB_GC(3, 2, 2);
  DIB_GC(4, 2, 2);
#undef DIB_GC
}

}  // extern "C"
