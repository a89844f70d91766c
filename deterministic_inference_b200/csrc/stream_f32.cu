// Kernels of models whose residual stream is kept in float32 whatever the engine's
// storage type is: token + learned position embedding, RMSNorm or layer norm of the float32 stream
// (alone, or after adding up to three scaled outputs to it), the scaled sum as a
// tensor, the xIELU activation and the soft cap of the logits.  All arithmetic is float32;
// inputs that come from a matrix product may be its split-k partial products.
#include "source.cuh"

// out[t] = table[ids[t]] + pos_table[positions[t]], float32
__global__ void embed_pos_kernel(const void* table, const void* pos_table, int dtype, const int* ids,
                                 const int* positions, float* out, int T, int W, int V, int P) {
  pdl_prologue();
  const int t = blockIdx.x;
  int id = ids[t], p = positions[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  p = p < 0 ? 0 : (p >= P ? P - 1 : p);
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    out[(long long)t * W + c] =
        __fadd_rn(load_as(table, dtype, (long long)id * W + c), load_as(pos_table, dtype, (long long)p * W + c));
}

// out[t] = table[ids[t]] * scale, float32
__global__ void embed_scale_kernel(const void* table, int dtype, const int* ids, float scale, float* out,
                                   int T, int W, int V) {
  pdl_prologue();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= V ? V - 1 : id);
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    out[(long long)t * W + c] = __fmul_rn(load_as(table, dtype, (long long)id * W + c), scale);
}

// One block per row: residual[row] += x[row] / sqrt(mean(x[row]^2) + eps_x) * wx (+ bias), the
// normed output of the part before added to the stream without being rounded; then, when out is
// given, out[row] = residual[row] / sqrt(mean(residual[row]^2) + eps) * w (w null: out[row] =
// residual[row], not normed).  x null: only the bias is added.  VPT > 0: a thread keeps its VPT elements of the row in registers (W <= VPT * blockDim.x),
// so the row is read once; VPT == 0: any width, the row is read again for every pass.  Both add a
// row's squares in the same order (a thread its own elements in ascending order, then the block's sum).
template <int VPT>
__global__ void stream_normed_add_kernel(float* residual, Source x, const float* wx, float eps_x,
                                         const float* bias, const float* w, void* out, int out_dtype,
                                         int W, float eps) {
  __shared__ float scratch[32];
  pdl_prologue(x.p);
  const long long base = (long long)blockIdx.x * W;
  constexpr int N = VPT > 0 ? VPT : 1;
  float xv[N], rv[N];
  float rx = 0.f;
  if (VPT > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      xv[i] = (x.p != nullptr && c < W) ? source_load(x, base + c) : 0.f;
      rv[i] = c < W ? residual[base + c] : 0.f;
    }
  }
  if (x.p != nullptr) {
    float sx = 0.f;
    if (VPT > 0) {
#pragma unroll
      for (int i = 0; i < N; ++i) sx = __fmaf_rn(xv[i], xv[i], sx);
    } else {
      for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const float v = source_load(x, base + c);
        sx = __fmaf_rn(v, v, sx);
      }
    }
    rx = 1.0f / sqrtf(block_sum(sx, scratch) / (float)W + eps_x);
  }
  float ss = 0.f;
  if (VPT > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) {
        float r = rv[i];
        if (x.p != nullptr) r = __fadd_rn(r, xv[i] * rx * wx[c]);
        if (bias != nullptr) r = __fadd_rn(r, bias[c]);
        residual[base + c] = r;
        rv[i] = r;
        ss = __fmaf_rn(r, r, ss);
      }
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      float r = residual[base + c];
      if (x.p != nullptr) r = __fadd_rn(r, source_load(x, base + c) * rx * wx[c]);
      if (bias != nullptr) r = __fadd_rn(r, bias[c]);
      residual[base + c] = r;
      ss = __fmaf_rn(r, r, ss);
    }
  }
  if (out == nullptr) return;
  if (w == nullptr) {
    // no norm: out is the updated stream itself in out's type
    if (VPT > 0) {
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < W) store_as(out, out_dtype, base + c, rv[i]);
      }
    } else {
      for (int c = threadIdx.x; c < W; c += blockDim.x) store_as(out, out_dtype, base + c, residual[base + c]);
    }
    return;
  }
  const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
  if (VPT > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) store_as(out, out_dtype, base + c, rv[i] * rstd * w[c]);
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x)
      store_as(out, out_dtype, base + c, residual[base + c] * rstd * w[c]);
  }
}

// [gate | up] rows of width 2I -> I: g = min(gate, limit), u = clamp(up, -limit, limit),
// y = g * sigmoid(alpha * g) * (u + 1)
__global__ void limited_gate_kernel(Source gu, float limit, float alpha, void* out, int out_dtype,
                                    int rows, int I) {
  pdl_prologue(gu.p);
  const long long n = (long long)rows * I;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / I, c = i % I;
    const float g = fminf(source_load(gu, r * 2 * I + c), limit);
    const float u = fminf(fmaxf(source_load(gu, r * 2 * I + I + c), -limit), limit);
    store_as(out, out_dtype, i, g * sigmoid_f32(alpha * g) * (u + 1.0f));
  }
}

// One block per row.  TERMS > 0: residual[row] += a0 * x0[row] (+ a1 * x1[row]) first, the
// terms added in their order; then out[row] = residual[row] / sqrt(mean(residual[row]^2) + eps)
// * w.  The sum of squares is taken by a block of a width that depends on W alone, a thread's elements in
// ascending order.  VPT > 0: a thread keeps its VPT elements of the row in registers (W <= VPT *
// blockDim.x); the order of the sums is the same.  AHEAD: splits whose loads are issued together (0 where no
// term is split: fewer registers, more rows in flight).
template <int TERMS, int VPT, int AHEAD>
__global__ void stream_norm_kernel(float* residual, Source x0, float a0, Source x1, float a1,
                                   const float* w, void* out, int out_dtype, int W, float eps) {
  __shared__ float scratch[32];
  pdl_prologue(x0.p, x1.p, residual);
  const long long base = (long long)blockIdx.x * W;
  float ss = 0.f;
  if (VPT > 0) {
    constexpr int N = VPT > 0 ? VPT : 1;
    float r[N], v[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      r[i] = c < W ? residual[base + c] : 0.f;
    }
    if (TERMS >= 1) {
      source_load_strided<N, AHEAD>(x0, base, threadIdx.x, blockDim.x, W, v);
#pragma unroll
      for (int i = 0; i < N; ++i) r[i] = __fmaf_rn(a0, v[i], r[i]);
    }
    if (TERMS >= 2) {
      source_load_strided<N, AHEAD>(x1, base, threadIdx.x, blockDim.x, W, v);
#pragma unroll
      for (int i = 0; i < N; ++i) r[i] = __fmaf_rn(a1, v[i], r[i]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) {
        if (TERMS >= 1) residual[base + c] = r[i];
        ss = __fmaf_rn(r[i], r[i], ss);
      }
    }
    if (out == nullptr) return;
    const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) store_as(out, out_dtype, base + c, r[i] * rstd * w[c]);
    }
    return;
  }
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float r = residual[base + c];
    if (TERMS >= 1) r = __fmaf_rn(a0, source_load(x0, base + c), r);
    if (TERMS >= 2) r = __fmaf_rn(a1, source_load(x1, base + c), r);
    if (TERMS >= 1) residual[base + c] = r;
    ss = __fmaf_rn(r, r, ss);
  }
  const float total = block_sum(ss, scratch);
  const float rstd = 1.0f / sqrtf(total / (float)W + eps);
  if (out == nullptr) return;
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    store_as(out, out_dtype, base + c, residual[base + c] * rstd * w[c]);
}

// One block per row, every term normed before it joins the stream:
// residual[row] += a0 * x0[row] / sqrt(mean(x0[row]^2) + e0) * w0 (+ a1 * x1[row] / sqrt(mean(x1[row]^2) + e1) * w1),
// the terms' sum taken first and then added, nothing rounded below float32; then, when out is given,
// out[row] = residual[row] / sqrt(mean(residual[row]^2) + eps) * w.  A term without a weight (w0 null)
// joins as a0 * x0.  The block's width depends on W alone.
__global__ void stream_norm_normed_terms_kernel(float* residual, int terms, Source x0, float a0, const float* w0,
                                                float e0, Source x1, float a1, const float* w1, float e1,
                                                const float* w, void* out, int out_dtype, int W, float eps) {
  __shared__ float scratch[32];
  pdl_prologue(x0.p, x1.p);
  const long long base = (long long)blockIdx.x * W;
  float r0 = 1.f, r1 = 1.f;
  if (w0 != nullptr) {
    float s = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = source_load(x0, base + c);
      s = __fmaf_rn(v, v, s);
    }
    r0 = 1.0f / sqrtf(block_sum(s, scratch) / (float)W + e0);
  }
  if (terms >= 2 && w1 != nullptr) {
    float s = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = source_load(x1, base + c);
      s = __fmaf_rn(v, v, s);
    }
    r1 = 1.0f / sqrtf(block_sum(s, scratch) / (float)W + e1);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = source_load(x0, base + c);
    if (w0 != nullptr) v = v * r0 * w0[c];
    float sum = __fmul_rn(a0, v);
    if (terms >= 2) {
      float u = source_load(x1, base + c);
      if (w1 != nullptr) u = u * r1 * w1[c];
      sum = __fmaf_rn(a1, u, sum);
    }
    const float r = __fadd_rn(residual[base + c], sum);
    residual[base + c] = r;
    ss = __fmaf_rn(r, r, ss);
  }
  if (out == nullptr) return;
  const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    store_as(out, out_dtype, base + c, residual[base + c] * rstd * w[c]);
}

// One block per row: stream[row] += sum_k a_k * n_k(x_k[row] + bias_k), the terms' sum taken first (in
// their order) and then added, nothing rounded below float32; n_k(v) = v / sqrt(mean(v^2) + e_k) * w_k
// where the term has a weight, v where it has none.  Then, when out is given, out[row] = the stream
// itself (norm_kind 0), its RMS norm stream / sqrt(mean(stream^2) + eps) * w (1), or its layer norm
// (stream - mean) / sqrt(mean((stream - mean)^2) + eps) * w (2).
// The block's width depends on W alone, and a sum over a row is a thread's own elements in ascending order,
// then the block's; VPT > 0 keeps a thread's elements in registers, VPT 0 reads them again.
struct StreamTerm {
  Source x;
  float a;
  const float* bias;
  const float* w;
  float eps;
};
constexpr int STREAM_TERMS = 3;
struct StreamTerms {
  StreamTerm t[STREAM_TERMS];
  int n;
};

// block_sum of several values at once (each in block_sum's order); scratch holds 32 floats a value
__device__ __forceinline__ void block_sums(float (&v)[STREAM_TERMS], float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int k = 0; k < STREAM_TERMS; ++k) v[k] = warp_sum(v[k]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int k = 0; k < STREAM_TERMS; ++k) scratch[k * 32 + warp] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < STREAM_TERMS; ++k) {
    float total = 0.f;
    for (int w = 0; w < nwarps; ++w) total += scratch[k * 32 + w];
    v[k] = total;
  }
}

template <int VPT, int AHEAD>
__global__ void stream_terms_kernel(float* stream, StreamTerms terms, int norm_kind, const float* w, void* out,
                                    int out_dtype, int W, float eps) {
  __shared__ float scratch[32 * STREAM_TERMS];
  pdl_prologue(stream, terms.t[0].x.p, terms.t[1].x.p, terms.t[2].x.p);
  const long long base = (long long)blockIdx.x * W;
  const float width = (float)W;
  if (VPT > 0) {
    constexpr int N = VPT > 0 ? VPT : 1;
    float r[N], v[STREAM_TERMS][N], f[STREAM_TERMS];
    // every term's loads before the first is used
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      r[i] = c < W ? stream[base + c] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < STREAM_TERMS; ++k)
      if (k < terms.n) source_load_strided<N, AHEAD>(terms.t[k].x, base, threadIdx.x, blockDim.x, W, v[k]);
    bool any = false;
#pragma unroll
    for (int k = 0; k < STREAM_TERMS; ++k) {
      f[k] = 0.f;                           // a normed term's squares, then its factor
      if (k >= terms.n) continue;
      const StreamTerm& t = terms.t[k];
      if (t.bias != nullptr) {
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < W) v[k][i] = __fadd_rn(v[k][i], t.bias[c]);
        }
      }
      if (t.w != nullptr) {
        any = true;
#pragma unroll
        for (int i = 0; i < N; ++i) f[k] = __fmaf_rn(v[k][i], v[k][i], f[k]);
      }
    }
    if (any) {
      block_sums(f, scratch);
#pragma unroll
      for (int k = 0; k < STREAM_TERMS; ++k) {
        if (k >= terms.n || terms.t[k].w == nullptr) continue;
        const StreamTerm& t = terms.t[k];
        const float rs = 1.0f / sqrtf(f[k] / width + t.eps);
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int c = threadIdx.x + i * blockDim.x;
          if (c < W) v[k][i] = __fmul_rn(__fmul_rn(v[k][i], rs), t.w[c]);
        }
      }
    }
    float sum[N];
#pragma unroll
    for (int i = 0; i < N; ++i) sum[i] = 0.f;
#pragma unroll
    for (int k = 0; k < STREAM_TERMS; ++k)
      if (k < terms.n) {
#pragma unroll
        for (int i = 0; i < N; ++i) sum[i] = __fmaf_rn(terms.t[k].a, v[k][i], sum[i]);
      }
    float first = 0.f;                      // the row's sum (layer norm) or its squares' (RMS norm)
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) {
        if (terms.n > 0) {
          r[i] = __fadd_rn(r[i], sum[i]);
          stream[base + c] = r[i];
        }
        first = norm_kind == 2 ? __fadd_rn(first, r[i]) : __fmaf_rn(r[i], r[i], first);
      }
    }
    if (out == nullptr) return;
    float mean = 0.f, rstd = 1.f;
    if (norm_kind == 1) rstd = 1.0f / sqrtf(block_sum(first, scratch) / width + eps);
    if (norm_kind == 2) {
      mean = block_sum(first, scratch) / width;
      float sq = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < W) {
          const float d = __fsub_rn(r[i], mean);
          sq = __fmaf_rn(d, d, sq);
        }
      }
      rstd = 1.0f / sqrtf(block_sum(sq, scratch) / width + eps);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < W) store_as(out, out_dtype, base + c, norm_kind == 0 ? r[i] : __fsub_rn(r[i], mean) * rstd * w[c]);
    }
    return;
  }
  float f[STREAM_TERMS];
#pragma unroll
  for (int k = 0; k < STREAM_TERMS; ++k) {
    f[k] = 1.f;
    if (k >= terms.n || terms.t[k].w == nullptr) continue;
    const StreamTerm& t = terms.t[k];
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      float v = source_load(t.x, base + c);
      if (t.bias != nullptr) v = __fadd_rn(v, t.bias[c]);
      ss = __fmaf_rn(v, v, ss);
    }
    f[k] = 1.0f / sqrtf(block_sum(ss, scratch) / width + t.eps);
  }
  float first = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float r = stream[base + c], sum = 0.f;
#pragma unroll
    for (int k = 0; k < STREAM_TERMS; ++k) {
      if (k >= terms.n) break;
      const StreamTerm& t = terms.t[k];
      float v = source_load(t.x, base + c);
      if (t.bias != nullptr) v = __fadd_rn(v, t.bias[c]);
      if (t.w != nullptr) v = __fmul_rn(__fmul_rn(v, f[k]), t.w[c]);
      sum = __fmaf_rn(t.a, v, sum);
    }
    if (terms.n > 0) {
      r = __fadd_rn(r, sum);
      stream[base + c] = r;
    }
    first = norm_kind == 2 ? __fadd_rn(first, r) : __fmaf_rn(r, r, first);
  }
  if (out == nullptr) return;
  float mean = 0.f, rstd = 1.f;
  if (norm_kind == 1) rstd = 1.0f / sqrtf(block_sum(first, scratch) / width + eps);
  if (norm_kind == 2) {
    mean = block_sum(first, scratch) / width;
    float sq = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float d = __fsub_rn(stream[base + c], mean);
      sq = __fmaf_rn(d, d, sq);
    }
    rstd = 1.0f / sqrtf(block_sum(sq, scratch) / width + eps);
  }
  for (int c = threadIdx.x; c < W; c += blockDim.x)
    store_as(out, out_dtype, base + c, norm_kind == 0 ? stream[base + c] : __fsub_rn(stream[base + c], mean) * rstd * w[c]);
}

// out = a0 * x0 (+ a1 * x1), float32
__global__ void weighted_sum_kernel(Source x0, float a0, Source x1, float a1, int terms, float* out,
                                    long long n) {
  pdl_prologue();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x) {
    float r = __fmul_rn(a0, source_load(x0, i));
    if (terms >= 2) r = __fmaf_rn(a1, source_load(x1, i), r);
    out[i] = r;
  }
}

// xIELU: z > 0: ap z^2 + z / 2;  z <= 0: an (exp(z) - 1 - z) + z / 2
__global__ void xielu_kernel(Source z, float ap, float an, void* out, int out_dtype, long long n) {
  pdl_prologue();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x) {
    const float x = source_load(z, i);
    const float y = x > 0.f ? __fmaf_rn(__fmul_rn(ap, x), x, 0.5f * x)
                            : __fmaf_rn(an, expm1f(x) - x, 0.5f * x);
    store_as(out, out_dtype, i, y);
  }
}

// out = max(z, 0)^2
__global__ void squared_relu_kernel(Source z, void* out, int out_dtype, long long n) {
  pdl_prologue(z.p);
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x) {
    const float x = fmaxf(source_load(z, i), 0.f);
    store_as(out, out_dtype, i, x * x);
  }
}

// x = cap * tanh(x / cap), in place
__global__ void softcap_kernel(float* x, float cap, long long n) {
  pdl_prologue();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

// x = x * a, in place
__global__ void scale_kernel(float* x, float a, long long n) {
  pdl_prologue();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n;
       i += (long long)gridDim.x * blockDim.x)
    x[i] = __fmul_rn(x[i], a);
}

static inline int flat_grid(long long n, int block) {
  long long g = (n + block - 1) / block;
  return (int)(g > 148 * 16 ? 148 * 16 : (g < 1 ? 1 : g));
}

extern "C" {

int dib_embed_pos(const void* table, const void* pos_table, int dtype, const int* ids,
                  const int* positions, float* out, int T, int W, int V, int P, cudaStream_t st) {
  if (T == 0) return DIB_OK;
  if (dtype != 0 && dtype != 1) return DIB_BAD_DTYPE;
  if (W < 1 || V < 1 || P < 1) return DIB_BAD_SIZE;
  dib_launch(embed_pos_kernel, dim3(T), dim3(W >= 1024 ? 256 : 128), 0, st, table, pos_table, dtype, ids,
             positions, out, T, W, V, P);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_embed_scale(const void* table, int dtype, const int* ids, float scale, float* out, int T, int W,
                    int V, cudaStream_t st) {
  if (T == 0) return DIB_OK;
  if (dtype != 0 && dtype != 1) return DIB_BAD_DTYPE;
  if (W < 1 || V < 1) return DIB_BAD_SIZE;
  dib_launch(embed_scale_kernel, dim3(T), dim3(W >= 1024 ? 256 : 128), 0, st, table, dtype, ids, scale, out,
             T, W, V);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// x null: no normed term; bias null: none; out null: the stream is updated and nothing is normed.
int dib_stream_normed_add(float* residual, const void* x, int kind, int splits, long long stride,
                          const float* wx, float eps_x, const float* bias, const float* w, void* out,
                          int out_dtype, int rows, int W, float eps, cudaStream_t st) {
  if (rows == 0) return DIB_OK;
  if (W < 1) return DIB_BAD_SIZE;
  if (out != nullptr && out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  const dim3 grid(rows), block(W >= 2048 ? 512 : (W >= 512 ? 256 : 128));
  const Source src = make_source(x, kind, splits, stride);
  const int per_thread = (W + (int)block.x - 1) / (int)block.x;
#define DIB_SNA(VPT) \
  dib_launch(stream_normed_add_kernel<VPT>, grid, block, 0, st, residual, src, wx, eps_x, bias, w, out, out_dtype, W, eps)
  if (per_thread <= 4) DIB_SNA(4);
  else if (per_thread <= 8) DIB_SNA(8);
  else if (per_thread <= 16) DIB_SNA(16);
  else DIB_SNA(0);
#undef DIB_SNA
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_limited_gate(const void* gu, int kind, int splits, long long stride, float limit, float alpha,
                     void* out, int out_dtype, int rows, int I, cudaStream_t st) {
  if (rows == 0) return DIB_OK;
  if (I < 1) return DIB_BAD_SIZE;
  if (out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  dib_launch(limited_gate_kernel, dim3(flat_grid((long long)rows * I, 256)), dim3(256), 0, st,
             make_source(gu, kind, splits, stride), limit, alpha, out, out_dtype, rows, I);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// terms 0: norm of the stream alone.  x kinds: 0 float32 (splits >= 1), 1 bfloat16.
// out may be null (terms > 0): the stream is updated and nothing is normed.
int dib_stream_norm(float* residual, int terms, const void* x0, int kind0, int splits0, long long stride0,
                    float a0, const void* x1, int kind1, int splits1, long long stride1, float a1,
                    const float* w, void* out, int out_dtype, int rows, int W, float eps,
                    cudaStream_t st) {
  if (rows == 0) return DIB_OK;
  if (W < 1 || terms < 0 || terms > 2) return DIB_BAD_SIZE;
  if (out != nullptr && out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  const Source s0 = make_source(x0, kind0, splits0, stride0), s1 = make_source(x1, kind1, splits1, stride1);
  const dim3 grid(rows), block(W >= 2048 ? 512 : (W >= 512 ? 256 : 128));
  const int per_thread = (W + (int)block.x - 1) / (int)block.x;
  const bool split = (terms >= 1 && s0.splits > 1) || (terms >= 2 && s1.splits > 1);
#define DIB_SN(TERMS, VPT, AHEAD) \
  dib_launch(stream_norm_kernel<TERMS, VPT, AHEAD>, grid, block, 0, st, residual, s0, a0, s1, a1, w, out, out_dtype, W, eps)
  // (wide rows without a split: the form that reads again has a third of the registers, so more rows in flight)
#define DIB_SNV(TERMS, A4, A8)                    \
  if (per_thread <= 4) DIB_SN(TERMS, 4, A4);      \
  else if (A8 > 0 && per_thread <= 8) DIB_SN(TERMS, 8, (A8 > 0 ? A8 : 1)); \
  else DIB_SN(TERMS, 0, 0)
  if (terms == 0) { DIB_SNV(0, 0, 0); }
  else if (terms == 1 && split) { DIB_SNV(1, 4, 2); }
  else if (terms == 1) { DIB_SNV(1, 0, 0); }
  else if (split) { DIB_SNV(2, 4, 2); }
  else { DIB_SNV(2, 0, 0); }
#undef DIB_SNV
#undef DIB_SN
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// Terms that are normed on their way into the stream (w0 / w1 null: that term joins as it is).
// out null: the stream is updated and nothing is normed.
int dib_stream_norm_normed_terms(float* residual, int terms, const void* x0, int kind0, int splits0, long long stride0,
                                 float a0, const float* w0, float e0, const void* x1, int kind1, int splits1,
                                 long long stride1, float a1, const float* w1, float e1, const float* w, void* out,
                                 int out_dtype, int rows, int W, float eps, cudaStream_t st) {
  if (rows == 0) return DIB_OK;
  if (W < 1 || terms < 1 || terms > 2) return DIB_BAD_SIZE;
  if (out != nullptr && (w == nullptr || (out_dtype != 0 && out_dtype != 1))) return DIB_BAD_DTYPE;
  const Source s0 = make_source(x0, kind0, splits0, stride0), s1 = make_source(x1, kind1, splits1, stride1);
  const dim3 grid(rows), block(W >= 2048 ? 512 : (W >= 512 ? 256 : 128));
  dib_launch(stream_norm_normed_terms_kernel, grid, block, 0, st, residual, terms, s0, a0, w0, e0, s1, a1, w1, e1, w,
             out, out_dtype, W, eps);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

// Up to three terms (see stream_terms_kernel).  x null with terms == 0.  out null: the stream is updated
// only.  norm_kind 0: out is the stream in out's type; 1: its RMS norm; 2: its layer norm.
int dib_stream_terms(float* stream, int terms, const void* x0, int kind0, int splits0, long long stride0, float a0,
                     const float* b0, const float* w0, float e0, const void* x1, int kind1, int splits1,
                     long long stride1, float a1, const float* b1, const float* w1, float e1, const void* x2, int kind2,
                     int splits2, long long stride2, float a2, const float* b2, const float* w2, float e2, int norm_kind,
                     const float* w, void* out, int out_dtype, int rows, int W, float eps, cudaStream_t st) {
  if (rows == 0) return DIB_OK;
  if (W < 1 || terms < 0 || terms > STREAM_TERMS || norm_kind < 0 || norm_kind > 2) return DIB_BAD_SIZE;
  if (out != nullptr && ((norm_kind > 0 && w == nullptr) || (out_dtype != 0 && out_dtype != 1))) return DIB_BAD_DTYPE;
  StreamTerms t;
  t.n = terms;
  t.t[0] = {make_source(x0, kind0, splits0, stride0), a0, b0, w0, e0};
  t.t[1] = {make_source(x1, kind1, splits1, stride1), a1, b1, w1, e1};
  t.t[2] = {make_source(x2, kind2, splits2, stride2), a2, b2, w2, e2};
  bool split = false;
  for (int k = 0; k < terms; ++k) split = split || t.t[k].x.splits > 1;
  const dim3 grid(rows), block(W >= 2048 ? 512 : (W >= 512 ? 256 : 128));
  const int per_thread = (W + (int)block.x - 1) / (int)block.x;
#define DIB_ST(VPT, AHEAD) dib_launch(stream_terms_kernel<VPT, AHEAD>, grid, block, 0, st, stream, t, norm_kind, w, out, out_dtype, W, eps)
  if (per_thread <= 4 && split) DIB_ST(4, 4);
  else if (per_thread <= 4) DIB_ST(4, 0);
  else if (per_thread <= 8 && split) DIB_ST(8, 2);
  else if (per_thread <= 8) DIB_ST(8, 0);
  else DIB_ST(0, 0);
#undef DIB_ST
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_weighted_sum(int terms, const void* x0, int kind0, int splits0, long long stride0, float a0,
                     const void* x1, int kind1, int splits1, long long stride1, float a1, float* out,
                     long long n, cudaStream_t st) {
  if (n == 0) return DIB_OK;
  if (terms < 1 || terms > 2) return DIB_BAD_SIZE;
  dib_launch(weighted_sum_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, st,
             make_source(x0, kind0, splits0, stride0), a0, make_source(x1, kind1, splits1, stride1), a1, terms,
             out, n);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_xielu(const void* z, int kind, int splits, long long stride, float ap, float an, void* out,
              int out_dtype, long long n, cudaStream_t st) {
  if (n == 0) return DIB_OK;
  if (out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  dib_launch(xielu_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, st, make_source(z, kind, splits, stride), ap,
             an, out, out_dtype, n);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_squared_relu(const void* z, int kind, int splits, long long stride, void* out, int out_dtype, long long n,
                     cudaStream_t st) {
  if (n == 0) return DIB_OK;
  if (out_dtype != 0 && out_dtype != 1) return DIB_BAD_DTYPE;
  dib_launch(squared_relu_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, st, make_source(z, kind, splits, stride), out,
             out_dtype, n);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_scale(float* x, float a, long long n, cudaStream_t st) {
  if (n == 0) return DIB_OK;
  dib_launch(scale_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, st, x, a, n);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

int dib_softcap(float* x, float cap, long long n, cudaStream_t st) {
  if (n == 0) return DIB_OK;
  dib_launch(softcap_kernel, dim3(flat_grid(n, 256)), dim3(256), 0, st, x, cap, n);
  DIB_CHECK_LAUNCH();
  return DIB_OK;
}

}  // extern "C"
