// Elementwise steps of a block whose sublayers read ONE norm of the residual row and whose results are
// scaled on their way into the float32 residual stream x:
//
// scaled_sum:       x <- x + mult * (y1 + y2)     (y2 may be absent); optionally also x in the compute
//                   type, for a product that reads the new row.
// gated_table_rows: g[t][j] = gelu_tanh(s[t][j]) * table[token[t]][offset + j]   (the per-layer part of a
//                   second embedding table, gated by a projection of the row), compute type out.
// norm_scaled_add:  x <- x + mult * y / sqrt(mean(y^2) + eps) * w    (an RMS norm of the branch's result,
//                   not of x); where rows lie on 16-byte borders it may go on to the norm that follows,
//                   out <- x / sqrt(mean(x^2) + eps2) * w2 in the compute type, without reading x again.
// All arithmetic is float32; one block per token for the norm, with a fixed reduction tree.
#include "common.cuh"
#include "partials.cuh"

template <typename T>
__global__ void __launch_bounds__(256)
scaled_sum_kernel(float* __restrict__ x, const float* __restrict__ y1, const float* __restrict__ y2, float mult,
                  T* __restrict__ xc, long long n) {
  pdl_launch();      // the product that follows may fetch its weights meanwhile
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float s = y1[i];
  if (y2 != nullptr) s += y2[i];
  const float v = fmaf(mult, s, x[i]);
  x[i] = v;
  if (xc != nullptr) xc[i] = from_f32<T>(v);
}

// The same for a few tokens whose sublayers left their last products as partials (either may instead
// be a plain buffer, the second may be absent): a row is shared out between gridDim.y blocks.
template <typename T>
__global__ void __launch_bounds__(256)
scaled_sum_partials_kernel(float* __restrict__ x, int E, const float* __restrict__ y1, const float* __restrict__ y2, float mult,
                           T* __restrict__ xc, const PartialLayout L1, const PartialLayout L2) {
  pdl_launch();      // the product that follows may fetch its weights meanwhile
  __shared__ PartialTable tab1, tab2;
  if (L1.ws != nullptr) build_partial_table(L1, tab1);
  if (L2.ws != nullptr) build_partial_table(L2, tab2);
  const int t = blockIdx.x;
  const int per = (E + gridDim.y - 1) / gridDim.y;
  const int lo = blockIdx.y * per, hi = min(E, lo + per);
  for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) {
    float s = L1.ws != nullptr ? partial_sum(L1, tab1, t, i) : y1[(size_t)t * E + i];
    if (L2.ws != nullptr) s += partial_sum(L2, tab2, t, i);
    else if (y2 != nullptr) s += y2[(size_t)t * E + i];
    const float v = fmaf(mult, s, x[(size_t)t * E + i]);
    x[(size_t)t * E + i] = v;
    if (xc != nullptr) xc[(size_t)t * E + i] = from_f32<T>(v);
  }
}

__device__ __forceinline__ float pb_gelu_tanh(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void __launch_bounds__(256)
gated_table_rows_kernel(const float* __restrict__ s, int lds, const T* __restrict__ table, int ldt, int n_vocab,
                        const int* __restrict__ token_ids, int offset, int dim, T* __restrict__ out, int ldo, int n_tokens,
                        int* __restrict__ err, const PartialLayout L) {
  pdl_launch();      // the product that follows may fetch its weights meanwhile
  __shared__ PartialTable tab;
  if (L.ws != nullptr) build_partial_table(L, tab);
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)n_tokens * dim) return;
  const int t = (int)(i / dim), j = (int)(i % dim);
  const int tok = token_ids[t];
  if (tok < 0 || tok >= n_vocab) {
    atomicExch(err, 1);
    return;
  }
  const float e = to_f32<T>(table[(size_t)tok * ldt + offset + j]);
  const float z = L.ws != nullptr ? partial_sum(L, tab, t, j) : s[(size_t)t * lds + j];
  out[(size_t)t * ldo + j] = from_f32<T>(pb_gelu_tanh(z) * e);
}

// y comes from a plain buffer or from partials; `hold`: the row is kept in shared memory (E floats)
// between the sum of squares and the update (always with partials; a wider row is read twice).
__global__ void __launch_bounds__(256)
norm_scaled_add_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, float mult, float eps,
                       int E, const PartialLayout L, int hold) {
  pdl_launch();      // the product that follows may fetch its weights meanwhile
  extern __shared__ float pb_row[];
  __shared__ float red[32];
  __shared__ PartialTable tab;
  if (L.ws != nullptr) build_partial_table(L, tab);
  const int t = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += blockDim.x) {
    const float v = L.ws != nullptr ? partial_sum(L, tab, t, i) : y[(size_t)t * E + i];
    if (hold) pb_row[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)E + eps);
  for (int i = threadIdx.x; i < E; i += blockDim.x) {
    const float v = hold ? pb_row[i] : y[(size_t)t * E + i];
    x[(size_t)t * E + i] = fmaf(mult, v * r * w[i], x[(size_t)t * E + i]);
  }
}

// Rows of E = 4 * (pieces) elements, at most PB_PIECES pieces a thread, kept in registers from the read to the last store.
constexpr int PB_PIECES = 4;
template <typename T>
__global__ void __launch_bounds__(1024)
norm_scaled_add_vec_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, float mult, float eps,
                           int E, const PartialLayout L, const float* __restrict__ w2, float eps2, T* __restrict__ out) {
  pdl_launch();      // the product that follows may fetch its weights meanwhile
  __shared__ float red[32];
  __shared__ PartialTable tab;
  if (L.ws != nullptr) build_partial_table(L, tab);
  const int t = blockIdx.x, n4 = E >> 2;
  float4 v[PB_PIECES], xo[PB_PIECES];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < PB_PIECES; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    v[k] = xo[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < n4) {
      xo[k] = *reinterpret_cast<const float4*>(x + (size_t)t * E + 4 * i);
      if (L.ws != nullptr) {
        v[k] = make_float4(partial_sum(L, tab, t, 4 * i), partial_sum(L, tab, t, 4 * i + 1), partial_sum(L, tab, t, 4 * i + 2),
                           partial_sum(L, tab, t, 4 * i + 3));
      } else {
        v[k] = *reinterpret_cast<const float4*>(y + (size_t)t * E + 4 * i);
      }
    }
    ss = fmaf(v[k].x, v[k].x, ss);
    ss = fmaf(v[k].y, v[k].y, ss);
    ss = fmaf(v[k].z, v[k].z, ss);
    ss = fmaf(v[k].w, v[k].w, ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)E + eps);
  float s2 = 0.f;
#pragma unroll
  for (int k = 0; k < PB_PIECES; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= n4) continue;
    const float4 g = *reinterpret_cast<const float4*>(w + 4 * i);
    xo[k].x = fmaf(mult, v[k].x * r * g.x, xo[k].x);
    xo[k].y = fmaf(mult, v[k].y * r * g.y, xo[k].y);
    xo[k].z = fmaf(mult, v[k].z * r * g.z, xo[k].z);
    xo[k].w = fmaf(mult, v[k].w * r * g.w, xo[k].w);
    *reinterpret_cast<float4*>(x + (size_t)t * E + 4 * i) = xo[k];
    s2 = fmaf(xo[k].x, xo[k].x, s2);
    s2 = fmaf(xo[k].y, xo[k].y, s2);
    s2 = fmaf(xo[k].z, xo[k].z, s2);
    s2 = fmaf(xo[k].w, xo[k].w, s2);
  }
  if (out == nullptr) return;
  s2 = block_sum(s2, red);
  const float r2 = 1.f / sqrtf(s2 / (float)E + eps2);
#pragma unroll
  for (int k = 0; k < PB_PIECES; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= n4) continue;
    const float4 g = *reinterpret_cast<const float4*>(w2 + 4 * i);
    const float a = xo[k].x * r2 * g.x, b = xo[k].y * r2 * g.y, c = xo[k].z * r2 * g.z, d = xo[k].w * r2 * g.w;
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(out + (size_t)t * E + 4 * i) = make_float4(a, b, c, d);
    } else {
      uint2 pk;
      pk.x = pack2<T>(a, b);
      pk.y = pack2<T>(c, d);
      *reinterpret_cast<uint2*>(out + (size_t)t * E + 4 * i) = pk;
    }
  }
}

static int pb_layout(const float* partials, const int* layout, int n_tokens, int width, PartialLayout* L) {
  *L = PartialLayout{nullptr, 0, 0, 0, 0};
  if (partials == nullptr) return 0;
  if (int r = partial_make_layout(partials, layout, L)) return r;
  FERRUM_CHECK_ARG(width <= L->tiles * 128 && n_tokens <= L->acc_cols, "the partials do not cover the rows");
  return 0;
}

// y1 / y2: float32 [n_tokens, E] buffers, or null where partials1 / partials2 (with their layouts) stand in.
FERRUM_API int ferrum_scaled_sum(float* x, const float* y1, const float* y2, float mult, void* xc, int dtype, int n_tokens,
                                 int E, const float* partials1, const int* layout1, const float* partials2,
                                 const int* layout2, cudaStream_t stream) {
  FERRUM_CHECK_ARG(y1 != nullptr || partials1 != nullptr, "scaled_sum: no first term");
  if (n_tokens == 0) return 0;
  if (partials1 != nullptr || partials2 != nullptr) {
    PartialLayout L1, L2;
    if (int r = pb_layout(partials1, layout1, n_tokens, E, &L1)) return r;
    if (int r = pb_layout(partials2, layout2, n_tokens, E, &L2)) return r;
    const int slices = n_tokens <= 64 ? max(1, min(16, E / 256)) : 1;
    FERRUM_DISPATCH_DTYPE(dtype, T, (scaled_sum_partials_kernel<T><<<dim3(n_tokens, slices), 256, 0, stream>>>(
        x, E, y1, y2, mult, (T*)xc, L1, L2)));
    FERRUM_CHECK_LAUNCH("scaled_sum_partials");
    return 0;
  }
  const long long n = (long long)n_tokens * E;
  FERRUM_DISPATCH_DTYPE(dtype, T, (scaled_sum_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, stream>>>(x, y1, y2, mult, (T*)xc, n)));
  FERRUM_CHECK_LAUNCH("scaled_sum");
  return 0;
}

FERRUM_API int ferrum_gated_table_rows(const float* s, int lds, const void* table, int ldt, int n_vocab, const int* token_ids,
                                       int offset, int dim, void* out, int ldo, int dtype, int n_tokens, int* err,
                                       const float* partials, const int* layout, cudaStream_t stream) {
  FERRUM_CHECK_ARG(dim > 0 && offset >= 0 && offset + dim <= ldt, "gated_table_rows: columns %d..%d are outside a row of %d",
                   offset, offset + dim, ldt);
  FERRUM_CHECK_ARG(s != nullptr || partials != nullptr, "gated_table_rows: no gate input");
  if (n_tokens == 0) return 0;
  PartialLayout L;
  if (int r = pb_layout(partials, layout, n_tokens, dim, &L)) return r;
  const long long n = (long long)n_tokens * dim;
  FERRUM_DISPATCH_DTYPE(dtype, T, (gated_table_rows_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, stream>>>(
      s, lds, (const T*)table, ldt, n_vocab, token_ids, offset, dim, (T*)out, ldo, n_tokens, err, L)));
  FERRUM_CHECK_LAUNCH("gated_table_rows");
  return 0;
}

constexpr int PB_MAX_ROW = 11264;      // floats of a row that the norm holds in shared memory

FERRUM_API int ferrum_norm_scaled_add_max_width() { return PB_MAX_ROW; }

static bool pb_vec(const float* x, const float* y, const float* w, int E) {
  return E % 4 == 0 && E <= 4096 * PB_PIECES && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)w) & 15) == 0;
}
// Whether norm_scaled_add can go on to a norm of the new rows (w2 and out as below).
FERRUM_API int ferrum_norm_scaled_add_can_norm(const float* x, const float* y, const float* w, int E, const float* w2, const void* out) {
  return pb_vec(x, y, w, E) && (((uintptr_t)w2 | (uintptr_t)out) & 15) == 0;
}

// out (may be null): [n_tokens][E] in the type `dtype`, the norm of the new rows with weight w2 and eps2.
FERRUM_API int ferrum_norm_scaled_add(float* x, const float* y, const float* w, float mult, float eps, int n_tokens, int E,
                                      const float* partials, const int* layout, const float* w2, float eps2, void* out, int dtype,
                                      cudaStream_t stream) {
  FERRUM_CHECK_ARG(y != nullptr || partials != nullptr, "norm_scaled_add: no input");
  FERRUM_CHECK_ARG(E > 0 && (partials == nullptr || E <= PB_MAX_ROW), "norm_scaled_add: a row of %d from partials is wider than %d",
                   E, PB_MAX_ROW);
  if (n_tokens == 0) return 0;
  PartialLayout L;
  if (int r = pb_layout(partials, layout, n_tokens, E, &L)) return r;
  if (pb_vec(x, y, w, E)) {
    FERRUM_CHECK_ARG(out == nullptr || (w2 != nullptr && (((uintptr_t)w2 | (uintptr_t)out) & 15) == 0), "norm_scaled_add: the norm's operands are unaligned");
    // a few rows: a piece a thread; many: four, so that several rows share an SM
    const int n4 = E / 4, most = n_tokens <= 64 ? n4 : (n4 + PB_PIECES - 1) / PB_PIECES;
    const int threads = min(1024, max((most + 31) / 32 * 32, (n4 + 32 * PB_PIECES - 1) / (32 * PB_PIECES) * 32));
    FERRUM_DISPATCH_DTYPE(dtype, T, (norm_scaled_add_vec_kernel<T><<<n_tokens, threads, 0, stream>>>(x, y, w, mult, eps, E, L, w2, eps2, (T*)out)));
    FERRUM_CHECK_LAUNCH("norm_scaled_add");
    return 0;
  }
  FERRUM_CHECK_ARG(out == nullptr, "norm_scaled_add: rows that are not on 16-byte borders take no norm after the sum");
  const int hold = E <= PB_MAX_ROW;
  norm_scaled_add_kernel<<<n_tokens, 256, hold ? (size_t)E * 4 : 0, stream>>>(x, y, w, mult, eps, E, L, hold);
  FERRUM_CHECK_LAUNCH("norm_scaled_add");
  return 0;
}
