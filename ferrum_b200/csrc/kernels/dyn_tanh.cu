// Kernels of designs whose norm is a dynamic tanh and whose units are not gated.
//
// dyn_tanh: out[r, i] = tanh(alpha * x[src(r), i]) * w[i] + b[i] with src(r) = rows ? rows[r] : r.  No
// statistics of the row enter, so a row may be cut anywhere.  Whatever sum into the residual row is still
// open is made on the way (x is then updated in place): a product left in partials (partials.cuh), or the
// weighted sum of a token's expert rows (moe.cu).
//
// embedding_bigram: out[t] = scale * table[id] + pairs[row] with row = (previous id * mul_prev + id * mul_cur)
// mod n_pairs, and row n_pairs for a sequence's first token.  The previous id of a portion's first token is the
// request's state (one integer per slot).
//
// unit_act: out = act(x) in the compute type for the middle of an ungated feed-forward, from float32 rows or
// from a product left in partials.
#include "common.cuh"
#include "partials.cuh"

// ================================================================= dynamic tanh
struct ExpertRows {
  const float* rows;         // null: none
  int ld;
  const int* row_of;         // [T * top]
  const float* weight_of;    // [T * top] or null
  int top;
};
constexpr int DT_MAX_TOP = 8;
constexpr int DT_THREADS = 256;

template <typename TOut> __device__ __forceinline__ void dt_store4(TOut* p, float4 v) {
  uint2 pk;
  pk.x = pack2<TOut>(v.x, v.y);
  pk.y = pack2<TOut>(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = pk;
}
template <> __device__ __forceinline__ void dt_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }

// A thread owns one column and one row: few rows, and rows that are not 16-byte multiples.
template <typename TOut>
__global__ void __launch_bounds__(DT_THREADS)
dyn_tanh_kernel(float* __restrict__ x, const float* __restrict__ alpha, const float* __restrict__ w, const float* __restrict__ b,
                TOut* __restrict__ out, const int* __restrict__ rows, int E, const PartialLayout L, const ExpertRows X) {
  __shared__ PartialTable tab;
  if (L.ws != nullptr) build_partial_table(L, tab);
  const int r = blockIdx.x, i = blockIdx.y * DT_THREADS + threadIdx.x;
  pdl_launch();
  // (parameters are not written by any kernel of the stream: they may be fetched before the wait)
  const float a = *alpha, wi = i < E ? w[i] : 0.f, bi = i < E ? b[i] : 0.f;
  pdl_wait();
  if (i >= E) return;
  const int src = rows ? rows[r] : r;
  float* const p = x + (size_t)src * E + i;
  float v = *p;
  if (L.ws != nullptr) {
    v += partial_sum(L, tab, src, i);
    *p = v;
  } else if (X.rows != nullptr) {
    float e[DT_MAX_TOP];
#pragma unroll
    for (int j = 0; j < DT_MAX_TOP; ++j) {
      e[j] = 0.f;
      if (j < X.top) {
        const int row = X.row_of[(size_t)src * X.top + j];
        if (row >= 0) e[j] = X.rows[(size_t)row * X.ld + i] * (X.weight_of != nullptr ? X.weight_of[(size_t)src * X.top + j] : 1.f);
      }
    }
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < DT_MAX_TOP; ++j) s += e[j];
    v += s;
    *p = v;
  }
  out[(size_t)r * E + i] = from_f32<TOut>(tanhf(a * v) * wi + bi);
}

// Many rows: a thread keeps w and b of four columns and walks every gridDim.x-th row.
template <typename TOut, bool EXPERTS>
__global__ void __launch_bounds__(DT_THREADS)
dyn_tanh_vec_kernel(float* __restrict__ x, const float* __restrict__ alpha, const float* __restrict__ w, const float* __restrict__ b,
                    TOut* __restrict__ out, const int* __restrict__ rows, int n_rows, int E, const ExpertRows X) {
  const int i = (blockIdx.y * DT_THREADS + threadIdx.x) * 4;
  pdl_launch();
  const bool in = i < E;
  const float a = *alpha;
  const float4 w4 = in ? *reinterpret_cast<const float4*>(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 b4 = in ? *reinterpret_cast<const float4*>(b + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  pdl_wait();
  if (!in) return;
  for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
    const int src = rows ? rows[r] : r;
    float4* const p = reinterpret_cast<float4*>(x + (size_t)src * E + i);
    float4 v = *p;
    if constexpr (EXPERTS) {
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < DT_MAX_TOP; ++j) {
        if (j < X.top) {
          const int row = X.row_of[(size_t)src * X.top + j];
          const float f = X.weight_of != nullptr ? X.weight_of[(size_t)src * X.top + j] : 1.f;
          if (row >= 0) {
            const float4 e = *reinterpret_cast<const float4*>(X.rows + (size_t)row * X.ld + i);
            s.x += e.x * f, s.y += e.y * f, s.z += e.z * f, s.w += e.w * f;
          }
        }
      }
      v.x += s.x, v.y += s.y, v.z += s.z, v.w += s.w;
      *p = v;
    }
    dt_store4<TOut>(out + (size_t)r * E + i, make_float4(tanhf(a * v.x) * w4.x + b4.x, tanhf(a * v.y) * w4.y + b4.y,
                                                         tanhf(a * v.z) * w4.z + b4.z, tanhf(a * v.w) * w4.w + b4.w));
  }
}

constexpr int DT_FEW_ROWS = 64;

// x: float32 [*, E], updated in place where a sum is pending (partials or expert rows, not both).  out [n_rows, E] dense.
FERRUM_API int ferrum_dyn_tanh(float* x, const float* alpha, const float* w, const float* b, void* out, int out_dtype, const int* rows,
                               int n_rows, int E, const float* partials, const int* layout, const float* ex_rows, int ex_ld,
                               const int* ex_row_of, const float* ex_weight_of, int ex_top, cudaStream_t stream) {
  FERRUM_CHECK_ARG(n_rows >= 0 && E > 0 && alpha && w && b, "dyn_tanh: bad arguments");
  FERRUM_CHECK_ARG(partials == nullptr || ex_rows == nullptr, "dyn_tanh: one pending sum at a time");
  FERRUM_CHECK_ARG(ex_rows == nullptr || (ex_row_of != nullptr && ex_top > 0 && ex_top <= DT_MAX_TOP && ex_ld >= E), "dyn_tanh: bad expert rows");
  if (n_rows == 0) return 0;
  PartialLayout L{nullptr, 0, 0, 0, 0};
  if (partials != nullptr) {
    if (int r = partial_make_layout(partials, layout, &L)) return r;
    FERRUM_CHECK_ARG(E <= L.tiles * 128, "dyn_tanh: the partials do not cover the rows");
  }
  const ExpertRows X{ex_rows, ex_ld, ex_row_of, ex_weight_of, ex_top};
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (partials == nullptr && n_rows > DT_FEW_ROWS && E % 4 == 0 && al(x) && al(w) && al(b) && al(out) && al(ex_rows) && ex_ld % 4 == 0) {
    const int chunks = (E + DT_THREADS * 4 - 1) / (DT_THREADS * 4);
    const dim3 grid(max(1, min(n_rows, 148 * 8 / chunks)), chunks);
    FERRUM_DISPATCH_DTYPE(out_dtype, T, {
      if (ex_rows != nullptr) launch_kernel(dyn_tanh_vec_kernel<T, true>, grid, dim3(DT_THREADS), 0, stream, x, alpha, w, b, (T*)out, rows, n_rows, E, X);
      else launch_kernel(dyn_tanh_vec_kernel<T, false>, grid, dim3(DT_THREADS), 0, stream, x, alpha, w, b, (T*)out, rows, n_rows, E, X);
    });
    FERRUM_CHECK_LAUNCH("dyn_tanh");
    return 0;
  }
  const dim3 grid(n_rows, (E + DT_THREADS - 1) / DT_THREADS);
  FERRUM_DISPATCH_DTYPE(out_dtype, T, launch_kernel(dyn_tanh_kernel<T>, grid, dim3(DT_THREADS), 0, stream, x, alpha, w, b, (T*)out, rows, E, L, X));
  FERRUM_CHECK_LAUNCH("dyn_tanh");
  return 0;
}

// ================================================================= embedding of a token and of its pair with the one before
// One block per token.  The block of a portion's first token reads the request's state (the id before the portion) and
// then leaves the portion's last id there: nobody else touches that entry, so nothing races.
template <typename T>
__global__ void __launch_bounds__(DT_THREADS)
embedding_bigram_kernel(const T* __restrict__ table, int V, float scale, const T* __restrict__ pairs, int n_pairs, long long mul_prev,
                        long long mul_cur, const int* __restrict__ ids, const int* __restrict__ positions, const int* __restrict__ req_of_token,
                        const int* __restrict__ q_start, const int* __restrict__ slots, int* __restrict__ last_id, float* __restrict__ out,
                        int E, int* __restrict__ err) {
  __shared__ int pair_row;
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < V;
  if (threadIdx.x == 0) {
    if (!ok) atomicExch(err, 1);
    const int r = req_of_token[t], first = q_start[r];
    long long before = 0;
    if (t == first) {
      int* const mine = last_id + slots[r];
      before = *mine;
      *mine = ids[q_start[r + 1] - 1];
    } else {
      before = ids[t - 1];
    }
    long long row = (before * mul_prev + (long long)id * mul_cur) % n_pairs;
    if (row < 0) row += n_pairs;
    pair_row = positions[t] == 0 ? n_pairs : (int)row;
  }
  __syncthreads();
  const T* a = table + (size_t)(ok ? id : 0) * E;
  const T* b = pairs + (size_t)pair_row * E;
  float* o = out + (size_t)t * E;
  for (int i = threadIdx.x; i < E; i += DT_THREADS) o[i] = ok ? to_f32<T>(a[i]) * scale + to_f32<T>(b[i]) : 0.f;
}

// table [V, E] and pairs [n_pairs + 1, E] of one type; last_id: int [slots], read for a portion that does not start a sequence.
FERRUM_API int ferrum_embedding_bigram(const void* table, int V, float scale, const void* pairs, int n_pairs, long long mul_prev,
                                       long long mul_cur, int dtype, const int* ids, const int* positions, const int* req_of_token,
                                       const int* q_start, const int* slots, int* last_id, float* out, int n_tokens, int E, int* err_flag,
                                       cudaStream_t stream) {
  FERRUM_CHECK_ARG(n_tokens >= 0 && E > 0 && V > 0 && n_pairs > 0 && last_id != nullptr, "embedding_bigram: bad arguments");
  if (n_tokens == 0) return 0;
  FERRUM_DISPATCH_DTYPE(dtype, T, launch_kernel(embedding_bigram_kernel<T>, dim3(n_tokens), dim3(DT_THREADS), 0, stream, (const T*)table, V, scale,
                                                (const T*)pairs, n_pairs, mul_prev, mul_cur, ids, positions, req_of_token, q_start, slots,
                                                last_id, out, E, err_flag));
  FERRUM_CHECK_LAUNCH("embedding_bigram");
  return 0;
}

// ================================================================= the activation of an ungated unit
template <typename T>
__global__ void __launch_bounds__(DT_THREADS)
unit_act_kernel(const float* __restrict__ x, int ldx, T* __restrict__ out, int ldo, int F, const PartialLayout L) {
  __shared__ PartialTable tab;
  if (L.ws != nullptr) build_partial_table(L, tab);
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x;
  for (int f = blockIdx.y * DT_THREADS + threadIdx.x; f < F; f += gridDim.y * DT_THREADS) {
    const float v = L.ws != nullptr ? partial_sum(L, tab, t, f) : x[(size_t)t * ldx + f];
    out[(size_t)t * ldo + f] = from_f32<T>(relu_squared(v));
  }
}

// out[t, f] = relu(v)^2 with v = x[t, f], or the sum of a product left in partials.
FERRUM_API int ferrum_unit_act(const float* x, int ldx, void* out, int out_dtype, int ldo, int n_tokens, int F, const float* partials,
                               const int* layout, cudaStream_t stream) {
  FERRUM_CHECK_ARG(n_tokens >= 0 && F > 0 && ldo >= F && (partials != nullptr || (x != nullptr && ldx >= F)), "unit_act: bad arguments");
  if (n_tokens == 0) return 0;
  PartialLayout L{nullptr, 0, 0, 0, 0};
  if (partials != nullptr) {
    if (int r = partial_make_layout(partials, layout, &L)) return r;
    FERRUM_CHECK_ARG(F <= L.tiles * 128 && n_tokens <= L.acc_cols, "unit_act: the partials do not cover the rows");
  }
  const dim3 grid(n_tokens, min((F + DT_THREADS - 1) / DT_THREADS, 64));
  FERRUM_DISPATCH_DTYPE(out_dtype, T, launch_kernel(unit_act_kernel<T>, grid, dim3(DT_THREADS), 0, stream, x, ldx, (T*)out, ldo, F, L));
  FERRUM_CHECK_LAUNCH("unit_act");
  return 0;
}
