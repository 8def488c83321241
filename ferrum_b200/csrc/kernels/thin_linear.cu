// y = x W^T for a product with few output features (a router, the first matrix of a low-rank pair, the gate of a
// per-layer token input): too few tiles for the tensor-core product, whose CTAs would each walk a sliver of K and
// then wait for one another's sums.  Here a block of 256 threads owns 8 tokens and NF features: a thread takes the
// 16-byte pieces of K at 8 tid, 8 tid + 2048, ..., keeps the 8 x NF float32 sums in registers, and the block adds them
// in one fixed tree, so a result depends on K alone, never on what else is in the batch.
//
// The epilogue stores float32 or the compute type, or applies the token input's gate:
// out[t][n] = gelu_tanh(z) * table[token[t]][offset + n].
#include "common.cuh"

constexpr int TL_THREADS = 256, TL_TOKENS = 8;

struct ThinEpilogue {
  int kind;                  // 0: float32; 1: compute type; 2: gelu_tanh(z) * table entry, compute type
  void* out;
  int ldo;
  const void* table;
  int ldt, n_vocab, offset;
  const int* token_ids;
  int* err;
};

template <typename T>
__device__ __forceinline__ void tl_unpack(const uint4& raw, float (&v)[8]) {
  const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = to_f32<T>(e[i]);
}

template <typename T, int NF>
__global__ void __launch_bounds__(TL_THREADS)
thin_linear_kernel(const T* __restrict__ x, int ldx, const T* __restrict__ w, int K, int N, int n_tokens, const ThinEpilogue ep) {
  pdl_launch();
  constexpr int NV = TL_TOKENS * NF;
  __shared__ float part[TL_THREADS / 32][NV];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * NF, t0 = blockIdx.y * TL_TOKENS;
  const int nt = min(TL_TOKENS, n_tokens - t0);
  float acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  const T* xr[TL_TOKENS];
  const T* wr[NF];
#pragma unroll
  for (int i = 0; i < TL_TOKENS; ++i) xr[i] = x + (size_t)(t0 + min(i, nt - 1)) * ldx;     // (rows past the last repeat it and are dropped)
#pragma unroll
  for (int j = 0; j < NF; ++j) wr[j] = w + (size_t)min(n0 + j, N - 1) * K;
  for (int k = tid * 8; k < K; k += TL_THREADS * 8) {
    uint4 xraw[TL_TOKENS];
#pragma unroll
    for (int i = 0; i < TL_TOKENS; ++i) xraw[i] = *reinterpret_cast<const uint4*>(xr[i] + k);
#pragma unroll
    for (int j = 0; j < NF; ++j) {
      const uint4 wraw = *reinterpret_cast<const uint4*>(wr[j] + k);
      float wv[8];
      tl_unpack<T>(wraw, wv);
#pragma unroll
      for (int i = 0; i < TL_TOKENS; ++i) {
        float xv[8];
        tl_unpack<T>(xraw[i], xv);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i * NF + j] = fmaf(xv[e], wv[e], acc[i * NF + j]);
      }
    }
  }
  // the 32 lanes of a warp: each exchange halves the values a lane keeps, then plain sums
  int first = 0;             // the first value this lane still holds
  {
    int n = NV;
#pragma unroll
    for (int m = 16; m >= 1; m >>= 1) {
      if (n > 1) {
        n >>= 1;
        const bool up = (lane & m) != 0;
#pragma unroll
        for (int i = 0; i < NV / 2; ++i) {
          if (i < n) {
            const float send = up ? acc[i] : acc[i + n], keep = up ? acc[i + n] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
          }
        }
        first += up ? n : 0;
      } else {
        acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], m);
      }
    }
  }
  constexpr int LEFT = NV > 32 ? NV / 32 : 1, DUP = NV < 32 ? 32 / NV : 1;
  if (lane % DUP == 0) {
#pragma unroll
    for (int i = 0; i < LEFT; ++i) part[warp][first + i] = acc[i];
  }
  __syncthreads();
  if (tid < NV) {
    const int i = tid / NF, n = n0 + tid % NF;
    if (i < nt && n < N) {
      float s = 0.f;
#pragma unroll
      for (int wp = 0; wp < TL_THREADS / 32; ++wp) s += part[wp][tid];
      const size_t o = (size_t)(t0 + i) * ep.ldo + n;
      if (ep.kind == 0) {
        reinterpret_cast<float*>(ep.out)[o] = s;
      } else if (ep.kind == 1) {
        reinterpret_cast<T*>(ep.out)[o] = from_f32<T>(s);
      } else {
        const int tok = ep.token_ids[t0 + i];
        if (tok < 0 || tok >= ep.n_vocab) {
          atomicExch(ep.err, 1);
        } else {
          const float g = 0.5f * s * (1.f + tanhf(0.7978845608028654f * (s + 0.044715f * s * s * s)));
          reinterpret_cast<T*>(ep.out)[o] = from_f32<T>(g * to_f32<T>(reinterpret_cast<const T*>(ep.table)[(size_t)tok * ep.ldt + ep.offset + n]));
        }
      }
    }
  }
}

// Products for which this kernel is the one to take: a few features, and either a few tokens or so few features that
// the tokens' rows are read once.
FERRUM_API int ferrum_thin_linear_supported(const void* x, int ldx, const void* w, int dtype, int n_tokens, int N, int K) {
  if (!ferrum_is_16bit(dtype) || K % 8 != 0 || ldx % 8 != 0 || ((uintptr_t)x & 15) != 0 || ((uintptr_t)w & 15) != 0) return 0;
  return (n_tokens <= 16 && N <= 512) || (n_tokens <= 64 && N <= 64) || N <= 16;
}

// table == null: out is float32 (kind 0) or the compute type (kind 1); else kind 2, see the top.
FERRUM_API int ferrum_thin_linear(const void* x, int ldx, const void* w, int dtype, int n_tokens, int N, int K, int kind, void* out, int ldo,
                                  const void* table, int ldt, int n_vocab, int offset, const int* token_ids, int* err, cudaStream_t stream) {
  FERRUM_CHECK_ARG(ferrum_is_16bit(dtype) && N > 0 && K > 0 && K % 8 == 0 && ldx % 8 == 0 && ldx >= K && ldo >= N &&
                   (((uintptr_t)x | (uintptr_t)w) & 15) == 0, "thin_linear: rows are not on 16-byte borders, or sizes do not agree");
  FERRUM_CHECK_ARG(kind >= 0 && kind <= 2 && (kind != 2 || (table != nullptr && token_ids != nullptr && offset >= 0 && offset + N <= ldt)),
                   "thin_linear: bad epilogue");
  if (n_tokens == 0) return 0;
  const ThinEpilogue ep{kind, out, ldo, table, ldt, n_vocab, offset, token_ids, err};
  const int chunks = (n_tokens + TL_TOKENS - 1) / TL_TOKENS;
  FERRUM_CHECK_ARG(chunks <= 65535, "thin_linear: too many tokens");
  // a few tokens: two features a block, so that the blocks cover the GPU; many: eight, so that the rows are read once or twice
  if (n_tokens <= 64) {
    FERRUM_DISPATCH_16BIT(dtype, T, (thin_linear_kernel<T, 2><<<dim3((N + 1) / 2, chunks), TL_THREADS, 0, stream>>>((const T*)x, ldx, (const T*)w, K, N,
                                                                                                                  n_tokens, ep)));
  } else {
    FERRUM_DISPATCH_16BIT(dtype, T, (thin_linear_kernel<T, 8><<<dim3((N + 7) / 8, chunks), TL_THREADS, 0, stream>>>((const T*)x, ldx, (const T*)w, K, N,
                                                                                                                  n_tokens, ep)));
  }
  FERRUM_CHECK_LAUNCH("thin_linear");
  return 0;
}
