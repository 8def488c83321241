// Recurrences over a matrix per head whose rows decay each at a rate of their own: S (D x Dv, float32, zero before
// a sequence's first token), a decay a_t in [0, 1] per head and key channel, keys k and queries q of D, values v of Dv:
//
//   after the write    S <- diag(a_t) S + k v^T;   o = c * S^T q                        (gated linear attention)
//   with a bonus       o = c * (S + diag(u) k v^T)^T q;   S <- diag(a_t) S + k v^T      (the RWKV form: the current token
//                                                         enters the read-out through u instead of through the state)
//
// channel_decay_scan walks a portion's tokens.  The update of an element needs nothing from its neighbours, so a lane
// keeps an 8 x 8 piece of the state (eight rows of eight columns) in registers and every step is three packed
// two-wide multiply-adds per pair of rows: the rows come in pairs because a, k and q then arrive packed from shared
// memory.  RL lanes side by side hold a column's rows (D <= 8 RL) and meet once per token and column in a fixed
// shuffle tree; a warp holds (32 / RL) * 8 columns.  Tokens are staged by cp.async, the next chunk on its way
// meanwhile.
//
// Long portions are cut into segments that run side by side: (1) every segment but a portion's last is walked from a
// zero state without read-outs, which leaves its own contribution and the product of its decays; (2) one pass over the
// elements chains them, start of the next = (product of decays) start + contribution, from the state of the request;
// (3) the walk proper starts every segment from its true state.  Only products of decays in [0, 1] are ever formed, so
// nothing overflows however fast a channel forgets.  A token's result depends on the cut only through the order of
// float32 sums.
//
// channel_decay_gate makes the decays from a low-rank projection: z = W2 act(low) + bias in float32 with float32
// inputs, then a = exp(-exp(z)) or sigmoid(z)^(1/tau).
//
// token_shift_mix makes the inputs of projections that see a blend of a row with the one before it.
#include "common.cuh"

typedef unsigned long long cd_pair;      // two float32 side by side in a 64-bit register

__device__ __forceinline__ cd_pair cd_pack(float lo, float hi) {
  cd_pair r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void cd_unpack(cd_pair p, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(p)); }
__device__ __forceinline__ cd_pair cd_mul(cd_pair a, cd_pair b) {
  cd_pair r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ cd_pair cd_fma(cd_pair a, cd_pair b, cd_pair c) {
  cd_pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

template <int BYTES>
__device__ __forceinline__ void cd_cp_async(float* smem, const float* gmem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(a), "l"(gmem), "n"(BYTES) : "memory");
}
__device__ __forceinline__ void cd_cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cd_cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

struct ChannelDecayArgs {
  const float *q, *k, *v, *dec;          // rows of tokens; head h at h * D (v: h * Dv)
  int ldq, ldk, ldv, ldd;
  const float* bonus;                    // [H * D], or null
  float out_scale;
  float* state;                          // [slots][state_stride]; head h at h * D * Dv, element (d, j) at d * Dv + j
  long long state_stride;
  const int *q_start, *slots;
  int n_reqs;
  float* o;
  int ldo;
  int H, D, Dv;
  int seg_len;                           // tokens per segment; 0: a portion is walked in one piece
  float *seg_state, *seg_dec;            // [segment][H][D * Dv], [segment][H][D]
  int vec;                               // rows, offsets and state on 16-byte borders: copies of four floats
};

// Segment `item` of the step: its request, its number within the portion, and how many the portion has (n = 0: past the last).
struct CdSegment { int req, seg, n; };
__device__ __forceinline__ CdSegment cd_find_segment(const int* q_start, int n_reqs, int seg_len, int item) {
  int left = item;
  for (int r = 0; r < n_reqs; ++r) {
    const int n = (q_start[r + 1] - q_start[r] + seg_len - 1) / seg_len;
    if (left < n) return CdSegment{r, left, n};
    left -= n;
  }
  return CdSegment{0, 0, 0};
}

constexpr int CD_WARPS = 4;              // warps of a block at most (fewer when the columns are fewer)

// MODE 0: read-out after the write; 1: with a bonus; 2: no read-out, from zero (a segment's own contribution).
template <int RL, int MODE>
__global__ void __launch_bounds__(CD_WARPS * 32, 3)
channel_decay_scan_kernel(const ChannelDecayArgs A) {
  constexpr int DP = 8 * RL, WC = (32 / RL) * 8, CB = CD_WARPS * WC, TC = RL <= 16 ? 8 : 4;
  constexpr bool LOCAL = MODE == 2, BONUS = MODE == 1;
  __shared__ __align__(16) float sa[2][TC][DP], sk[2][TC][DP], sq[LOCAL ? 1 : 2][LOCAL ? 1 : TC][LOCAL ? 4 : DP], sv[2][TC][CB];
  __shared__ CdSegment seg_smem;
  const int tid = threadIdx.x, nthreads = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane % RL, co = lane / RL;
  const int D = A.D, Dv = A.Dv, h = blockIdx.y;
  const int cols0 = blockIdx.x * (nthreads / 32) * WC;            // the block's first column
  const int j0 = cols0 + warp * WC + co * 8;                      // the lane's
  CdSegment sg{(int)blockIdx.z, 0, 1};
  if (A.seg_len > 0) {
    if (tid == 0) seg_smem = cd_find_segment(A.q_start, A.n_reqs, A.seg_len, blockIdx.z);
    __syncthreads();
    sg = seg_smem;
    if (sg.n == 0 || (LOCAL && sg.seg == sg.n - 1)) return;       // past the last segment; the last one's contribution nobody needs
  }
  int t0 = A.q_start[sg.req], t1 = A.q_start[sg.req + 1];
  if (A.seg_len > 0) {
    t0 += sg.seg * A.seg_len;
    t1 = min(t1, t0 + A.seg_len);
  }
  const bool last = sg.seg == sg.n - 1;
  const size_t head = (size_t)h * D * Dv;
  float* const mine = A.state + (long long)A.slots[sg.req] * A.state_stride + head;
  float* const scratch = A.seg_len > 0 ? A.seg_state + (size_t)blockIdx.z * A.H * D * Dv + head : nullptr;
  // padding (rows past D, columns past Dv) is zero in both buffers and stays so: the copies never touch it
  for (int i = tid; i < 2 * TC * DP; i += nthreads) {
    (&sa[0][0][0])[i] = 0.f;
    (&sk[0][0][0])[i] = 0.f;
    if (!LOCAL) (&sq[0][0][0])[i] = 0.f;
  }
  for (int i = tid; i < 2 * TC * CB; i += nthreads) (&sv[0][0][0])[i] = 0.f;
  __syncthreads();
  const int ncols = min((nthreads / 32) * WC, Dv - cols0);
  auto stage = [&](int c0, int b) {              // a chunk's rows on their way into buffer b
    const int nt = min(TC, t1 - c0);
    if (A.vec) {
      const int pd = D / 4, pv = ncols / 4, per = (LOCAL ? 2 : 3) * pd + pv;
      for (int idx = tid; idx < nt * per; idx += nthreads) {
        const int tk = idx / per;
        int i = idx - tk * per;
        const size_t t = (size_t)(c0 + tk);
        if (i < pv) {
          cd_cp_async<16>(&sv[b][tk][4 * i], A.v + t * A.ldv + (size_t)h * Dv + cols0 + 4 * i);
        } else if ((i -= pv) < pd) {
          cd_cp_async<16>(&sa[b][tk][4 * i], A.dec + t * A.ldd + (size_t)h * D + 4 * i);
        } else if ((i -= pd) < pd) {
          cd_cp_async<16>(&sk[b][tk][4 * i], A.k + t * A.ldk + (size_t)h * D + 4 * i);
        } else if (!LOCAL) {
          i -= pd;
          cd_cp_async<16>(&sq[b][tk][4 * i], A.q + t * A.ldq + (size_t)h * D + 4 * i);
        }
      }
    } else {
      const int per = (LOCAL ? 2 : 3) * D + ncols;
      for (int idx = tid; idx < nt * per; idx += nthreads) {
        const int tk = idx / per;
        int i = idx - tk * per;
        const size_t t = (size_t)(c0 + tk);
        if (i < ncols) {
          cd_cp_async<4>(&sv[b][tk][i], A.v + t * A.ldv + (size_t)h * Dv + cols0 + i);
        } else if ((i -= ncols) < D) {
          cd_cp_async<4>(&sa[b][tk][i], A.dec + t * A.ldd + (size_t)h * D + i);
        } else if ((i -= D) < D) {
          cd_cp_async<4>(&sk[b][tk][i], A.k + t * A.ldk + (size_t)h * D + i);
        } else if (!LOCAL) {
          i -= D;
          cd_cp_async<4>(&sq[b][tk][i], A.q + t * A.ldq + (size_t)h * D + i);
        }
      }
    }
    cd_cp_async_commit();
  };
  if (t0 < t1) stage(t0, 0);
  // A lane's rows are two runs of four (4 rg .. and 4 RL + 4 rg ..): the lanes' 16-byte reads of a token's row then lie
  // side by side.  Pair p holds rows row(2 p), row(2 p) + 1.
  auto row = [&](int i) { return (i >> 2) * 4 * RL + 4 * rg + (i & 3); };
  cd_pair S[8][4], P[4];
#pragma unroll
  for (int p = 0; p < 4; ++p) {
    P[p] = cd_pack(1.f, 1.f);
    float e[2][8];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int d = row(2 * p + half);
      const float* src = (sg.n > 1 ? scratch : mine) + (size_t)d * Dv + j0;
#pragma unroll
      for (int c = 0; c < 8; ++c) e[half][c] = 0.f;
      if (!LOCAL && d < D) {
        if (A.vec) {
          if (j0 < Dv) *reinterpret_cast<float4*>(&e[half][0]) = *reinterpret_cast<const float4*>(src);
          if (j0 + 4 < Dv) *reinterpret_cast<float4*>(&e[half][4]) = *reinterpret_cast<const float4*>(src + 4);
        } else {
#pragma unroll
          for (int c = 0; c < 8; ++c)
            if (j0 + c < Dv) e[half][c] = src[c];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < 8; ++c) S[c][p] = cd_pack(e[0][c], e[1][c]);
  }
  cd_pair ub[4];
  if (BONUS) {
#pragma unroll
    for (int p = 0; p < 4; ++p) {
      const int d = row(2 * p);
      ub[p] = cd_pack(d < D ? A.bonus[(size_t)h * D + d] : 0.f, d + 1 < D ? A.bonus[(size_t)h * D + d + 1] : 0.f);
    }
  }
  cd_cp_async_wait_all();
  __syncthreads();
  int b = 0;
  for (int c0 = t0; c0 < t1; c0 += TC, b ^= 1) {
    const int nt = min(TC, t1 - c0);
    if (c0 + TC < t1) stage(c0 + TC, b ^ 1);     // (that buffer was last read before the barrier that ended the chunk before)
#pragma unroll 2
    for (int tk = 0; tk < nt; ++tk) {
      const ulonglong2 al = *reinterpret_cast<const ulonglong2*>(&sa[b][tk][4 * rg]), ah = *reinterpret_cast<const ulonglong2*>(&sa[b][tk][4 * RL + 4 * rg]);
      const ulonglong2 kl = *reinterpret_cast<const ulonglong2*>(&sk[b][tk][4 * rg]), kh = *reinterpret_cast<const ulonglong2*>(&sk[b][tk][4 * RL + 4 * rg]);
      const cd_pair a[4] = {al.x, al.y, ah.x, ah.y}, k[4] = {kl.x, kl.y, kh.x, kh.y};
      cd_pair q[4];
      if (!LOCAL) {
        const ulonglong2 ql = *reinterpret_cast<const ulonglong2*>(&sq[b][tk][4 * rg]), qh = *reinterpret_cast<const ulonglong2*>(&sq[b][tk][4 * RL + 4 * rg]);
        q[0] = ql.x, q[1] = ql.y, q[2] = qh.x, q[3] = qh.y;
      }
      const float4 v0 = *reinterpret_cast<const float4*>(&sv[b][tk][warp * WC + co * 8]), v1 = *reinterpret_cast<const float4*>(&sv[b][tk][warp * WC + co * 8 + 4]);
      const float v[8] = {v0.x, v0.y, v0.z, v0.w, v1.x, v1.y, v1.z, v1.w};
      float u[8];
      float w = 0.f;
      if (BONUS) {                               // the lane's part of (u k) . q, which multiplies v in every column
        cd_pair ws = cd_mul(cd_mul(ub[0], k[0]), q[0]);
#pragma unroll
        for (int p = 1; p < 4; ++p) ws = cd_fma(cd_mul(ub[p], k[p]), q[p], ws);
        float lo, hi;
        cd_unpack(ws, lo, hi);
        w = lo + hi;
      }
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const cd_pair vv = cd_pack(v[c], v[c]);
        cd_pair us = 0ull;
#pragma unroll
        for (int p = 0; p < 4; ++p) {
          if (BONUS) us = cd_fma(S[c][p], q[p], us);
          S[c][p] = cd_fma(a[p], S[c][p], cd_mul(k[p], vv));
          if (MODE == 0) us = cd_fma(S[c][p], q[p], us);
        }
        if (!LOCAL) {
          float lo, hi;
          cd_unpack(us, lo, hi);
          u[c] = BONUS ? fmaf(w, v[c], lo + hi) : lo + hi;
        }
      }
      if (LOCAL) {
#pragma unroll
        for (int p = 0; p < 4; ++p) P[p] = cd_mul(P[p], a[p]);
      } else {
        // the RL lanes of a column meet: each halving of the columns is one exchange, then plain sums
        int n = 8, col = 0;
#pragma unroll
        for (int m = RL / 2; m >= 1; m >>= 1) {
          if (n > 1) {
            const bool up = (rg & m) != 0;
            n >>= 1;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              if (i < n) {
                const float send = up ? u[i] : u[i + n], keep = up ? u[i + n] : u[i];
                u[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
              }
            }
            col += up ? n : 0;
          } else {
            u[0] += __shfl_xor_sync(0xffffffffu, u[0], m);
          }
        }
        constexpr int LEFT = RL >= 8 ? 1 : 8 / RL;               // columns a lane ends up with
        constexpr int DUP = RL > 8 ? RL / 8 : 1;                 // lanes that end up with the same column
        if (rg % DUP == 0) {
          float* dst = A.o + (size_t)(c0 + tk) * A.ldo + (size_t)h * Dv + j0 + col;
#pragma unroll
          for (int i = 0; i < LEFT; ++i)
            if (j0 + col + i < Dv) dst[i] = u[i] * A.out_scale;
        }
      }
    }
    cd_cp_async_wait_all();
    __syncthreads();
  }
  if (!LOCAL && !last) return;
  float* const dst0 = LOCAL ? scratch : mine;
#pragma unroll
  for (int p = 0; p < 4; ++p) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int d = row(2 * p + half);
      if (d >= D) continue;
      float e[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        float lo, hi;
        cd_unpack(S[c][p], lo, hi);
        e[c] = half ? hi : lo;
      }
      float* dst = dst0 + (size_t)d * Dv + j0;
      if (A.vec) {
        if (j0 < Dv) *reinterpret_cast<float4*>(dst) = make_float4(e[0], e[1], e[2], e[3]);
        if (j0 + 4 < Dv) *reinterpret_cast<float4*>(dst + 4) = make_float4(e[4], e[5], e[6], e[7]);
      } else {
#pragma unroll
        for (int c = 0; c < 8; ++c)
          if (j0 + c < Dv) dst[c] = e[c];
      }
      if (LOCAL && j0 == 0) {
        float lo, hi;
        cd_unpack(P[p], lo, hi);
        A.seg_dec[((size_t)blockIdx.z * A.H + h) * D + d] = half ? hi : lo;
      }
    }
  }
}

// The segments' start states, in place of their contributions: one thread per state element and request.
__global__ void __launch_bounds__(256)
channel_decay_chain_kernel(const ChannelDecayArgs A) {
  const int r = blockIdx.z, h = blockIdx.y;
  const int n = (A.q_start[r + 1] - A.q_start[r] + A.seg_len - 1) / A.seg_len;
  if (n <= 1) return;
  int first = 0;
  for (int i = 0; i < r; ++i) first += (A.q_start[i + 1] - A.q_start[i] + A.seg_len - 1) / A.seg_len;
  const int e = blockIdx.x * 256 + threadIdx.x;
  if (e >= A.D * A.Dv) return;
  const size_t hs = (size_t)A.H * A.D * A.Dv, off = (size_t)h * A.D * A.Dv + e;
  float s = A.state[(long long)A.slots[r] * A.state_stride + off];
  const float* dec = A.seg_dec + ((size_t)first * A.H + h) * A.D + e / A.Dv;
  float* st = A.seg_state + (size_t)first * hs + off;
  constexpr int BATCH = 8;                       // (the last segment has no contribution: nothing of it is read)
  for (int i0 = 0; i0 < n; i0 += BATCH) {
    float own[BATCH], p[BATCH];
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const bool have = i0 + i < n - 1;
      own[i] = have ? st[(size_t)(i0 + i) * hs] : 0.f;
      p[i] = have ? dec[(size_t)(i0 + i) * A.H * A.D] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      if (i0 + i < n) st[(size_t)(i0 + i) * hs] = s;
      s = fmaf(p[i], s, own[i]);
    }
  }
}

constexpr int CD_MAX_D = 256;

template <int RL>
static int cd_launch(const ChannelDecayArgs& a, int segments, int n_items, cudaStream_t stream) {
  constexpr int WC = (32 / RL) * 8;
  const int warps = min(CD_WARPS, (a.Dv + WC - 1) / WC);
  const dim3 grid((a.Dv + warps * WC - 1) / (warps * WC), a.H, n_items);
  if (segments) {
    channel_decay_scan_kernel<RL, 2><<<grid, warps * 32, 0, stream>>>(a);
    FERRUM_CHECK_LAUNCH("channel_decay_scan (contributions)");
    channel_decay_chain_kernel<<<dim3((a.D * a.Dv + 255) / 256, a.H, a.n_reqs), 256, 0, stream>>>(a);
    FERRUM_CHECK_LAUNCH("channel_decay_chain");
  }
  if (a.bonus != nullptr) channel_decay_scan_kernel<RL, 1><<<grid, warps * 32, 0, stream>>>(a);
  else channel_decay_scan_kernel<RL, 0><<<grid, warps * 32, 0, stream>>>(a);
  FERRUM_CHECK_LAUNCH("channel_decay_scan");
  return 0;
}

// Columns that one block of the walk covers, for the caller that picks the length of the segments.
FERRUM_API int ferrum_channel_decay_block_columns(int D, int Dv) {
  const int RL = D <= 32 ? 4 : D <= 64 ? 8 : D <= 128 ? 16 : 32;
  const int WC = (32 / RL) * 8;
  return min(CD_WARPS, (Dv + WC - 1) / WC) * WC;
}

// q, k, v, dec: float32 rows of n_tokens tokens (strides ld*; heads of D, or Dv, side by side); bonus: [H * D] or null;
// state: [slots][state_stride] float32 rows whose first H * D * Dv floats are S; o: [n_tokens][ldo] receives
// out_scale * the read-outs.  seg_len > 0: portions are cut into segments of that many tokens; seg_state and seg_dec
// then hold n_segments * H * D * Dv and n_segments * H * D floats, n_segments >= the sum over the portions of
// ceil(length / seg_len).
FERRUM_API int ferrum_channel_decay(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* dec, int ldd,
                                    const float* bonus, float out_scale, int n_tokens, int n_reqs, const int* q_start, const int* slots,
                                    int H, int D, int Dv, float* state, long long state_stride, int seg_len, int n_segments,
                                    float* seg_state, float* seg_dec, float* o, int ldo, cudaStream_t stream) {
  FERRUM_CHECK_ARG(H > 0 && D > 0 && D <= CD_MAX_D && Dv > 0, "channel_decay: bad head sizes H=%d D=%d Dv=%d", H, D, Dv);
  FERRUM_CHECK_ARG(ldq >= H * D && ldk >= H * D && ldd >= H * D && ldv >= H * Dv && ldo >= H * Dv && state_stride >= (long long)H * D * Dv,
                   "channel_decay: a row is too short");
  FERRUM_CHECK_ARG(seg_len >= 0 && (seg_len == 0 || (n_segments > 0 && seg_state != nullptr && seg_dec != nullptr)), "channel_decay: bad segments");
  const int items = seg_len > 0 ? n_segments : n_reqs;
  FERRUM_CHECK_ARG(items <= 65535 && n_reqs <= 65535 && H <= 65535, "channel_decay: too many requests, segments or heads");
  if (n_tokens == 0 || n_reqs == 0) return 0;
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const int vec = D % 4 == 0 && Dv % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 && ldd % 4 == 0 && state_stride % 4 == 0 && al(q) &&
                  al(k) && al(v) && al(dec) && al(state) && (seg_state == nullptr || al(seg_state));
  const ChannelDecayArgs a{q, k, v, dec, ldq, ldk, ldv, ldd, bonus, out_scale, state, state_stride, q_start, slots, n_reqs, o, ldo,
                           H, D, Dv, seg_len, seg_state, seg_dec, vec};
  if (D <= 32) return cd_launch<4>(a, seg_len > 0, items, stream);
  if (D <= 64) return cd_launch<8>(a, seg_len > 0, items, stream);
  if (D <= 128) return cd_launch<16>(a, seg_len > 0, items, stream);
  return cd_launch<32>(a, seg_len > 0, items, stream);
}

// ------------------------------------------------------------------ decays from a low-rank projection
// z[t][n] = sum_r W2[n][r] act(low[t][r]) + bias[n]; out = exp(-exp(z)) (kind 0) or sigmoid(z)^(1/tau) (kind 1).
__device__ __forceinline__ float cd_gate(float z, int kind, float inv_tau) {
  return kind == 0 ? expf(-expf(z)) : expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau);
}

// A few tokens: a block of 8 tokens x 32 channels, a thread per pair; the tokens' low-rank rows wait in shared memory
// (CD_GATE_ROWS elements at a time) and a channel's weights come straight from memory, eight at a time where they are aligned.
constexpr int CD_GATE_ROWS = 128;
template <typename T>
__global__ void __launch_bounds__(256)
channel_decay_gate_few_kernel(const float* __restrict__ low, int ldl, int rank, int act_tanh, const T* __restrict__ w2, const float* __restrict__ bias,
                              int kind, float inv_tau, int n_tokens, int N, float* __restrict__ out, int ldo, int vec) {
  __shared__ __align__(16) float sl[8][CD_GATE_ROWS];
  const int tid = threadIdx.x, c = blockIdx.x * 32 + (tid & 31), i = tid >> 5;
  const int t0 = blockIdx.y * 8;
  const T* wr = w2 + (size_t)min(c, N - 1) * rank;
  float acc = 0.f;
  for (int k0 = 0; k0 < rank; k0 += CD_GATE_ROWS) {
    const int n = min(CD_GATE_ROWS, rank - k0);
    for (int idx = tid; idx < 8 * n; idx += 256) {
      const int m = idx / n, k = idx % n;
      const float v = t0 + m < n_tokens ? low[(size_t)(t0 + m) * ldl + k0 + k] : 0.f;
      sl[m][k] = act_tanh ? tanhf(v) : v;
    }
    __syncthreads();
    if (vec) {                       // (rank is a multiple of 8, and so is n)
      for (int k = 0; k < n; k += 8) {
        float wv[8];
        if constexpr (sizeof(T) == 4) {
          *reinterpret_cast<float4*>(&wv[0]) = *reinterpret_cast<const float4*>(wr + k0 + k);
          *reinterpret_cast<float4*>(&wv[4]) = *reinterpret_cast<const float4*>(wr + k0 + k + 4);
        } else {
          const uint4 raw = *reinterpret_cast<const uint4*>(wr + k0 + k);
          const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
          for (int j = 0; j < 8; ++j) wv[j] = to_f32<T>(e[j]);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) acc = fmaf(sl[i][k + j], wv[j], acc);
      }
    } else {
      for (int k = 0; k < n; ++k) acc = fmaf(sl[i][k], to_f32<T>(wr[k0 + k]), acc);
    }
    __syncthreads();
  }
  if (c < N && t0 + i < n_tokens) out[(size_t)(t0 + i) * ldo + c] = cd_gate(acc + bias[c], kind, inv_tau);
}

// Many tokens: a block makes 64 tokens x 64 channels, 4 x 4 a thread, the inner size in steps of 32 through shared memory.
template <typename T>
__global__ void __launch_bounds__(256)
channel_decay_gate_kernel(const float* __restrict__ low, int ldl, int rank, int act_tanh, const T* __restrict__ w2, const float* __restrict__ bias,
                          int kind, float inv_tau, int n_tokens, int N, float* __restrict__ out, int ldo) {
  constexpr int KC = 32, TN = 64, TM = 64, MT = 4;
  __shared__ __align__(16) float sl[KC][TM + 4], sw[KC][TN + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int n0 = blockIdx.x * TN, t0 = blockIdx.y * TM;
  float acc[MT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < rank; k0 += KC) {
    for (int idx = tid; idx < TM * KC; idx += 256) {
      const int m = idx / KC, k = idx % KC;
      float v = (t0 + m < n_tokens && k0 + k < rank) ? low[(size_t)(t0 + m) * ldl + k0 + k] : 0.f;
      sl[k][m] = act_tanh ? tanhf(v) : v;
    }
    for (int idx = tid; idx < TN * KC; idx += 256) {
      const int n = idx / KC, k = idx % KC;
      sw[k][n] = (n0 + n < N && k0 + k < rank) ? to_f32<T>(w2[(size_t)(n0 + n) * rank + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < KC; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&sl[k][4 * ty]), bv = *reinterpret_cast<const float4*>(&sw[k][4 * tx]);
      const float a[4] = {av.x, av.y, av.z, av.w}, b[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const int t = t0 + 4 * ty + i;
    if (t >= n_tokens) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + 4 * tx + j;
      if (n < N) out[(size_t)t * ldo + n] = cd_gate(acc[i][j] + bias[n], kind, inv_tau);
    }
  }
}

FERRUM_API int ferrum_channel_decay_gate(const float* low, int ldl, int rank, int act_tanh, const void* w2, int dtype, const float* bias, int kind,
                                         float inv_tau, int n_tokens, int N, float* out, int ldo, cudaStream_t stream) {
  FERRUM_CHECK_ARG(rank > 0 && N > 0 && ldl >= rank && ldo >= N && (kind == 0 || kind == 1), "channel_decay_gate: bad sizes");
  if (n_tokens == 0) return 0;
  const bool few = n_tokens <= 32;
  const dim3 grid(few ? (N + 31) / 32 : (N + 63) / 64, few ? (n_tokens + 7) / 8 : (n_tokens + 63) / 64);
  FERRUM_CHECK_ARG(grid.y <= 65535, "channel_decay_gate: too many tokens");
  const int vec = rank % 8 == 0 && ((uintptr_t)w2 & 15) == 0;
  if (few)
    FERRUM_DISPATCH_DTYPE(dtype, T, (channel_decay_gate_few_kernel<T><<<grid, 256, 0, stream>>>(low, ldl, rank, act_tanh, (const T*)w2, bias, kind,
                                                                                               inv_tau, n_tokens, N, out, ldo, vec)));
  else
    FERRUM_DISPATCH_DTYPE(dtype, T, (channel_decay_gate_kernel<T><<<grid, 256, 0, stream>>>(low, ldl, rank, act_tanh, (const T*)w2, bias, kind,
                                                                                           inv_tau, n_tokens, N, out, ldo)));
  FERRUM_CHECK_LAUNCH("channel_decay_gate");
  return 0;
}

// ------------------------------------------------------------------ blends of a row with the one before it
// out[i][t] = x[t] + (x[t - 1] - x[t]) * mu[i], float32 arithmetic, rounded once.  The row before a portion's first token
// is the request's (float32, in its state row; zero before a sequence starts); the thread that reads an element of it
// puts the portion's last row there, so nobody else touches it.  counts[0 .. n_counts - 1] = n_tokens: what a grouped
// product over the blends wants.
template <typename T, int V>
__global__ void __launch_bounds__(128)
token_shift_mix_kernel(const T* __restrict__ x, int ldx, int E, const float* __restrict__ mu, int n_mix, const int* __restrict__ q_start,
                       const int* __restrict__ req_of_token, const int* __restrict__ slots, float* __restrict__ prev, long long prev_stride,
                       T* __restrict__ out, int n_tokens, int* __restrict__ counts, int n_counts) {
  const int t = blockIdx.x;
  if (t == 0 && blockIdx.y == 0 && (int)threadIdx.x < n_counts) counts[threadIdx.x] = n_tokens;
  const int e = (blockIdx.y * 128 + threadIdx.x) * V;
  if (e >= E) return;
  const int r = req_of_token[t];
  const bool first = t == q_start[r];
  float* const p = prev + (long long)slots[r] * prev_stride + e;
  auto load = [&](int row, float (&v)[V]) {
    const T* src = x + (size_t)row * ldx + e;
    if constexpr (V == 4) {
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(src);
      } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(src);
        const T* w = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = to_f32<T>(w[i]);
      }
    } else {
      v[0] = to_f32<T>(src[0]);
    }
  };
  float cur[V], before[V];
  load(t, cur);
  if (first) {
    float fin[V];
    load(q_start[r + 1] - 1, fin);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      before[i] = p[i];
      p[i] = fin[i];
    }
  } else {
    load(t - 1, before);
  }
  for (int m = 0; m < n_mix; ++m) {
    const float* w = mu + (size_t)m * E + e;
    T* dst = out + ((size_t)m * n_tokens + t) * E + e;
    float v[V];
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = fmaf(before[i] - cur[i], w[i], cur[i]);
    if constexpr (V == 4) {
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(dst) = *reinterpret_cast<float4*>(v);
      } else {
        uint2 pk;
        pk.x = pack2<T>(v[0], v[1]);
        pk.y = pack2<T>(v[2], v[3]);
        *reinterpret_cast<uint2*>(dst) = pk;
      }
    } else {
      dst[0] = from_f32<T>(v[0]);
    }
  }
}

// x: [n_tokens][ldx] in the type `dtype`; mu: float32 [n_mix][E]; prev: float32, element e of slot s at s * prev_stride + e;
// out: [n_mix][n_tokens][E] in the same type as x.
FERRUM_API int ferrum_token_shift_mix(const void* x, int ldx, int dtype, int E, const float* mu, int n_mix, const int* q_start,
                                      const int* req_of_token, const int* slots, float* prev, long long prev_stride, void* out, int n_tokens,
                                      int* counts, int n_counts, cudaStream_t stream) {
  FERRUM_CHECK_ARG(E > 0 && n_mix > 0 && ldx >= E && prev_stride >= E && n_counts >= 0 && n_counts <= 128, "token_shift_mix: bad sizes");
  if (n_tokens == 0) return 0;
  const bool vec = E % 4 == 0 && ldx % 4 == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)out & 15) == 0;
  const int per = vec ? 512 : 128;
  const dim3 grid(n_tokens, (E + per - 1) / per);
  FERRUM_CHECK_ARG(grid.y <= 65535, "token_shift_mix: rows are too wide");
  if (vec)
    FERRUM_DISPATCH_DTYPE(dtype, T, (token_shift_mix_kernel<T, 4><<<grid, 128, 0, stream>>>((const T*)x, ldx, E, mu, n_mix, q_start, req_of_token,
                                                                                           slots, prev, prev_stride, (T*)out, n_tokens, counts, n_counts)));
  else
    FERRUM_DISPATCH_DTYPE(dtype, T, (token_shift_mix_kernel<T, 1><<<grid, 128, 0, stream>>>((const T*)x, ldx, E, mu, n_mix, q_start, req_of_token,
                                                                                           slots, prev, prev_stride, (T*)out, n_tokens, counts, n_counts)));
  FERRUM_CHECK_LAUNCH("token_shift_mix");
  return 0;
}
