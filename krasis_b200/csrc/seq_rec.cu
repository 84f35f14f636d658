// Ragged-batch sequence operators, third part: linear recurrences with per-sequence state slots and the small row kernels of
// designs that run several mixers side by side, average their residual stream over depth or keep several copies of it.
//
//   gla_scan / gla_reg     gated linear attention, S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t per head, with one decay per key
//                          channel alpha = sigmoid(z)^(1 / tau); the state of a (sequence, head, slice of value columns) lives in
//                          registers: a generic form (P lanes share a column and each keeps dk / P of its rows) and, for key sizes
//                          32 / 64 / 128 / 256, a form with lane = column, warp = slice of rows and cp.async token tiles
//                          the generic form also serves the matrix memory of mLSTM, S <- keep_t S + add_t k_t v_t^T with one pair of numbers
//                          per token and head and a further column of ones whose read-out is the normaliser
//   mlstm_reg              the matrix memory for the same key sizes: a lane holds a tile of rows x columns, a warp of its own the key sum
//   mlstm_gates            log gates of mLSTM and their running maximum m_t = max(f_t + m_(t-1), i_t) by a (sum, maximum) scan; keep and add
//                          relative to m_t
//   rglru_scan             real-gated linear recurrent unit: per channel S <- a_t S + sqrt(1 - a_t^2) i_t u_t, times gelu of the other branch;
//                          warps own pieces of the time axis and meet once per tile
//   split_blocks           fp32 rows as a bf16 high and low part side by side, grouped per block of channels: a block-diagonal product of
//                          fp32 inputs on the tensor cores
//   selective_scan         S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n, y_c = sum_n S[c, n] C_n + D_c x_c, times silu(z);
//                          the lanes of a channel keep its states in registers; their pieces of y meet in shared memory once per tile
//   head_norm_gate         per head: o (/ a divisor per head) / rms(o) * w (optional) times silu or sigmoid of a gate column (optional)
//   rms_rows               RMS norm of a column range of strided fp32 rows
//   branch_merge           c (a / rms(a) * wa + b / rms(b) * wb): two mixers that read the same input, each normed, averaged
//   depth_mix              the residual stream as a learned weighted sum of the embedding output and every layer's result, fused with
//                          the residual add that completes the newest result and with the next norm
//   stream_mix             several copies of the residual stream: every copy becomes a weighted sum of all copies plus a share of the
//                          sublayer's output, fused with the weighted sum the next sublayer reads and with its norm
//
// Precision: decays, step sizes, softplus / exponentials, states, norms and every accumulation are fp32; `dt` selects storage only.
#include "seq_common.cuh"

namespace kb2seq {

constexpr int kRecThreads = 256, kRecTok = 16;

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------------ gated linear attention
// q, k [T, ld] (H x dk columns from q_off / k_off), v (H x dv from v_off), decay_in [T, lda] (H x dk logits, + decay_bias).
// Block (sequence s, head h, slice of CB value columns).  Lane l of a warp: column l % CW, key slice p = l / CW of P = 32 / CW;
// thread rows are i = p + P ii, ii < KR.  Tokens are staged kRecTok at a time as (alpha, k, q) triples in shared memory.
// SC (matrix memory): alpha = keep[t, h] for all rows, the keys are multiplied by add[t, h], and column dv of ones keeps the key sum in
// nstate [slots][H][dk]; its read-out becomes den[t, h] = max(|n . q|, exp(-mx[t, h])) + 1e-6.
struct MemoryGates {
  const float* keep;       // [T, H]
  const float* add;
  const float* mx;
  float* nstate;
  float* den;              // [T, H]
};
__device__ __forceinline__ float memory_den(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + 1e-6f; }
template <int KR, bool SC>
__global__ void __launch_bounds__(kRecThreads) gla_scan_kernel(const float* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                                                               const float* __restrict__ decay_in, long long lda,
                                                               const float* __restrict__ decay_bias, float inv_tau, float q_scale, int H,
                                                               int dk, int dv, int P, float* __restrict__ state, const int* __restrict__ cu,
                                                               const int* __restrict__ slots, float* __restrict__ out, MemoryGates mg) {
  extern __shared__ __align__(16) float sm[];
  float4* akq = reinterpret_cast<float4*>(sm);              // [kRecTok][dk]
  const int CW = 32 / P, CB = (kRecThreads / 32) * CW;
  float* vs = sm + 4 * kRecTok * dk;                        // [kRecTok][CB]
  const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CB;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int p = lane / CW, cl = warp * CW + lane % CW, c = c0 + cl;
  const bool ones = SC && c == dv, live = c < dv || ones;
  const int row0 = cu[s], n = cu[s + 1] - row0;
  float* S = ones ? mg.nstate + ((long long)slots[s] * H + h) * dk : state + ((long long)slots[s] * H + h) * dk * dv + c;
  const int pitch = ones ? 1 : dv;
  float st[KR];
#pragma unroll
  for (int ii = 0; ii < KR; ++ii) {
    const int i = p + P * ii;
    st[ii] = (live && i < dk) ? S[(long long)i * pitch] : 0.f;
  }
  for (int t0 = 0; t0 < n; t0 += kRecTok) {
    const int nt = min(kRecTok, n - t0);
    __syncthreads();
    for (int e = tid; e < nt * dk; e += kRecThreads) {
      const int tt = e / dk, i = e - tt * dk;
      const long long t = row0 + t0 + tt;
      float4 f;
      f.y = qkv[t * ld + k_off + h * dk + i];
      if constexpr (SC) {
        f.x = mg.keep[t * H + h];
        f.y *= mg.add[t * H + h];
      } else {
        const float z = decay_in[t * lda + h * dk + i] + (decay_bias ? decay_bias[h * dk + i] : 0.f);
        f.x = expf(-softplus_f(-z) * inv_tau);              // sigmoid(z)^(1 / tau)
      }
      f.z = qkv[t * ld + q_off + h * dk + i] * q_scale;
      f.w = 0.f;
      akq[e] = f;
    }
    for (int e = tid; e < nt * CB; e += kRecThreads) {
      const int tt = e / CB, cc = e - tt * CB;
      vs[e] = c0 + cc < dv ? qkv[(long long)(row0 + t0 + tt) * ld + v_off + h * dv + c0 + cc] : (SC && c0 + cc == dv ? 1.f : 0.f);
    }
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      const float v = vs[tt * CB + cl];
      const float4* row = akq + tt * dk;
      float o = 0.f;
#pragma unroll
      for (int ii = 0; ii < KR; ++ii) {
        const int i = p + P * ii;
        if (i < dk) {
          const float4 f = row[i];
          st[ii] = fmaf(st[ii], f.x, f.y * v);
          o = fmaf(st[ii], f.z, o);
        }
      }
      for (int off = CW; off < 32; off <<= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
      const long long th = (long long)(row0 + t0 + tt) * H + h;
      if (p == 0 && live) {
        if (ones) mg.den[th] = memory_den(o, mg.mx[th]);
        else out[th * dv + c] = o;
      }
    }
  }
#pragma unroll
  for (int ii = 0; ii < KR; ++ii) {
    const int i = p + P * ii;
    if (live && i < dk) S[(long long)i * pitch] = st[ii];
  }
}

// The same recurrence for key sizes 32, 64, 128 and 256 with value sizes that are multiples of 32 (the sizes of real models): a block
// owns 32 value columns of a (sequence, head); lane = column, so that the state moves in whole 128-byte rows; warp w keeps rows
// [w DK / 8, (w + 1) DK / 8) of its column in registers.  A token's alpha, k and q values are the same address for every lane (one
// shared-memory transaction per 16 bytes); tiles of kGlaTile tokens arrive by cp.async, double-buffered, from the projection itself and
// from the decays that gla_decay_kernel wrote; the warps' pieces of S^T q meet in shared memory once per tile.  No barrier inside a token.
__global__ void gla_decay_kernel(const float* __restrict__ decay_in, long long lda, const float* __restrict__ decay_bias, float inv_tau,
                                 long long T, int n, float* __restrict__ alpha) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= T * n) return;
  const long long t = i / n;
  const int c = (int)(i - t * n);
  const float z = decay_in[t * lda + c] + (decay_bias ? decay_bias[c] : 0.f);
  alpha[i] = expf(-softplus_f(-z) * inv_tau);
}

__device__ __forceinline__ void rec_cp_async16(void* smem_dst, const void* gmem_src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ void rec_cp_async4(void* smem_dst, const void* gmem_src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ void rec_cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void rec_cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

constexpr int kGlaTile = 8, kGlaWarps = 8;
template <int DK>
__global__ void __launch_bounds__(32 * kGlaWarps) gla_reg_kernel(const float* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                                                                 const float* __restrict__ alpha, float q_scale, int H, int dv,
                                                                 float* __restrict__ state, const int* __restrict__ cu,
                                                                 const int* __restrict__ slots, float* __restrict__ out) {
  constexpr int P = kGlaWarps, NT = 32 * P, Q = DK / P;
  extern __shared__ __align__(16) float sm[];
  float* as = sm;                                   // [2][kGlaTile][DK]
  float* ks = as + 2 * kGlaTile * DK;
  float* qs = ks + 2 * kGlaTile * DK;
  float* vs = qs + 2 * kGlaTile * DK;               // [2][kGlaTile][32]
  float* os_part = vs + 2 * kGlaTile * 32;          // [kGlaTile][P][32]
  const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 32;
  const int tid = threadIdx.x, lane = tid & 31, piece = tid >> 5;
  const int t0 = cu[s], n = cu[s + 1] - cu[s];
  float* Sg = state + ((long long)slots[s] * H + h) * DK * dv;
  float S[Q];
#pragma unroll
  for (int ii = 0; ii < Q; ++ii) S[ii] = Sg[(long long)(piece * Q + ii) * dv + j0 + lane];

  auto load_tile = [&](int buf, int b0) {
    const int nt = min(kGlaTile, n - b0);
    for (int c = tid; c < nt * (DK / 4); c += NT) {                  // 16-byte chunks of the alpha, k and q rows
      const int tt = c / (DK / 4), cc = c - tt * (DK / 4);
      const long long row = t0 + b0 + tt;
      const int dst = (buf * kGlaTile + tt) * DK + cc * 4;
      rec_cp_async16(as + dst, alpha + (row * H + h) * DK + cc * 4);
      rec_cp_async16(ks + dst, qkv + row * ld + k_off + h * DK + cc * 4);
      rec_cp_async16(qs + dst, qkv + row * ld + q_off + h * DK + cc * 4);
    }
    for (int c = tid; c < nt * 8; c += NT) {
      const int tt = c >> 3, cc = c & 7;
      rec_cp_async16(vs + (buf * kGlaTile + tt) * 32 + cc * 4, qkv + (long long)(t0 + b0 + tt) * ld + v_off + h * dv + j0 + cc * 4);
    }
    rec_cp_async_commit();
  };

  load_tile(0, 0);
  int buf = 0;
  for (int b0 = 0; b0 < n; b0 += kGlaTile, buf ^= 1) {
    const int nt = min(kGlaTile, n - b0);
    rec_cp_async_wait_all();
    __syncthreads();                                  // tile `buf` is in place; everyone is done with the other buffer and with os_part
    if (b0 + kGlaTile < n) load_tile(buf ^ 1, b0 + kGlaTile);
    for (int tt = 0; tt < nt; ++tt) {
      const int base = (buf * kGlaTile + tt) * DK + piece * Q;
      const float4* a4 = reinterpret_cast<const float4*>(as + base);
      const float4* k4 = reinterpret_cast<const float4*>(ks + base);
      const float4* q4 = reinterpret_cast<const float4*>(qs + base);
      const float vv = vs[(buf * kGlaTile + tt) * 32 + lane];
      float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
      for (int ii = 0; ii < Q / 4; ++ii) {
        const float4 ar = a4[ii], kr = k4[ii], qr = q4[ii];
        S[4 * ii] = fmaf(S[4 * ii], ar.x, kr.x * vv);
        S[4 * ii + 1] = fmaf(S[4 * ii + 1], ar.y, kr.y * vv);
        S[4 * ii + 2] = fmaf(S[4 * ii + 2], ar.z, kr.z * vv);
        S[4 * ii + 3] = fmaf(S[4 * ii + 3], ar.w, kr.w * vv);
        a0 = fmaf(S[4 * ii], qr.x, a0);
        a1 = fmaf(S[4 * ii + 1], qr.y, a1);
        a2 = fmaf(S[4 * ii + 2], qr.z, a2);
        a3 = fmaf(S[4 * ii + 3], qr.w, a3);
      }
      os_part[(tt * P + piece) * 32 + lane] = (a0 + a1) + (a2 + a3);
    }
    __syncthreads();
    for (int i = tid; i < nt * 32; i += NT) {
      const int tt = i >> 5, c = i & 31;
      float o = 0.f;
#pragma unroll
      for (int p = 0; p < P; ++p) o += os_part[(tt * P + p) * 32 + c];
      out[((long long)(t0 + b0 + tt) * H + h) * dv + j0 + c] = o * q_scale;
    }
  }
#pragma unroll
  for (int ii = 0; ii < Q; ++ii) Sg[(long long)(piece * Q + ii) * dv + j0 + lane] = S[ii];
}

// ------------------------------------------------------------------------------------------------ matrix memory (mLSTM)
// Log gates per (token, head): i = cap tanh((zi + bi) / cap), f = logsigmoid(cap tanh((zf + bf) / cap)); the running maximum
// m_t = max(f_t + m_(t-1), i_t); keep = exp(f_t + m_(t-1) - m_t), add = exp(i_t - m_t).  A block per (sequence, head), a thread per token
// of the tile: (F, M) pairs compose as (F1 + F2, max(M1 + F2, M2)), so m_t = max(F + m_0, M) over the prefix.  Everything in fp64; m_t is
// rounded to fp32 at every token and keep / add are taken relative to the rounded values: the matrix and its maximum agree exactly
// wherever a prompt is cut, and the rounding of m cancels.
constexpr int kGateThreads = 1024;
__device__ __forceinline__ double softplus_d(double z) { return z > 40.0 ? z : log1p(exp(z)); }
__global__ void __launch_bounds__(kGateThreads) mlstm_gates_kernel(const float* __restrict__ proj, long long ld, int i_off, int f_off,
                                                                   const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap,
                                                                   int H, float* __restrict__ mstate, const int* __restrict__ cu,
                                                                   const int* __restrict__ slots, float* __restrict__ keep,
                                                                   float* __restrict__ add, float* __restrict__ mx) {
  __shared__ double wF[32], wM[32];
  __shared__ float ms[kGateThreads + 1];             // ms[1 + k]: m of the tile's token k, ms[0]: m before the tile
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = cu[s], n = cu[s + 1] - t0;
  float* mp = mstate + (long long)slots[s] * H + h;
  const double c = cap, bi = i_bias ? i_bias[h] : 0.f, bf = f_bias ? f_bias[h] : 0.f;
  float m0 = *mp;
  for (int b0 = 0; b0 < n; b0 += blockDim.x) {
    const int nt = min((int)blockDim.x, n - b0);
    const long long t = t0 + b0 + tid;
    double f = 0.0, i = -1e300;                      // a place without a token: the neutral pair
    if (tid < nt) {
      i = c * tanh(((double)proj[t * ld + i_off + h] + bi) / c);
      f = -softplus_d(-c * tanh(((double)proj[t * ld + f_off + h] + bf) / c));
    }
    double F = f, M = i;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmax(Mp + F, M);
        F += Fp;
      }
    }
    if (lane == 31) {
      wF[warp] = F;
      wM[warp] = M;
    }
    if (tid == 0) ms[0] = m0;
    __syncthreads();
    double m = m0;                                   // the maximum ahead of this warp's first token
    for (int w = 0; w < warp; ++w) m = fmax(wF[w] + m, wM[w]);
    m = fmax(F + m, M);
    ms[1 + tid] = (float)m;
    __syncthreads();
    if (tid < nt) {
      const double prev = ms[tid], cur = ms[1 + tid];
      keep[t * H + h] = (float)exp(f + prev - cur);
      add[t * H + h] = (float)exp(i - cur);
      mx[t * H + h] = ms[1 + tid];
    }
    m0 = ms[nt];
    __syncthreads();
  }
  if (tid == 0) *mp = m0;
}

// two fp32 lanes of one 64-bit register (packed FMA of sm_100)
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float sum2(uint64_t v) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
  return lo + hi;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// The recurrence of the matrix memory in registers: a block owns 32 value columns of a (sequence, head); warp w keeps DK / 8 rows of them, a
// lane a tile of R rows x CPL columns (128 keys: 4 x 4), so that a 16-byte read of k, q or v serves several state elements; row pairs sit in
// 64-bit registers.  Tiles of kMemTile tokens arrive by cp.async, kMemStages deep (the recurrence of a tile is shorter than a trip to memory).
// The lanes' and warps' pieces of S^T q meet in shared memory while the next tile runs: one barrier per tile.  In the first block of a head
// (blockIdx.z == 0) one more warp keeps the key sum, DK / 32 rows per lane.
constexpr int kMemTile = 8, kMemWarps = 8, kMemStages = 4, kMemUnroll = 2;
static_assert(kMemTile == kMemWarps, "the read-outs take a warp per token of the tile");
template <int DK> struct MemShape {
  static constexpr int Q = DK / kMemWarps;             // rows of a warp
  static constexpr int RG = DK == 32 ? 2 : 4;          // row groups of its lanes; 32 / RG column groups of CPL = RG columns
  static constexpr int R = Q / RG, CPL = RG;
  static constexpr int kFloats = kMemStages * kMemTile * (2 * DK + 32 + 4) + 2 * kMemTile * (kMemWarps * RG * 32 + 32 + 1);
};
template <int N> __device__ __forceinline__ void ld_vec(const float* p, float* v) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      const float4 f = *reinterpret_cast<const float4*>(p + 4 * i);
      v[4 * i] = f.x; v[4 * i + 1] = f.y; v[4 * i + 2] = f.z; v[4 * i + 3] = f.w;
    }
  } else if constexpr (N == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = p[0];
  }
}
template <int N> __device__ __forceinline__ void st_vec(float* p, const float* v) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}
template <int DK>
__global__ void __launch_bounds__(32 * (kMemWarps + 1), 1) mlstm_reg_kernel(const float* __restrict__ qkv, long long ld, int q_off, int k_off, int v_off,
                                                                   float q_scale, int H, int dv, float* __restrict__ state,
                                                                   const int* __restrict__ cu, const int* __restrict__ slots,
                                                                   float* __restrict__ out, MemoryGates mg) {
  using M = MemShape<DK>;
  constexpr int P = kMemWarps, NT = 32 * (P + 1), Q = M::Q, R = M::R, CPL = M::CPL, RG = M::RG, NP = P * RG, KR = DK / 32;
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                                      // [kMemStages][kMemTile][DK]
  float* qs = ks + kMemStages * kMemTile * DK;
  float* vs = qs + kMemStages * kMemTile * DK;         // [kMemStages][kMemTile][32]
  float* os_part = vs + kMemStages * kMemTile * 32;    // [2][kMemTile][NP][32]
  float* n_part = os_part + 2 * kMemTile * NP * 32;    // [2][kMemTile][32]
  float* m_part = n_part + 2 * kMemTile * 32;          // [2][kMemTile]: m of the token
  float* gs = m_part + 2 * kMemTile;                       // [kMemStages][kMemTile][4]: keep, add, mx, -
  const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 32;
  const int tid = threadIdx.x, lane = tid & 31, piece = tid >> 5;
  const int rg = lane / (32 / RG), row0 = piece * Q + rg * R, col0 = (lane % (32 / RG)) * CPL;
  const int t0 = cu[s], n = cu[s + 1] - cu[s];
  const long long head = (long long)slots[s] * H + h;
  float* Sg = state + head * DK * dv + (long long)row0 * dv + j0 + col0;
  uint64_t S[R / 2][CPL];                              // S[i][c]: rows row0 + 2 i, row0 + 2 i + 1 of column col0 + c
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    float lo[CPL] = {}, hi[CPL] = {};
    if (piece < P) {
      ld_vec<CPL>(Sg + (long long)(2 * i) * dv, lo);
      ld_vec<CPL>(Sg + (long long)(2 * i + 1) * dv, hi);
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) S[i][c] = pack2(lo[c], hi[c]);
  }
  const bool sums = blockIdx.z == 0 && piece == P;     // the warp of the key sum: rows lane KR .. lane KR + KR - 1
  float* Ng = mg.nstate + head * DK + lane * KR;
  float nsum[KR];
#pragma unroll
  for (int i = 0; i < KR; ++i) nsum[i] = sums ? Ng[i] : 0.f;

  auto load_tile = [&](int buf, int b0) {
    const int nt = min(kMemTile, n - b0);
    for (int c = tid; c < nt * (DK / 4); c += NT) {                  // 16-byte chunks of the k and q rows
      const int tt = c / (DK / 4), cc = c - tt * (DK / 4);
      const float* row = qkv + (long long)(t0 + b0 + tt) * ld + h * DK + cc * 4;
      const int dst = (buf * kMemTile + tt) * DK + cc * 4;
      rec_cp_async16(ks + dst, row + k_off);
      rec_cp_async16(qs + dst, row + q_off);
    }
    if (tid < nt * 8) {
      const int tt = tid >> 3, cc = tid & 7;
      rec_cp_async16(vs + (buf * kMemTile + tt) * 32 + cc * 4, qkv + (long long)(t0 + b0 + tt) * ld + v_off + h * dv + j0 + cc * 4);
    }
    if (tid < 4 * nt && (tid & 3) < 3)
      rec_cp_async4(gs + buf * kMemTile * 4 + tid, ((tid & 3) == 0 ? mg.keep : (tid & 3) == 1 ? mg.add : mg.mx) + (long long)(t0 + b0 + (tid >> 2)) * H + h);
  };
#pragma unroll
  for (int st = 0; st < kMemStages - 1; ++st) {
    if (st * kMemTile < n) load_tile(st, st * kMemTile);
    rec_cp_async_commit();
  }
  // read-out of the tile that starts at b0: a warp per token, a lane per column
  auto read_out = [&](int b0, int half) {
    if (piece >= min(kMemTile, n - b0)) return;
    const long long th = (long long)(t0 + b0 + piece) * H + h;
    float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
    const float* pp = os_part + (half * kMemTile + piece) * NP * 32 + lane;
#pragma unroll
    for (int p = 0; p < NP; p += 4) {
      o0 += pp[p * 32];
      o1 += pp[p * 32 + 32];
      o2 += pp[p * 32 + 64];
      o3 += pp[p * 32 + 96];
    }
    out[th * dv + j0 + lane] = ((o0 + o1) + (o2 + o3)) * q_scale;
    if (blockIdx.z == 0) {
      const float nq = warp_sum(n_part[(half * kMemTile + piece) * 32 + lane]);
      if (lane == 0) mg.den[th] = memory_den(nq * q_scale, m_part[half * kMemTile + piece]);
    }
  };
  int buf = 0, half = 0;
  for (int b0 = 0; b0 < n; b0 += kMemTile, buf = buf + 1 == kMemStages ? 0 : buf + 1, half ^= 1) {
    const int nt = min(kMemTile, n - b0), ahead = b0 + (kMemStages - 1) * kMemTile;
    asm volatile("cp.async.wait_group %0;" ::"n"(kMemStages - 2) : "memory");
    __syncthreads();                                   // tile `buf` and the pieces of the tile before it are in place; everyone is done with that tile's inputs
    if (ahead < n) load_tile(buf == 0 ? kMemStages - 1 : buf - 1, ahead);
    rec_cp_async_commit();                             // a group per tile, empty at the end: the wait above counts groups
    if (b0 > 0) read_out(b0 - kMemTile, half ^ 1);
    auto token = [&](int tt, float* o) {
      const int at = buf * kMemTile + tt;
      float kf[R], qf[R], v[CPL];
      ld_vec<R>(ks + at * DK + row0, kf);
      ld_vec<R>(qs + at * DK + row0, qf);
      ld_vec<CPL>(vs + at * 32 + col0, v);
      const float2 g = *reinterpret_cast<const float2*>(gs + at * 4);
      const uint64_t keep = pack2(g.x, g.x);
      uint64_t k2[R / 2], q2[R / 2];
#pragma unroll
      for (int i = 0; i < R / 2; ++i) {
        k2[i] = pack2(kf[2 * i], kf[2 * i + 1]);
        q2[i] = pack2(qf[2 * i], qf[2 * i + 1]);
      }
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const float va = v[c] * g.y;
        const uint64_t v2 = pack2(va, va);
        uint64_t acc = 0;
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
          S[i][c] = fma2(S[i][c], keep, mul2(k2[i], v2));
          acc = i == 0 ? mul2(S[i][c], q2[i]) : fma2(S[i][c], q2[i], acc);
        }
        o[c] = sum2(acc);
      }
    };
    auto keep_piece = [&](int tt, const float* o) { st_vec<CPL>(os_part + ((half * kMemTile + tt) * NP + piece * RG + rg) * 32 + col0, o); };
    if (sums) {
#pragma unroll 2
      for (int tt = 0; tt < nt; ++tt) {
        const int at = buf * kMemTile + tt;
        float kf[KR], qf[KR], o = 0.f;
        ld_vec<KR>(ks + at * DK + lane * KR, kf);
        ld_vec<KR>(qs + at * DK + lane * KR, qf);
        const float2 g = *reinterpret_cast<const float2*>(gs + at * 4);
#pragma unroll
        for (int i = 0; i < KR; ++i) {
          nsum[i] = fmaf(nsum[i], g.x, kf[i] * g.y);
          o = fmaf(nsum[i], qf[i], o);
        }
        n_part[(half * kMemTile + tt) * 32 + lane] = o;
        if (lane == 0) m_part[half * kMemTile + tt] = gs[at * 4 + 2];
      }
    } else if (piece == P) {
      // nothing to keep in the other blocks
    } else if (nt == kMemTile) {
#pragma unroll
      for (int t4 = 0; t4 < kMemTile; t4 += kMemUnroll) {     // stores after kMemUnroll tokens, so that their loads are in flight together
        float o[kMemUnroll][CPL];
#pragma unroll
        for (int tt = 0; tt < kMemUnroll; ++tt) token(t4 + tt, o[tt]);
#pragma unroll
        for (int tt = 0; tt < kMemUnroll; ++tt) keep_piece(t4 + tt, o[tt]);
      }
    } else {
      for (int tt = 0; tt < nt; ++tt) {
        float o[CPL];
        token(tt, o);
        keep_piece(tt, o);
      }
    }
  }
  __syncthreads();
  if (n > 0) read_out((n - 1) / kMemTile * kMemTile, half ^ 1);
  if (sums) {
#pragma unroll
    for (int i = 0; i < KR; ++i) Ng[i] = nsum[i];
  }
  if (piece == P) return;
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    float lo[CPL], hi[CPL];
#pragma unroll
    for (int c = 0; c < CPL; ++c) asm("mov.b64 {%0, %1}, %2;" : "=f"(lo[c]), "=f"(hi[c]) : "l"(S[i][c]));
    st_vec<CPL>(Sg + (long long)(2 * i) * dv, lo);
    st_vec<CPL>(Sg + (long long)(2 * i + 1) * dv, hi);
  }
}

// ------------------------------------------------------------------------------------------------ real-gated linear recurrent unit
// u [T, ldu]: convolved inputs of C channels in blocks of bs; z: gate products, the pair of channel c = b bs + j at z + t ldz + b zb + j
// (recurrence gate) and + bs (input gate); y [T, ldy] the other branch.  Per channel
//   log a = rate sigmoid(z_r + r_bias),  S <- a S + sqrt(1 - a^2) sigmoid(z_i + i_bias) u,  out = S gelu_tanh(y + y_bias).
// a = 1 + expm1(log a) and 1 - a^2 = -expm1 (2 + expm1): exact where a is next to one.  A block owns CG groups of 32 channels (lane = channel)
// of a sequence; warp w of the NW warps of a group takes tokens [TOK w, TOK w + TOK) of a tile, composes its (a, b) pairs from S = 0, and the
// warps' compositions meet in shared memory once per tile.  The next tile's inputs are in registers before this one's are used.
// NW = 1 serves steps of single tokens.
constexpr int kRgWarps = 16, kRgTok = 8, kRgGroups = 4;
__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.f, 1.f + expf(-z)); }      // both ends come out right: exp = inf gives 0
__device__ __forceinline__ float sqrt_approx(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// y gelu's factor: 0.5 (1 + tanh(t)) = sigmoid(2 t)
__device__ __forceinline__ float gelu_tanh_f(float y) { return y * sigmoid_f(1.5957691216057308f * y * fmaf(0.044715f * y, y, 1.f)); }
template <int NW, int CG, int TOK>
__global__ void __launch_bounds__(32 * NW * CG, 1) rglru_scan_kernel(const float* __restrict__ u, long long ldu, const float* __restrict__ z,
                                                                   long long ldz, long long zb, const float* __restrict__ y, long long ldy,
                                                                   const float* __restrict__ r_bias, const float* __restrict__ i_bias,
                                                                   const float* __restrict__ y_bias, const float* __restrict__ rate_c, int C, int bs,
                                                                   float* __restrict__ state, const int* __restrict__ cu,
                                                                   const int* __restrict__ slots, void* __restrict__ out, int dt_out) {
  __shared__ float Aw[2][CG][NW][32], Bw[2][CG][NW][32];
  const int s = blockIdx.x, lane = threadIdx.x & 31, grp = (threadIdx.x >> 5) / NW, warp = (threadIdx.x >> 5) % NW;
  const int c = (blockIdx.y * CG + grp) * 32 + lane;
  const bool live = c < C;
  const int row0 = cu[s], n = cu[s + 1] - row0;
  float* Sp = state + (long long)slots[s] * C + c;
  float carry = live ? *Sp : 0.f;
  const float rb = live && r_bias ? r_bias[c] : 0.f, ib = live && i_bias ? i_bias[c] : 0.f, yb = live && y_bias ? y_bias[c] : 0.f;
  const float rate = live ? rate_c[c] : 0.f;
  const int blk = live ? c / bs : 0;
  // rows of the next tile's first token of this warp; the tile's tokens lie a row stride apart
  const long long first = row0 + warp * TOK;
  const float* zp = z + blk * zb + (c - blk * bs) + first * ldz;
  const float* up = u + first * ldu + c;
  const float* yp = y + first * ldy + c;
  struct In { float u, r, i, y; };
  In cur[TOK], nxt[TOK];
  auto load = [&](In* in, int b0) {
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      const int tt = b0 + warp * TOK + k;
      in[k] = {0.f, 0.f, 0.f, 0.f};
      if (live && tt < n) in[k] = {up[k * ldu], zp[k * ldz], zp[k * ldz + bs], yp[k * ldy]};
    }
    up += NW * TOK * ldu;
    zp += NW * TOK * ldz;
    yp += NW * TOK * ldy;
  };
  load(cur, 0);
  int buf = 0;
  for (int b0 = 0; b0 < n; b0 += NW * TOK, buf ^= 1) {
    if (b0 + NW * TOK < n) load(nxt, b0 + NW * TOK);
    float a[TOK], b[TOK], A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      a[k] = 1.f;                                     // a place without a token leaves the state as it is
      b[k] = 0.f;
      if (live && b0 + warp * TOK + k < n) {
        const float e = expm1f(rate * sigmoid_f(cur[k].r + rb));
        a[k] = 1.f + e;
        b[k] = sqrt_approx(-e * (2.f + e)) * sigmoid_f(cur[k].i + ib) * cur[k].u;
      }
      A *= a[k];
      B = fmaf(a[k], B, b[k]);
    }
    float mine = carry;
    if constexpr (NW == 1) {
      carry = fmaf(A, carry, B);
    } else {
      Aw[buf][grp][warp][lane] = A;
      Bw[buf][grp][warp][lane] = B;
      __syncthreads();                                // one barrier per tile: the other buffer is written only after the next one
      float S = carry;
#pragma unroll
      for (int w = 0; w < NW; ++w) {
        if (w == warp) mine = S;
        S = fmaf(Aw[buf][grp][w][lane], S, Bw[buf][grp][w][lane]);
      }
      carry = S;
    }
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      const int tt = b0 + warp * TOK + k;
      mine = fmaf(a[k], mine, b[k]);
      if (live && tt < n) st_dt(out, dt_out, (long long)(row0 + tt) * C + c, mine * gelu_tanh_f(cur[k].y + yb));
      cur[k] = nxt[k];
    }
  }
  if (warp == 0 && live) *Sp = carry;
}

// u [T, ldu] fp32 -> out [blocks][Tp][2 bs] bf16: row (b, t) holds the channels of block b as [high | low], high + low = u up to 2^-17 |u|
__global__ void __launch_bounds__(256) split_blocks_kernel(const float* __restrict__ u, long long ldu, long long T, long long Tp, int blocks, int bs,
                                                           bf16* __restrict__ out) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;     // a pair of channels
  const int half = bs >> 1;
  if (i >= T * blocks * half) return;
  const long long t = i / (blocks * half);
  const int r = (int)(i - t * blocks * half), b = r / half, j = (r - b * half) * 2;
  const float v0 = u[t * ldu + b * bs + j], v1 = u[t * ldu + b * bs + j + 1];
  const __nv_bfloat162 hi = __floats2bfloat162_rn(v0, v1);
  const float2 back = __bfloat1622float2(hi);
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v0 - back.x, v1 - back.y);
  bf16* row = out + (b * Tp + t) * 2 * bs + j;
  *reinterpret_cast<__nv_bfloat162*>(row) = hi;
  *reinterpret_cast<__nv_bfloat162*>(row + bs) = lo;
}

// ------------------------------------------------------------------------------------------------ selective scan
// x [T, ldx] (inner channels after convolution and activation), dt_in [T, ldd] (+ dt_bias, then softplus), bc [T, ldb] = [B: N | C: N]
// from b_off, z [T, ldz] from z_off, A_log [inner, N], D [inner].  Block (sequence, group of CB channels); lane l: state slice
// p = l % P, channel l / P of the warp; thread states are n = p + P ii, ii < NR.
__device__ __forceinline__ float ex2_approx_ftz(float x) {       // 2^x, MUFU.EX2 (2 ulp, as exp2f); results below 2^-126 become 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Tiles of kRecTok tokens arrive by cp.async, double-buffered (dt input, x, z of the block's channels; B and C of the token), so that
// the loads of the next tile run under the recurrence of this one.  Per tile: step sizes (softplus) once per (token, channel); the
// recurrence with nothing but shared memory and registers inside and no exchange between lanes; then the lanes' pieces of y are summed,
// D x added, the gate applied and the rows written.
template <int NR>
__global__ void __launch_bounds__(kRecThreads) selective_scan_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ dt_in,
                                                                     long long ldd, const float* __restrict__ dt_bias,
                                                                     const float* __restrict__ bc, long long ldb, int b_off,
                                                                     const float* __restrict__ z, long long ldz, int z_off,
                                                                     const float* __restrict__ A_log, const float* __restrict__ Dw, int inner,
                                                                     int N, int P, float* __restrict__ state, const int* __restrict__ cu,
                                                                     const int* __restrict__ slots, void* __restrict__ out, int dt_out) {
  extern __shared__ __align__(16) float sm[];
  const int CW = 32 / P, CB = (kRecThreads / 32) * CW;
  float* bcs = sm;                                   // [2][kRecTok][2 N]: B | C of the token
  float* dts = bcs + 2 * kRecTok * 2 * N;            // [2][kRecTok][CB]: dt input, then the step size
  float* xs = dts + 2 * kRecTok * CB;                // [2][kRecTok][CB]
  float* zs = xs + 2 * kRecTok * CB;                 // [2][kRecTok][CB]
  float* yp = zs + 2 * kRecTok * CB;                 // [kRecTok][CB][P + 1]: every lane's piece of y, summed once per tile (odd pitch: no bank conflicts)
  const int s = blockIdx.x, c0 = blockIdx.y * CB;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int p = lane % P, cl = warp * CW + lane / P, c = c0 + cl;   // tid == cl * P + p
  const bool live = c < inner;
  const int row0 = cu[s], n = cu[s + 1] - row0;
  float* S = state + (long long)slots[s] * inner * N;
  float st[NR], a[NR];
#pragma unroll
  for (int ii = 0; ii < NR; ++ii) {
    const int j = p + P * ii;
    const bool ok = live && j < N;
    st[ii] = ok ? S[(long long)c * N + j] : 0.f;
    a[ii] = ok ? -expf(A_log[(long long)c * N + j]) * 1.4426950408889634f : 0.f;      // A log2(e): exp(dt A) = 2^(dt a)
  }
  const int cb_shift = __ffs(CB) - 1;                // CB = 256 / P is a power of two: rows and channels of a tile by shift and mask

  auto load_tile = [&](int buf, int b0) {
    const int nt = min(kRecTok, n - b0);
    for (int e = tid; e < nt * 2 * N; e += kRecThreads) {
      const int tt = e / (2 * N), j = e - tt * 2 * N;
      rec_cp_async4(bcs + (buf * kRecTok + tt) * 2 * N + j, bc + (long long)(row0 + b0 + tt) * ldb + b_off + j);
    }
    for (int e = tid; e < nt * CB; e += kRecThreads) {
      const int tt = e >> cb_shift, cc = e & (CB - 1);
      if (c0 + cc >= inner) continue;
      const long long t = row0 + b0 + tt;
      const int dst = (buf * kRecTok + tt) * CB + cc;
      rec_cp_async4(dts + dst, dt_in + t * ldd + c0 + cc);
      rec_cp_async4(xs + dst, x + t * ldx + c0 + cc);
      rec_cp_async4(zs + dst, z + t * ldz + z_off + c0 + cc);
    }
    rec_cp_async_commit();
  };

  load_tile(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += kRecTok, buf ^= 1) {
    const int nt = min(kRecTok, n - t0);
    rec_cp_async_wait_all();
    __syncthreads();                                 // tile `buf` is in place; everyone is done with the other buffer and with yp
    if (t0 + kRecTok < n) load_tile(buf ^ 1, t0 + kRecTok);
    for (int e = tid; e < nt * CB; e += kRecThreads) {
      const int cc = e & (CB - 1);
      if (c0 + cc >= inner) continue;
      float* d = dts + buf * kRecTok * CB + e;
      *d = softplus_f(*d + dt_bias[c0 + cc]);
    }
    __syncthreads();
    if (live) {
      const float* dp = dts + buf * kRecTok * CB + cl;
      const float* xq = xs + buf * kRecTok * CB + cl;
      const float* row = bcs + buf * kRecTok * 2 * N + p;
      float* yq = yp + cl * (P + 1) + p;
      const int ypitch = CB * (P + 1);
#pragma unroll 4
      for (int tt = 0; tt < nt; ++tt, dp += CB, xq += CB, row += 2 * N, yq += ypitch) {
        const float dtv = *dp;
        const float dtx = dtv * *xq;
        float y = 0.f;
#pragma unroll
        for (int ii = 0; ii < NR; ++ii) {
          if (p + P * ii < N) {                      // a[] is A log2(e): one MUFU per state update
            st[ii] = fmaf(ex2_approx_ftz(dtv * a[ii]), st[ii], dtx * row[P * ii]);
            y = fmaf(st[ii], row[N + P * ii], y);
          }
        }
        *yq = y;
      }
    }
    __syncthreads();
    for (int e = tid; e < nt * CB; e += kRecThreads) {
      const int tt = e >> cb_shift, cc = e & (CB - 1);
      if (c0 + cc >= inner) continue;
      const float* pieces = yp + (tt * CB + cc) * (P + 1);
      float y = 0.f;
      for (int q = 0; q < P; ++q) y += pieces[q];
      const int src = (buf * kRecTok + tt) * CB + cc;
      y = fmaf(Dw[c0 + cc], xs[src], y);
      st_dt(out, dt_out, (long long)(row0 + t0 + tt) * inner + c0 + cc, y * silu(zs[src]));
    }
  }
#pragma unroll
  for (int ii = 0; ii < NR; ++ii) {
    const int j = p + P * ii;
    if (live && j < N) S[(long long)c * N + j] = st[ii];
  }
}

// ------------------------------------------------------------------------------------------------ row kernels
// out[t, h, :] = o[t, h, :] (/ den[t, h]) (/ rms * w[:] if w) (* act(gate[t, h dv + :]) if gate); a warp per (token, head).  gate_act 0: silu,
// 1: sigmoid.  w_heads: w [H dv], weights of their own for every head
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, long long ldo, const float* __restrict__ w, float eps,
                                                             const float* __restrict__ gate, long long ldg, int gate_act, int H, int dv,
                                                             long long T, void* __restrict__ out, int dt_out,
                                                             const float* __restrict__ den, int w_heads) {
  const long long wi = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wi >= T * H) return;
  const long long t = wi / H;
  const int h = (int)(wi - t * H);
  const float* row = o + t * ldo + (long long)h * dv;
  const float dinv = den != nullptr ? 1.f / den[wi] : 1.f;
  float rstd = dinv;
  if (w != nullptr) {
    float ss = 0.f;
    for (int j = lane; j < dv; j += 32) {
      const float v = row[j] * dinv;
      ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    rstd = dinv / sqrtf(ss / (float)dv + eps);
    if (w_heads) w += (long long)h * dv;
  }
  for (int j = lane; j < dv; j += 32) {
    float v = row[j] * rstd;
    if (w != nullptr) v *= w[j];
    if (gate != nullptr) {
      const float gz = gate[t * ldg + h * dv + j];
      v *= gate_act ? 1.f / (1.f + expf(-gz)) : silu(gz);
    }
    st_dt(out, dt_out, wi * dv + j, v);
  }
}

// the same for value sizes that are multiples of 4 up to 128 NV and 16-byte rows: a lane keeps its columns in registers
template <int NV>
__global__ void __launch_bounds__(256) head_norm_gate_vec_kernel(const float* __restrict__ o, long long ldo, const float* __restrict__ w, float eps,
                                                                 const float* __restrict__ gate, long long ldg, int gate_act, int H, int dv,
                                                                 long long T, void* __restrict__ out, int dt_out, const float* __restrict__ den,
                                                                 int w_heads) {
  const long long wi = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wi >= T * H) return;
  const long long t = wi / H;
  const int h = (int)(wi - t * H);
  const float* row = o + t * ldo + (long long)h * dv;
  const float* gr = gate != nullptr ? gate + t * ldg + (long long)h * dv : nullptr;
  float4 v[NV], g[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = (lane + 32 * i) * 4;
    v[i] = j < dv ? *reinterpret_cast<const float4*>(row + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (gr != nullptr && j < dv) g[i] = *reinterpret_cast<const float4*>(gr + j);
  }
  const float dinv = den != nullptr ? 1.f / den[wi] : 1.f;
  float rstd = dinv;
  if (w != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const float a = v[i].x * dinv, b = v[i].y * dinv, c = v[i].z * dinv, d = v[i].w * dinv;
      ss = fmaf(a, a, ss);
      ss = fmaf(b, b, ss);
      ss = fmaf(c, c, ss);
      ss = fmaf(d, d, ss);
    }
    rstd = dinv / sqrtf(warp_sum(ss) / (float)dv + eps);
    if (w_heads) w += (long long)h * dv;
  }
  auto act = [&](float z) { return gate_act ? 1.f / (1.f + expf(-z)) : silu(z); };
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int j = (lane + 32 * i) * 4;
    if (j >= dv) continue;
    float4 r = make_float4(v[i].x * rstd, v[i].y * rstd, v[i].z * rstd, v[i].w * rstd);
    if (w != nullptr) {
      const float4 ww = *reinterpret_cast<const float4*>(w + j);
      r.x *= ww.x; r.y *= ww.y; r.z *= ww.z; r.w *= ww.w;
    }
    if (gr != nullptr) {
      r.x *= act(g[i].x); r.y *= act(g[i].y); r.z *= act(g[i].z); r.w *= act(g[i].w);
    }
    if (dt_out) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
      uint2 p;
      p.x = *reinterpret_cast<const uint32_t*>(&lo);
      p.y = *reinterpret_cast<const uint32_t*>(&hi);
      *reinterpret_cast<uint2*>((bf16*)out + wi * dv + j) = p;
    } else {
      *reinterpret_cast<float4*>((float*)out + wi * dv + j) = r;
    }
  }
}

// out[t, :n] = in[t, :n] / rms * w; a block per row
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* __restrict__ in, long long ld_in, int n, const float* __restrict__ w,
                                                       float eps, void* __restrict__ out, int dt_out, long long ld_out) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const float* r = in + t * ld_in;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(r[i], r[i], ss);
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) st_dt(out, dt_out, t * ld_out + i, r[i] * rstd * w[i]);
}

// out[t] = coef (a[t] / rms(a[t]) * wa + b[t] / rms(b[t]) * wb)
__global__ void __launch_bounds__(256) branch_merge_kernel(const float* __restrict__ a, const float* __restrict__ b, const float* __restrict__ wa,
                                                           const float* __restrict__ wb, float eps, float coef, float* __restrict__ out, int W) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const float* ra = a + t * W;
  const float* rb = b + t * W;
  float sa = 0.f, sb = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    sa = fmaf(ra[i], ra[i], sa);
    sb = fmaf(rb[i], rb[i], sb);
  }
  sa = block_sum(sa, red);
  sb = block_sum(sb, red);
  const float fa = 1.f / sqrtf(sa / (float)W + eps), fb = 1.f / sqrtf(sb / (float)W + eps);
  for (int i = threadIdx.x; i < W; i += blockDim.x) out[t * W + i] = coef * (ra[i] * fa * wa[i] + rb[i] * fb * wb[i]);
}

// stack [n][T][W]: results 0 .. n - 2 are there; result n - 1 = x + y (y may be null) is stored; then x <- sum_j coef[j] stack[j] and
// h = x / rms(x) * w (w may be null: no h)
__global__ void __launch_bounds__(256) depth_mix_kernel(float* __restrict__ stack, long long stride, int n, const float* __restrict__ coef,
                                                        float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w,
                                                        void* __restrict__ h, int dt_h, int W, float eps) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  float* xr = x + t * W;
  float ss = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float newest = xr[i] + (y ? y[t * W + i] : 0.f);
    stack[(long long)(n - 1) * stride + t * W + i] = newest;
    float acc = 0.f;
    for (int j = 0; j < n - 1; ++j) acc = fmaf(coef[j], stack[(long long)j * stride + t * W + i], acc);
    acc = fmaf(coef[n - 1], newest, acc);
    xr[i] = acc;
    ss = fmaf(acc, acc, ss);
  }
  if (w == nullptr) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)W + eps);
  for (int i = threadIdx.x; i < W; i += blockDim.x) st_dt(h, dt_h, t * W + i, xr[i] * rstd * w[i]);
}

// xs [T][n][W]: n copies of the residual stream per token, one block per token.  A thread keeps its columns of all copies in registers, so
// the copies are read and written once; the row of u waits in shared memory for the norm.  NS: the number of copies (0: n, up to 32);
// V: columns per access (4 needs W % 4 == 0 and 16-byte rows).
constexpr int kMaxStreams = 32;
template <int V> struct Cols { float v[V]; };
template <int V> __device__ __forceinline__ Cols<V> ld_cols(const float* p) {
  Cols<V> c;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    c.v[0] = f.x; c.v[1] = f.y; c.v[2] = f.z; c.v[3] = f.w;
  } else {
    c.v[0] = p[0];
  }
  return c;
}
template <int V> __device__ __forceinline__ void st_cols(float* p, const Cols<V>& c) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
  else p[0] = c.v[0];
}
template <int NS, int V>
__global__ void __launch_bounds__(256) stream_mix_kernel(float* __restrict__ xs, int n_rt, const float* __restrict__ x0,
                                                         const float* __restrict__ y, const float* __restrict__ mix,
                                                         const float* __restrict__ out, const float* __restrict__ read,
                                                         const float* __restrict__ w, float w_shift, void* __restrict__ h, int dt_h, int W,
                                                         float eps) {
  constexpr int N = NS > 0 ? NS : kMaxStreams, U = NS > 0 ? NS : 1;      // the generic form keeps its loops over the copies rolled
  extern __shared__ __align__(16) float u_row[];           // [W]
  __shared__ float cm[N * N], co[N], cr[N], red[32];
  const int n = NS > 0 ? NS : n_rt;
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < n * n; i += blockDim.x) cm[i] = y != nullptr ? mix[i] : 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    co[i] = y != nullptr ? out[i] : 0.f;
    cr[i] = read != nullptr ? read[i] : 1.f;
  }
  __syncthreads();
  float* xt = xs + t * n * W;
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < W; d += blockDim.x * V) {
    Cols<V> x[N], u;
    if (x0 != nullptr) {
      const Cols<V> e = ld_cols<V>(x0 + t * W + d);
#pragma unroll U
      for (int s = 0; s < N; ++s) if (s < n) x[s] = e;
    } else {
#pragma unroll U
      for (int s = 0; s < N; ++s) if (s < n) x[s] = ld_cols<V>(xt + (long long)s * W + d);
    }
#pragma unroll
    for (int c = 0; c < V; ++c) u.v[c] = 0.f;
    if (y != nullptr) {
      const Cols<V> yv = ld_cols<V>(y + t * W + d);
#pragma unroll U
      for (int q = 0; q < N; ++q) {
        if (q < n) {
          Cols<V> r;
#pragma unroll
          for (int c = 0; c < V; ++c) r.v[c] = 0.f;
#pragma unroll U
          for (int s = 0; s < N; ++s)
            if (s < n) {
#pragma unroll
              for (int c = 0; c < V; ++c) r.v[c] = fmaf(cm[s * n + q], x[s].v[c], r.v[c]);
            }
#pragma unroll
          for (int c = 0; c < V; ++c) {
            r.v[c] = fmaf(co[q], yv.v[c], r.v[c]);
            u.v[c] = fmaf(cr[q], r.v[c], u.v[c]);
          }
          st_cols<V>(xt + (long long)q * W + d, r);
        }
      }
    } else {
#pragma unroll U
      for (int s = 0; s < N; ++s)
        if (s < n) {
#pragma unroll
          for (int c = 0; c < V; ++c) u.v[c] = fmaf(cr[s], x[s].v[c], u.v[c]);
          if (x0 != nullptr) st_cols<V>(xt + (long long)s * W + d, x[s]);
        }
    }
    st_cols<V>(u_row + d, u);
#pragma unroll
    for (int c = 0; c < V; ++c) ss = fmaf(u.v[c], u.v[c], ss);
  }
  if (h == nullptr) return;
  float rstd = 1.f;
  if (w != nullptr) rstd = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  for (int d = threadIdx.x * V; d < W; d += blockDim.x * V) {       // a thread reads back the columns it wrote
    Cols<V> u = ld_cols<V>(u_row + d);
    if (w != nullptr) {
      const Cols<V> wv = ld_cols<V>(w + d);
#pragma unroll
      for (int c = 0; c < V; ++c) u.v[c] = u.v[c] * rstd * (w_shift + wv.v[c]);
    }
    if (dt_h == 0) {
      st_cols<V>((float*)h + t * W + d, u);
    } else if constexpr (V == 4) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(u.v[0], u.v[1]), hi = __floats2bfloat162_rn(u.v[2], u.v[3]);
      uint2 o;
      o.x = *reinterpret_cast<const uint32_t*>(&lo);
      o.y = *reinterpret_cast<const uint32_t*>(&hi);
      *reinterpret_cast<uint2*>((bf16*)h + t * W + d) = o;
    } else {
      ((bf16*)h)[t * W + d] = __float2bfloat16_rn(u.v[0]);
    }
  }
}

static int pow2_at_least(int v) {
  int p = 1;
  while (p < v) p <<= 1;
  return p;
}

// Generic scan: P lanes share a value column, each keeps at most 32 (16 for small heads) of its rows; more lanes where the columns would
// leave warps idle.
template <bool SC>
static int launch_gla_scan(const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay_in, long long lda,
                           const float* decay_bias, float inv_tau, float q_scale, int S, int H, int dk, int dv, float* state, const int* cu,
                           const int* slots, float* out, const MemoryGates& mg, cudaStream_t st) {
  const int cols = dv + (SC ? 1 : 0);
  int P = 1;
  while ((dk + P - 1) / P > 32) P <<= 1;
  while (P < 32 && (kRecThreads / 32) * (32 / P) / 2 >= cols && (dk + P - 1) / P > 4) P <<= 1;
  const int KR = (dk + P - 1) / P;
  const int CB = (kRecThreads / 32) * (32 / P);
  const size_t smem = (size_t)(4 * kRecTok * dk + kRecTok * CB) * 4;
  dim3 grid(S, H, (cols + CB - 1) / CB);
  if (smem > 48 * 1024) {
    SEQ_CUDA(cudaFuncSetAttribute(gla_scan_kernel<32, SC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SEQ_CUDA(cudaFuncSetAttribute(gla_scan_kernel<16, SC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  }
  if (KR <= 16)
    gla_scan_kernel<16, SC><<<grid, kRecThreads, smem, st>>>(qkv, ld, q_off, k_off, v_off, decay_in, lda, decay_bias, inv_tau, q_scale, H, dk, dv,
                                                             P, state, cu, slots, out, mg);
  else
    gla_scan_kernel<32, SC><<<grid, kRecThreads, smem, st>>>(qkv, ld, q_off, k_off, v_off, decay_in, lda, decay_bias, inv_tau, q_scale, H, dk, dv,
                                                             P, state, cu, slots, out, mg);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

template <int DK>
static int launch_mlstm_reg(const float* qkv, long long ld, int q_off, int k_off, int v_off, float q_scale, int S, int H, int dv, float* state,
                            const int* cu, const int* slots, float* out, const MemoryGates& mg, cudaStream_t st) {
  const size_t smem = (size_t)MemShape<DK>::kFloats * 4;
  if (smem > 48 * 1024) SEQ_CUDA(cudaFuncSetAttribute(mlstm_reg_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  mlstm_reg_kernel<DK><<<dim3(S, H, dv / 32), 32 * (kMemWarps + 1), smem, st>>>(qkv, ld, q_off, k_off, v_off, q_scale, H, dv, state, cu, slots, out, mg);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

template <int DK>
static int launch_gla_reg(const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* alpha, float q_scale, int S, int H,
                          int dv, float* state, const int* cu, const int* slots, float* out, cudaStream_t st) {
  const size_t smem = (size_t)(3 * 2 * kGlaTile * DK + 2 * kGlaTile * 32 + kGlaTile * kGlaWarps * 32) * 4;
  if (smem > 48 * 1024) SEQ_CUDA(cudaFuncSetAttribute(gla_reg_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  gla_reg_kernel<DK><<<dim3(S, H, dv / 32), 32 * kGlaWarps, smem, st>>>(qkv, ld, q_off, k_off, v_off, alpha, q_scale, H, dv, state, cu, slots, out);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

}  // namespace kb2seq

using namespace kb2seq;

extern "C" {

KB2SEQ_API int kb2_seq_gla(const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay_in, long long lda,
                           const float* decay_bias, float tau, float q_scale, int T, int S, int H, int dk, int dv, float* state,
                           const int* cu, const int* slots, float* scratch, float* out, void* stream) {
  if (!qkv || !decay_in || !state || !cu || !slots || !out || T <= 0 || S <= 0 || H <= 0 || dk <= 0 || dv <= 0 || !(tau > 0.f))
    return failf(KB2SEQ_ERR_VALUE, "gla: bad argument");
  if (dk > 1024) return failf(KB2SEQ_ERR_VALUE, "gla: key size %d > 1024", dk);
  if (H > 65535) return failf(KB2SEQ_ERR_VALUE, "gla: too many heads");
  const bool aligned = ((uintptr_t)qkv & 15) == 0 && (ld & 3) == 0 && (q_off & 3) == 0 && (k_off & 3) == 0 && (v_off & 3) == 0 &&
                       scratch != nullptr && ((uintptr_t)scratch & 15) == 0;
  if (aligned && (dk == 32 || dk == 64 || dk == 128 || dk == 256) && dv % 32 == 0 && dv / 32 <= 65535) {
    cudaStream_t st0 = (cudaStream_t)stream;
    const long long ne = (long long)T * H * dk;
    gla_decay_kernel<<<(unsigned)((ne + 255) / 256), 256, 0, st0>>>(decay_in, lda, decay_bias, 1.f / tau, T, H * dk, scratch);
    SEQ_LAUNCHED();
    if (dk == 32) return launch_gla_reg<32>(qkv, ld, q_off, k_off, v_off, scratch, q_scale, S, H, dv, state, cu, slots, out, st0);
    if (dk == 64) return launch_gla_reg<64>(qkv, ld, q_off, k_off, v_off, scratch, q_scale, S, H, dv, state, cu, slots, out, st0);
    if (dk == 128) return launch_gla_reg<128>(qkv, ld, q_off, k_off, v_off, scratch, q_scale, S, H, dv, state, cu, slots, out, st0);
    return launch_gla_reg<256>(qkv, ld, q_off, k_off, v_off, scratch, q_scale, S, H, dv, state, cu, slots, out, st0);
  }
  return launch_gla_scan<false>(qkv, ld, q_off, k_off, v_off, decay_in, lda, decay_bias, 1.f / tau, q_scale, S, H, dk, dv, state, cu, slots, out,
                                MemoryGates{}, (cudaStream_t)stream);
}

KB2SEQ_API int kb2_seq_mlstm(const float* proj, long long ld, int q_off, int k_off, int v_off, int i_off, int f_off, const float* i_bias,
                             const float* f_bias, float cap, float q_scale, int T, int S, int H, int dk, int dv, float* state, float* nstate,
                             float* mstate, const int* cu, const int* slots, float* scratch, float* out, float* den, void* stream) {
  if (!proj || !state || !nstate || !mstate || !cu || !slots || !scratch || !out || !den || T <= 0 || S <= 0 || H <= 0 || dk <= 0 || dv <= 0 ||
      !(cap > 0.f))
    return failf(KB2SEQ_ERR_VALUE, "mlstm: bad argument");
  if (dk > 1024) return failf(KB2SEQ_ERR_VALUE, "mlstm: key size %d > 1024", dk);
  if (H > 65535) return failf(KB2SEQ_ERR_VALUE, "mlstm: too many heads");
  cudaStream_t st = (cudaStream_t)stream;
  float* keep = scratch;
  float* add = keep + (long long)T * H;
  float* mx = add + (long long)T * H;
  const int threads = T >= kGateThreads ? kGateThreads : (T + 31) / 32 * 32;
  mlstm_gates_kernel<<<dim3(S, H), threads, 0, st>>>(proj, ld, i_off, f_off, i_bias, f_bias, cap, H, mstate, cu, slots, keep, add, mx);
  SEQ_LAUNCHED();
  const MemoryGates mg{keep, add, mx, nstate, den};
  const bool aligned = (((uintptr_t)proj | (uintptr_t)state) & 15) == 0 && (ld & 3) == 0 && (q_off & 3) == 0 && (k_off & 3) == 0 &&
                       (v_off & 3) == 0;
  if (aligned && (dk == 32 || dk == 64 || dk == 128 || dk == 256) && dv % 32 == 0 && dv / 32 <= 65535) {
#define KB2_MEM(DKV) launch_mlstm_reg<DKV>(proj, ld, q_off, k_off, v_off, q_scale, S, H, dv, state, cu, slots, out, mg, st)
    if (dk == 32) return KB2_MEM(32);
    if (dk == 64) return KB2_MEM(64);
    if (dk == 128) return KB2_MEM(128);
    return KB2_MEM(256);
#undef KB2_MEM
  }
  return launch_gla_scan<true>(proj, ld, q_off, k_off, v_off, nullptr, 0, nullptr, 1.f, q_scale, S, H, dk, dv, state, cu, slots, out, mg, st);
}

KB2SEQ_API int kb2_seq_rglru(const float* u, long long ldu, const float* z, long long ldz, long long zb, const float* y, long long ldy,
                             const float* r_bias, const float* i_bias, const float* y_bias, const float* rate, int T, int S, int C, int bs,
                             float* state, const int* cu, const int* slots, void* out, int dt_out, void* stream) {
  if (!u || !z || !y || !rate || !state || !cu || !slots || !out || T <= 0 || S <= 0 || C <= 0 || bs <= 0 || C % bs || bad_dt(dt_out))
    return failf(KB2SEQ_ERR_VALUE, "rglru: bad argument");
  if ((C + 31) / 32 > 65535) return failf(KB2SEQ_ERR_VALUE, "rglru: too many channels");
  const int groups = (C + 31) / 32;
  if (T - S + 1 <= 2)                                  // no portion is longer than two tokens
    rglru_scan_kernel<1, kRgGroups, 2><<<dim3(S, (groups + kRgGroups - 1) / kRgGroups), 32 * kRgGroups, 0, (cudaStream_t)stream>>>(
        u, ldu, z, ldz, zb, y, ldy, r_bias, i_bias, y_bias, rate, C, bs, state, cu, slots, out, dt_out);
  else
    rglru_scan_kernel<kRgWarps, 1, kRgTok><<<dim3(S, groups), 32 * kRgWarps, 0, (cudaStream_t)stream>>>(
        u, ldu, z, ldz, zb, y, ldy, r_bias, i_bias, y_bias, rate, C, bs, state, cu, slots, out, dt_out);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_split_blocks(const float* u, long long ldu, int T, int T_pad, int blocks, int bs, void* out, void* stream) {
  if (!u || !out || T <= 0 || T_pad < T || blocks <= 0 || bs <= 0 || (bs & 1)) return failf(KB2SEQ_ERR_VALUE, "split_blocks: bad argument");
  const long long n = (long long)T * blocks * (bs / 2);
  split_blocks_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(u, ldu, T, T_pad, blocks, bs, (bf16*)out);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_selective_scan(const float* x, long long ldx, const float* dt_in, long long ldd, const float* dt_bias, const float* bc,
                                      long long ldb, int b_off, const float* z, long long ldz, int z_off, const float* A_log,
                                      const float* D, int T, int S, int inner, int N, float* state, const int* cu, const int* slots,
                                      void* out, int dt_out, void* stream) {
  if (!x || !dt_in || !dt_bias || !bc || !z || !A_log || !D || !state || !cu || !slots || !out || T <= 0 || S <= 0 || inner <= 0 || N <= 0 ||
      bad_dt(dt_out))
    return failf(KB2SEQ_ERR_VALUE, "selective_scan: bad argument");
  if (N > 256) return failf(KB2SEQ_ERR_VALUE, "selective_scan: state size %d > 256", N);
  const int NR = N <= 32 ? 1 : (N <= 64 ? 2 : (N <= 128 ? 4 : 8));
  const int P = pow2_at_least((N + NR - 1) / NR);
  const int CB = (kRecThreads / 32) * (32 / P);
  const size_t smem = (size_t)(2 * kRecTok * 2 * N + 3 * 2 * kRecTok * CB + kRecTok * CB * (P + 1)) * 4;
  dim3 grid(S, (inner + CB - 1) / CB);
  cudaStream_t st = (cudaStream_t)stream;
#define KB2_SCAN(NRV)                                                                                                                  \
  if (smem > 48 * 1024) SEQ_CUDA(cudaFuncSetAttribute(selective_scan_kernel<NRV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
  selective_scan_kernel<NRV><<<grid, kRecThreads, smem, st>>>(x, ldx, dt_in, ldd, dt_bias, bc, ldb, b_off, z, ldz, z_off, A_log, D, inner, N, \
                                                              P, state, cu, slots, out, dt_out)
  if (NR == 1) { KB2_SCAN(1); } else if (NR == 2) { KB2_SCAN(2); } else if (NR == 4) { KB2_SCAN(4); } else { KB2_SCAN(8); }
#undef KB2_SCAN
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_head_norm_gate(const float* o, long long ldo, const float* w, float eps, const float* gate, long long ldg, int gate_act,
                                      int T, int H, int dv, void* out, int dt_out, const float* den, int w_heads, void* stream) {
  if (!o || !out || T <= 0 || H <= 0 || dv <= 0 || bad_dt(dt_out) || gate_act < 0 || gate_act > 1)
    return failf(KB2SEQ_ERR_VALUE, "head_norm_gate: bad argument");
  const long long nw = (long long)T * H;
  const uintptr_t all = (uintptr_t)o | (uintptr_t)w | (uintptr_t)gate | (uintptr_t)out;
  if (dv % 4 == 0 && dv <= 512 && ldo % 4 == 0 && ldg % 4 == 0 && !(all & 15)) {
#define KB2_HN(NV)                                                                                                                          \
  head_norm_gate_vec_kernel<NV><<<(unsigned)((nw + 7) / 8), 256, 0, (cudaStream_t)stream>>>(o, ldo, w, eps, gate, ldg, gate_act, H, dv, T, out, dt_out, \
                                                                                           den, w_heads)
    if (dv <= 128) KB2_HN(1); else if (dv <= 256) KB2_HN(2); else KB2_HN(4);
#undef KB2_HN
    SEQ_LAUNCHED();
    return KB2SEQ_OK;
  }
  head_norm_gate_kernel<<<(unsigned)((nw + 7) / 8), 256, 0, (cudaStream_t)stream>>>(o, ldo, w, eps, gate, ldg, gate_act, H, dv, T, out, dt_out, den,
                                                                                      w_heads);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_rms_rows(const float* in, long long ld_in, int n, const float* w, float eps, void* out, int dt_out, long long ld_out,
                                int T, void* stream) {
  if (!in || !w || !out || T <= 0 || n <= 0 || bad_dt(dt_out)) return failf(KB2SEQ_ERR_VALUE, "rms_rows: bad argument");
  rms_rows_kernel<<<T, 256, 0, (cudaStream_t)stream>>>(in, ld_in, n, w, eps, out, dt_out, ld_out);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_branch_merge(const float* a, const float* b, const float* wa, const float* wb, float eps, float coef, float* out, int T,
                                    int W, void* stream) {
  if (!a || !b || !wa || !wb || !out || T <= 0 || W <= 0) return failf(KB2SEQ_ERR_VALUE, "branch_merge: bad argument");
  branch_merge_kernel<<<T, 256, 0, (cudaStream_t)stream>>>(a, b, wa, wb, eps, coef, out, W);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_depth_mix(float* stack, long long stride, int n, const float* coef, float* x, const float* y, const float* w, void* h,
                                 int dt_h, int T, int W, float eps, void* stream) {
  if (!stack || !coef || !x || n <= 0 || T <= 0 || W <= 0 || (w && (!h || bad_dt(dt_h)))) return failf(KB2SEQ_ERR_VALUE, "depth_mix: bad argument");
  depth_mix_kernel<<<T, 256, 0, (cudaStream_t)stream>>>(stack, stride, n, coef, x, y, w, h, dt_h, W, eps);
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

KB2SEQ_API int kb2_seq_stream_mix(float* xs, int n, const float* x0, const float* y, const float* mix, const float* out, const float* read,
                                  const float* w, float w_shift, void* h, int dt_h, int T, int W, float eps, void* stream) {
  if (!xs || n < 1 || n > kMaxStreams || T <= 0 || W <= 0 || (y && (!mix || !out)) || (w && !h) || (h && bad_dt(dt_h)))
    return failf(KB2SEQ_ERR_VALUE, "stream_mix: bad argument (n=%d T=%d W=%d)", n, T, W);
  const size_t smem = (size_t)W * 4;
  if (smem > 200 * 1024) return failf(KB2SEQ_ERR_VALUE, "stream_mix: width %d too large", W);
  const uintptr_t all = (uintptr_t)xs | (uintptr_t)x0 | (uintptr_t)y | (uintptr_t)w | (uintptr_t)h;
  const bool vec = W % 4 == 0 && !(all & 15);
  cudaStream_t s = (cudaStream_t)stream;
#define KB2_SM(NSV, VV)                                                                                                              \
  do {                                                                                                                               \
    if (smem > 40 * 1024) SEQ_CUDA(cudaFuncSetAttribute(stream_mix_kernel<NSV, VV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    stream_mix_kernel<NSV, VV><<<T, 256, smem, s>>>(xs, n, x0, y, mix, out, read, w, w_shift, h, dt_h, W, eps);                      \
  } while (0)
  if (!vec) KB2_SM(0, 1);
  else switch (n) {
    case 1: KB2_SM(1, 4); break;
    case 2: KB2_SM(2, 4); break;
    case 3: KB2_SM(3, 4); break;
    case 4: KB2_SM(4, 4); break;
    case 8: KB2_SM(8, 4); break;
    default: KB2_SM(0, 1); break;
  }
#undef KB2_SM
  SEQ_LAUNCHED();
  return KB2SEQ_OK;
}

}  // extern "C"
