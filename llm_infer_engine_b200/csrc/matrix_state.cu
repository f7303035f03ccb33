// Recurrences over a matrix state per head, S [D, Dv] float32, in which every key channel has a decay of its own, the
// state is read before it is updated, or what is written depends on what the state holds:
//
//   FORM 0 (key decay)   S <- diag(a_t) S + k_t v_t^T;                 o_t = S^T q_t           gated linear attention
//   FORM 1 (bonus)       o_t = (S + diag(b) k_t v_t^T)^T q_t;          S <- diag(a_t) S + k_t v_t^T     time mixing
//   FORM 2 (delta rule)  S <- g_t S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
//
// Packed tokens: sequence s of the step owns rows cu_q[s] .. cu_q[s+1]-1, its state lives in row seq_slot[s] of a
// [slots, H, D, Dv] tensor, is read at the start of a piece and written at its end. Decays, states, what is read from them
// and its norm are float32 in both precisions; what the projections make has the activation type.
//
//   low_rank_gate   a[t, c] = exp(-softplus(-z) / tau) = sigmoid(z)^(1/tau), or exp(-exp(z)) with a tanh inside, of
//                   z = B x_t + b, x_t a few numbers per token
//   delta_prepare   unit-length q and k per head, beta = sigmoid(.), g = exp(-exp(A_log) softplus(. + dt_bias)), q . k
//   channel_scan    pieces of any length: a sequence's tokens in order, its columns and heads side by side
//   state_step      one token per sequence, with everything around the recurrence in the same kernel: gates or unit
//                   vectors, the recurrence, the norm of what is read and its silu gate
//   shift_mix       x + (x_prev - x) (.) mu_s for several mu_s at once, x_prev the previous token's x
#include "common.cuh"
#include <math.h>

namespace llmie {

__device__ __forceinline__ float sigmoidf_(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float siluf_(float z) { return z / (1.f + expf(-z)); }

constexpr int kFormKeyDecay = 0, kFormBonus = 1, kFormDelta = 2;

// The decay of a key channel from its pre-activation z.
__device__ __forceinline__ float key_decay(float z, int mode, float inv_tau) {
  return mode == 0 ? expf(-softplusf_(-z) * inv_tau) : expf(-expf(z));
}

// ------------------------------------------------------------------------------------------ gates of whole pieces
constexpr int kGateTokens = 16;

// grid (channel tiles of 128, token tiles of kGateTokens); x rows of R numbers, ld apart; Bt float32 [R, N].
template <typename T>
__global__ void __launch_bounds__(128)
low_rank_gate_kernel(const T* __restrict__ x, int ld, const float* __restrict__ Bt, const float* __restrict__ bias,
                     float* __restrict__ out, int R, int N, int n_tokens, int mode, float inv_tau) {
  extern __shared__ float gate_smem[];                          // [R][kGateTokens]
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.y * kGateTokens, n = min(kGateTokens, n_tokens - t0);
  for (int i = threadIdx.x; i < R * kGateTokens; i += blockDim.x) {
    const int tt = i % kGateTokens, r = i / kGateTokens;
    const float v = tt < n ? to_f32(x[(size_t)(t0 + tt) * ld + r]) : 0.f;
    gate_smem[i] = mode == 1 ? tanhf(v) : v;
  }
  __syncthreads();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= N) return;
  float z[kGateTokens];
  const float b = bias[c];
#pragma unroll
  for (int tt = 0; tt < kGateTokens; ++tt) z[tt] = b;
  for (int r = 0; r < R; ++r) {
    const float w = Bt[(size_t)r * N + c];
    const float4* xr = reinterpret_cast<const float4*>(gate_smem + r * kGateTokens);
#pragma unroll
    for (int k = 0; k < kGateTokens / 4; ++k) {
      const float4 v = xr[k];
      z[4 * k] = fmaf(w, v.x, z[4 * k]);
      z[4 * k + 1] = fmaf(w, v.y, z[4 * k + 1]);
      z[4 * k + 2] = fmaf(w, v.z, z[4 * k + 2]);
      z[4 * k + 3] = fmaf(w, v.w, z[4 * k + 3]);
    }
  }
#pragma unroll
  for (int tt = 0; tt < kGateTokens; ++tt)
    if (tt < n) out[(size_t)(t0 + tt) * N + c] = key_decay(z[tt], mode, inv_tau);
}

// A block per token; its warps take the G key heads in turn. qkv rows [q : G D | k : G D | ...] of TC, ld apart (what the
// convolutions leave); ba rows hold b at b_off and a at a_off, H numbers each. q is also multiplied by q_scale.
// qn, kn float32 [T, G D]; scal float32 [T, H, 2] = (beta, g); qk float32 [T, G] = q . k of the results.
template <typename TC, typename TP>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const TC* __restrict__ qkv, int ld, const TP* __restrict__ ba, int ba_ld, int b_off, int a_off,
                     const float* __restrict__ A, const float* __restrict__ dt_bias, float eps, float q_scale,
                     float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ scal, float* __restrict__ qk,
                     int H, int G, int D) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const TC* row = qkv + t * ld;
  for (int g = warp; g < G; g += warps) {
    const TC* qr = row + (size_t)g * D;
    const TC* kr = row + (size_t)(G + g) * D;
    float qq = 0.f, kk = 0.f, dot = 0.f;
    for (int i = lane; i < D; i += 32) {
      const float q = to_f32(qr[i]), k = to_f32(kr[i]);
      qq = fmaf(q, q, qq);
      kk = fmaf(k, k, kk);
      dot = fmaf(q, k, dot);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    dot = warp_sum(dot);
    const float rq = q_scale / sqrtf(qq + eps), rk = 1.f / sqrtf(kk + eps);
    for (int i = lane; i < D; i += 32) {
      qn[(t * G + g) * D + i] = to_f32(qr[i]) * rq;
      kn[(t * G + g) * D + i] = to_f32(kr[i]) * rk;
    }
    if (lane == 0) qk[t * G + g] = dot * rq * rk;
  }
  const TP* bar = ba + t * ba_ld;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    scal[(t * H + h) * 2] = sigmoidf_(to_f32(bar[b_off + h]));
    scal[(t * H + h) * 2 + 1] = expf(-A[h] * softplusf_(to_f32(bar[a_off + h]) + dt_bias[h]));
  }
}

// ------------------------------------------------------------------------------------------ the previous token's input
// out[s][t][c] = x + (x_prev - x) mu[s][c], s < n_mix; x_prev of a piece's first token is prev[slot][c]. grid (column
// blocks, tokens). `single`: one token per sequence, and prev receives it (in other steps the caller stores it afterwards).
template <typename T>
__global__ void shift_mix_kernel(const T* __restrict__ x, float* prev, const float* __restrict__ mu,
                                 const int* __restrict__ cu_q, const int* __restrict__ tok_seq,
                                 const int* __restrict__ seq_slot, T* __restrict__ out, int n_mix, int d, int n_tokens,
                                 int single) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= d) return;
  for (int t = blockIdx.y; t < n_tokens; t += gridDim.y) {
    const int seq = tok_seq[t];
    float* ps = prev + (size_t)seq_slot[seq] * d + c;
    const float now = to_f32(x[(size_t)t * d + c]);
    const float before = t > cu_q[seq] ? to_f32(x[(size_t)(t - 1) * d + c]) : *ps;
    const float step = before - now;
    for (int s = 0; s < n_mix; ++s)
      out[((size_t)s * n_tokens + t) * d + c] = from_f32<T>(fmaf(step, mu[(size_t)s * d + c], now));
    if (single) *ps = now;
  }
}

// The same, eight channels a thread (d % 8 == 0, 16-byte aligned rows).
template <typename T>
__global__ void shift_mix8_kernel(const T* __restrict__ x, float* prev, const float* __restrict__ mu,
                                  const int* __restrict__ cu_q, const int* __restrict__ tok_seq,
                                  const int* __restrict__ seq_slot, T* __restrict__ out, int n_mix, int d, int n_tokens,
                                  int single) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= d) return;
  for (int t = blockIdx.y; t < n_tokens; t += gridDim.y) {
    const int seq = tok_seq[t];
    float* ps = prev + (size_t)seq_slot[seq] * d + c;
    float now[8], step[8];
    load8(x + (size_t)t * d + c, now);
    if (t > cu_q[seq]) load8(x + (size_t)(t - 1) * d + c, step);
    else load8(ps, step);
#pragma unroll
    for (int e = 0; e < 8; ++e) step[e] -= now[e];
    for (int s = 0; s < n_mix; ++s) {
      float m[8];
      load8(mu + (size_t)s * d + c, m);
#pragma unroll
      for (int e = 0; e < 8; ++e) m[e] = fmaf(step[e], m[e], now[e]);
      store8(out + ((size_t)s * n_tokens + t) * d + c, m);
    }
    if (single) store8(ps, now);
  }
}

// ------------------------------------------------------------------------------------------ pieces of any length
// What the scan and the one-token step read and write.
struct StateArgs {
  const void* q;            // rows of G * D of TQ, q_ld apart, times q_scale
  const void* k;            // likewise, k_ld apart
  const void* v;            // rows of H * Dv of TV, v_ld apart
  const float* gate;        // FORM 0, 1: decays float32 [T, G * D]
  const float* bonus;       // FORM 1: float32 [G * D]
  const float* scal;        // FORM 2: float32 [T, H, 2] = (beta, g)
  const float* qk;          // FORM 2: float32 [T, G] = q . k
  float* state;             // [slots, H, D, Dv]
  const int* cu_q;
  const int* seq_slot;
  float* o;                 // float32 [T, H * Dv]
  int q_ld, k_ld, v_ld, H, G, D, Dv, vec;
  float q_scale;
  float* ws;                // long pieces in chunks side by side: [n_seqs, n_chunks, H, D, Dv], else null
  float* prod;              // ... and the products of the chunks' decays, [n_seqs, n_chunks, H, D]
  int chunk, n_chunks;      // tokens a chunk (a multiple of the tile), chunks of the longest piece (1: whole pieces)
};

// Four adjacent elements as float32; entries from `left` on are zeros. `vec`: one aligned access.
template <typename T>
__device__ __forceinline__ float4 load_row4(const T* p, int left, bool vec) {
  if (vec) {
    if (left <= 0) return make_float4(0.f, 0.f, 0.f, 0.f);
    if (sizeof(T) == 4) return *reinterpret_cast<const float4*>(p);
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
  }
  return make_float4(left > 0 ? to_f32(p[0]) : 0.f, left > 1 ? to_f32(p[1]) : 0.f, left > 2 ? to_f32(p[2]) : 0.f,
                     left > 3 ? to_f32(p[3]) : 0.f);
}

// Asks for four adjacent elements into shared memory, behind this thread's next commit; entries from `left` on become
// zeros. Without `vec` (one aligned access) they are loaded and stored here and now.
template <typename T>
__device__ __forceinline__ void stage_row4(T* dst, const T* src, int left, bool vec) {
  if (vec) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int n = left > 0 ? (int)(4 * sizeof(T)) : 0;
    if (sizeof(T) == 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
    return;
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) dst[e] = e < left ? src[e] : from_f32<T>(0.f);
}

constexpr int kScanTile = 8;           // tokens staged at a time

// Pairs of float32 in one register pair (two adjacent rows of a column): one instruction works on both.
using pair_t = unsigned long long;
__device__ __forceinline__ pair_t pair_of(float lo, float hi) {
  pair_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 pair_split(pair_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ float pair_sum(pair_t v) { const float2 f = pair_split(v); return f.x + f.y; }
__device__ __forceinline__ pair_t pair_fma(pair_t a, pair_t b, pair_t c) {
  pair_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ pair_t pair_mul(pair_t a, pair_t b) {
  pair_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// The shape of a scan: a thread keeps C adjacent columns and R rows of them, S lanes share a column, NT threads a block.
template <int C_, int R_, int S_, int NT_>
struct ScanShape {
  static constexpr int C = C_, R = R_, S = S_, NT = NT_;
};

// How a block of the scan lays out shared memory, in bytes: a ring of raw tiles, then two tiles in float32.
template <typename TQ, typename TV, int FORM, typename SH>
struct ScanLayout {
  static constexpr int DP = SH::R * SH::S;                       // rows, padded
  static constexpr int COLS = SH::NT / SH::S * SH::C;
  static constexpr int NARR = FORM == kFormDelta ? 2 : 3;        // q, k (, decays)
  static constexpr int RUNS = kScanTile * DP / 4;                // runs of four in one staged array
  static constexpr int STAGES = DP > 256 ? 2 : 4;
  static constexpr int RAW_Q = RUNS * 4 * (int)sizeof(TQ);
  static constexpr int RAW_G = FORM == kFormDelta ? 0 : RUNS * 16;
  static constexpr int RAW_V = kScanTile * COLS * (int)sizeof(TV);
  static constexpr int RAW = 2 * RAW_Q + RAW_G + RAW_V + kScanTile * 16;
  static constexpr int TILE = kScanTile * (NARR * DP + COLS + 4) * 4;
  static constexpr size_t BYTES = (size_t)STAGES * RAW + 2 * TILE;
};

// grid (column tiles, heads, sequences). C adjacent columns of the state are S lanes' work; lane s of them keeps the rows
// 4 (s + S i) + e, i < R / 4, e < 4, in registers over the whole piece, so that an entry of a key, query or decay that is
// read from shared memory serves C columns. Tiles of kScanTile tokens' decays, keys, queries and values travel through a
// ring of raw tiles (asynchronous copies, a few tiles ahead; every thread waits for, and converts, what it asked for
// itself) into one of two float32 tiles, the next while the current one is worked on. Tokens behind the piece's end are
// staged as ones that leave the state as it is. What the eight tokens of a tile read from the state is reduced over the
// lanes together: a step halves the number of values and of lanes.
//
// Long pieces of forms 0 and 1, whose end state is linear in the start state: a piece is cut into chunks, grid z =
// (sequence, chunk). OUT false runs every chunk but a sequence's last from a zero state, without outputs, and leaves its
// end state in ws[c + 1] and the product of its decays in prod[c + 1]; a chain over the chunks makes ws[c] the state that
// chunk c starts from; OUT true runs every chunk from there.
template <typename TQ, typename TV, int FORM, typename SH, bool OUT>
__global__ void __launch_bounds__(SH::NT) channel_scan_kernel(const StateArgs a) {
  using L = ScanLayout<TQ, TV, FORM, SH>;
  constexpr int C = SH::C, R = SH::R, S = SH::S, NT = SH::NT;
  constexpr int DP = L::DP, COLS = L::COLS, RUNS = L::RUNS, STAGES = L::STAGES;
  constexpr int NV = (RUNS + NT - 1) / NT;
  constexpr int CG = 32 / S;                                    // groups of columns a warp
  constexpr int VRUNS = kScanTile * COLS / 4;
  constexpr int VV = (VRUNS + NT - 1) / NT;
  constexpr int P = R / 2;                                      // pairs of rows a thread
  extern __shared__ __align__(16) char scan_smem[];
  pdl_launch_dependents();
  const int tid = threadIdx.x;
  const int s = tid & (S - 1), col = tid / S * C;
  const int j0 = blockIdx.x * COLS, j = j0 + col;
  const int h = blockIdx.y, g = h / (a.H / a.G);
  const int seq = blockIdx.z / a.n_chunks, chunk = blockIdx.z - seq * a.n_chunks;
  const int D = a.D, Dv = a.Dv;
  float4 bo[FORM == kFormBonus ? R / 4 : 1];
  if (FORM == kFormBonus) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
      const int row = 4 * (s + S * i);
      bo[i] = load_row4<float>(a.bonus + (size_t)g * D + row, D - row, false);
    }
  }
  pdl_wait();
  const int seq_end = a.cu_q[seq + 1];
  const int t0 = a.cu_q[seq] + chunk * a.chunk, t1 = a.n_chunks > 1 ? min(t0 + a.chunk, seq_end) : seq_end;
  if (t0 >= t1) return;
  if (!OUT && t1 >= seq_end) return;                            // nobody needs the last chunk's end state
  const TQ* qb = reinterpret_cast<const TQ*>(a.q) + (size_t)g * D;
  const TQ* kb = reinterpret_cast<const TQ*>(a.k) + (size_t)g * D;
  const float* gb = FORM == kFormDelta ? nullptr : a.gate + (size_t)g * D;
  const TV* vb = reinterpret_cast<const TV*>(a.v) + (size_t)h * Dv;
  const size_t GD = (size_t)a.G * D;
  auto raw_q = [&](int st) { return reinterpret_cast<TQ*>(scan_smem + st * L::RAW); };
  auto raw_k = [&](int st) { return reinterpret_cast<TQ*>(scan_smem + st * L::RAW + L::RAW_Q); };
  auto raw_g = [&](int st) { return reinterpret_cast<float*>(scan_smem + st * L::RAW + 2 * L::RAW_Q); };
  auto raw_v = [&](int st) { return reinterpret_cast<TV*>(scan_smem + st * L::RAW + 2 * L::RAW_Q + L::RAW_G); };
  auto raw_s = [&](int st) { return reinterpret_cast<float*>(scan_smem + st * L::RAW + 2 * L::RAW_Q + L::RAW_G + L::RAW_V); };
  auto ask = [&](int t, int st) {                               // tile of tokens t .. into the ring's place st
    if (t < t1) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int run = tid + i * NT;
        if (run < RUNS) {
          const int tt = run / (DP / 4), row = (run % (DP / 4)) * 4;
          const int left = t + tt < t1 ? D - row : 0;
          const size_t tok = t + tt < t1 ? t + tt : t1 - 1;
          const int at = left > 0 ? row : 0;
          stage_row4<TQ>(raw_q(st) + run * 4, qb + tok * a.q_ld + at, left, a.vec & 1);
          stage_row4<TQ>(raw_k(st) + run * 4, kb + tok * a.k_ld + at, left, a.vec & 1);
          if (FORM != kFormDelta) stage_row4<float>(raw_g(st) + run * 4, gb + tok * GD + at, left, a.vec & 1);
        }
      }
#pragma unroll
      for (int i = 0; i < VV; ++i) {
        const int run = tid + i * NT;
        if (run < VRUNS) {
          const int tt = run / (COLS / 4), jj = j0 + (run % (COLS / 4)) * 4;
          const int left = t + tt < t1 ? Dv - jj : 0;
          const size_t tok = t + tt < t1 ? t + tt : t1 - 1;
          stage_row4<TV>(raw_v(st) + run * 4, vb + tok * a.v_ld + (left > 0 ? jj : 0), left, a.vec & 2);
        }
      }
      if (FORM == kFormDelta && tid < kScanTile && t + tid < t1) {
        const size_t tok = t + tid;
        const unsigned d = (unsigned)__cvta_generic_to_shared(raw_s(st) + tid * 4);
        asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(d), "l"(a.scal + (tok * a.H + h) * 2) : "memory");
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d + 8), "l"(a.qk + tok * a.G + g) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float4 fq[NV], fk[NV], fg[FORM == kFormDelta ? 1 : NV], fv[VV], fs;
  auto take = [&](int st) {                                     // this thread's part of a raw tile, as float32
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int run = tid + i * NT;
      if (run < RUNS) {
        fq[i] = load_row4<TQ>(raw_q(st) + run * 4, 4, true);
        fk[i] = load_row4<TQ>(raw_k(st) + run * 4, 4, true);
        if (FORM != kFormDelta) fg[i] = load_row4<float>(raw_g(st) + run * 4, 4, true);
      }
    }
#pragma unroll
    for (int i = 0; i < VV; ++i)
      if (tid + i * NT < VRUNS) fv[i] = load_row4<TV>(raw_v(st) + (tid + i * NT) * 4, 4, true);
    if (FORM == kFormDelta && tid < kScanTile) fs = *reinterpret_cast<const float4*>(raw_s(st) + tid * 4);
  };
  auto tile = [&](int buf) { return reinterpret_cast<float*>(scan_smem + STAGES * L::RAW + buf * L::TILE); };
  auto put = [&](int t, int buf) {
    float *sq = tile(buf), *sk = sq + kScanTile * DP, *sg = sk + kScanTile * DP, *sv = sq + L::NARR * kScanTile * DP,
          *sc = sv + kScanTile * COLS;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int run = tid + i * NT;
      if (run < RUNS) {
        reinterpret_cast<float4*>(sq)[run] = make_float4(fq[i].x * a.q_scale, fq[i].y * a.q_scale, fq[i].z * a.q_scale,
                                                         fq[i].w * a.q_scale);
        reinterpret_cast<float4*>(sk)[run] = fk[i];
        if (FORM != kFormDelta)
          reinterpret_cast<float4*>(sg)[run] = t + run / (DP / 4) < t1 ? fg[i] : make_float4(1.f, 1.f, 1.f, 1.f);
      }
    }
#pragma unroll
    for (int i = 0; i < VV; ++i)
      if (tid + i * NT < VRUNS) reinterpret_cast<float4*>(sv)[tid + i * NT] = fv[i];
    if (FORM == kFormDelta && tid < kScanTile)
      reinterpret_cast<float4*>(sc)[tid] = t + tid < t1 ? fs : make_float4(0.f, 1.f, 0.f, 0.f);
  };
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) ask(t0 + i * kScanTile, i);
  const size_t place = ((size_t)seq * a.n_chunks + chunk) * a.H + h;              // of (sequence, chunk, head)
  float* st = a.state + (((size_t)a.seq_slot[seq] * a.H + h) * D) * Dv + j;
  const float* start = OUT && a.n_chunks > 1 ? a.ws + place * D * Dv + j : st;
  pair_t St[C][P];                                              // pair p of column c: rows row_of(p) and the next
  auto row_of = [&](int p) { return 4 * (s + S * (p / 2)) + 2 * (p & 1); };
#pragma unroll
  for (int p = 0; p < P; ++p)
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int row = row_of(p);
      const bool ok = OUT && j + c < Dv;
      St[c][p] = pair_of(ok && row < D ? start[(size_t)row * Dv + c] : 0.f,
                         ok && row + 1 < D ? start[(size_t)(row + 1) * Dv + c] : 0.f);
    }
  pair_t decays[OUT ? 1 : P];                                   // the product of the chunk's decays
#pragma unroll
  for (int p = 0; p < (OUT ? 1 : P); ++p) decays[p] = pair_of(1.f, 1.f);
  asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
  take(0);
  put(t0, 0);
  __syncthreads();
  int ring = 0, buf = 0;                                        // the current tile's places
  for (int t = t0; t < t1; t += kScanTile, buf ^= 1) {
    const int n = min(kScanTile, t1 - t);
    const bool more = t + kScanTile < t1;
    // the place of the tile before the current one is free: this thread has converted its part of it
    ask(t + (STAGES - 1) * kScanTile, (ring + STAGES - 1) % STAGES);
    ring = (ring + 1) % STAGES;
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    if (more) take(ring);
    const float *sq = tile(buf), *sk = sq + kScanTile * DP, *sg = sk + kScanTile * DP,
                *sv = sq + L::NARR * kScanTile * DP, *sc = sv + kScanTile * COLS;
    float acc[kScanTile * C];                                   // token tt, column c at tt * C + c
    float part[FORM == kFormBonus ? S / 4 : 1];                 // the bonus's share of q . k: a warp's groups take turns
    if (FORM == kFormBonus && OUT) {
      const int cg = (tid & 31) / S;
#pragma unroll
      for (int m = 0; m < S / 4; ++m) {
        const int tt = cg + CG * m;
        float p = 0.f;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          const float4 q = reinterpret_cast<const float4*>(sq + tt * DP)[s + S * i];
          const float4 k = reinterpret_cast<const float4*>(sk + tt * DP)[s + S * i];
          p = fmaf(q.x * bo[i].x, k.x, p);
          p = fmaf(q.y * bo[i].y, k.y, p);
          p = fmaf(q.z * bo[i].z, k.z, p);
          p = fmaf(q.w * bo[i].w, k.w, p);
        }
        part[m] = p;
      }
    }
#pragma unroll
    for (int tt = 0; tt < kScanTile; ++tt) {
      const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(sq + tt * DP) + s;
      const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(sk + tt * DP) + s;
      const ulonglong2* g2 = reinterpret_cast<const ulonglong2*>(sg + tt * DP) + s;
      float v[C];
      if constexpr (C == 4) {
        const float4 f = *reinterpret_cast<const float4*>(sv + tt * COLS + col);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
      } else {
        const float2 f = *reinterpret_cast<const float2*>(sv + tt * COLS + col);
        v[0] = f.x; v[1] = f.y;
      }
      if constexpr (FORM == kFormDelta) {
        pair_t held[C], read[C], kk[P];
#pragma unroll
        for (int c = 0; c < C; ++c) held[c] = read[c] = 0ull;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          const ulonglong2 k = k2[S * i], q = q2[S * i];
          kk[2 * i] = k.x;
          kk[2 * i + 1] = k.y;
#pragma unroll
          for (int c = 0; c < C; ++c) {
            held[c] = pair_fma(k.x, St[c][2 * i], held[c]);
            held[c] = pair_fma(k.y, St[c][2 * i + 1], held[c]);
            read[c] = pair_fma(q.x, St[c][2 * i], read[c]);
            read[c] = pair_fma(q.y, St[c][2 * i + 1], read[c]);
          }
        }
        const float4 scal = reinterpret_cast<const float4*>(sc)[tt];            // beta, g, q . k
        const pair_t g = pair_of(scal.y, scal.y);
        float h1[C];
#pragma unroll
        for (int c = 0; c < C; ++c) h1[c] = pair_sum(held[c]);
#pragma unroll
        for (int off = 1; off < S; off <<= 1)
#pragma unroll
          for (int c = 0; c < C; ++c) h1[c] += __shfl_xor_sync(0xffffffffu, h1[c], off);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const float u = scal.x * (v[c] - scal.y * h1[c]);
          acc[tt * C + c] = scal.y * pair_sum(read[c]) + (s == 0 ? u * scal.z : 0.f);
          const pair_t uu = pair_of(u, u);
#pragma unroll
          for (int p = 0; p < P; ++p) St[c][p] = pair_fma(g, St[c][p], pair_mul(kk[p], uu));
        }
      } else {
        pair_t r[C], vv[C];
        float bonus = 0.f;
        if (FORM == kFormBonus && OUT)
          bonus = CG == 1 ? part[tt] : __shfl_sync(0xffffffffu, part[tt / CG], (tt % CG) * S + s);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          r[c] = FORM == kFormBonus ? pair_of(bonus * v[c], 0.f) : 0ull;
          vv[c] = pair_of(v[c], v[c]);
        }
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
          ulonglong2 q;
          if (OUT) q = q2[S * i];
          const ulonglong2 k = k2[S * i], f = g2[S * i];
          if (!OUT) {
            decays[2 * i % (OUT ? 1 : P)] = pair_mul(decays[2 * i % (OUT ? 1 : P)], f.x);
            decays[(2 * i + 1) % (OUT ? 1 : P)] = pair_mul(decays[(2 * i + 1) % (OUT ? 1 : P)], f.y);
          }
#pragma unroll
          for (int c = 0; c < C; ++c) {
            pair_t &lo = St[c][2 * i], &hi = St[c][2 * i + 1];
            if (FORM == kFormBonus && OUT) r[c] = pair_fma(q.y, hi, pair_fma(q.x, lo, r[c]));
            lo = pair_fma(f.x, lo, pair_mul(k.x, vv[c]));
            hi = pair_fma(f.y, hi, pair_mul(k.y, vv[c]));
            if (FORM == kFormKeyDecay && OUT) r[c] = pair_fma(q.y, hi, pair_fma(q.x, lo, r[c]));
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) acc[tt * C + c] = pair_sum(r[c]);
      }
    }
    if constexpr (OUT) {
      // 8 C sums over the group's S lanes: step b hands over the half of the values that bit b of the lane does not name
      constexpr int VALUES = kScanTile * C;
      int first = 0;                                              // which of the values this lane ends with
#pragma unroll
      for (int b = 0; (1 << b) < S; ++b) {
        const int left = VALUES >> (b + 1);
        if (left > 0) {
          const bool up = (s >> b) & 1;
#pragma unroll
          for (int i = 0; i < VALUES / 2; ++i)
            if (i < left)
              acc[i] = (up ? acc[i + left] : acc[i]) + __shfl_xor_sync(0xffffffffu, up ? acc[i] : acc[i + left], 1 << b);
          first += up ? left : 0;
        } else {
          acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1 << b);
        }
      }
      constexpr int KEPT = VALUES >= S ? VALUES / S : 1;
      if (s < VALUES) {
#pragma unroll
        for (int i = 0; i < KEPT; ++i) {
          const int tt = (first + i) / C, c = (first + i) % C;
          if (tt < n && j + c < Dv) a.o[(size_t)(t + tt) * a.H * Dv + (size_t)h * Dv + j + c] = acc[i];
        }
      }
    }
    if (more) put(t + kScanTile, buf ^ 1);
    __syncthreads();
  }
  if (OUT && t1 < seq_end) return;                              // the slot's state is the last chunk's to write
  float* end = OUT ? st : a.ws + (place + a.H) * D * Dv + j;
#pragma unroll
  for (int p = 0; p < P; ++p)
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int row = row_of(p);
      const float2 f = pair_split(St[c][p]);
      if (j + c < Dv && row < D) end[(size_t)row * Dv + c] = f.x;
      if (j + c < Dv && row + 1 < D) end[(size_t)(row + 1) * Dv + c] = f.y;
    }
  if (!OUT && blockIdx.x == 0 && col == 0) {
#pragma unroll
    for (int p = 0; p < (OUT ? 1 : P); ++p) {
      const int row = row_of(p);
      const float2 f = pair_split(decays[p]);
      if (row < D) a.prod[(place + a.H) * D + row] = f.x;
      if (row + 1 < D) a.prod[(place + a.H) * D + row + 1] = f.y;
    }
  }
}

// The chain over a sequence's chunks, a thread per element of the state: ws[0] = the slot's state, ws[c] = prod[c] (.)
// ws[c - 1] + ws[c], so that ws[c] is where chunk c starts.
__global__ void channel_chain_kernel(const StateArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y;
  const size_t n_state = (size_t)a.H * a.D * a.Dv, n_rows = (size_t)a.H * a.D;
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= n_state) return;
  const int nc = (a.cu_q[seq + 1] - a.cu_q[seq] + a.chunk - 1) / a.chunk;
  if (nc <= 0) return;
  float S = a.state[(size_t)a.seq_slot[seq] * n_state + e];
  float* w = a.ws + (size_t)seq * a.n_chunks * n_state + e;
  const float* d = a.prod + (size_t)seq * a.n_chunks * n_rows + e / a.Dv;
  w[0] = S;
  constexpr int U = 4;                                          // loads of the next chunks ahead of the chain
  for (int c0 = 1; c0 < nc; c0 += U) {
    float x[U], f[U];
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (c0 + i < nc) {
        x[i] = w[(size_t)(c0 + i) * n_state];
        f[i] = d[(size_t)(c0 + i) * n_rows];
      }
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (c0 + i < nc) {
        S = fmaf(f[i], S, x[i]);
        w[(size_t)(c0 + i) * n_state] = S;
      }
  }
}

// ------------------------------------------------------------------------------------------ one token per sequence
// What the one-token step needs besides StateArgs: what decays or rates are made of, and what becomes of the reading.
struct StepArgs {
  const void* x;            // FORM 0, 1: rows of R numbers of x_dtype, x_ld apart (the low-rank product's first half)
  const float* Bt;          // [R, G * D]
  const float* gate_bias;   // [G * D]
  const void* ba;           // FORM 2: rows of TP with b at b_off and a at a_off
  const float* A;           // FORM 2: exp(A_log), [H]
  const float* dt_bias;     // FORM 2: [H]
  const float* norm_w;      // head h uses norm_w[h * norm_stride ..]
  const void* z;            // the output gate, rows of H * Dv of TP, z_ld apart
  void* out;                // [T, H * Dv] of TP
  int x_ld, x_dtype, R, mode, ba_ld, b_off, a_off, norm_stride, z_ld;
  float inv_tau, unit_eps, norm_eps;
};

constexpr int kStepRows = 8;             // rows a thread keeps between the two passes of the delta rule

// grid (heads, sequences). A thread owns V adjacent columns (4 where the value size allows) and every RG-th row, RG the
// block's threads over the columns' threads, so that a warp's accesses to the state are whole rows side by side.
template <typename TQ, typename TP, int FORM, int V>
__global__ void __launch_bounds__(512, 2) state_step_kernel(const StateArgs a, const StepArgs p) {
  extern __shared__ __align__(16) float step_smem[];           // q [D] | k [D] | decays [D] | u [Dv] | partial sums
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, g = h / (a.H / a.G), D = a.D, Dv = a.Dv;
  const int NT = blockDim.x, tid = threadIdx.x;
  const int nc = Dv / V, RG = NT / nc;
  const int rg = tid / nc, c = (tid - rg * nc) * V;
  const bool works = rg < RG;
  const size_t t = a.cu_q[seq];
  float* st = a.state + (((size_t)a.seq_slot[seq] * a.H + h) * D) * Dv + c;
  auto load_state = [&](int row, float (&x)[V]) {
    if (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(st + (size_t)row * Dv);
      x[0] = v.x; x[1 % V] = v.y; x[2 % V] = v.z; x[3 % V] = v.w;
    } else {
      x[0] = st[(size_t)row * Dv];
    }
  };
  auto store_state = [&](int row, const float (&x)[V]) {
    if (V == 4) *reinterpret_cast<float4*>(st + (size_t)row * Dv) = make_float4(x[0], x[1 % V], x[2 % V], x[3 % V]);
    else st[(size_t)row * Dv] = x[0];
  };
  // the first rows are asked for before anything else is worked out
  float S[kStepRows][V];
#pragma unroll
  for (int i = 0; i < kStepRows; ++i)
    if (works && rg + i * RG < D) load_state(rg + i * RG, S[i]);
  float *sq = step_smem, *sk = sq + D, *sg = sk + D, *su = sg + D, *part = su + Dv;
  const TQ* qr = reinterpret_cast<const TQ*>(a.q) + t * a.q_ld + (size_t)g * D;
  const TQ* kr = reinterpret_cast<const TQ*>(a.k) + t * a.k_ld + (size_t)g * D;
  const TQ* vr = reinterpret_cast<const TQ*>(a.v) + t * a.v_ld + (size_t)h * Dv;
  float beta = 0.f, gt = 0.f, qk = 0.f;                         // FORM 2
  float bonus = 0.f;                                            // FORM 1: sum of q b k
  if (FORM == kFormDelta) {
    float s0 = 0.f, s1 = 0.f, s2 = 0.f;
    for (int i = tid; i < D; i += NT) {
      const float q = to_f32(qr[i]), k = to_f32(kr[i]);
      sq[i] = q;
      sk[i] = k;
      s0 = fmaf(q, q, s0);
      s1 = fmaf(k, k, s1);
      s2 = fmaf(q, k, s2);
    }
    s0 = block_sum(s0, red);
    s1 = block_sum(s1, red);
    s2 = block_sum(s2, red);
    const float rq = a.q_scale / sqrtf(s0 + p.unit_eps), rk = 1.f / sqrtf(s1 + p.unit_eps);
    for (int i = tid; i < D; i += NT) {                         // each thread its own entries
      sq[i] *= rq;
      sk[i] *= rk;
    }
    qk = s2 * rq * rk;
    const TP* bar = reinterpret_cast<const TP*>(p.ba) + t * p.ba_ld;
    beta = sigmoidf_(to_f32(bar[p.b_off + h]));
    gt = expf(-p.A[h] * softplusf_(to_f32(bar[p.a_off + h]) + p.dt_bias[h]));
  } else {
    const size_t GD = (size_t)a.G * D;
    float s0 = 0.f;
    for (int i = tid; i < D; i += NT) {
      const size_t ch = (size_t)g * D + i;
      float z = p.gate_bias[ch];
      for (int r = 0; r < p.R; ++r) {
        float x = p.x_dtype == LLMIE_F32 ? reinterpret_cast<const float*>(p.x)[t * p.x_ld + r]
                                         : to_f32(reinterpret_cast<const __nv_bfloat16*>(p.x)[t * p.x_ld + r]);
        if (p.mode == 1) x = tanhf(x);
        z = fmaf(p.Bt[(size_t)r * GD + ch], x, z);
      }
      const float q = to_f32(qr[i]) * a.q_scale, k = to_f32(kr[i]);
      sg[i] = key_decay(z, p.mode, p.inv_tau);
      sq[i] = q;
      sk[i] = k;
      if (FORM == kFormBonus) s0 = fmaf(q * a.bonus[ch], k, s0);
    }
    if (FORM == kFormBonus) bonus = block_sum(s0, red);
  }
  __syncthreads();
  float v[V], acc[V], held[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    v[e] = works ? to_f32(vr[c + e]) : 0.f;
    acc[e] = held[e] = 0.f;
  }
  for (int base = rg; base < D; base += kStepRows * RG) {
    if (!works) break;
    if (base != rg) {
#pragma unroll
      for (int i = 0; i < kStepRows; ++i)
        if (base + i * RG < D) load_state(base + i * RG, S[i]);
    }
#pragma unroll
    for (int i = 0; i < kStepRows; ++i) {
      const int row = base + i * RG;
      if (row < D) {
        const float q = sq[row], k = sk[row];
        const float f = FORM == kFormDelta ? 0.f : sg[row];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          if (FORM == kFormDelta) held[e] = fmaf(k, S[i][e], held[e]);
          if (FORM != kFormKeyDecay) acc[e] = fmaf(q, S[i][e], acc[e]);
          if (FORM != kFormDelta) S[i][e] = fmaf(f, S[i][e], k * v[e]);
          if (FORM == kFormKeyDecay) acc[e] = fmaf(q, S[i][e], acc[e]);
        }
        if (FORM != kFormDelta) store_state(row, S[i]);
      }
    }
  }
  float* part2 = part + RG * Dv;
  if (works) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      part[rg * Dv + c + e] = acc[e];
      if (FORM == kFormDelta) part2[rg * Dv + c + e] = held[e];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < Dv; j += NT) {
    float o = 0.f;
    for (int r = 0; r < RG; ++r) o += part[r * Dv + j];
    if (FORM == kFormBonus) o = fmaf(bonus, to_f32(vr[j]), o);
    if (FORM == kFormDelta) {
      float k = 0.f;
      for (int r = 0; r < RG; ++r) k += part2[r * Dv + j];
      const float u = beta * (to_f32(vr[j]) - gt * k);
      su[j] = u;
      o = fmaf(u, qk, gt * o);
    }
    part[j] = o;                                                // row 0 of the partial sums: column j is this thread's
    ss = fmaf(o, o, ss);
  }
  ss = block_sum(ss, red);                                      // its barriers also publish u
  const float rn = 1.f / sqrtf(ss / (float)Dv + p.norm_eps);
  const TP* zr = reinterpret_cast<const TP*>(p.z) + t * p.z_ld + (size_t)h * Dv;
  TP* yr = reinterpret_cast<TP*>(p.out) + (t * a.H + h) * Dv;
  for (int j = tid; j < Dv; j += NT)
    yr[j] = from_f32<TP>(part[j] * rn * p.norm_w[(size_t)h * p.norm_stride + j] * siluf_(to_f32(zr[j])));
  if (FORM != kFormDelta || !works) return;
  const float* u = su + c;
  const bool kept = D <= kStepRows * RG;                        // every row is still in registers
  for (int base = rg; base < D; base += kStepRows * RG) {
#pragma unroll
    for (int i = 0; i < kStepRows; ++i) {
      const int row = base + i * RG;
      if (row < D) {
        if (!kept) load_state(row, S[i]);
        const float k = sk[row];
#pragma unroll
        for (int e = 0; e < V; ++e) S[i][e] = fmaf(gt, S[i][e], k * u[e]);
        store_state(row, S[i]);
      }
    }
  }
}

}  // namespace llmie

using namespace llmie;

static inline bool dtype_ok(int dt) { return dt == LLMIE_F32 || dt == LLMIE_BF16; }

// x rows of R numbers of x_dtype, ld apart; Bt float32 [R, N]; bias float32 [N]; out float32 [T, N].
// mode 0: out = sigmoid(z)^inv_tau; mode 1: out = exp(-exp(z)) with tanh applied to x first. R up to 512.
extern "C" int llmie_low_rank_gate(const void* x, int ld, const float* Bt, const float* bias, float* out, int R, int N,
                                   int n_tokens, int mode, float inv_tau, int x_dtype, cudaStream_t stream) {
  if (!x || !Bt || !bias || !out || R <= 0 || N <= 0 || ld < R || n_tokens < 0 || mode < 0 || mode > 1)
    return LLMIE_ERR_BAD_ARG;
  if (!dtype_ok(x_dtype)) return LLMIE_ERR_DTYPE;
  const long long tiles = ((long long)n_tokens + kGateTokens - 1) / kGateTokens;
  if (R > 512 || tiles > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
  const dim3 grid((N + 127) / 128, (unsigned)tiles), block(128);
  const size_t smem = (size_t)R * kGateTokens * sizeof(float);
  if (x_dtype == LLMIE_F32)
    launch_k(low_rank_gate_kernel<float>, grid, block, smem, stream, (const float*)x, ld, Bt, bias, out, R, N, n_tokens,
             mode, inv_tau);
  else
    launch_k(low_rank_gate_kernel<__nv_bfloat16>, grid, block, smem, stream, (const __nv_bfloat16*)x, ld, Bt, bias, out,
             R, N, n_tokens, mode, inv_tau);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// See delta_prepare_kernel. A = exp(A_log), dt_bias float32 [H].
extern "C" int llmie_delta_prepare(const void* qkv, int ld, int qkv_dtype, const void* ba, int ba_ld, int b_off, int a_off,
                                   int ba_dtype, const float* A, const float* dt_bias, float eps, float q_scale, float* qn,
                                   float* kn, float* scal, float* qk, int n_tokens, int H, int G, int D,
                                   cudaStream_t stream) {
  if (!qkv || !ba || !A || !dt_bias || !qn || !kn || !scal || !qk || n_tokens < 0 || H <= 0 || G <= 0 || H % G || D <= 0 ||
      ld < 2 * G * D || b_off < 0 || a_off < 0 || ba_ld < b_off + H || ba_ld < a_off + H)
    return LLMIE_ERR_BAD_ARG;
  if (!dtype_ok(qkv_dtype) || !dtype_ok(ba_dtype)) return LLMIE_ERR_DTYPE;
  if (n_tokens == 0) return LLMIE_OK;
  const dim3 grid(n_tokens), block(128);
#define LLMIE_PREP(TC, TP)                                                                                              \
  launch_k(delta_prepare_kernel<TC, TP>, grid, block, 0, stream, (const TC*)qkv, ld, (const TP*)ba, ba_ld, b_off, a_off, \
           A, dt_bias, eps, q_scale, qn, kn, scal, qk, H, G, D)
  if (qkv_dtype == LLMIE_F32 && ba_dtype == LLMIE_F32) LLMIE_PREP(float, float);
  else if (qkv_dtype == LLMIE_F32) LLMIE_PREP(float, __nv_bfloat16);
  else if (ba_dtype == LLMIE_F32) LLMIE_PREP(__nv_bfloat16, float);
  else LLMIE_PREP(__nv_bfloat16, __nv_bfloat16);
#undef LLMIE_PREP
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// x [T, d] of `dtype`; prev float32 [slots, d]; mu float32 [n_mix, d]; out [n_mix, T, d] of `dtype`.
extern "C" int llmie_shift_mix(const void* x, float* prev, const float* mu, const int* cu_q, const int* tok_seq,
                               const int* seq_slot, void* out, int n_mix, int d, int n_tokens, int single, int dtype,
                               cudaStream_t stream) {
  if (!x || !prev || !mu || !out || n_mix <= 0 || d <= 0 || n_tokens < 0) return LLMIE_ERR_BAD_ARG;
  if (!dtype_ok(dtype)) return LLMIE_ERR_DTYPE;
  if (n_tokens == 0) return LLMIE_OK;
  const bool by8 = d % 8 == 0 && aligned16(x) && aligned16(prev) && aligned16(mu) && aligned16(out);
  const int units = by8 ? d / 8 : d, threads = units >= 128 ? 128 : (units + 31) / 32 * 32;
  const dim3 grid((units + threads - 1) / threads, n_tokens < 32768 ? n_tokens : 32768), block(threads);
#define LLMIE_SHIFT(K, T) \
  launch_k(K<T>, grid, block, 0, stream, (const T*)x, prev, mu, cu_q, tok_seq, seq_slot, (T*)out, n_mix, d, n_tokens, single)
  if (dtype == LLMIE_F32) {
    if (by8) LLMIE_SHIFT(shift_mix8_kernel, float);
    else LLMIE_SHIFT(shift_mix_kernel, float);
  } else {
    if (by8) LLMIE_SHIFT(shift_mix8_kernel, __nv_bfloat16);
    else LLMIE_SHIFT(shift_mix_kernel, __nv_bfloat16);
  }
#undef LLMIE_SHIFT
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

template <typename TQ, typename TV, int FORM, typename SH>
static int channel_scan_launch(const StateArgs& a, int n_seqs, cudaStream_t stream) {
  using L = ScanLayout<TQ, TV, FORM, SH>;
  auto kernel = channel_scan_kernel<TQ, TV, FORM, SH, true>;
  const dim3 grid((a.Dv + L::COLS - 1) / L::COLS, a.H, n_seqs * a.n_chunks), block(SH::NT);
  if (L::BYTES > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L::BYTES);
    if (e != cudaSuccess) return (int)e;
  }
  if constexpr (FORM != kFormDelta) {
    if (a.n_chunks > 1) {
      auto first = channel_scan_kernel<TQ, TV, FORM, SH, false>;
      if (L::BYTES > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L::BYTES);
        if (e != cudaSuccess) return (int)e;
      }
      launch_k(first, grid, block, L::BYTES, stream, a);
      const size_t n_state = (size_t)a.H * a.D * a.Dv;
      launch_k(channel_chain_kernel, dim3((unsigned)((n_state + 255) / 256), n_seqs), dim3(256), 0, stream, a);
    }
  }
  launch_k(kernel, grid, block, L::BYTES, stream, a);
  return LLMIE_OK;
}

// Four columns a thread where tokens do not wait for one another. The delta rule does: every token's write needs a sum over
// the rows first, so fewer lanes share a column there, unless the step has too few warps to hide that sum behind one another
// (which lanes add what then depends on how many sequences a step has; a float32 engine always takes the first way).
template <typename TQ, typename TV, int FORM>
static int channel_scan_sizes(const StateArgs& a, int n_seqs, cudaStream_t stream) {
  if constexpr (FORM == kFormDelta) {
    if (a.D <= 32) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 8, 4, 32>>(a, n_seqs, stream);
    if constexpr (sizeof(TV) == 2) {
      const long long warps = (long long)n_seqs * a.H * ((a.Dv + 31) / 32) * (a.D <= 64 ? 2 : 4);
      if (a.D <= 64 && warps < 900) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 8, 8, 128>>(a, n_seqs, stream);
      if (a.D > 64 && a.D <= 128 && warps < 900)
        return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 8, 16, 256>>(a, n_seqs, stream);
    }
    if (a.D <= 64) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 16, 4, 64>>(a, n_seqs, stream);
    if (a.D <= 128) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 16, 8, 128>>(a, n_seqs, stream);
    if (a.D <= 256) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 16, 16, 128>>(a, n_seqs, stream);
    return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 16, 32, 128>>(a, n_seqs, stream);
  } else {
    if (a.D <= 32) return channel_scan_launch<TQ, TV, FORM, ScanShape<4, 4, 8, 32>>(a, n_seqs, stream);
    if (a.D <= 64) return channel_scan_launch<TQ, TV, FORM, ScanShape<4, 4, 16, 64>>(a, n_seqs, stream);
    if (a.D <= 128) return channel_scan_launch<TQ, TV, FORM, ScanShape<4, 4, 32, 128>>(a, n_seqs, stream);
    if (a.D <= 256) return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 8, 32, 128>>(a, n_seqs, stream);
    return channel_scan_launch<TQ, TV, FORM, ScanShape<2, 16, 32, 128>>(a, n_seqs, stream);
  }
}

static inline bool aligned_rows(const void* p, int ld, int dt) {
  return ld % 4 == 0 && (reinterpret_cast<uintptr_t>(p) & (dt == LLMIE_F32 ? 15u : 7u)) == 0;
}

// q, k (rows q_ld, k_ld apart) of q_dtype, v (v_ld apart) of v_dtype; form 0 and 1: gate float32 [T, G D] (form 1 also
// bonus float32 [G D]); form 2: scal, qk as delta_prepare leaves them. state float32 [slots, H, D, Dv] is read and written;
// o float32 [T, H Dv]. D up to 512. ws null: whole pieces (the only way for form 2); otherwise chunks of `chunk` tokens side
// by side, n_chunks >= ceil(longest piece / chunk), ws float32 [n_seqs, n_chunks, H, D, Dv] and prod float32
// [n_seqs, n_chunks, H, D] scratch.
extern "C" int llmie_channel_scan(const void* q, int q_ld, const void* k, int k_ld, int q_dtype, float q_scale,
                                  const void* v, int v_ld, int v_dtype, const float* gate, const float* bonus,
                                  const float* scal, const float* qk, float* state, const int* cu_q, const int* seq_slot,
                                  float* o, float* ws, float* prod, int chunk, int n_chunks, int n_seqs, int H, int G, int D,
                                  int Dv, int form, cudaStream_t stream) {
  if (!q || !k || !v || !state || !o || n_seqs < 0 || H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || q_ld < G * D ||
      k_ld < G * D || v_ld < H * Dv || form < 0 || form > 2)
    return LLMIE_ERR_BAD_ARG;
  if ((form != 2 && !gate) || (form == 1 && !bonus) || (form == 2 && (!scal || !qk))) return LLMIE_ERR_BAD_ARG;
  if (!dtype_ok(q_dtype) || !dtype_ok(v_dtype)) return LLMIE_ERR_DTYPE;
  if (ws && (form == 2 || !prod || chunk <= 0 || chunk % kScanTile || n_chunks <= 0)) return LLMIE_ERR_BAD_ARG;
  if (!ws) { chunk = 0; n_chunks = 1; }
  if (D > 512 || H > 65535 || (long long)n_seqs * n_chunks > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_seqs == 0) return LLMIE_OK;
  const bool vec = D % 4 == 0 && aligned_rows(q, q_ld, q_dtype) && aligned_rows(k, k_ld, q_dtype) &&
                   (form == 2 || aligned_rows(gate, G * D, LLMIE_F32));
  const bool vec_v = Dv % 4 == 0 && aligned_rows(v, v_ld, v_dtype);
  const StateArgs a{q, k, v, gate, bonus, scal, qk, state, cu_q, seq_slot, o, q_ld, k_ld, v_ld, H, G, D, Dv,
                    (vec ? 1 : 0) | (vec_v ? 2 : 0), q_scale, ws, prod, chunk, n_chunks};
  if (form == 2 && (reinterpret_cast<uintptr_t>(scal) & 7u)) return LLMIE_ERR_ALIGNMENT;
  int rc = LLMIE_ERR_DTYPE;
#define LLMIE_SCAN_FORM(TQ, TV)                                                \
  rc = form == 0   ? channel_scan_sizes<TQ, TV, kFormKeyDecay>(a, n_seqs, stream) \
       : form == 1 ? channel_scan_sizes<TQ, TV, kFormBonus>(a, n_seqs, stream)    \
                   : LLMIE_ERR_DTYPE
  if (form == 2) {                                              // unit vectors are always float32
    if (q_dtype != LLMIE_F32) return LLMIE_ERR_DTYPE;
    rc = v_dtype == LLMIE_F32 ? channel_scan_sizes<float, float, kFormDelta>(a, n_seqs, stream)
                              : channel_scan_sizes<float, __nv_bfloat16, kFormDelta>(a, n_seqs, stream);
  } else if (q_dtype == LLMIE_F32 && v_dtype == LLMIE_F32) {
    LLMIE_SCAN_FORM(float, float);
  } else if (q_dtype == LLMIE_BF16 && v_dtype == LLMIE_BF16) {
    LLMIE_SCAN_FORM(__nv_bfloat16, __nv_bfloat16);
  }
#undef LLMIE_SCAN_FORM
  if (rc != LLMIE_OK) return rc;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// The threads of a step's block, or 0 where the sizes do not fit one.
static int step_threads(int D, int Dv, int V) {
  const int nc = Dv / V;
  int nt = 128;
  while (nt < 512 && (nt < nc || D > kStepRows * (nt / nc))) nt *= 2;
  return nt >= nc ? nt : 0;
}

static size_t step_smem(int D, int Dv, int V, int nt) {
  return sizeof(float) * (3 * (size_t)D + Dv + 2 * (size_t)(nt / (Dv / V)) * Dv);
}

static int step_columns(int Dv, const void* state) { return Dv % 4 == 0 && aligned16(state) ? 4 : 1; }

// 1 where llmie_state_step takes these sizes.
extern "C" int llmie_state_step_ok(int D, int Dv) {
  const int V = Dv % 4 == 0 ? 4 : 1;
  const int nt = step_threads(D, Dv, V);
  return nt && step_smem(D, Dv, V, nt) <= 48 * 1024 && D <= 2048;
}

// One token per sequence, everything around the recurrence included; q, k, v of q_dtype (float32 for form 2, dtype
// otherwise); x (of x_dtype), Bt, gate_bias, mode, inv_tau as in llmie_low_rank_gate (forms 0, 1); ba, A, dt_bias as in
// llmie_delta_prepare (form 2); then out = o / sqrt(mean(o^2) + eps over a head) * norm_w * silu(z), head h with
// norm_w[h * norm_stride ..]; z (z_ld apart), ba and out of `dtype`.
extern "C" int llmie_state_step(const void* q, int q_ld, const void* k, int k_ld, int q_dtype, float q_scale, const void* v,
                                int v_ld, const float* bonus, float* state, const int* cu_q, const int* seq_slot,
                                const void* x, int x_ld, int x_dtype, const float* Bt, const float* gate_bias, int R,
                                int mode, float inv_tau, const void* ba, int ba_ld, int b_off, int a_off, const float* A,
                                const float* dt_bias, float unit_eps, const float* norm_w, int norm_stride, float norm_eps,
                                const void* z, int z_ld, void* out, int dtype, int n_seqs, int H, int G, int D, int Dv,
                                int form, cudaStream_t stream) {
  if (!q || !k || !v || !state || !z || !out || !norm_w || n_seqs < 0 || H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 ||
      q_ld < G * D || k_ld < G * D || v_ld < H * Dv || z_ld < H * Dv || form < 0 || form > 2)
    return LLMIE_ERR_BAD_ARG;
  if (form != 2 && (!x || !Bt || !gate_bias || R <= 0 || x_ld < R || mode < 0 || mode > 1)) return LLMIE_ERR_BAD_ARG;
  if (form == 1 && !bonus) return LLMIE_ERR_BAD_ARG;
  if (form == 2 && (!ba || !A || !dt_bias || b_off < 0 || a_off < 0 || ba_ld < b_off + H || ba_ld < a_off + H))
    return LLMIE_ERR_BAD_ARG;
  if (!dtype_ok(dtype) || !dtype_ok(q_dtype) || (form != 2 && (!dtype_ok(x_dtype) || q_dtype != dtype)) ||
      (form == 2 && q_dtype != LLMIE_F32))
    return LLMIE_ERR_DTYPE;
  if (n_seqs == 0) return LLMIE_OK;
  const int V = step_columns(Dv, state);
  const int nt = step_threads(D, Dv, V);
  if (!nt || n_seqs > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const size_t smem = step_smem(D, Dv, V, nt);
  if (smem > 48 * 1024) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const StateArgs a{q, k, v, nullptr, bonus, nullptr, nullptr, state, cu_q, seq_slot, nullptr, q_ld, k_ld, v_ld, H, G, D,
                    Dv, 0, q_scale, nullptr, nullptr, 0, 1};
  const StepArgs p{x, Bt, gate_bias, ba, A, dt_bias, norm_w, z, out, x_ld, x_dtype, R, mode, ba_ld, b_off, a_off,
                   norm_stride, z_ld, inv_tau, unit_eps, norm_eps};
  const dim3 grid(H, n_seqs), block(nt);
#define LLMIE_STEP(TQ, TP, FORM)                                                                 \
  do {                                                                                           \
    if (V == 4) launch_k(state_step_kernel<TQ, TP, FORM, 4>, grid, block, smem, stream, a, p);   \
    else launch_k(state_step_kernel<TQ, TP, FORM, 1>, grid, block, smem, stream, a, p);          \
  } while (0)
  if (dtype == LLMIE_F32) {
    if (form == 0) LLMIE_STEP(float, float, kFormKeyDecay);
    else if (form == 1) LLMIE_STEP(float, float, kFormBonus);
    else LLMIE_STEP(float, float, kFormDelta);
  } else {
    if (form == 0) LLMIE_STEP(__nv_bfloat16, __nv_bfloat16, kFormKeyDecay);
    else if (form == 1) LLMIE_STEP(__nv_bfloat16, __nv_bfloat16, kFormBonus);
    else LLMIE_STEP(float, __nv_bfloat16, kFormDelta);
  }
#undef LLMIE_STEP
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}
