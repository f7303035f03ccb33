// Mixers that carry a fixed-size state from token to token instead of reading a cache of keys: a gated linear
// recurrence over a matrix state per head, and a gated linear recurrent unit over a vector state behind a short causal
// convolution. Everything that enters a recurrence (gates, decays, the state, the norms of what is read) is float32 in
// both precisions; the projections that feed the kernels have the activation type.
//
// Packed tokens: sequence s of the step owns rows cu_q[s] .. cu_q[s+1]-1, its state lives in row seq_slot[s] of a
// [slots, ...] float32 tensor and is read at the start and written at the end, so a sequence fed in pieces, or token
// by token, goes through exactly the same arithmetic as one fed whole.
//
//   matrix_gates       q = silu(q_raw), f = l + (1 - l) sigmoid(f_raw + b)           element-wise, float32 out
//   matrix_scan        S <- diag(f_t) S + (1 - f_t) v_t^T ; o_t = S^T q_t            S [dim, vdim] per head
//                      keyed form (a decay per head given): S <- a_h S + k_t v_t^T   linear attention with a constant decay
//                      stepped form (a decay and a factor per token and head): S <- a_t S + (c_t k_t) v_t^T, keys and
//                      queries shared by groups of heads (a state space model)
//   act_columns        float32 copies of up to three runs of columns of the projections, through an activation
//   matrix_scan_chunked  the same for long pieces, cut into chunks that run side by side (below)
//   head_rmsnorm       o / sqrt(mean(o^2) + eps) * w over each head's vdim (or over the whole row), w shared by the heads
//                      or with a weight per column, optionally times sigmoid(gate) or silu(gate)
//   causal_conv        u_t = act(b + sum_j taps[:, K-1-j] x_(t-j)), x before the step from the state's last K-1 inputs
//   conv_state_store   the last K-1 inputs after the step (a one-token step's causal_conv writes them itself)
//   unit_gate_values   a = exp(-c r softplus(lam)), drive = sqrt(1 - a^2) i u, r and i sigmoids of given pre-activations
//   unit_scan          S <- a_t S + drive_t ; out_t = S act(y_raw + b) ; the new conv state
//   unit_scan_chunked  the same for long pieces, 32 chunks of a sequence side by side in one block
//
// Long pieces. Both recurrences are linear in the state, S_end = A S_start + B with A the product of the chunk's gates
// and B what the chunk makes from a zero state. So a piece is cut into chunks; every chunk is run from zero (A and B),
// the chunks' true starting states follow from a short chain over the chunks, and every chunk is run again from its
// start, now with outputs. Twice the arithmetic, all of it float32 and in token order within a chunk; what differs
// from the token-by-token order is the rounding of the chain's steps only.
#include "common.cuh"
#include <math.h>

namespace llmie {

__device__ __forceinline__ float sigmoidf_(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------ matrix state
template <typename T>
__global__ void matrix_gates_kernel(const T* __restrict__ proj, int ld, int q_off, int f_off,
                                    const float* __restrict__ f_bias, const float* __restrict__ lower,
                                    float* __restrict__ q_out, float* __restrict__ f_out, int n, size_t total) {
  pdl_launch_dependents();
  pdl_wait();
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < total; i += stride) {
    const size_t t = i / n;
    const int c = (int)(i - t * n);
    const T* row = proj + t * ld;
    const float q = to_f32(row[q_off + c]);
    const float z = to_f32(row[f_off + c]) + f_bias[c];
    const float l = lower[c];
    q_out[i] = q * sigmoidf_(q);
    f_out[i] = l + (1.f - l) * sigmoidf_(z);
  }
}

constexpr int kScanThreads = 128;
constexpr int kScanR = 16;          // state rows a thread keeps at most (one column a thread)
constexpr int kScanRWide = 8;       // ... when it owns four columns

// grid (column tiles, heads, sequences). A thread owns C adjacent columns (C = 1, or 4 when the value size allows) of its
// head's state and the rows [s R, (s+1) R) of them, S = slices (a power of two up to 32, lanes that differ in their low
// bits), R = ceil(dim / S) <= RMAX. With four columns a thread every gate, key and query entry that is loaded serves
// four state entries: the kernel is bound by what the first-level cache delivers otherwise. The next token's gate, query
// and values are requested before the current token's products.
// FORM 1 (keyed): with `head_decay` (float32 [H]) the update is S <- head_decay[h] S + k_t v_t^T with the keys k_t in the
// place of fg. FORM 2 (stepped): head_decay and key_factor are float32 [T, H], S <- head_decay[t, h] S + (key_factor[t, h]
// k_t) v_t^T, and qa and fg have G <= H heads, each shared by H / G heads of the state. FORM 0: fg holds gates, G = H.
// MODE 0: a sequence's whole piece, from the slot's state to the slot's state. MODE 1 and 2 work on chunk c =
// blockIdx.z % NC of sequence blockIdx.z / NC, L tokens each, with ws float32 [n_seqs, NC, H, D, Dv] and decay float32
// [n_seqs, NC, H, D]: MODE 1 runs a chunk that is not the sequence's last from a zero state, without outputs, and leaves
// its end state in ws[c + 1] and the product of its gates in decay[c + 1]; MODE 2 runs a chunk from ws[c] with outputs,
// and the last one writes the slot's state.
template <typename T, int MODE, int C, int RMAX, int FORM>
__global__ void __launch_bounds__(kScanThreads)
matrix_scan_kernel(const float* __restrict__ qa, const float* __restrict__ fg, const T* __restrict__ v, int v_ld,
                   float* __restrict__ state, const int* __restrict__ cu_q, const int* __restrict__ seq_slot,
                   float* __restrict__ o, int H, int D, int Dv, int S, int R, int write_state,
                   float* __restrict__ ws, float* __restrict__ decay, int L, int NC,
                   const float* __restrict__ head_decay, const float* __restrict__ key_factor, int G) {
  pdl_launch_dependents();
  // keyed forms: fg holds keys k_t instead of gates, and every row of head h has the same gate
  constexpr bool keyed = FORM != 0, stepped = FORM == 2;
  const float dh = FORM == 1 ? head_decay[blockIdx.y] : 0.f;   // a constant of the model: no kernel writes it
  pdl_wait();
  const int s = threadIdx.x & (S - 1);
  const int col = threadIdx.x / S;
  const int j = (blockIdx.x * (kScanThreads / S) + col) * C;   // Dv is a multiple of C
  const int h = blockIdx.y;
  const int seq = MODE == 0 ? blockIdx.z : blockIdx.z / NC;
  const int chunk = MODE == 0 ? 0 : blockIdx.z - seq * NC;
  const bool live = j < Dv;
  const int jj = live ? j : Dv - C;
  const int i0 = s * R;
  const int seq_end = cu_q[seq + 1];
  const int t0 = MODE == 0 ? cu_q[seq] : cu_q[seq] + chunk * L;
  const int t1 = MODE == 0 ? seq_end : min(t0 + L, seq_end);
  if (MODE == 1 && t1 >= seq_end) return;          // the last chunk (or none at all): nobody needs its end state
  if (MODE == 2 && t0 >= seq_end) return;
  const int slot = seq_slot[seq];
  float* st = state + (((size_t)slot * H + h) * D) * Dv + jj;
  const size_t HDDv = (size_t)H * D * Dv;
  const float* start = MODE == 2 ? ws + ((size_t)seq * NC + chunk) * HDDv + ((size_t)h * D) * Dv + jj : st;
  float St[RMAX][C];
#pragma unroll
  for (int r = 0; r < RMAX; ++r)
#pragma unroll
    for (int c = 0; c < C; ++c)
      St[r][c] = (MODE != 1 && r < R && i0 + r < D) ? start[(size_t)(i0 + r) * Dv + c] : 0.f;
  float f[RMAX], q[RMAX], vj[C];
  const size_t HD = (size_t)G * D;
  const int hq = stepped ? h / (H / G) : h;
  float dt_gate = 0.f, dt_factor = 0.f;             // stepped form: the next token's decay and key factor
  auto fetch = [&](int t) {
    const float* fr = fg + (size_t)t * HD + (size_t)hq * D + i0;
    const float* qr = qa + (size_t)t * HD + (size_t)hq * D + i0;
    if (stepped) {
      dt_gate = head_decay[(size_t)t * H + h];
      dt_factor = key_factor[(size_t)t * H + h];
    }
#pragma unroll
    for (int r = 0; r < RMAX; ++r) {
      const bool ok = r < R && i0 + r < D;
      f[r] = ok ? fr[r] : 0.f;
      if (MODE != 1) q[r] = ok ? qr[r] : 0.f;
    }
#pragma unroll
    for (int c = 0; c < C; ++c) vj[c] = to_f32(v[(size_t)t * v_ld + (size_t)h * Dv + jj + c]);
  };
  float prod[RMAX];                                 // MODE 1: the product of the chunk's gates
#pragma unroll
  for (int r = 0; r < RMAX; ++r) prod[r] = 1.f;
  if (t0 < t1) fetch(t0);
  for (int t = t0; t < t1; ++t) {
    float cf[RMAX], cq[RMAX], cv[C], acc[C];
#pragma unroll
    for (int c = 0; c < C; ++c) { cv[c] = vj[c]; acc[c] = 0.f; }
#pragma unroll
    for (int r = 0; r < RMAX; ++r) { cf[r] = f[r]; cq[r] = MODE != 1 ? q[r] : 0.f; }
    const float tg = dt_gate, tf = dt_factor;
    if (t + 1 < t1) fetch(t + 1);
#pragma unroll
    for (int r = 0; r < RMAX; ++r) {
      const float gate = stepped ? tg : (keyed ? dh : cf[r]);
      const float write = stepped ? tf * cf[r] : (keyed ? cf[r] : 1.f - cf[r]);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        St[r][c] = fmaf(gate, St[r][c], write * cv[c]);
        if (MODE != 1) acc[c] = fmaf(St[r][c], cq[r], acc[c]);
      }
      if (MODE == 1) prod[r] *= gate;
    }
    if (MODE != 1) {
#pragma unroll
      for (int c = 0; c < C; ++c) {
        for (int off = 1; off < S; off <<= 1) acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], off);
        if (s == 0 && live) o[(size_t)t * H * Dv + (size_t)h * Dv + j + c] = acc[c];
      }
    }
  }
  if (MODE == 1) {
    float* end = ws + ((size_t)seq * NC + chunk + 1) * HDDv + ((size_t)h * D) * Dv + jj;
    float* dec = decay + (((size_t)seq * NC + chunk + 1) * H + h) * D;
#pragma unroll
    for (int r = 0; r < RMAX; ++r)
      if (r < R && i0 + r < D) {
        if (live) {
#pragma unroll
          for (int c = 0; c < C; ++c) end[(size_t)(i0 + r) * Dv + c] = St[r][c];
        }
        if (blockIdx.x == 0 && col == 0) dec[i0 + r] = prod[r];
      }
    return;
  }
  if (write_state && live && t1 >= seq_end) {
#pragma unroll
    for (int r = 0; r < RMAX; ++r)
      if (r < R && i0 + r < D) {
#pragma unroll
        for (int c = 0; c < C; ++c) st[(size_t)(i0 + r) * Dv + c] = St[r][c];
      }
  }
}

// How a head's state is cut among threads: C columns a thread, S slices of R rows.
struct ScanShape { int C, S, R; };
static inline ScanShape scan_shape(int D, int Dv) {
  ScanShape g;
  // four columns a thread where the value size is a multiple of four and fills a block's threads that way (a narrow
  // state would leave threads without columns); one column a thread otherwise
  int s4 = 1;
  while (s4 * kScanRWide < D) s4 <<= 1;
  g.C = (Dv % 4 == 0 && s4 <= 32 && (kScanThreads / s4) * 4 <= Dv) ? 4 : 1;
  const int rmax = g.C == 4 ? kScanRWide : kScanR;
  g.S = 1;
  while (g.S * rmax < D) g.S <<= 1;
  g.R = (D + g.S - 1) / g.S;
  return g;
}

// The chain over a sequence's chunks, a thread per element of the state: ws[0] = the slot's state and
// ws[c] = decay[c] (.) ws[c - 1] + ws[c] for the chunks the sequence has, so that ws[c] is where chunk c starts.
__global__ void matrix_scan_chain_kernel(const float* __restrict__ state, const int* __restrict__ cu_q,
                                         const int* __restrict__ seq_slot, float* __restrict__ ws,
                                         const float* __restrict__ decay, int H, int D, int Dv, int L, int NC) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y;
  const size_t HDDv = (size_t)H * D * Dv;
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= HDDv) return;
  const int n = cu_q[seq + 1] - cu_q[seq];
  const int nc = (n + L - 1) / L;
  if (nc <= 0) return;
  const size_t hi = e / Dv;                         // (head, row) of the element
  float S = state[(size_t)seq_slot[seq] * HDDv + e];
  float* w = ws + (size_t)seq * NC * HDDv + e;
  const float* d = decay + (size_t)seq * NC * H * D + hi;
  w[0] = S;
  for (int c = 1; c < nc; ++c) {
    S = fmaf(d[(size_t)c * H * D], S, w[(size_t)c * HDDv]);
    w[(size_t)c * HDDv] = S;
  }
}

// sigmoid(z), or silu(z) = z sigmoid(z)
__device__ __forceinline__ float gate_factor(float z, int silu) { return (silu ? z : 1.f) / (1.f + expf(-z)); }

// a warp per (token, head): o float32 [T, H * Dv] -> y of the activation type. `gate` (rows gate_ld apart, null = none):
// the result is multiplied by sigmoid(gate) (or silu) of the same place. An item may also be a token's whole row (Dv = the
// row). The weights repeat every w_items items (1: all heads share them).
template <typename T>
__global__ void head_rmsnorm_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps,
                                    T* __restrict__ y, int Dv, size_t n_items, const T* __restrict__ gate, int gate_ld,
                                    int items_per_row, int silu, int w_items) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t item = (size_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= n_items) return;
  if (w_items > 1) w += (item % w_items) * Dv;
  const float* row = o + item * Dv;
  float ss = 0.f;
  for (int i = lane; i < Dv; i += 32) { const float x = row[i]; ss = fmaf(x, x, ss); }
  ss = warp_sum(ss);
  const float r = 1.f / sqrtf(ss / (float)Dv + eps);
  if (!gate) {
    for (int i = lane; i < Dv; i += 32) y[item * Dv + i] = from_f32<T>(row[i] * r * w[i]);
    return;
  }
  const size_t t = item / items_per_row;
  const T* gr = gate + t * gate_ld + (item - t * items_per_row) * Dv;
  for (int i = lane; i < Dv; i += 32)
    y[item * Dv + i] = from_f32<T>(row[i] * r * w[i] * gate_factor(to_f32(gr[i]), silu));
}

// The same for wide items (a token's whole row of concatenated heads): a block per item, so that a one-token step's few
// rows are not each one warp's work. Dv % 4 == 0 and 16-byte aligned rows: four elements a thread and access.
template <typename T>
__global__ void __launch_bounds__(256)
row_rmsnorm_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps, T* __restrict__ y, int Dv,
                   const T* __restrict__ gate, int gate_ld, int items_per_row, int silu, int w_items) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const size_t item = blockIdx.x;
  if (w_items > 1) w += (item % w_items) * Dv;
  const float4* row = reinterpret_cast<const float4*>(o + item * Dv);
  const int n4 = Dv >> 2;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n4; i += blockDim.x) {
    const float4 x = row[i];
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)Dv + eps);
  const size_t t = item / items_per_row;
  const T* gr = gate ? gate + t * gate_ld + (item - t * items_per_row) * Dv : nullptr;
  T* yr = y + item * Dv;
  for (int i = threadIdx.x; i < n4; i += blockDim.x) {
    const float4 x = row[i];
    const float4 wv = reinterpret_cast<const float4*>(w)[i];
    float v[4] = {x.x * r * wv.x, x.y * r * wv.y, x.z * r * wv.z, x.w * r * wv.w};
    if (gr) {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = v[e] * gate_factor(to_f32(gr[4 * i + e]), silu);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) yr[4 * i + e] = from_f32<T>(v[e]);
  }
}

// Float32 copies of up to three runs of columns of proj [T, ld], each through the activation `act`:
// out_k[t, c] = act(proj[t, off_k + c]), c < n_k. (What a linear-attention layer reads of its projections.)
template <typename T>
__global__ void act_columns_kernel(const T* __restrict__ proj, int ld, int off0, int n0, float* __restrict__ out0,
                                   int off1, int n1, float* __restrict__ out1, int off2, int n2,
                                   float* __restrict__ out2, int act, size_t total) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = n0 + n1 + n2;
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < total; i += stride) {
    const size_t t = i / n;
    int c = (int)(i - t * n);
    const T* row = proj + t * ld;
    if (c < n0) { out0[t * n0 + c] = apply_act(to_f32(row[off0 + c]), act); continue; }
    c -= n0;
    if (c < n1) { out1[t * n1 + c] = apply_act(to_f32(row[off1 + c]), act); continue; }
    c -= n1;
    out2[t * n2 + c] = apply_act(to_f32(row[off2 + c]), act);
  }
}

// ------------------------------------------------------------------------------------------ vector state
constexpr int kMaxTaps = 16;

// A thread is V adjacent channels over a run of consecutive packed tokens. x = proj[:, x_off + c] + x_bias; inputs before
// the step come from conv_state [slots, K-1, C] (the last K-1 inputs of the sequence so far, zeros at its start). Oldest
// input first: a fixed order of summation.
// `act`: an activation of the result. `single`: every sequence of the step brings one token, so a channel's inputs are
// this thread's alone and it also writes the new conv_state (in other steps conv_state_store does).
template <typename TP, int V>
__device__ __forceinline__ void conv_input(const TP* p, const float (&xb)[V], float (&x)[V]) {
  if (V == 4) {
    if (sizeof(TP) == 4) {
      const float4 r = *reinterpret_cast<const float4*>(p);
      x[0] = r.x; x[1 % V] = r.y; x[2 % V] = r.z; x[3 % V] = r.w;
    } else {
      const uint2 r = *reinterpret_cast<const uint2*>(p);
      const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
      const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
      x[0] = lo.x; x[1 % V] = lo.y; x[2 % V] = hi.x; x[3 % V] = hi.y;
    }
  } else {
    x[0] = to_f32(p[0]);
  }
#pragma unroll
  for (int e = 0; e < V; ++e) x[e] += xb[e];
}

template <typename TO, int V>
__device__ __forceinline__ void conv_output(TO* dst, const float (&a)[V]) {
  if (V == 4 && sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(dst) = make_float4(a[0], a[1 % V], a[2 % V], a[3 % V]);
  } else if (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1 % V]), hi = __floats2bfloat162_rn(a[2 % V], a[3 % V]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(dst) = raw;
  } else {
    dst[0] = from_f32<TO>(a[0]);
  }
}

// TILE: tokens a thread works on. A tile that lies within one sequence (nearly all do) asks for its TILE + K - 1 inputs at
// once; one that crosses from a sequence into the next goes token by token, with all K inputs of each.
template <typename TP, typename TO, int KM, int V, int TILE>
__global__ void causal_conv_kernel(const TP* __restrict__ proj, int ld, int x_off, const float* __restrict__ x_bias,
                                   const float* __restrict__ taps, const float* __restrict__ conv_bias,
                                   float* conv_state, const int* __restrict__ cu_q,
                                   const int* __restrict__ tok_seq, const int* __restrict__ seq_slot,
                                   TO* __restrict__ u, int C, int K, int n_tokens, int act, int single) {
  pdl_launch_dependents();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  float tp[KM][V], xb[V], cb[V];                      // tp[i]: the taps of the inputs i tokens back
  auto load_v = [&](const float* src, float (&v)[V]) {          // weights: no kernel writes them
    if (V == 4) {
      const float4 r = *reinterpret_cast<const float4*>(src + c);
      v[0] = r.x; v[1 % V] = r.y; v[2 % V] = r.z; v[3 % V] = r.w;
    } else {
      v[0] = src[c];
    }
  };
#pragma unroll
  for (int e = 0; e < V; ++e) xb[e] = cb[e] = 0.f;
#pragma unroll
  for (int i = 0; i < KM; ++i)
    if (i < K) load_v(taps + (size_t)(K - 1 - i) * C, tp[i]);
  if (x_bias) load_v(x_bias, xb);
  if (conv_bias) load_v(conv_bias, cb);
  pdl_wait();
  const int ta = blockIdx.x * TILE, tb = min(ta + TILE, n_tokens);
  constexpr int W = KM - 1;
  float x[TILE + W][V];                               // x[W + j]: the input of token t0 + j
  // the rows in front of the tile are asked for with the tile's own, before it is known whose they are
  {
    const TP* src = proj + (size_t)ta * ld + x_off + c;
#pragma unroll
    for (int j = 0; j < TILE; ++j)
      if (ta + j < tb) conv_input<TP, V>(src + (size_t)j * ld, xb, x[W + j]);
#pragma unroll
    for (int i = 1; i < KM; ++i)
      if (i < K && ta - i >= 0) conv_input<TP, V>(src - (size_t)i * ld, xb, x[W - i]);
  }
  const bool whole = TILE == 1 || tok_seq[ta] == tok_seq[tb - 1];
  for (int t0 = ta; t0 < tb; t0 += whole ? TILE : 1) {
    const int seq = tok_seq[t0];
    const int p = t0 - cu_q[seq];                     // place within this step's piece of the sequence
    const int n = whole ? tb - t0 : 1;
    const TP* src = proj + (size_t)t0 * ld + x_off + c;
    if (!whole) conv_input<TP, V>(src, xb, x[W]);
    float* cs = conv_state + (size_t)seq_slot[seq] * (K - 1) * C + c;
#pragma unroll
    for (int i = 1; i < KM; ++i) {
      if (i < K) {
        if (p - i >= 0) {
          if (!whole) conv_input<TP, V>(src - (size_t)i * ld, xb, x[W - i]);
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) x[W - i][e] = cs[(size_t)(K - 1 + p - i) * C + e];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < TILE; ++j) {
      if (j < n) {
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          acc[e] = cb[e];
#pragma unroll
          for (int i = KM - 1; i >= 0; --i)
            if (i < K) acc[e] = fmaf(tp[i][e], x[W + j - i][e], acc[e]);
        }
        if (sizeof(TO) == 2 && act == 4) {            // silu in front of a store that keeps 8 bits of it
#pragma unroll
          for (int e = 0; e < V; ++e) acc[e] = acc[e] * __fdividef(1.f, 1.f + __expf(-acc[e]));
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) acc[e] = apply_act(acc[e], act);
        }
        conv_output<TO, V>(u + (size_t)(t0 + j) * C + c, acc);
      }
    }
    if (single) {                                     // K - 1 inputs, the oldest first
#pragma unroll
      for (int i = 0; i + 1 < KM; ++i)
        if (i + 1 < K) {
#pragma unroll
          for (int e = 0; e < V; ++e) cs[(size_t)(K - 2 - i) * C + e] = x[W - i][e];
        }
    }
  }
}

// The convolution's new state: a thread per (sequence, channel) leaves the last K-1 inputs of the sequence, this step's
// and before them what the state held.
template <typename T>
__global__ void conv_state_store_kernel(const T* __restrict__ proj, int ld, int x_off, const float* __restrict__ x_bias,
                                        float* __restrict__ conv_state, const int* __restrict__ cu_q,
                                        const int* __restrict__ seq_slot, int C, int K) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y;
  if (c >= C) return;
  const int t0 = cu_q[seq], n = cu_q[seq + 1] - t0;
  float* cs = conv_state + (size_t)seq_slot[seq] * (K - 1) * C + c;
  const float xb = x_bias ? x_bias[c] : 0.f;
  float keep[kMaxTaps];
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k) {
    if (k < K - 1) {
      const int m = n - (K - 1) + k;                  // place within the step, negative = before it
      keep[k] = m >= 0 ? to_f32(proj[(size_t)(t0 + m) * ld + x_off + c]) + xb : cs[(size_t)(K - 1 + m) * C];
    }
  }
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k)
    if (k < K - 1) cs[(size_t)k * C] = keep[k];
}

// gates [T, groups * 2 * bw]: per group the pre-activations of r (bw) and then of i (bw). In place: r's place receives
// a = exp(-c r softplus(lam)), i's place the drive sqrt(1 - a^2) * i * u.
__global__ void unit_gate_values_kernel(float* __restrict__ gates, const float* __restrict__ u,
                                        const float* __restrict__ r_bias, const float* __restrict__ i_bias,
                                        const float* __restrict__ lam, float c_decay, int C, int bw, size_t total) {
  pdl_launch_dependents();
  pdl_wait();
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < total; i += stride) {
    const size_t t = i / C;
    const int c = (int)(i - t * C);
    const int g = c / bw, e = c - g * bw;
    float* gr = gates + t * 2 * C + (size_t)g * 2 * bw + e;
    const float r = sigmoidf_(gr[0] + r_bias[c]);
    const float in = sigmoidf_(gr[bw] + i_bias[c]);
    const float log_a = -c_decay * r * softplusf_(lam[c]);
    const float a = expf(log_a);
    gr[0] = a;
    gr[bw] = sqrtf(-expm1f(2.f * log_a)) * (in * u[i]);     // 1 - a^2 without cancellation near a = 1
  }
}

// a thread per (sequence, channel): the recurrence over the step's tokens, the output gate act(y_raw + y_bias), and
// the new state of the recurrence and of the convolution.
template <typename T>
__global__ void unit_scan_kernel(const float* __restrict__ gates, const T* __restrict__ proj, int ld, int y_off,
                                 int x_off, const float* __restrict__ y_bias, const float* __restrict__ x_bias,
                                 int act, float* __restrict__ state, float* __restrict__ conv_state,
                                 const int* __restrict__ cu_q, const int* __restrict__ seq_slot, T* __restrict__ out,
                                 int C, int bw, int K, int write_state) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y;
  if (c >= C) return;
  const int t0 = cu_q[seq], t1 = cu_q[seq + 1];
  const int slot = seq_slot[seq];
  const int g = c / bw, e = c - g * bw;
  const float yb = y_bias ? y_bias[c] : 0.f;
  float S = state[(size_t)slot * C + c];
  const float* gr = gates + (size_t)g * 2 * bw + e;
  constexpr int U = 4;
  int t = t0;
  for (; t + U <= t1; t += U) {
    float a[U], d[U], y[U];
#pragma unroll
    for (int k = 0; k < U; ++k) {
      a[k] = gr[(size_t)(t + k) * 2 * C];
      d[k] = gr[(size_t)(t + k) * 2 * C + bw];
      y[k] = apply_act(to_f32(proj[(size_t)(t + k) * ld + y_off + c]) + yb, act);
    }
#pragma unroll
    for (int k = 0; k < U; ++k) {
      S = fmaf(a[k], S, d[k]);
      out[(size_t)(t + k) * C + c] = from_f32<T>(S * y[k]);
    }
  }
  for (; t < t1; ++t) {
    S = fmaf(gr[(size_t)t * 2 * C], S, gr[(size_t)t * 2 * C + bw]);
    out[(size_t)t * C + c] = from_f32<T>(S * apply_act(to_f32(proj[(size_t)t * ld + y_off + c]) + yb, act));
  }
  if (!write_state) return;
  state[(size_t)slot * C + c] = S;
  // the last K-1 inputs of the sequence: this step's, and before them what the state held
  float* cs = conv_state + (size_t)slot * (K - 1) * C + c;
  const int n = t1 - t0;
  const float xb = x_bias ? x_bias[c] : 0.f;
  float keep[kMaxTaps];
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k) {
    if (k < K - 1) {
      const int m = n - (K - 1) + k;                  // place within the step, negative = before it
      keep[k] = m >= 0 ? to_f32(proj[(size_t)(t0 + m) * ld + x_off + c]) + xb : cs[(size_t)(K - 1 + m) * C];
    }
  }
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k)
    if (k < K - 1) cs[(size_t)k * C] = keep[k];
}

// The same recurrence for long pieces: a block is 32 channels by kUnitChunks chunks of one sequence. Every thread runs
// its chunk from zero (the product of its a's and what it makes), the first warp chains the chunks' starting states in
// shared memory, and every thread runs its chunk again from its start, now with outputs.
constexpr int kUnitChunks = 32;

template <typename T>
__global__ void __launch_bounds__(32 * kUnitChunks)
unit_scan_chunked_kernel(const float* __restrict__ gates, const T* __restrict__ proj, int ld, int y_off, int x_off,
                         const float* __restrict__ y_bias, const float* __restrict__ x_bias, int act,
                         float* __restrict__ state, float* __restrict__ conv_state, const int* __restrict__ cu_q,
                         const int* __restrict__ seq_slot, T* __restrict__ out, int C, int bw, int K, int write_state) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sA[kUnitChunks][33], sB[kUnitChunks][33];
  const int cx = threadIdx.x, ky = threadIdx.y;
  const int c = blockIdx.x * 32 + cx;
  const int seq = blockIdx.y;
  const bool live = c < C;
  const int cc = live ? c : C - 1;
  const int t0 = cu_q[seq], t1 = cu_q[seq + 1];
  const int n = t1 - t0;
  const int L = (n + kUnitChunks - 1) / kUnitChunks;
  const int a0 = min(t0 + ky * L, t1), a1 = min(a0 + L, t1);
  const int slot = seq_slot[seq];
  const int g = cc / bw, e = cc - g * bw;
  const float* gr = gates + (size_t)g * 2 * bw + e;
  constexpr int U = 4;
  {
    float A = 1.f, B = 0.f;
    int t = a0;
    for (; t + U <= a1; t += U) {
      float a[U], d[U];
#pragma unroll
      for (int k = 0; k < U; ++k) {
        a[k] = gr[(size_t)(t + k) * 2 * C];
        d[k] = gr[(size_t)(t + k) * 2 * C + bw];
      }
#pragma unroll
      for (int k = 0; k < U; ++k) {
        A *= a[k];
        B = fmaf(a[k], B, d[k]);
      }
    }
    for (; t < a1; ++t) {
      const float a = gr[(size_t)t * 2 * C];
      A *= a;
      B = fmaf(a, B, gr[(size_t)t * 2 * C + bw]);
    }
    sA[ky][cx] = A;
    sB[ky][cx] = B;
  }
  __syncthreads();
  if (ky == 0) {                                       // sB[k] becomes where chunk k starts
    float S = state[(size_t)slot * C + cc];
    for (int k = 0; k < kUnitChunks; ++k) {
      const float next = fmaf(sA[k][cx], S, sB[k][cx]);
      sB[k][cx] = S;
      S = next;
    }
    if (write_state && live) state[(size_t)slot * C + c] = S;
  }
  __syncthreads();
  if (live) {
    const float yb = y_bias ? y_bias[c] : 0.f;
    float S = sB[ky][cx];
    int t = a0;
    for (; t + U <= a1; t += U) {
      float a[U], d[U], y[U];
#pragma unroll
      for (int k = 0; k < U; ++k) {
        a[k] = gr[(size_t)(t + k) * 2 * C];
        d[k] = gr[(size_t)(t + k) * 2 * C + bw];
        y[k] = apply_act(to_f32(proj[(size_t)(t + k) * ld + y_off + c]) + yb, act);
      }
#pragma unroll
      for (int k = 0; k < U; ++k) {
        S = fmaf(a[k], S, d[k]);
        out[(size_t)(t + k) * C + c] = from_f32<T>(S * y[k]);
      }
    }
    for (; t < a1; ++t) {
      S = fmaf(gr[(size_t)t * 2 * C], S, gr[(size_t)t * 2 * C + bw]);
      out[(size_t)t * C + c] = from_f32<T>(S * apply_act(to_f32(proj[(size_t)t * ld + y_off + c]) + yb, act));
    }
  }
  if (!write_state || !live || ky != 0) return;
  // the last K-1 inputs of the sequence: this step's, and before them what the state held
  float* cs = conv_state + (size_t)slot * (K - 1) * C + c;
  const float xb = x_bias ? x_bias[c] : 0.f;
  float keep[kMaxTaps];
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k) {
    if (k < K - 1) {
      const int m = n - (K - 1) + k;                  // place within the step, negative = before it
      keep[k] = m >= 0 ? to_f32(proj[(size_t)(t0 + m) * ld + x_off + c]) + xb : cs[(size_t)(K - 1 + m) * C];
    }
  }
#pragma unroll
  for (int k = 0; k < kMaxTaps; ++k)
    if (k < K - 1) cs[(size_t)k * C] = keep[k];
}

}  // namespace llmie

using namespace llmie;

static inline unsigned sweep_blocks(size_t total, int threads) {
  size_t b = (total + threads - 1) / threads;
  return (unsigned)(b > 148 * 16 ? 148 * 16 : (b ? b : 1));
}

// proj [T, ld] of `dtype` holds the raw query projection at column q_off and the raw gate projection at f_off, n
// columns each; f_bias, lower float32 [n]; q_out, f_out float32 [T, n].
extern "C" int llmie_matrix_gates(const void* proj, int ld, int q_off, int f_off, const float* f_bias, const float* lower,
                                  float* q_out, float* f_out, int n_tokens, int n, int dtype, cudaStream_t stream) {
  if (n_tokens < 0 || n <= 0 || q_off < 0 || f_off < 0 || ld < q_off + n || ld < f_off + n) return LLMIE_ERR_BAD_ARG;
  if (!f_bias || !lower) return LLMIE_ERR_BAD_ARG;
  if (n_tokens == 0) return LLMIE_OK;
  const size_t total = (size_t)n_tokens * n;
  const dim3 grid(sweep_blocks(total, 256)), block(256);
  if (dtype == LLMIE_F32)
    launch_k(matrix_gates_kernel<float>, grid, block, 0, stream, (const float*)proj, ld, q_off, f_off, f_bias, lower,
             q_out, f_out, n, total);
  else if (dtype == LLMIE_BF16)
    launch_k(matrix_gates_kernel<__nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)proj, ld, q_off, f_off,
             f_bias, lower, q_out, f_out, n, total);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// What one of the scans reads and writes, whatever its form.
struct ScanArgs {
  const float* qa;
  const float* fg;
  const void* v;
  int v_ld;
  float* state;
  const int* cu_q;
  const int* seq_slot;
  float* o;
  int n_seqs, H, D, Dv, write_state;
  const float* head_decay;     // FORM 1: [H], FORM 2: [T, H], FORM 0: null
  const float* key_factor;     // FORM 2: [T, H], else null
  int G;                       // heads of qa and fg
  float* ws;                   // chunked: scratch, else null
  float* decay;
  int chunk, n_chunks;
};

template <typename T, int C, int RM, int FORM>
static void matrix_scan_launch(const ScanArgs& a, const ScanShape& g, cudaStream_t stream) {
  const int cols = (kScanThreads / g.S) * C;
  const bool chunked = a.ws != nullptr;
  const dim3 grid((a.Dv + cols - 1) / cols, a.H, a.n_seqs * (chunked ? a.n_chunks : 1)), block(kScanThreads);
#define LLMIE_SCAN_ARGS                                                                                                   \
  grid, block, 0, stream, a.qa, a.fg, (const T*)a.v, a.v_ld, a.state, a.cu_q, a.seq_slot, a.o, a.H, a.D, a.Dv, g.S, g.R, \
      a.write_state, a.ws, a.decay, a.chunk, a.n_chunks, a.head_decay, a.key_factor, a.G
  if (!chunked) {
    launch_k(matrix_scan_kernel<T, 0, C, RM, FORM>, LLMIE_SCAN_ARGS);
    return;
  }
  launch_k(matrix_scan_kernel<T, 1, C, RM, FORM>, LLMIE_SCAN_ARGS);
  const size_t HDDv = (size_t)a.H * a.D * a.Dv;
  launch_k(matrix_scan_chain_kernel, dim3((unsigned)((HDDv + 255) / 256), a.n_seqs), dim3(256), 0, stream,
           (const float*)a.state, a.cu_q, a.seq_slot, a.ws, (const float*)a.decay, a.H, a.D, a.Dv, a.chunk, a.n_chunks);
  launch_k(matrix_scan_kernel<T, 2, C, RM, FORM>, LLMIE_SCAN_ARGS);
#undef LLMIE_SCAN_ARGS
}

template <int FORM>
static int matrix_scan_entry(const ScanArgs& a, int dtype, cudaStream_t stream) {
  if (a.n_seqs < 0 || a.H <= 0 || a.D <= 0 || a.Dv <= 0 || a.v_ld < a.H * a.Dv || a.G <= 0 || a.H % a.G)
    return LLMIE_ERR_BAD_ARG;
  if (a.ws && (a.chunk <= 0 || a.n_chunks <= 0 || !a.decay)) return LLMIE_ERR_BAD_ARG;
  if (a.D > 32 * kScanR) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (a.n_seqs == 0) return LLMIE_OK;
  if (a.H > 65535 || a.n_seqs > 65535 || (a.ws && (long long)a.n_seqs * a.n_chunks > 65535)) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const ScanShape g = scan_shape(a.D, a.Dv);
  if (dtype == LLMIE_F32) {
    if (g.C == 4) matrix_scan_launch<float, 4, kScanRWide, FORM>(a, g, stream);
    else matrix_scan_launch<float, 1, kScanR, FORM>(a, g, stream);
  } else if (dtype == LLMIE_BF16) {
    if (g.C == 4) matrix_scan_launch<__nv_bfloat16, 4, kScanRWide, FORM>(a, g, stream);
    else matrix_scan_launch<__nv_bfloat16, 1, kScanR, FORM>(a, g, stream);
  } else {
    return LLMIE_ERR_DTYPE;
  }
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// qa, fg float32 [T, H * D]; v rows of H * Dv elements of `dtype`, v_ld apart; state float32 [slots, H, D, Dv];
// o float32 [T, H * Dv]. D up to 512.
// head_decay float32 [H] or null: with it, fg holds keys and S <- head_decay[h] S + k_t v_t^T.
extern "C" int llmie_matrix_scan_ex(const float* qa, const float* fg, const void* v, int v_ld, float* state,
                                    const int* cu_q, const int* seq_slot, float* o, int n_seqs, int H, int D, int Dv,
                                    int write_state, int dtype, const float* head_decay, cudaStream_t stream) {
  const ScanArgs a{qa, fg, v, v_ld, state, cu_q, seq_slot, o, n_seqs, H, D, Dv, write_state, head_decay, nullptr, H,
                   nullptr, nullptr, 0, 1};
  return head_decay ? matrix_scan_entry<1>(a, dtype, stream) : matrix_scan_entry<0>(a, dtype, stream);
}

// llmie_matrix_scan_ex for long pieces: chunks of `chunk` tokens run side by side. n_chunks >= ceil(longest piece /
// chunk); ws float32 [n_seqs, n_chunks, H, D, Dv] and decay float32 [n_seqs, n_chunks, H, D] are scratch.
extern "C" int llmie_matrix_scan_chunked_ex(const float* qa, const float* fg, const void* v, int v_ld, float* state,
                                            const int* cu_q, const int* seq_slot, float* o, float* ws, float* decay,
                                            int n_seqs, int H, int D, int Dv, int chunk, int n_chunks, int write_state,
                                            int dtype, const float* head_decay, cudaStream_t stream) {
  if (!ws || !decay) return LLMIE_ERR_BAD_ARG;
  const ScanArgs a{qa, fg, v, v_ld, state, cu_q, seq_slot, o, n_seqs, H, D, Dv, write_state, head_decay, nullptr, H,
                   ws, decay, chunk, n_chunks};
  return head_decay ? matrix_scan_entry<1>(a, dtype, stream) : matrix_scan_entry<0>(a, dtype, stream);
}

// The stepped form: qa (queries) and fg (keys) float32 [T, G * D], shared by H / G heads each; decay and factor per token
// and head, float32 [T, H]: S <- token_decay S + (key_factor k) v^T. ws null: unchunked, else as above.
extern "C" int llmie_matrix_scan_stepped(const float* qa, const float* fg, const void* v, int v_ld, float* state,
                                         const int* cu_q, const int* seq_slot, float* o, float* ws, float* decay,
                                         int n_seqs, int H, int G, int D, int Dv, int chunk, int n_chunks,
                                         int write_state, int dtype, const float* token_decay, const float* key_factor,
                                         cudaStream_t stream) {
  if (!token_decay || !key_factor) return LLMIE_ERR_BAD_ARG;
  const ScanArgs a{qa, fg, v, v_ld, state, cu_q, seq_slot, o, n_seqs, H, D, Dv, write_state, token_decay, key_factor, G,
                   ws, decay, chunk, n_chunks};
  return matrix_scan_entry<2>(a, dtype, stream);
}

// proj [T, ld] of `dtype`; out_k float32 [T, n_k] = act(proj[:, off_k : off_k + n_k]) for up to three runs (n_k = 0: unused).
extern "C" int llmie_act_columns(const void* proj, int ld, int off0, int n0, float* out0, int off1, int n1, float* out1,
                                 int off2, int n2, float* out2, int act, int n_tokens, int dtype, cudaStream_t stream) {
  if (n_tokens < 0 || n0 <= 0 || n1 < 0 || n2 < 0 || off0 < 0 || off1 < 0 || off2 < 0) return LLMIE_ERR_BAD_ARG;
  if (ld < off0 + n0 || (n1 && ld < off1 + n1) || (n2 && ld < off2 + n2)) return LLMIE_ERR_BAD_ARG;
  if (!out0 || (n1 && !out1) || (n2 && !out2)) return LLMIE_ERR_BAD_ARG;
  if (n_tokens == 0) return LLMIE_OK;
  const size_t total = (size_t)n_tokens * (n0 + n1 + n2);
  const dim3 grid(sweep_blocks(total, 256)), block(256);
  if (dtype == LLMIE_F32)
    launch_k(act_columns_kernel<float>, grid, block, 0, stream, (const float*)proj, ld, off0, n0, out0, off1, n1, out1,
             off2, n2, out2, act, total);
  else if (dtype == LLMIE_BF16)
    launch_k(act_columns_kernel<__nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)proj, ld, off0, n0, out0,
             off1, n1, out1, off2, n2, out2, act, total);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// o float32 [n_items, Dv] (an item = a token's head); w float32 [Dv]; y [n_items, Dv] of `dtype`.
// gate (of `dtype`, rows gate_ld apart, items_per_row items a row) or null: y is also multiplied by sigmoid(gate), or by
// silu(gate) with `silu`. w_items > 1: w float32 [w_items, Dv], item i uses row i % w_items.
extern "C" int llmie_head_rmsnorm_ex(const float* o, const float* w, float eps, void* y, long long n_items, int Dv,
                                     int dtype, const void* gate, int gate_ld, int items_per_row, int silu, int w_items,
                                     cudaStream_t stream) {
  if (n_items < 0 || Dv <= 0 || w_items <= 0 || (gate && (items_per_row <= 0 || gate_ld < items_per_row * Dv))) return LLMIE_ERR_BAD_ARG;
  if (n_items == 0) return LLMIE_OK;
  if (Dv >= 512 && Dv % 4 == 0 && aligned16(o) && aligned16(w) && n_items <= 0x7fffffffLL) {
    // wide items: a block each
    const dim3 grid((unsigned)n_items), block(Dv >= 1024 ? 256 : 128);
    if (dtype == LLMIE_F32)
      launch_k(row_rmsnorm_kernel<float>, grid, block, 0, stream, o, w, eps, (float*)y, Dv, (const float*)gate, gate_ld,
               items_per_row, silu, w_items);
    else if (dtype == LLMIE_BF16)
      launch_k(row_rmsnorm_kernel<__nv_bfloat16>, grid, block, 0, stream, o, w, eps, (__nv_bfloat16*)y, Dv,
               (const __nv_bfloat16*)gate, gate_ld, items_per_row, silu, w_items);
    else
      return LLMIE_ERR_DTYPE;
    LLMIE_LAUNCH_CHECK();
    return LLMIE_OK;
  }
  const int warps = 4;
  const long long blocks = (n_items + warps - 1) / warps;
  if (blocks > 0x7fffffffLL) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const dim3 grid((unsigned)blocks), block(warps * 32);
  if (dtype == LLMIE_F32)
    launch_k(head_rmsnorm_kernel<float>, grid, block, 0, stream, o, w, eps, (float*)y, Dv, (size_t)n_items,
             (const float*)gate, gate_ld, items_per_row, silu, w_items);
  else if (dtype == LLMIE_BF16)
    launch_k(head_rmsnorm_kernel<__nv_bfloat16>, grid, block, 0, stream, o, w, eps, (__nv_bfloat16*)y, Dv,
             (size_t)n_items, (const __nv_bfloat16*)gate, gate_ld, items_per_row, silu, w_items);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

extern "C" int llmie_head_rmsnorm_gated(const float* o, const float* w, float eps, void* y, long long n_items, int Dv,
                                        int dtype, const void* gate, int gate_ld, int items_per_row,
                                        cudaStream_t stream) {
  return llmie_head_rmsnorm_ex(o, w, eps, y, n_items, Dv, dtype, gate, gate_ld, items_per_row, 0, 1, stream);
}

extern "C" int llmie_head_rmsnorm(const float* o, const float* w, float eps, void* y, long long n_items, int Dv,
                                  int dtype, cudaStream_t stream) {
  return llmie_head_rmsnorm_ex(o, w, eps, y, n_items, Dv, dtype, nullptr, 0, 1, 0, 1, stream);
}

template <typename TP, typename TO>
static void causal_conv_launch(const TP* proj, int ld, int x_off, const float* x_bias, const float* taps,
                               const float* conv_bias, float* conv_state, const int* cu_q, const int* tok_seq,
                               const int* seq_slot, TO* u, int n_tokens, int C, int K, int act, int single,
                               cudaStream_t stream) {
  const bool by4 = K <= 4 && C % 4 == 0 && ld % 4 == 0 && x_off % 4 == 0 && aligned16(proj) && aligned16(u) && aligned16(taps) &&
                   (!x_bias || aligned16(x_bias)) && (!conv_bias || aligned16(conv_bias));
  const int units = by4 ? C / 4 : C;
  const int threads = units >= 128 ? 128 : ((units + 31) / 32) * 32;
#define LLMIE_CONV_LAUNCH(KM, V, TILE)                                                                                   \
  launch_k(causal_conv_kernel<TP, TO, KM, V, TILE>, dim3((n_tokens + TILE - 1) / TILE, (units + threads - 1) / threads), \
           dim3(threads), 0, stream, proj, ld, x_off, x_bias, taps, conv_bias, conv_state, cu_q, tok_seq, seq_slot, u, C, \
           K, n_tokens, act, single)
  if (!by4) {
    if (n_tokens >= 64 && !single) LLMIE_CONV_LAUNCH(kMaxTaps, 1, 4);
    else LLMIE_CONV_LAUNCH(kMaxTaps, 1, 1);
  } else if (single || n_tokens < 64) {
    LLMIE_CONV_LAUNCH(4, 4, 1);
  } else if (n_tokens < 512) {
    LLMIE_CONV_LAUNCH(4, 4, 4);
  } else {
    LLMIE_CONV_LAUNCH(4, 4, 8);
  }
#undef LLMIE_CONV_LAUNCH
}

// proj [T, ld] of `dtype` with the convolution's input at column x_off (C columns); x_bias, conv_bias float32 [C] or
// null; taps float32 [K, C] (the last row multiplies the current token); conv_state float32 [slots, K-1, C];
// u [T, C] of u_dtype = act(convolution), act a code of apply_act. single != 0: every sequence brings one token and the
// new conv_state is written too.
extern "C" int llmie_causal_conv_ex(const void* proj, int ld, int x_off, const float* x_bias, const float* taps,
                                    const float* conv_bias, float* conv_state, const int* cu_q, const int* tok_seq,
                                    const int* seq_slot, void* u, int u_dtype, int n_tokens, int C, int K, int act,
                                    int single, int dtype, cudaStream_t stream) {
  if (n_tokens < 0 || C <= 0 || K <= 0 || x_off < 0 || ld < x_off + C || act < 0 || act > 4) return LLMIE_ERR_BAD_ARG;
  if (K > kMaxTaps || C > 65535 * 32) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
#define LLMIE_CONV(TP, TO)                                                                                              \
  causal_conv_launch<TP, TO>((const TP*)proj, ld, x_off, x_bias, taps, conv_bias, conv_state, cu_q, tok_seq, seq_slot,  \
                             (TO*)u, n_tokens, C, K, act, single, stream)
  if (dtype == LLMIE_F32 && u_dtype == LLMIE_F32) LLMIE_CONV(float, float);
  else if (dtype == LLMIE_BF16 && u_dtype == LLMIE_F32) LLMIE_CONV(__nv_bfloat16, float);
  else if (dtype == LLMIE_BF16 && u_dtype == LLMIE_BF16) LLMIE_CONV(__nv_bfloat16, __nv_bfloat16);
  else if (dtype == LLMIE_F32 && u_dtype == LLMIE_BF16) LLMIE_CONV(float, __nv_bfloat16);
  else return LLMIE_ERR_DTYPE;
#undef LLMIE_CONV
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// The state a convolution leaves behind after a step of any pieces (see conv_state_store_kernel); K >= 2.
extern "C" int llmie_conv_state_store(const void* proj, int ld, int x_off, const float* x_bias, float* conv_state,
                                      const int* cu_q, const int* seq_slot, int n_seqs, int C, int K, int dtype,
                                      cudaStream_t stream) {
  if (n_seqs < 0 || C <= 0 || K < 2 || x_off < 0 || ld < x_off + C) return LLMIE_ERR_BAD_ARG;
  if (K > kMaxTaps || n_seqs > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_seqs == 0) return LLMIE_OK;
  const dim3 grid((C + 127) / 128, n_seqs), block(128);
  if (dtype == LLMIE_F32)
    launch_k(conv_state_store_kernel<float>, grid, block, 0, stream, (const float*)proj, ld, x_off, x_bias, conv_state,
             cu_q, seq_slot, C, K);
  else if (dtype == LLMIE_BF16)
    launch_k(conv_state_store_kernel<__nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)proj, ld, x_off, x_bias,
             conv_state, cu_q, seq_slot, C, K);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// gates float32 [T, 2 C] (per group of bw channels: r's pre-activations, then i's), changed in place into (a, drive);
// u float32 [T, C]; r_bias, i_bias, lam float32 [C].
extern "C" int llmie_unit_gate_values(float* gates, const float* u, const float* r_bias, const float* i_bias,
                                      const float* lam, float c_decay, int n_tokens, int C, int bw,
                                      cudaStream_t stream) {
  if (n_tokens < 0 || C <= 0 || bw <= 0 || C % bw) return LLMIE_ERR_BAD_ARG;
  if (n_tokens == 0) return LLMIE_OK;
  const size_t total = (size_t)n_tokens * C;
  launch_k(unit_gate_values_kernel, dim3(sweep_blocks(total, 256)), dim3(256), 0, stream, gates, u, r_bias, i_bias, lam,
           c_decay, C, bw, total);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// gates as left by llmie_unit_gate_values; proj [T, ld] of `dtype` with the output gate's raw projection at y_off and
// the convolution's input at x_off; state float32 [slots, C]; conv_state float32 [slots, K-1, C]; out [T, C] of `dtype`.
// chunked != 0: the form for long pieces (every sequence's piece in 32 chunks side by side).
extern "C" int llmie_unit_scan(const float* gates, const void* proj, int ld, int y_off, int x_off, const float* y_bias,
                               const float* x_bias, int act, float* state, float* conv_state, const int* cu_q,
                               const int* seq_slot, void* out, int n_seqs, int C, int bw, int K, int write_state,
                               int chunked, int dtype, cudaStream_t stream) {
  if (n_seqs < 0 || C <= 0 || bw <= 0 || C % bw || K <= 0 || y_off < 0 || x_off < 0 || ld < y_off + C || ld < x_off + C)
    return LLMIE_ERR_BAD_ARG;
  if (act < 0 || act > 4) return LLMIE_ERR_BAD_ARG;
  if (K > kMaxTaps) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_seqs == 0) return LLMIE_OK;
  if (n_seqs > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (chunked) {
    const dim3 grid((C + 31) / 32, n_seqs), block(32, kUnitChunks);
    if (dtype == LLMIE_F32)
      launch_k(unit_scan_chunked_kernel<float>, grid, block, 0, stream, gates, (const float*)proj, ld, y_off, x_off,
               y_bias, x_bias, act, state, conv_state, cu_q, seq_slot, (float*)out, C, bw, K, write_state);
    else if (dtype == LLMIE_BF16)
      launch_k(unit_scan_chunked_kernel<__nv_bfloat16>, grid, block, 0, stream, gates, (const __nv_bfloat16*)proj, ld,
               y_off, x_off, y_bias, x_bias, act, state, conv_state, cu_q, seq_slot, (__nv_bfloat16*)out, C, bw, K,
               write_state);
    else
      return LLMIE_ERR_DTYPE;
    LLMIE_LAUNCH_CHECK();
    return LLMIE_OK;
  }
  const int threads = C >= 128 ? 128 : ((C + 31) / 32) * 32;
  const dim3 grid((C + threads - 1) / threads, n_seqs), block(threads);
  if (dtype == LLMIE_F32)
    launch_k(unit_scan_kernel<float>, grid, block, 0, stream, gates, (const float*)proj, ld, y_off, x_off, y_bias,
             x_bias, act, state, conv_state, cu_q, seq_slot, (float*)out, C, bw, K, write_state);
  else if (dtype == LLMIE_BF16)
    launch_k(unit_scan_kernel<__nv_bfloat16>, grid, block, 0, stream, gates, (const __nv_bfloat16*)proj, ld, y_off,
             x_off, y_bias, x_bias, act, state, conv_state, cu_q, seq_slot, (__nv_bfloat16*)out, C, bw, K, write_state);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}
