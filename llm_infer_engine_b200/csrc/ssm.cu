// A state space layer with a scalar decay per token and head (the recurrence of Mamba-2). Per head h with P value columns
// and a state S [N, P] (float32, zero at a sequence's start, carried per slot), group g = h / (H / G):
//
//   dt_t = softplus(raw_t + dt_bias)          a_t = exp(-A dt_t),  A > 0 a number per head
//   S <- a_t S + B_t (dt_t x_t)^T              y_t = S^T C_t + D x_t              B, C [N] shared by a group's heads
//
// x, B and C are columns of one buffer xbc [T, H P + 2 G N] (what the convolution in front leaves), raw is a column of the
// input projection, and so is z of the gated norm.
//
//   ssm_steps          dt and a as float32 [T, H] (for the scan of recurrent.cu, whose stepped form is this recurrence)
//   ssm_step           steps in which every sequence brings one token: one pass over the state
//   ssm_scan           prompts of the bfloat16 engine on the tensor cores, 64 tokens at a time (below)
//   gated_group_norm   (y + D x) silu(z), then a root mean square over each of several equal runs of columns, weight
//
// ssm_scan. Within a chunk of Q = 64 tokens, with cum_i = sum_(k <= i) -A dt_k (float32, from the chunk's start; kept in base 2):
//   y_i   = sum_(j <= i) (C_i . B_j) exp(cum_i - cum_j) dt_j x_j  +  exp(cum_i) C_i^T S_prev  +  D x_i
//   S_new = exp(cum_last) S_prev + sum_j B_j (exp(cum_last - cum_j) dt_j x_j)^T
// three matrix products and one more for the scores. A block walks over one sequence's chunks in order for one head and
// PS of its value columns, the state in its accumulator registers all the way: a state is read and written once. The
// operands B, C and x are bfloat16 as the convolution leaves them; what the recurrence itself makes (the weighted scores,
// the weighted x, the state) enters a product as the sum of TWO bfloat16 numbers, high and low half, so that no factor of
// the recurrence is rounded to 8 bits: its relative error is 2^-17. Accumulators are float32.
#include "common.cuh"
#include <math.h>

namespace llmie {

__device__ __forceinline__ float ssm_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T>
__global__ void ssm_steps_kernel(const T* __restrict__ proj, int ld, int dt_off, const float* __restrict__ dt_bias,
                                 const float* __restrict__ A, float* __restrict__ dt, float* __restrict__ decay, int H,
                                 int total) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int t = i / H, h = i - t * H;
  const float d = ssm_softplus(to_f32(proj[(size_t)t * ld + dt_off + h]) + dt_bias[h]);
  dt[i] = d;
  decay[i] = expf(-A[h] * d);
}

// ------------------------------------------------------------------------------------------ one token a sequence
constexpr int kStepThreads = 256;
constexpr int kStepUnroll = 8;

struct SsmArgs {
  const void* proj;            // the input projection; the raw step of head h at column dt_off + h
  int ld, dt_off;
  const float* dt_bias;        // [H]
  const float* A;              // [H]
  const float* Dskip;          // [H]
  float* state;                // [slots, H, N, P]
  const int* cu_q;
  const int* seq_slot;
  int H, G, N, P, xbc_ld, write_state;
};

// grid (H * column tiles, sequences). V adjacent columns a thread; CT threads beside each other cover a row's part of the
// tile, RT = kStepThreads / CT rows are worked on side by side. The first rows of the state are requested before the
// wait for the previous kernel: the state was last written a whole step ago.
template <typename TP, int V>
__global__ void __launch_bounds__(kStepThreads)
ssm_step_kernel(const SsmArgs p, const float* __restrict__ xbc, float* __restrict__ y, int CT, int RT, int ctiles) {
  extern __shared__ float st_smem[];                // B [N], C [N], then RT x CT partial sums of V
  __shared__ float step_dt, step_decay;
  pdl_launch_dependents();
  const int h = blockIdx.x / ctiles, ctile = blockIdx.x - h * ctiles;
  const int seq = blockIdx.y;
  const int ct = threadIdx.x % CT, rt = threadIdx.x / CT;
  const int col = (ctile * CT + ct) * V;
  const bool live = rt < RT && col < p.P;
  const int slot = p.seq_slot[seq];
  float* st = p.state + ((size_t)slot * p.H + h) * p.N * p.P + col;
  float S[kStepUnroll][V];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int u = 0; u < kStepUnroll; ++u) {
      const int r = r0 + u * RT;
      if (live && r < p.N) {
        if (V == 4) {
          const float4 v = *reinterpret_cast<const float4*>(st + (size_t)r * p.P);
          S[u][0] = v.x; S[u][1 % V] = v.y; S[u][2 % V] = v.z; S[u][3 % V] = v.w;
        } else {
          S[u][0] = st[(size_t)r * p.P];
        }
      }
    }
  };
  fetch(rt);
  const float bias = p.dt_bias[h], A = p.A[h], Dh = p.Dskip[h];
  pdl_wait();
  const int t = p.cu_q[seq];
  const float* row = xbc + (size_t)t * p.xbc_ld;
  const int inner = p.H * p.P, g = h / (p.H / p.G);
  float* Bs = st_smem;
  float* Cs = Bs + p.N;
  float* red = Cs + p.N;
  for (int i = threadIdx.x; i < p.N; i += kStepThreads) {
    Bs[i] = row[inner + g * p.N + i];
    Cs[i] = row[inner + p.G * p.N + g * p.N + i];
  }
  if (threadIdx.x == 0) {
    const float d = ssm_softplus(to_f32(reinterpret_cast<const TP*>(p.proj)[(size_t)t * p.ld + p.dt_off + h]) + bias);
    step_dt = d;
    step_decay = expf(-A * d);
  }
  float x[V], acc[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    x[e] = live ? row[h * p.P + col + e] : 0.f;
    acc[e] = 0.f;
  }
  __syncthreads();
  const float dt = step_dt, decay = step_decay;
  for (int r0 = rt; r0 < p.N; r0 += kStepUnroll * RT) {
    if (r0 != rt) fetch(r0);
#pragma unroll
    for (int u = 0; u < kStepUnroll; ++u) {
      const int r = r0 + u * RT;
      if (live && r < p.N) {
        const float kb = dt * Bs[r], kc = Cs[r];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          S[u][e] = fmaf(decay, S[u][e], kb * x[e]);
          acc[e] = fmaf(S[u][e], kc, acc[e]);
        }
        if (p.write_state) {
          if (V == 4)
            *reinterpret_cast<float4*>(st + (size_t)r * p.P) = make_float4(S[u][0], S[u][1 % V], S[u][2 % V], S[u][3 % V]);
          else
            st[(size_t)r * p.P] = S[u][0];
        }
      }
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e)
    if (rt < RT) red[(rt * CT + ct) * V + e] = acc[e];
  __syncthreads();
  for (int i = threadIdx.x; i < CT * V; i += kStepThreads) {
    const int c = ctile * CT * V + i;
    if (c >= p.P) continue;
    float s = 0.f;
    for (int k = 0; k < RT; ++k) s += red[k * CT * V + i];
    y[(size_t)t * inner + h * p.P + c] = fmaf(Dh, row[h * p.P + c], s);
  }
}

// ------------------------------------------------------------------------------------------ prompts, tensor cores
constexpr int kSsmQ = 64;          // tokens a chunk
constexpr int kSsmThreads = 128;   // four warps, 16 tokens of a chunk each

__device__ __forceinline__ void ssm_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ssm_ldm(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ssm_ldm_t(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 2^x by the special-function unit (relative error about 2^-22)
__device__ __forceinline__ float ssm_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two floats as (high, low) pairs of bfloat16: v = high + low up to 2^-17 of v
__device__ __forceinline__ void ssm_split(float v0, float v1, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - back.x, v1 - back.y);
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = *reinterpret_cast<const unsigned*>(&l);
}
// 16 bytes from global memory into shared memory, or zeros (src is not read then)
__device__ __forceinline__ void ssm_copy16(unsigned dst, const void* src, bool real) {
  const int n = real ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

template <int NT, int PS>
struct SsmTile {
  static constexpr int NP = NT + 8, XP = PS + 8;            // row pitches: 16 bytes more than a row, against bank conflicts
  static constexpr int kB = kSsmQ * NP, kX = kSsmQ * XP;    // elements of a staged tile of B (or C), of x
  static constexpr int kStage = 2 * kB + kX;                // B, C, x
  static constexpr int kS = NT * XP;                        // the state as a product's operand, one half
  static constexpr int kElems = 2 * kStage + 2 * kX + 2 * kS;
  static constexpr int kSmem = kElems * 2;
};

// grid (value tiles, H, sequences). NT: rows of the state, N rounded up; PS: value columns a block.
template <typename TP, typename TO, int NT, int PS>
__global__ void __launch_bounds__(kSsmThreads)
ssm_scan_kernel(const SsmArgs p, const __nv_bfloat16* __restrict__ xbc, TO* __restrict__ y) {
  using Tile = SsmTile<NT, PS>;
  constexpr int NP = Tile::NP, XP = Tile::XP;
  constexpr int MT = (NT + 63) / 64;                        // 16-row tiles of the state a warp owns
  constexpr int PT = PS / 8;                                // 8-column tiles of the values
  extern __shared__ __align__(16) unsigned char ssm_smem[];
  // per token of a chunk, for this chunk and the next in turn: the sum of the decays' logarithms (base 2), the step, and
  // the weight of the token's x in the state after the chunk
  __shared__ __align__(16) float2 s_tok[2][kSsmQ];
  __shared__ float s_xw[2][kSsmQ];
  __nv_bfloat16* stage0 = reinterpret_cast<__nv_bfloat16*>(ssm_smem);
  __nv_bfloat16* xw_hi = stage0 + 2 * Tile::kStage;         // [64][XP] exp(cum_last - cum_j) dt_j x_j
  __nv_bfloat16* xw_lo = xw_hi + Tile::kX;
  __nv_bfloat16* s_hi = xw_lo + Tile::kX;                   // [NT][XP] the state before the chunk
  __nv_bfloat16* s_lo = s_hi + Tile::kS;

  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int p0 = blockIdx.x * PS, h = blockIdx.y, seq = blockIdx.z;
  const int N = p.N, P = p.P;
  const float dt_bias = p.dt_bias[h], A = p.A[h], Dh = p.Dskip[h];
  pdl_wait();
  const int t_begin = p.cu_q[seq], t_end = p.cu_q[seq + 1];
  if (t_begin >= t_end) return;
  const int inner = p.H * P, grp = h / (p.H / p.G);
  const __nv_bfloat16* gx = xbc + h * P + p0;
  const __nv_bfloat16* gB = xbc + inner + grp * N;
  const __nv_bfloat16* gC = gB + p.G * N;
  const TP* graw = reinterpret_cast<const TP*>(p.proj) + p.dt_off + h;
  const int n_chunks = (t_end - t_begin + kSsmQ - 1) / kSsmQ;

  auto issue = [&](int chunk, int stage) {
    const int t0 = t_begin + chunk * kSsmQ;
    const unsigned bd = (unsigned)__cvta_generic_to_shared(stage0 + stage * Tile::kStage);
    const unsigned cd = bd + Tile::kB * 2, xd = cd + Tile::kB * 2;
    constexpr int kPer = NT / 8;
    for (int i = tid; i < kSsmQ * kPer; i += kSsmThreads) {
      const int r = i / kPer, ch = i % kPer;
      const bool real = t0 + r < t_end && ch * 8 < N;
      const size_t off = real ? (size_t)(t0 + r) * p.xbc_ld + ch * 8 : 0;
      ssm_copy16(bd + (r * NP + ch * 8) * 2, gB + off, real);
      ssm_copy16(cd + (r * NP + ch * 8) * 2, gC + off, real);
    }
    for (int i = tid; i < kSsmQ * PT; i += kSsmThreads) {
      const int r = i / PT, ch = i % PT;
      const bool real = t0 + r < t_end && p0 + ch * 8 < P;
      ssm_copy16(xd + (r * XP + ch * 8) * 2, gx + (real ? (size_t)(t0 + r) * p.xbc_ld + ch * 8 : 0), real);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0, 0);

  // Warp 0 works out the steps of a chunk, two tokens a lane, one chunk ahead; their raw values are asked for another
  // chunk ahead of that. Tokens beyond the piece: dt = 0, no decay.
  const float A2 = -A * 1.4426950408889634f;
  float raw0 = 0.f, raw1 = 0.f;
  auto fetch_raw = [&](int chunk) {
    const int t = t_begin + chunk * kSsmQ + 2 * lane;
    if (t < t_end) raw0 = to_f32(graw[(size_t)t * p.ld]);
    if (t + 1 < t_end) raw1 = to_f32(graw[(size_t)(t + 1) * p.ld]);
  };
  auto make_steps = [&](int chunk) {
    const int t = t_begin + chunk * kSsmQ + 2 * lane, buf = chunk & 1;
    const float d0 = t < t_end ? ssm_softplus(raw0 + dt_bias) : 0.f;
    const float d1 = t + 1 < t_end ? ssm_softplus(raw1 + dt_bias) : 0.f;
    const float l0 = A2 * d0, l1 = A2 * d1;
    float sum = l0 + l1;                              // of this lane's two, then up to and including them
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    float before = __shfl_up_sync(0xffffffffu, sum, 1);
    if (lane == 0) before = 0.f;
    const float c0 = before + l0, c1 = c0 + l1;
    const float last = __shfl_sync(0xffffffffu, c1, 31);
    s_tok[buf][2 * lane] = make_float2(c0, d0);
    s_tok[buf][2 * lane + 1] = make_float2(c1, d1);
    s_xw[buf][2 * lane] = exp2f(last - c0) * d0;
    s_xw[buf][2 * lane + 1] = exp2f(last - c1) * d1;
  };
  if (warp == 0) {
    fetch_raw(0);
    make_steps(0);
    fetch_raw(1);
  }

  // the state: warp w owns rows w * 16 + mt * 64 .. + 15; as a product's operand it lies in shared memory in two halves
  float* st = p.state + ((size_t)p.seq_slot[seq] * p.H + h) * N * P + p0;
  float S[MT][PT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int pt = 0; pt < PT; ++pt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int n = warp * 16 + mt * 64 + g + 8 * e, c = pt * 8 + 2 * t4;
        float2 v = make_float2(0.f, 0.f);
        if (n < N && p0 + c < P) v = *reinterpret_cast<const float2*>(st + (size_t)n * P + c);
        S[mt][pt][2 * e] = v.x;
        S[mt][pt][2 * e + 1] = v.y;
      }
  auto publish_state = [&]() {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const int n = warp * 16 + mt * 64 + g;
      if (warp * 16 + mt * 64 < NT) {
#pragma unroll
        for (int pt = 0; pt < PT; ++pt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            unsigned hi, lo;
            ssm_split(S[mt][pt][2 * e], S[mt][pt][2 * e + 1], hi, lo);
            const int off = (n + 8 * e) * XP + pt * 8 + 2 * t4;
            *reinterpret_cast<unsigned*>(s_hi + off) = hi;
            *reinterpret_cast<unsigned*>(s_lo + off) = lo;
          }
      }
    }
  };
  publish_state();

  const int lm_row = lane & 15, lm_hi = (lane >> 4) * 8;                       // ldmatrix: A from row-major rows
  const int lt_r = (lane & 7) + ((lane >> 4) & 1) * 8, lt_c = ((lane >> 3) & 1) * 8;   // A from its transpose
  const int lb_r = (lane & 7) + ((lane >> 4) & 1) * 8, lb_c = ((lane >> 3) & 1) * 8;   // B, two 8-column tiles, k contiguous
  const int lv_r = (lane & 7) + ((lane >> 3) & 1) * 8, lv_c = ((lane >> 4) & 1) * 8;   // B, two 8-column tiles, n contiguous
  for (int chunk = 0; chunk < n_chunks; ++chunk) {
    const int t0 = t_begin + chunk * kSsmQ;
    const __nv_bfloat16* Bs = stage0 + (chunk & 1) * Tile::kStage;
    const __nv_bfloat16* Cs = Bs + Tile::kB;
    const __nv_bfloat16* Xs = Cs + Tile::kB;
    const float2* tok = s_tok[chunk & 1];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                         // this chunk is here; nobody works on the one before any more
    if (chunk + 1 < n_chunks) {
      issue(chunk + 1, (chunk + 1) & 1);
      if (warp == 0) {
        make_steps(chunk + 1);
        fetch_raw(chunk + 2);
      }
    }
    const float cum_last = tok[kSsmQ - 1].x;
    // ---- x weighted for the state's update
    for (int i = tid; i < kSsmQ * (PS / 2); i += kSsmThreads) {
      const int r = i / (PS / 2), c = (i % (PS / 2)) * 2;
      const float w = s_xw[chunk & 1][r];
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Xs + r * XP + c));
      unsigned hi, lo;
      ssm_split(w * x.x, w * x.y, hi, lo);
      *reinterpret_cast<unsigned*>(xw_hi + r * XP + c) = hi;
      *reinterpret_cast<unsigned*>(xw_lo + r * XP + c) = lo;
    }
    // ---- scores C B^T for this warp's 16 tokens against tokens up to its last, and C S_prev
    float sc[8][4], yc[PT][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
    for (int pt = 0; pt < PT; ++pt) yc[pt][0] = yc[pt][1] = yc[pt][2] = yc[pt][3] = 0.f;
    const unsigned c_addr = (unsigned)__cvta_generic_to_shared(Cs + (warp * 16 + lm_row) * NP + lm_hi);
    const unsigned b_addr = (unsigned)__cvta_generic_to_shared(Bs + lb_r * NP + lb_c);
    const unsigned sh_addr = (unsigned)__cvta_generic_to_shared(s_hi + lv_r * XP + lv_c);
    const unsigned sl_addr = (unsigned)__cvta_generic_to_shared(s_lo + lv_r * XP + lv_c);
#pragma unroll 2
    for (int k0 = 0; k0 < NT; k0 += 16) {
      unsigned a[4], b[4];
      ssm_ldm(a, c_addr + k0 * 2);
#pragma unroll
      for (int pr = 0; pr < 4; ++pr) {
        if (pr <= warp) {                                    // later tokens are masked out whole
          ssm_ldm(b, b_addr + (pr * 16 * NP + k0) * 2);
          ssm_mma(sc[2 * pr], a, b[0], b[1]);
          ssm_mma(sc[2 * pr + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int pp = 0; pp < PT / 2; ++pp) {
        ssm_ldm_t(b, sh_addr + (k0 * XP + pp * 16) * 2);
        ssm_mma(yc[2 * pp], a, b[0], b[1]);
        ssm_mma(yc[2 * pp + 1], a, b[2], b[3]);
        ssm_ldm_t(b, sl_addr + (k0 * XP + pp * 16) * 2);
        ssm_mma(yc[2 * pp], a, b[0], b[1]);
        ssm_mma(yc[2 * pp + 1], a, b[2], b[3]);
      }
    }
    const int i_lo = warp * 16 + g, i_hi = i_lo + 8;
    const float cum_lo = tok[i_lo].x, cum_hi = tok[i_hi].x;
    {
      const float e_lo = ssm_exp2(cum_lo), e_hi = ssm_exp2(cum_hi);
#pragma unroll
      for (int pt = 0; pt < PT; ++pt) {
        yc[pt][0] *= e_lo;
        yc[pt][1] *= e_lo;
        yc[pt][2] *= e_hi;
        yc[pt][3] *= e_hi;
      }
    }
    // ---- weighted scores (accumulator layout = the operand layout of the next product) times x
    const unsigned x_addr = (unsigned)__cvta_generic_to_shared(Xs + lv_r * XP + lv_c);
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk <= warp) {
        unsigned ah[4], al[4], b[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int j = kk * 16 + half * 8 + 2 * t4;
          const float4 cd = *reinterpret_cast<const float4*>(tok + j);     // (sum, step) of tokens j and j + 1
          const float* s = sc[2 * kk + half];
          float w0 = s[0] * (ssm_exp2(cum_lo - cd.x) * cd.y), w1 = s[1] * (ssm_exp2(cum_lo - cd.z) * cd.w);
          float w2 = s[2] * (ssm_exp2(cum_hi - cd.x) * cd.y), w3 = s[3] * (ssm_exp2(cum_hi - cd.z) * cd.w);
          if (kk == warp) {                                  // the diagonal tile: later tokens are not seen
            w0 = j <= i_lo ? w0 : 0.f;
            w1 = j + 1 <= i_lo ? w1 : 0.f;
            w2 = j <= i_hi ? w2 : 0.f;
            w3 = j + 1 <= i_hi ? w3 : 0.f;
          }
          ssm_split(w0, w1, ah[2 * half], al[2 * half]);
          ssm_split(w2, w3, ah[2 * half + 1], al[2 * half + 1]);
        }
#pragma unroll
        for (int pp = 0; pp < PT / 2; ++pp) {
          ssm_ldm_t(b, x_addr + (kk * 16 * XP + pp * 16) * 2);
          ssm_mma(yc[2 * pp], ah, b[0], b[1]);
          ssm_mma(yc[2 * pp + 1], ah, b[2], b[3]);
          ssm_mma(yc[2 * pp], al, b[0], b[1]);
          ssm_mma(yc[2 * pp + 1], al, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = e ? i_hi : i_lo;
      if (t0 + i < t_end) {
        TO* dst = y + (size_t)(t0 + i) * inner + h * P + p0;
#pragma unroll
        for (int pt = 0; pt < PT; ++pt) {
          const int c = pt * 8 + 2 * t4;
          if (p0 + c < P) {
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Xs + i * XP + c));
            const float v0 = fmaf(Dh, x.x, yc[pt][2 * e]), v1 = fmaf(Dh, x.y, yc[pt][2 * e + 1]);
            if (sizeof(TO) == 4)
              *reinterpret_cast<float2*>(dst + c) = make_float2(v0, v1);
            else
              *reinterpret_cast<__nv_bfloat162*>(dst + c) = __floats2bfloat162_rn(v0, v1);
          }
        }
      }
    }
    __syncthreads();                                         // the weighted x is complete
    // ---- the state after the chunk
    const float e_last = ssm_exp2(cum_last);
    const unsigned bt_addr = (unsigned)__cvta_generic_to_shared(Bs + lt_r * NP + lt_c + warp * 16);
    const unsigned xh_addr = (unsigned)__cvta_generic_to_shared(xw_hi + lv_r * XP + lv_c);
    const unsigned xl_addr = (unsigned)__cvta_generic_to_shared(xw_lo + lv_r * XP + lv_c);
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int pt = 0; pt < PT; ++pt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][pt][e] *= e_last;
#pragma unroll
    for (int j0 = 0; j0 < kSsmQ; j0 += 16) {
#pragma unroll
      for (int pp = 0; pp < PT / 2; ++pp) {
        unsigned bh[4], bl[4];
        ssm_ldm_t(bh, xh_addr + (j0 * XP + pp * 16) * 2);
        ssm_ldm_t(bl, xl_addr + (j0 * XP + pp * 16) * 2);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          if (warp * 16 + mt * 64 < NT) {
            unsigned a[4];
            ssm_ldm_t(a, bt_addr + (j0 * NP + mt * 64) * 2);
            ssm_mma(S[mt][2 * pp], a, bh[0], bh[1]);
            ssm_mma(S[mt][2 * pp + 1], a, bh[2], bh[3]);
            ssm_mma(S[mt][2 * pp], a, bl[0], bl[1]);
            ssm_mma(S[mt][2 * pp + 1], a, bl[2], bl[3]);
          }
        }
      }
    }
    publish_state();                                         // every warp has read the state before the chunk
  }
  if (!p.write_state) return;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int pt = 0; pt < PT; ++pt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int n = warp * 16 + mt * 64 + g + 8 * e, c = pt * 8 + 2 * t4;
        if (n < N && p0 + c < P)
          *reinterpret_cast<float2*>(st + (size_t)n * P + c) = make_float2(S[mt][pt][2 * e], S[mt][pt][2 * e + 1]);
      }
}

// ------------------------------------------------------------------------------------------ gated norm
// A block per (token, run of columns). y float32 [T, n]; z rows of n elements, z_ld apart. With `skip_d` the row is
// y + skip_d[c / P] * x[c] first (x float32, rows x_ld apart: for a scan that leaves the skip term out).
template <typename TZ, typename TO, int V>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, const TZ* __restrict__ z, int z_ld,
                                        const float* __restrict__ w, float eps, TO* __restrict__ out, int n, int size,
                                        const float* __restrict__ skip_x, int x_ld, const float* __restrict__ skip_d,
                                        int P) {
  extern __shared__ float row_smem[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int c0 = blockIdx.y * size;
  const float* yr = y + t * n + c0;
  const TZ* zr = z + t * z_ld + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < size; i += blockDim.x * V) {
    float yv[V], zv[V];
    if (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(yr + i);
      yv[0] = a.x; yv[1 % V] = a.y; yv[2 % V] = a.z; yv[3 % V] = a.w;
      if (sizeof(TZ) == 4) {
        const float4 b = *reinterpret_cast<const float4*>(zr + i);
        zv[0] = b.x; zv[1 % V] = b.y; zv[2 % V] = b.z; zv[3 % V] = b.w;
      } else {
        const uint2 r = *reinterpret_cast<const uint2*>(zr + i);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
        zv[0] = lo.x; zv[1 % V] = lo.y; zv[2 % V] = hi.x; zv[3 % V] = hi.y;
      }
    } else {
      yv[0] = yr[i];
      zv[0] = to_f32(zr[i]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      if (skip_d) yv[e] = fmaf(skip_d[(c0 + i + e) / P], skip_x[t * x_ld + c0 + i + e], yv[e]);
      const float v = yv[e] * (zv[e] / (1.f + expf(-zv[e])));
      row_smem[i + e] = v;
      ss = fmaf(v, v, ss);
    }
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)size + eps);
  for (int i = threadIdx.x * V; i < size; i += blockDim.x * V) {       // the thread's own values: no barrier
    TO* dst = out + t * n + c0 + i;
    if (V == 4) {
      const float4 wv = *reinterpret_cast<const float4*>(w + c0 + i);
      const float v0 = row_smem[i] * r * wv.x, v1 = row_smem[i + 1 % V] * r * wv.y, v2 = row_smem[i + 2 % V] * r * wv.z,
                  v3 = row_smem[i + 3 % V] * r * wv.w;
      if (sizeof(TO) == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(v0, v1, v2, v3);
      } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v0, v1), hi = __floats2bfloat162_rn(v2, v3);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned*>(&lo);
        raw.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(dst) = raw;
      }
    } else {
      dst[0] = from_f32<TO>(row_smem[i] * r * w[c0 + i]);
    }
  }
}

template <typename TZ, typename TO>
static int gated_group_norm_launch(const float* y, const void* z, int z_ld, const float* w, float eps, void* out,
                                   int n_tokens, int n, int groups, const float* skip_x, int x_ld, const float* skip_d,
                                   int P, cudaStream_t stream) {
  const int size = n / groups;
  const size_t smem = (size_t)size * sizeof(float);
  const bool by4 = size % 4 == 0 && z_ld % 4 == 0 && aligned16(y) && aligned16(w) && aligned16(out) &&
                   (reinterpret_cast<uintptr_t>(z) & (4 * sizeof(TZ) - 1)) == 0;
  int threads = (((by4 ? size / 4 : size) + 31) / 32) * 32;
  threads = threads > 256 ? 256 : threads;
  const dim3 grid(n_tokens, groups), block(threads);
  auto kernel = by4 ? gated_group_norm_kernel<TZ, TO, 4> : gated_group_norm_kernel<TZ, TO, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch_k(kernel, grid, block, smem, stream, y, (const TZ*)z, z_ld, w, eps, (TO*)out, n, size, skip_x, x_ld, skip_d, P);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

template <typename TP, typename TO, int NT, int PS>
static int ssm_scan_launch(const SsmArgs& a, const void* xbc, void* y, int n_seqs, cudaStream_t stream) {
  auto kernel = ssm_scan_kernel<TP, TO, NT, PS>;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SsmTile<NT, PS>::kSmem);
  if (e != cudaSuccess) return (int)e;
  launch_k(kernel, dim3((a.P + PS - 1) / PS, a.H, n_seqs), dim3(kSsmThreads), SsmTile<NT, PS>::kSmem, stream, a,
           (const __nv_bfloat16*)xbc, (TO*)y);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

template <typename TP, typename TO>
static int ssm_scan_dispatch(const SsmArgs& a, const void* xbc, void* y, int n_seqs, cudaStream_t stream) {
  const bool narrow = a.P <= 16;
  if (a.N <= 32) return narrow ? ssm_scan_launch<TP, TO, 32, 16>(a, xbc, y, n_seqs, stream) : ssm_scan_launch<TP, TO, 32, 32>(a, xbc, y, n_seqs, stream);
  if (a.N <= 64) return narrow ? ssm_scan_launch<TP, TO, 64, 16>(a, xbc, y, n_seqs, stream) : ssm_scan_launch<TP, TO, 64, 32>(a, xbc, y, n_seqs, stream);
  if (a.N <= 128) return narrow ? ssm_scan_launch<TP, TO, 128, 16>(a, xbc, y, n_seqs, stream) : ssm_scan_launch<TP, TO, 128, 32>(a, xbc, y, n_seqs, stream);
  return narrow ? ssm_scan_launch<TP, TO, 256, 16>(a, xbc, y, n_seqs, stream) : ssm_scan_launch<TP, TO, 256, 32>(a, xbc, y, n_seqs, stream);
}

}  // namespace llmie

using namespace llmie;

// proj [T, ld] of `dtype` with the raw steps at columns dt_off .. dt_off + H - 1; dt_bias, A float32 [H]; dt, decay float32
// [T, H].
extern "C" int llmie_ssm_steps(const void* proj, int ld, int dt_off, const float* dt_bias, const float* A, float* dt,
                               float* decay, int n_tokens, int H, int dtype, cudaStream_t stream) {
  if (n_tokens < 0 || H <= 0 || dt_off < 0 || ld < dt_off + H) return LLMIE_ERR_BAD_ARG;
  if ((long long)n_tokens * H > 0x7fffffffLL) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
  const int total = n_tokens * H;
  const dim3 grid((total + 255) / 256), block(256);
  if (dtype == LLMIE_F32)
    launch_k(ssm_steps_kernel<float>, grid, block, 0, stream, (const float*)proj, ld, dt_off, dt_bias, A, dt, decay, H, total);
  else if (dtype == LLMIE_BF16)
    launch_k(ssm_steps_kernel<__nv_bfloat16>, grid, block, 0, stream, (const __nv_bfloat16*)proj, ld, dt_off, dt_bias, A,
             dt, decay, H, total);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

static int ssm_args_ok(const SsmArgs& a, int n_seqs) {
  if (n_seqs < 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.N <= 0 || a.P <= 0 || a.dt_off < 0 || a.ld < a.dt_off + a.H ||
      a.xbc_ld < a.H * a.P + 2 * a.G * a.N)
    return LLMIE_ERR_BAD_ARG;
  if (n_seqs > 65535 || a.H > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  return LLMIE_OK;
}

// Every sequence of the step brings one token. xbc float32 rows [x: H P | B: G N | C: G N], xbc_ld apart; y float32
// [T, H P]; state float32 [slots, H, N, P] is updated in place (write_state); proj as in llmie_ssm_steps. N up to 4096.
extern "C" int llmie_ssm_step(const void* proj, int ld, int dt_off, const float* dt_bias, const float* A,
                              const float* Dskip, const float* xbc, int xbc_ld, float* state, const int* cu_q,
                              const int* seq_slot, float* y, int n_seqs, int H, int G, int N, int P, int write_state,
                              int proj_dtype, cudaStream_t stream) {
  const SsmArgs a{proj, ld, dt_off, dt_bias, A, Dskip, state, cu_q, seq_slot, H, G, N, P, xbc_ld, write_state};
  const int rc = ssm_args_ok(a, n_seqs);
  if (rc != LLMIE_OK) return rc;
  if (N > 4096) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_seqs == 0) return LLMIE_OK;
  const bool by4 = P % 4 == 0 && aligned16(state);
  const int V = by4 ? 4 : 1;
  const int units = P / V;
  int CT = 1;
  while (CT < units && CT < 64) CT <<= 1;
  if (units < CT) CT = units;                       // a row that is no power of two of units: some threads stay idle
  const int RT = kStepThreads / CT, ctiles = (units + CT - 1) / CT;
  const dim3 grid(H * ctiles, n_seqs), block(kStepThreads);
  const size_t smem = (size_t)(2 * N + RT * CT * V) * sizeof(float);
#define LLMIE_STEP(TP, VV) launch_k(ssm_step_kernel<TP, VV>, grid, block, smem, stream, a, xbc, y, CT, RT, ctiles)
  if (proj_dtype == LLMIE_F32) {
    if (by4) LLMIE_STEP(float, 4); else LLMIE_STEP(float, 1);
  } else if (proj_dtype == LLMIE_BF16) {
    if (by4) LLMIE_STEP(__nv_bfloat16, 4); else LLMIE_STEP(__nv_bfloat16, 1);
  } else {
    return LLMIE_ERR_DTYPE;
  }
#undef LLMIE_STEP
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

// Pieces of any length on the tensor cores. xbc bfloat16 rows [x | B | C], xbc_ld apart (a multiple of 8, 16-byte aligned);
// y float32 [T, H P]; state as above. N and P multiples of 8, N <= 256.
extern "C" int llmie_ssm_scan(const void* proj, int ld, int dt_off, const float* dt_bias, const float* A,
                              const float* Dskip, const void* xbc, int xbc_ld, float* state, const int* cu_q,
                              const int* seq_slot, float* y, int n_seqs, int H, int G, int N, int P, int write_state,
                              int proj_dtype, cudaStream_t stream) {
  const SsmArgs a{proj, ld, dt_off, dt_bias, A, Dskip, state, cu_q, seq_slot, H, G, N, P, xbc_ld, write_state};
  const int rc = ssm_args_ok(a, n_seqs);
  if (rc != LLMIE_OK) return rc;
  if (N % 8 || P % 8 || N > 256) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (xbc_ld % 8 || !aligned16(xbc) || !aligned16(state)) return LLMIE_ERR_ALIGNMENT;
  if (n_seqs == 0) return LLMIE_OK;
  if (proj_dtype == LLMIE_F32) return ssm_scan_dispatch<float, float>(a, xbc, y, n_seqs, stream);
  if (proj_dtype == LLMIE_BF16) return ssm_scan_dispatch<__nv_bfloat16, float>(a, xbc, y, n_seqs, stream);
  return LLMIE_ERR_DTYPE;
}

// out [T, n] of out_dtype = norm((y + skip) silu(z)) per run of n / groups columns, times w float32 [n]. y float32 [T, n];
// z rows of z_dtype, z_ld apart; skip_x (float32 rows, x_ld apart) and skip_d (float32 [n / P]) or both null.
extern "C" int llmie_gated_group_norm(const float* y, const void* z, int z_ld, int z_dtype, const float* w, float eps,
                                      void* out, int out_dtype, int n_tokens, int n, int groups, const float* skip_x,
                                      int x_ld, const float* skip_d, int P, cudaStream_t stream) {
  if (n_tokens < 0 || n <= 0 || groups <= 0 || n % groups || z_ld < n || !w || (!skip_x) != (!skip_d) ||
      (skip_d && (P <= 0 || n % P || x_ld < n)))
    return LLMIE_ERR_BAD_ARG;
  if ((size_t)(n / groups) * sizeof(float) > 200 * 1024 || groups > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
#define LLMIE_GGN(TZ, TO) \
  gated_group_norm_launch<TZ, TO>(y, z, z_ld, w, eps, out, n_tokens, n, groups, skip_x, x_ld, skip_d, P, stream)
  if (z_dtype == LLMIE_F32 && out_dtype == LLMIE_F32) return LLMIE_GGN(float, float);
  if (z_dtype == LLMIE_F32 && out_dtype == LLMIE_BF16) return LLMIE_GGN(float, __nv_bfloat16);
  if (z_dtype == LLMIE_BF16 && out_dtype == LLMIE_BF16) return LLMIE_GGN(__nv_bfloat16, __nv_bfloat16);
#undef LLMIE_GGN
  return LLMIE_ERR_DTYPE;
}
