// What stands between the q and k projections of an attention layer with a short convolution and its scores, in one
// kernel. For token t, head h of q or k and channel c (D channels a head), with u = the projection plus its bias:
//
//   y_t[c] = sum_(i < K) f_i[c] u_(t - i)[c]               a causal convolution per channel over time; inputs from before the
//                                                          step come from the slot's state (zeros in a new slot)
//   values = y                                             key heads only: the values ARE the keys as they stand here
//   n[c]   = y[c] / sqrt(mean_c(y^2) + eps) * w[c]         RMS norm per head, one weight [D] for all q heads, one for k
//   rotation of the first `rot` channels in pairs (2i, 2i + 1) by the token's position, (cos, sin) from a table
//
// q goes to an activation buffer, keys (normed, rotated) and values into the paged cache. All arithmetic is float32, one
// rounding at each store. A warp per (run of tokens, head); a lane owns channels 2 lane, 2 lane + 1 of every 64. In a step
// in which every sequence brings one token (`single`) the warp also writes the convolution's new state: its channels'
// inputs are its own. Other steps leave that to conv_state_store (recurrent.cu).
#include "common.cuh"

namespace llmie {

constexpr int kCaWarps = 2;
constexpr int kCaMaxTaps = 16;

struct ConvQkArgs {
  int ld;                        // elements between two rows of proj
  const float* bias;             // [C] or null, C = (n_q + n_kv) * D: q heads, then k heads
  const float* taps;             // [K, C], the last row multiplies the current token
  float* conv_state;             // [slots, K - 1, C]
  const float* q_w;              // [D]
  const float* k_w;              // [D]
  float eps;
  const float2* table;           // [positions, rot / 2] of (cos, sin)
  int table_len, rot;
  const int* cu_q;
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* block_table;
  int max_pages, page_size, n_tokens, n_q, n_kv, D, K, pair, by8, single;
};

// two neighbouring channels; `pair`: rows and heads begin on an even element, so that one access serves both
__device__ __forceinline__ void ca_load2(const float* p, bool pair, bool second, float& a, float& b) {
  if (pair) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    a = v.x;
    b = v.y;
  } else {
    a = p[0];
    b = second ? p[1] : 0.f;
  }
}
__device__ __forceinline__ void ca_load2(const __nv_bfloat16* p, bool pair, bool second, float& a, float& b) {
  if (pair) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    a = v.x;
    b = v.y;
  } else {
    a = to_f32(p[0]);
    b = second ? to_f32(p[1]) : 0.f;
  }
}
__device__ __forceinline__ void ca_store2(float* p, bool pair, bool second, float a, float b) {
  if (pair) {
    *reinterpret_cast<float2*>(p) = make_float2(a, b);
  } else {
    p[0] = a;
    if (second) p[1] = b;
  }
}
__device__ __forceinline__ void ca_store2(__nv_bfloat16* p, bool pair, bool second, float a, float b) {
  if (pair) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
  } else {
    p[0] = __float2bfloat16_rn(a);
    if (second) p[1] = __float2bfloat16_rn(b);
  }
}

// NP: runs of 64 channels a head has at most; KM: taps the registers hold; TILE: tokens a warp works on. A tile that lies
// within one sequence (nearly all do) asks for its TILE + K - 1 inputs at once; one that crosses from a sequence into the
// next goes token by token, with all K inputs of each.
template <typename TP, typename TO, int NP, int KM, int TILE>
__global__ void __launch_bounds__(kCaWarps * 32)
conv_qk_store_kernel(const TP* __restrict__ proj, TO* __restrict__ q_out, TO* __restrict__ k_cache,
                     TO* __restrict__ v_cache, const ConvQkArgs p) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int head = blockIdx.y * kCaWarps + (threadIdx.x >> 5);
  const int D = p.D, K = p.K;
  if (head >= p.n_q + p.n_kv) return;
  const bool is_q = head < p.n_q, pair = p.pair != 0;
  const int C = (p.n_q + p.n_kv) * D;
  const int base = head * D;                       // first channel of the head
  float tp[KM][2 * NP], b[2 * NP], nw[2 * NP];     // tp[i]: the tap of the input i tokens back
#pragma unroll
  for (int r = 0; r < 2 * NP; ++r) {
    const int c = 64 * (r >> 1) + 2 * lane + (r & 1);
    const bool ok = c < D;
#pragma unroll
    for (int i = 0; i < KM; ++i) tp[i][r] = ok && i < K ? p.taps[(size_t)(K - 1 - i) * C + base + c] : 0.f;
    b[r] = ok && p.bias ? p.bias[base + c] : 0.f;
    nw[r] = ok ? (is_q ? p.q_w[c] : p.k_w[c]) : 0.f;
  }
  pdl_wait();
  auto input = [&](const TP* row, float (&x)[2 * NP]) {
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int c = 64 * j + 2 * lane;
      x[2 * j] = x[2 * j + 1] = 0.f;
      if (c < D) {
        ca_load2(row + c, pair, c + 1 < D, x[2 * j], x[2 * j + 1]);
        x[2 * j] += b[2 * j];
        x[2 * j + 1] += b[2 * j + 1];
      }
    }
  };
  const int ta = blockIdx.x * TILE, tb = min(ta + TILE, p.n_tokens);
  const bool whole = TILE > 1 && p.tok_seq[ta] == p.tok_seq[tb - 1];
  for (int t0 = ta; t0 < tb; t0 += whole ? TILE : 1) {
    constexpr int W = KM - 1;
    float x[TILE + W][2 * NP];                     // x[W + j]: the input of token t0 + j
    const int seq = p.tok_seq[t0];
    const int at = t0 - p.cu_q[seq];               // place within this step's piece of the sequence
    const int slot = p.seq_slot[seq], pos0 = p.tok_pos[t0];
    const int n = whole ? tb - t0 : 1;
    const TP* src = proj + (size_t)t0 * p.ld + base;
#pragma unroll
    for (int j = 0; j < TILE; ++j)
      if (j < n) input(src + (size_t)j * p.ld, x[W + j]);
    float* cs = p.conv_state + (size_t)slot * (K - 1) * C + base;
#pragma unroll
    for (int i = 1; i < KM; ++i) {
      if (i < K && at - i >= 0) {
        input(src - (size_t)i * p.ld, x[W - i]);
      } else {
#pragma unroll
        for (int r = 0; r < 2 * NP; ++r) {
          const int c = 64 * (r >> 1) + 2 * lane + (r & 1);
          x[W - i][r] = i < K && c < D ? cs[(size_t)(K - 1 + at - i) * C + c] : 0.f;
        }
      }
    }
#pragma unroll
    for (int j = 0; j < TILE; ++j) {
      if (j < n) {
        float y[2 * NP], ss = 0.f;
#pragma unroll
        for (int r = 0; r < 2 * NP; ++r) {
          y[r] = 0.f;
#pragma unroll
          for (int i = KM - 1; i >= 0; --i)
            if (i < K) y[r] = fmaf(tp[i][r], x[W + j - i][r], y[r]);
          ss = fmaf(y[r], y[r], ss);
        }
        ss = warp_sum(ss);
        const float rstd = 1.f / sqrtf(ss / (float)D + p.eps);
        const int pos = pos0 + j;
        TO* dst;
        TO* vdst = nullptr;
        if (is_q) {
          dst = q_out + (size_t)(t0 + j) * p.n_q * D + base;
        } else {
          const int page = p.block_table[(size_t)slot * p.max_pages + pos / p.page_size];
          const size_t off = (((size_t)page * p.n_kv + head - p.n_q) * p.page_size + pos % p.page_size) * D;
          dst = k_cache + off;
          vdst = v_cache + off;
        }
        const float2* angle = p.table + (size_t)min(pos, p.table_len - 1) * (p.rot >> 1);
#pragma unroll
        for (int k = 0; k < NP; ++k) {
          const int c = 64 * k + 2 * lane;
          float n0 = y[2 * k] * rstd * nw[2 * k], n1 = y[2 * k + 1] * rstd * nw[2 * k + 1];
          if (c < p.rot) {                         // rot is even: a pair is rotated whole or not at all
            const float2 a = angle[c >> 1];
            const float u = n0, v = n1;
            n0 = u * a.x - v * a.y;
            n1 = v * a.x + u * a.y;
          }
          if (c < D) {
            ca_store2(dst + c, pair, c + 1 < D, n0, n1);
            if (vdst) ca_store2(vdst + c, pair, c + 1 < D, y[2 * k], y[2 * k + 1]);
          }
        }
      }
    }
    if (p.single) {                                // K - 1 inputs, the oldest first
#pragma unroll
      for (int i = 0; i + 1 < KM; ++i)
        if (i + 1 < K) {
#pragma unroll
          for (int r = 0; r < 2 * NP; ++r) {
            const int c = 64 * (r >> 1) + 2 * lane + (r & 1);
            if (c < D) cs[(size_t)(K - 2 - i) * C + c] = x[W - i][r];
          }
        }
    }
  }
}

// The same for head sizes that are multiples of 8: eight channels a lane in 16-byte accesses, LPH lanes (a power of two)
// per head and 32 / LPH heads a warp, so that what a token costs beside its channels (places, the page, the root mean
// square) is shared by the heads of a warp.
template <typename TP, typename TO, int LPH, int TILE>
__global__ void __launch_bounds__(kCaWarps * 32, 8)
conv_qk_store8_kernel(const TP* __restrict__ proj, TO* __restrict__ q_out, TO* __restrict__ k_cache,
                      TO* __restrict__ v_cache, const ConvQkArgs p, int page_shift) {
  constexpr int KM = 4, W = KM - 1, kHeads = 32 / LPH;
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int head = (blockIdx.y * kCaWarps + (threadIdx.x >> 5)) * kHeads + lane / LPH;
  const int c = (lane % LPH) * 8;                  // first of the lane's channels
  const int D = p.D, K = p.K, n_heads = p.n_q + p.n_kv;
  const bool live = head < n_heads && c < D;       // every lane stays for the sums over a head's lanes
  const bool is_q = head < p.n_q;
  const int C = n_heads * D;
  const int ch = live ? head * D + c : 0;
  float tp[KM][8], b[8], nw[8];
#pragma unroll
  for (int i = 0; i < KM; ++i)
    if (i < K) load8(p.taps + (size_t)(K - 1 - i) * C + ch, tp[i]);
#pragma unroll
  for (int e = 0; e < 8; ++e) b[e] = 0.f;
  if (p.bias) load8(p.bias + ch, b);
  load8((is_q ? p.q_w : p.k_w) + (live ? c : 0), nw);
  pdl_wait();
  const int ta = blockIdx.x * TILE, tb = min(ta + TILE, p.n_tokens);
  // the rows in front of the tile are asked for with the tile's own, before it is known whose they are
  float x[TILE + W][8];
#pragma unroll
  for (int j = 0; j < TILE; ++j)
    if (ta + j < tb) load8(proj + (size_t)(ta + j) * p.ld + ch, x[W + j]);
#pragma unroll
  for (int i = 1; i < KM; ++i)
    if (i < K && ta - i >= 0) load8(proj + (size_t)(ta - i) * p.ld + ch, x[W - i]);
  const bool whole = TILE == 1 || p.tok_seq[ta] == p.tok_seq[tb - 1];
  for (int t0 = ta; t0 < tb; t0 += whole ? TILE : 1) {
    const int seq = p.tok_seq[t0];
    const int at = t0 - p.cu_q[seq];
    const int slot = p.seq_slot[seq], pos0 = p.tok_pos[t0];
    const int n = whole ? tb - t0 : 1;
    const TP* src = proj + (size_t)t0 * p.ld + ch;
    float* cs = p.conv_state + (size_t)slot * (K - 1) * C + ch;
    if (!whole) load8(src, x[W]);
    bool old[KM];
#pragma unroll
    for (int i = 1; i < KM; ++i) {
      old[i] = i < K && at - i < 0;
      if (!whole && i < K && !old[i]) load8(src - (size_t)i * p.ld, x[W - i]);
      else if (old[i]) load8(cs + (size_t)(K - 1 + at - i) * C, x[W - i]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {                  // the state holds biased inputs
#pragma unroll
      for (int j = 0; j < TILE; ++j)
        if (j < n) x[W + j][e] += b[e];
#pragma unroll
      for (int i = 1; i < KM; ++i)
        if (i < K && !old[i]) x[W - i][e] += b[e];
    }
#pragma unroll
    for (int j = 0; j < TILE; ++j) {
      if (j < n) {
        float y[8], ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          y[e] = 0.f;
#pragma unroll
          for (int i = KM - 1; i >= 0; --i)
            if (i < K) y[e] = fmaf(tp[i][e], x[W + j - i][e], y[e]);
          ss = fmaf(y[e], y[e], ss);
        }
        if (!live) ss = 0.f;
#pragma unroll
        for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (live) {
          const float rstd = 1.f / sqrtf(ss / (float)D + p.eps);
          const int pos = pos0 + j;
          float v[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) v[e] = y[e] * rstd * nw[e];
          if (c < p.rot) {
            const float2* angle = p.table + (size_t)min(pos, p.table_len - 1) * (p.rot >> 1) + (c >> 1);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              if (c + 2 * k < p.rot) {             // rot is even: a pair is rotated whole or not at all
                const float2 a = angle[k];
                const float u = v[2 * k], w = v[2 * k + 1];
                v[2 * k] = u * a.x - w * a.y;
                v[2 * k + 1] = w * a.x + u * a.y;
              }
            }
          }
          if (is_q) {
            store8(q_out + ((size_t)(t0 + j) * p.n_q + head) * D + c, v);
          } else {
            const int page = p.block_table[(size_t)slot * p.max_pages + (pos >> page_shift)];
            const size_t off = ((((size_t)page * p.n_kv + head - p.n_q) << page_shift) + (pos & (p.page_size - 1))) * D + c;
            store8(k_cache + off, v);
            store8(v_cache + off, y);
          }
        }
      }
    }
    if (p.single && live) {
#pragma unroll
      for (int i = 0; i + 1 < KM; ++i)
        if (i + 1 < K) store8(cs + (size_t)(K - 2 - i) * C, x[W - i]);
    }
  }
}

template <typename TP, typename TO, int LPH>
static void conv_qk_launch8(const void* proj, void* q_out, void* k_cache, void* v_cache, const ConvQkArgs& a,
                            int page_shift, cudaStream_t stream) {
  const int per_block = kCaWarps * (32 / LPH), hb = (a.n_q + a.n_kv + per_block - 1) / per_block;
  if (a.n_tokens >= 256 && !a.single)
    launch_k(conv_qk_store8_kernel<TP, TO, LPH, 4>, dim3((a.n_tokens + 3) / 4, hb), dim3(kCaWarps * 32), 0, stream,
             (const TP*)proj, (TO*)q_out, (TO*)k_cache, (TO*)v_cache, a, page_shift);
  else
    launch_k(conv_qk_store8_kernel<TP, TO, LPH, 1>, dim3(a.n_tokens, hb), dim3(kCaWarps * 32), 0, stream,
             (const TP*)proj, (TO*)q_out, (TO*)k_cache, (TO*)v_cache, a, page_shift);
}

template <typename TP, typename TO, int NP>
static void conv_qk_launch(const void* proj, void* q_out, void* k_cache, void* v_cache, const ConvQkArgs& a,
                           cudaStream_t stream) {
#define LLMIE_CONV_QK(KM, TILE)                                                                                       \
  launch_k(conv_qk_store_kernel<TP, TO, NP, KM, TILE>,                                                                \
           dim3((a.n_tokens + TILE - 1) / TILE, (a.n_q + a.n_kv + kCaWarps - 1) / kCaWarps), dim3(kCaWarps * 32), 0,  \
           stream, (const TP*)proj, (TO*)q_out, (TO*)k_cache, (TO*)v_cache, a)
  const bool many = a.n_tokens >= 256 && !a.single;
  if (a.K > 4) LLMIE_CONV_QK(kCaMaxTaps, 1);
  else if (many && NP == 1) LLMIE_CONV_QK(4, (NP == 1 ? 8 : 4));
  else if (many) LLMIE_CONV_QK(4, 4);
  else LLMIE_CONV_QK(4, 1);
#undef LLMIE_CONV_QK
}

template <typename TP, typename TO>
static void conv_qk_dispatch(const void* proj, void* q_out, void* k_cache, void* v_cache, const ConvQkArgs& a,
                             cudaStream_t stream) {
  int shift = 0;
  while ((1 << shift) < a.page_size) ++shift;
  if (a.K <= 4 && a.by8 && (1 << shift) == a.page_size) {
    if (a.D <= 64) conv_qk_launch8<TP, TO, 8>(proj, q_out, k_cache, v_cache, a, shift, stream);
    else if (a.D <= 128) conv_qk_launch8<TP, TO, 16>(proj, q_out, k_cache, v_cache, a, shift, stream);
    else conv_qk_launch8<TP, TO, 32>(proj, q_out, k_cache, v_cache, a, shift, stream);
    return;
  }
  if (a.D <= 64) conv_qk_launch<TP, TO, 1>(proj, q_out, k_cache, v_cache, a, stream);
  else if (a.D <= 128) conv_qk_launch<TP, TO, 2>(proj, q_out, k_cache, v_cache, a, stream);
  else conv_qk_launch<TP, TO, 4>(proj, q_out, k_cache, v_cache, a, stream);
}

}  // namespace llmie

using namespace llmie;

// proj [T, ld] of proj_dtype holds the projections of the q heads and then of the k heads in its first (n_q + n_kv) * D
// columns; q_out [T, n_q * D] and the caches [pages, n_kv, page_size, D] are of out_dtype. D <= 256, K <= 16 taps, rot even
// and at most D. single != 0: every sequence brings one token and conv_state is written too.
extern "C" int llmie_conv_qk_store(const void* proj, int ld, const float* bias, const float* taps, float* conv_state,
                                   const float* q_w, const float* k_w, float eps, const float* table, int table_len,
                                   int rot, const int* cu_q, const int* tok_pos, const int* tok_seq, const int* seq_slot,
                                   const int* block_table, int max_pages, int page_size, void* q_out, void* k_cache,
                                   void* v_cache, int n_tokens, int n_q, int n_kv, int D, int K, int single,
                                   int proj_dtype, int out_dtype, cudaStream_t stream) {
  if (n_tokens < 0 || n_q <= 0 || n_kv <= 0 || D <= 0 || K <= 0 || rot < 0 || rot % 2 || rot > D || page_size <= 0 ||
      max_pages <= 0 || table_len <= 0 || ld < (n_q + n_kv) * D)
    return LLMIE_ERR_BAD_ARG;
  if (D > 256 || K > kCaMaxTaps) return LLMIE_ERR_UNSUPPORTED_SIZE;
  if (n_tokens == 0) return LLMIE_OK;
  const int pair = D % 2 == 0 && ld % 2 == 0 && aligned16(proj) && aligned16(q_out) && aligned16(k_cache) && aligned16(v_cache);
  const int by8 = pair && D % 8 == 0 && ld % 8 == 0 && aligned16(taps) && aligned16(conv_state) && aligned16(q_w) &&
                  aligned16(k_w) && (!bias || aligned16(bias));
  const ConvQkArgs a{ld, bias, taps, conv_state, q_w, k_w, eps, (const float2*)table, table_len, rot, cu_q, tok_pos,
                     tok_seq, seq_slot, block_table, max_pages, page_size, n_tokens, n_q, n_kv, D, K, pair, by8, single};
  if (proj_dtype == LLMIE_F32 && out_dtype == LLMIE_F32)
    conv_qk_dispatch<float, float>(proj, q_out, k_cache, v_cache, a, stream);
  else if (proj_dtype == LLMIE_F32 && out_dtype == LLMIE_BF16)
    conv_qk_dispatch<float, __nv_bfloat16>(proj, q_out, k_cache, v_cache, a, stream);
  else if (proj_dtype == LLMIE_BF16 && out_dtype == LLMIE_BF16)
    conv_qk_dispatch<__nv_bfloat16, __nv_bfloat16>(proj, q_out, k_cache, v_cache, a, stream);
  else
    return LLMIE_ERR_DTYPE;
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}
