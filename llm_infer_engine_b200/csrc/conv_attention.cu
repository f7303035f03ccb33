// What stands between the q and k projections of an attention layer with a short convolution and its scores, in one
// kernel. For token t, head h of q or k and channel c (D channels a head), with u = the projection plus its bias:
//
//   y_t[c] = sum_j taps[c, j] u_(t - K + 1 + j)[c]         a causal convolution per channel over time, zeros before the
//                                                          sequence; inputs from before the step come from the slot's state
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

constexpr int kCaWarps = 4;
constexpr int kCaMaxTaps = 16;

struct ConvQkArgs {
  int ld;                        // elements between two rows of proj
  const float* bias;             // [C] or null, C = (n_q + n_kv) * D: q heads, then k heads
  const float* taps;             // [C, K], the last column multiplies the current token
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
  int max_pages, page_size, n_tokens, n_q, n_kv, D, K, tile, single;
};

// NP: runs of 64 channels a head has at most; KM: taps the registers hold
template <typename TP, typename TO, int NP, int KM>
__global__ void __launch_bounds__(kCaWarps * 32)
conv_qk_store_kernel(const TP* __restrict__ proj, TO* __restrict__ q_out, TO* __restrict__ k_cache,
                     TO* __restrict__ v_cache, const ConvQkArgs p) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const int head = blockIdx.x * kCaWarps + (threadIdx.x >> 5);
  const int D = p.D, K = p.K;
  if (head >= p.n_q + p.n_kv) return;
  const bool is_q = head < p.n_q;
  const int C = (p.n_q + p.n_kv) * D;
  const int base = head * D;                       // first channel of the head
  float tp[KM][2 * NP], w[KM][2 * NP], b[2 * NP], nw[2 * NP];
#pragma unroll
  for (int i = 0; i < 2 * NP; ++i) {
    const int c = 64 * (i >> 1) + 2 * lane + (i & 1);
    const bool ok = c < D;
#pragma unroll
    for (int k = 0; k < KM; ++k) tp[k][i] = ok && k < K ? p.taps[(size_t)(base + c) * K + k] : 0.f;
    b[i] = ok && p.bias ? p.bias[base + c] : 0.f;
    nw[i] = ok ? (is_q ? p.q_w[c] : p.k_w[c]) : 0.f;
  }
  pdl_wait();
  const int ta = blockIdx.y * p.tile, tb = min(ta + p.tile, p.n_tokens);
  int prev_seq = -1;
  auto input = [&](int t, float (&x)[2 * NP]) {
    const TP* row = proj + (size_t)t * p.ld + base;
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      const int c = 64 * (i >> 1) + 2 * lane + (i & 1);
      x[i] = c < D ? to_f32(row[c]) + b[i] : 0.f;
    }
  };
  for (int t = ta; t < tb; ++t) {
    const int seq = p.tok_seq[t];
    const int at = t - p.cu_q[seq];                // place within this step's piece of the sequence
    const int slot = p.seq_slot[seq];
    const int pos = p.tok_pos[t];
    if (seq != prev_seq || at == 0) {
      const float* old = p.conv_state + (size_t)slot * (K - 1) * C + base;
#pragma unroll
      for (int k = 0; k < KM; ++k) {
        if (k < K) {
          const int m = at - (K - 1 - k);          // w[k] is the input K - 1 - k tokens back
          if (m >= 0) {
            input(t - (K - 1 - k), w[k]);
          } else {
#pragma unroll
            for (int i = 0; i < 2 * NP; ++i) {
              const int c = 64 * (i >> 1) + 2 * lane + (i & 1);
              w[k][i] = c < D ? old[(size_t)(K - 1 + m) * C + c] : 0.f;
            }
          }
        }
      }
      prev_seq = seq;
    } else {
#pragma unroll
      for (int k = 0; k + 1 < KM; ++k)
        if (k + 1 < K) {
#pragma unroll
          for (int i = 0; i < 2 * NP; ++i) w[k][i] = w[k + 1][i];
        }
      float x[2 * NP];
      input(t, x);
#pragma unroll
      for (int k = 0; k < KM; ++k)
        if (k == K - 1) {
#pragma unroll
          for (int i = 0; i < 2 * NP; ++i) w[k][i] = x[i];
        }
    }
    float y[2 * NP], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      y[i] = 0.f;
#pragma unroll
      for (int k = 0; k < KM; ++k)
        if (k < K) y[i] = fmaf(tp[k][i], w[k][i], y[i]);
      ss = fmaf(y[i], y[i], ss);
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / (float)D + p.eps);
    TO* dst;
    TO* vdst = nullptr;
    if (is_q) {
      dst = q_out + (size_t)t * p.n_q * D + base;
    } else {
      const int page = p.block_table[(size_t)slot * p.max_pages + pos / p.page_size];
      const size_t off = (((size_t)page * p.n_kv + head - p.n_q) * p.page_size + pos % p.page_size) * D;
      dst = k_cache + off;
      vdst = v_cache + off;
    }
    const float2* cs = p.table + (size_t)min(pos, p.table_len - 1) * (p.rot >> 1);
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int c = 64 * j + 2 * lane;
      float n0 = y[2 * j] * r * nw[2 * j], n1 = y[2 * j + 1] * r * nw[2 * j + 1];
      if (c < p.rot) {                             // rot is even: a pair is rotated whole or not at all
        const float2 a = cs[c >> 1];
        const float u = n0, v = n1;
        n0 = u * a.x - v * a.y;
        n1 = v * a.x + u * a.y;
      }
      if (c < D) {
        dst[c] = from_f32<TO>(n0);
        if (vdst) vdst[c] = from_f32<TO>(y[2 * j]);
      }
      if (c + 1 < D) {
        dst[c + 1] = from_f32<TO>(n1);
        if (vdst) vdst[c + 1] = from_f32<TO>(y[2 * j + 1]);
      }
    }
    if (p.single) {
      float* ns = p.conv_state + (size_t)slot * (K - 1) * C + base;
#pragma unroll
      for (int k = 0; k + 1 < KM; ++k)
        if (k + 1 < K) {
#pragma unroll
          for (int i = 0; i < 2 * NP; ++i) {
            const int c = 64 * (i >> 1) + 2 * lane + (i & 1);
            if (c < D) ns[(size_t)k * C + c] = w[k + 1][i];
          }
        }
    }
  }
}

template <typename TP, typename TO, int NP>
static void conv_qk_launch(const void* proj, void* q_out, void* k_cache, void* v_cache, const ConvQkArgs& a,
                           cudaStream_t stream) {
  const dim3 grid((a.n_q + a.n_kv + kCaWarps - 1) / kCaWarps, (a.n_tokens + a.tile - 1) / a.tile), block(kCaWarps * 32);
  if (a.K <= 4)
    launch_k(conv_qk_store_kernel<TP, TO, NP, 4>, grid, block, 0, stream, (const TP*)proj, (TO*)q_out, (TO*)k_cache,
             (TO*)v_cache, a);
  else
    launch_k(conv_qk_store_kernel<TP, TO, NP, kCaMaxTaps>, grid, block, 0, stream, (const TP*)proj, (TO*)q_out,
             (TO*)k_cache, (TO*)v_cache, a);
}

template <typename TP, typename TO>
static void conv_qk_dispatch(const void* proj, void* q_out, void* k_cache, void* v_cache, const ConvQkArgs& a,
                             cudaStream_t stream) {
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
  const int tile = n_tokens >= 2048 ? 16 : (n_tokens >= 64 ? 4 : 1);
  if ((n_tokens + tile - 1) / tile > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const ConvQkArgs a{ld, bias, taps, conv_state, q_w, k_w, eps, (const float2*)table, table_len, rot, cu_q, tok_pos,
                     tok_seq, seq_slot, block_table, max_pages, page_size, n_tokens, n_q, n_kv, D, K, tile, single};
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
