// Causal attention for prompts on the 5th-generation tensor cores: tcgen05.mma with TMEM
// accumulators, operands brought in by TMA straight from the paged KV cache.
//
// The math is the reference's prefill kernel (src/flash_attn.py:42-82): scores q.k / sqrt(hd),
// causal mask, online softmax with float32 running max / sum, probabilities rounded to bfloat16
// for the product with V (:72), output accumulated in float32 and divided by the sum at the end
// (:82). Unlike the reference, K and V are never expanded to the query heads (:92-94): query head
// h simply reads key/value head h / (Hq / Hkv) from the cache, and a sequence may start at any
// position (the reference's mask is only right at position 0).
//
// One block = 128 consecutive query tokens of one sequence and one query head, 320 threads:
//   warp 0      TMA producer: the Q tile once, then for every tile of 128 keys the two cache pages
//               of K and of V ([64 keys, hd] each) into their stages
//   warp 1      owns TMEM (two score buffers of 128 columns); one lane issues S = Q K^T two key
//               tiles ahead, as soon as a buffer is free, and O_j = P_j V_j when P_j is there
//   warps 2..9  softmax, two threads per query row (each half of a key tile's columns and half of
//               the output's): read S from TMEM (tcgen05.ld), mask, running max and sum, write P
//               as bfloat16 into shared memory in the tensor core's swizzled operand layout; the
//               P.V tile of the PREVIOUS key tile is added to the output kept in registers in the
//               middle of this work, so that no thread ever waits for the second product
// V is used as an MN-major B operand (rows of the cache are keys, i.e. the K dimension of P.V),
// so nothing is transposed. Every barrier wait is bounded (tcgen05.cuh).
//
// Registers: a block has 10 warps, which the SM deals to its four schedulers in turn, so a scheduler
// may get three warps of each of two blocks. With more than 85 registers a thread (16,384 a scheduler
// / 6 warps / 32) a new block then finds no room beside a running one although half the SM is free,
// and the SM is refilled only when both of its blocks have ended: the head-size-64 kernel, which
// wants two blocks an SM, is therefore held at 80.
#include "tcgen05.cuh"
#include <math.h>

namespace llmie {
using namespace tc;

constexpr int kQTile = 128;       // query rows per block
constexpr int kKTile = 128;       // keys per step (two cache pages of 64)
constexpr int kSoftmaxThreads = 256;   // two per query row: each takes half of a key tile's columns
constexpr int kAttnThreads = 64 + kSoftmaxThreads;
constexpr int kSubTileBytes = 128 * 128;   // [128 rows x 64 bf16], 16 KB

template <int HD> struct AttnCfg {
  static constexpr int kSub = HD / 64;                       // 64-wide blocks of the head dimension
  // Two score buffers: S of the next key tile is computed while the softmax of the current one runs.
  // head size 64: two blocks share an SM (each 256 TMEM columns, 97 KB). The two score buffers fill the 256
  // columns, so the P.V tile of key tile j is written over S_j, which nobody reads any more once P_j is
  // complete; the buffer is free for S_j+2 when the P.V tile has been read out.
  // head size 128: one block per SM, 512 columns: the P.V tile has columns of its own.
  static constexpr int kSBufs = 2;
  static constexpr bool kPvAlias = HD == 64;
  static constexpr int kKStages = 2;
  static constexpr int kVStages = HD == 64 ? 1 : 2;
  static constexpr int kTmemCols = HD == 64 ? 256 : 512;
  static constexpr int kPvCol = 256;                         // TMEM column of the P.V tile if it has its own
  static constexpr int kMaxRegs = HD == 64 ? 80 : 168;   // 168: three warps of a block on one scheduler
  static constexpr int kQBytes = kSub * kSubTileBytes;
  static constexpr int kKvBytes = kSub * kSubTileBytes;      // one K (or V) tile of 128 keys
  static constexpr int kPBytes = 2 * kSubTileBytes;          // P: [128 rows x 128 keys] bf16
  static constexpr int kSmem = kQBytes + (kKStages + kVStages) * kKvBytes + kPBytes + 1024;
};

struct AttnShared {
  uint64_t q_full;
  uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
  uint64_t s_full[2], s_free[2];
  uint64_t p_ready, pv_full;
  uint32_t tmem_base;
  int abort;
  int last_lo;                     // the first key the tile's last query row may see: the latest among its rows
  // the two threads of a query row tell each other their maxima (and, at the end, their sums) through
  // shared memory; the two warps that share a quarter of the rows meet at an mbarrier of their own
  // (a bounded wait that sleeps in hardware, so a waiting warp does not take issue slots from its partner
  // on the same scheduler). Two value buffers in turn: a thread is never more than one exchange ahead.
  float row_val[2][2][128];
  uint64_t pair_bar[4];
};

// 2^x by the special-function unit (about 2 units in the last place; the probabilities are then
// rounded to bfloat16, whose last place is 2^16 times coarser)
__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Two float32 operations in one instruction (the packed forms of sm_100): what limits the softmax threads is
// the number of instructions they issue as much as the exponentials.
__device__ __forceinline__ uint64_t pair_of(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void split_pair(uint64_t p, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(p));
}
// (y0, y1) = (x0, x1) * b + c, each still one rounding
__device__ __forceinline__ void fma_pair(float& y0, float& y1, float x0, float x1, uint64_t b, uint64_t c) {
  uint64_t y;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(y) : "l"(pair_of(x0, x1)), "l"(b), "l"(c));
  split_pair(y, y0, y1);
}
__device__ __forceinline__ uint64_t add_pair(uint64_t a, float x0, float x1) {
  uint64_t y;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(y) : "l"(a), "l"(pair_of(x0, x1)));
  return y;
}

__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

// Options that change single scores, each off at 0 / null (kernels instantiated with SCORED = false never look at
// them): softcap c > 0 turns a scaled score s into c * tanh(s / c); dist_bias (float32 [n_q, bias_len]) adds a number per
// query head and distance (query position - key position; bias_len - 1 and more share the last entry) after the cap,
// unscaled; sink_vals (float32 [n_q]) is the sink's score per head instead of 0.
// sigmoid_bias (float32 [n_q]) is another kind of attention and has an instantiation of its own (SIGMOID): the weight
// of a visible key is sigmoid(scaled score + sigmoid_bias[head]), not normalised over the keys. No running maximum, no
// sum, nothing exchanged between a row's two threads, and the output is the accumulated P.V as it is; the mask, the
// P operand and the tensor-core protocol are the softmax kernel's.
struct ScoreOptions {
  float softcap;
  const float* dist_bias;
  int bias_len;
  const float* sink_vals;
  const float* sigmoid_bias;
};

__device__ __forceinline__ float tanh_approx(float x) {
  float y;
  asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int HD, bool SCORED, bool SIGMOID>
__global__ void __maxnreg__(SCORED && HD == 64 ? 96 : AttnCfg<HD>::kMaxRegs)
attention_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                            const __grid_constant__ CUtensorMap map_v, __nv_bfloat16* __restrict__ out,
                            const int* __restrict__ cu_q, const int* __restrict__ seq_slot,
                            const int* __restrict__ seq_start, const int* __restrict__ block_table, int max_pages,
                            int scratch_page, int n_q, int n_kv, float scale, int window, int keep_first, int sink,
                            const __nv_bfloat16* __restrict__ gate, int gate_ld, int* __restrict__ status,
                            const ScoreOptions so) {
  using Cfg = AttnCfg<HD>;
  extern __shared__ uint8_t smem_raw[];
  __shared__ AttnShared sh;
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* q_smem = base;
  uint8_t* k_smem = q_smem + Cfg::kQBytes;
  uint8_t* v_smem = k_smem + Cfg::kKStages * Cfg::kKvBytes;
  uint8_t* p_smem = v_smem + Cfg::kVStages * Cfg::kKvBytes;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, head = blockIdx.x;
  const int q_begin = cu_q[seq], q_len = cu_q[seq + 1] - q_begin;
  // Late query tiles see the most keys. Blocks are handed out in the order of blockIdx.x, then y: with
  // the head as x and the query tile (latest first) as y, every head's longest block starts first and
  // the short ones fill the end (longest-processing-time-first), instead of one head after another.
  const int t0 = (gridDim.y - 1 - blockIdx.y) * kQTile;
  if (t0 >= q_len) return;                         // uniform for the block: nothing was set up yet
  const int start = seq_start[seq];                // tokens the sequence held before this step
  const int hk = head / (n_q / n_kv);
  const int rows_here = min(kQTile, q_len - t0);
  // keys this tile of queries may see: [first_key, last_key]
  const int last_key = start + t0 + rows_here - 1;
  const int first_key = first_visible_key(start + t0, window);
  const int tile_lo = first_key / kKTile, tile_hi = last_key / kKTile;
  // With kept first keys (keys below keep_first stay visible behind the window) the key tiles that hold them come
  // first, as far as they lie below the window's tiles; then the window's tiles. tile_of(jt) is the key tile of step jt.
  const int n_kept = (window > 0 && keep_first > 0) ? min((keep_first + kKTile - 1) / kKTile, tile_lo) : 0;
  const int n_tiles = n_kept + tile_hi - tile_lo + 1;
  auto tile_of = [&](int jt) { return jt < n_kept ? jt : tile_lo + jt - n_kept; };

  // One thread is the TMA producer. K and V of a key tile are the two cache pages that hold its 128 keys.
  const int* pages = block_table + (size_t)seq_slot[seq] * max_pages;
  auto load_k = [&](int jt) {
    const int ks = jt % Cfg::kKStages;
    const int lp = tile_of(jt) * 2;              // logical pages of this key tile
    const int last_page = last_key / 64;         // pages beyond the sequence's last key are not mapped
    const int pg0 = pages[lp];
    const int pg1 = (lp + 1 <= last_page && lp + 1 < max_pages) ? pages[lp + 1] : scratch_page;
    uint8_t* kd = k_smem + ks * Cfg::kKvBytes;
    mbar_arrive_expect_tx(&sh.k_full[ks], Cfg::kKvBytes);
    for (int sub = 0; sub < Cfg::kSub; ++sub) {
      tma_load_2d(kd + sub * kSubTileBytes, &map_k, sub * 64, (pg0 * n_kv + hk) * 64, &sh.k_full[ks]);
      tma_load_2d(kd + sub * kSubTileBytes + 8192, &map_k, sub * 64, (pg1 * n_kv + hk) * 64, &sh.k_full[ks]);
    }
  };
  auto load_v = [&](int jt) {
    const int vs = jt % Cfg::kVStages;
    const int lp = tile_of(jt) * 2;
    const int last_page = last_key / 64;
    const int pg0 = pages[lp];
    const int pg1 = (lp + 1 <= last_page && lp + 1 < max_pages) ? pages[lp + 1] : scratch_page;
    uint8_t* vd = v_smem + vs * Cfg::kKvBytes;
    mbar_arrive_expect_tx(&sh.v_full[vs], Cfg::kKvBytes);
    for (int sub = 0; sub < Cfg::kSub; ++sub) {
      tma_load_2d(vd + sub * kSubTileBytes, &map_v, sub * 64, (pg0 * n_kv + hk) * 64, &sh.v_full[vs]);
      tma_load_2d(vd + sub * kSubTileBytes + 8192, &map_v, sub * 64, (pg1 * n_kv + hk) * 64, &sh.v_full[vs]);
    }
  };

  if (threadIdx.x == 0) {
    mbar_init(&sh.q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&sh.k_full[s], 1);
      mbar_init(&sh.k_empty[s], 1);
      mbar_init(&sh.v_full[s], 1);
      mbar_init(&sh.v_empty[s], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&sh.s_full[b], 1);
      mbar_init(&sh.s_free[b], kSoftmaxThreads);
    }
    mbar_init(&sh.p_ready, kSoftmaxThreads);
    mbar_init(&sh.pv_full, 1);
    for (int i = 0; i < 4; ++i) mbar_init(&sh.pair_bar[i], 64);
    sh.abort = 0;
    sh.last_lo = first_visible_key(start + t0 + kQTile - 1, window);
    fence_mbar_init();
    // The first loads leave at once, while warp 1 still asks for tensor memory: only this thread touches the
    // barriers they complete on until the block has met below.
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
    mbar_arrive_expect_tx(&sh.q_full, Cfg::kQBytes);
    for (int sub = 0; sub < Cfg::kSub; ++sub)
      tma_load_2d(q_smem + sub * kSubTileBytes, &map_q, head * HD + sub * 64, q_begin + t0, &sh.q_full);
    load_k(0);
    load_v(0);
  }
  if (warp == 1) {
    tmem_alloc(&sh.tmem_base, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = sh.tmem_base;
  volatile int* abort = &sh.abort;
#define LLMIE_FAIL(code) do { if (!*abort) { *abort = 1; atomicExch(status, (code)); } } while (0)

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer (tile 0 is on its way)
    if (lane == 0) {
      int issued = 1;
      for (int jt = 1; jt < n_tiles; ++jt) {
        const int ks = jt % Cfg::kKStages, vs = jt % Cfg::kVStages;
        if (jt >= Cfg::kKStages && !mbar_wait(&sh.k_empty[ks], ((jt / Cfg::kKStages) - 1) & 1, abort)) {
          LLMIE_FAIL(kStatusTimeoutEmpty);
          break;
        }
        load_k(jt);
        if (jt >= Cfg::kVStages && !mbar_wait(&sh.v_empty[vs], ((jt / Cfg::kVStages) - 1) & 1, abort)) {
          LLMIE_FAIL(kStatusTimeoutEmpty);
          issued = jt + 1;                         // K of this tile is in flight
          break;
        }
        load_v(jt);
        issued = jt + 1;
      }
      if (*abort) {   // let copies that are still in flight land before the block gives its memory up
        for (unsigned spin = 0; spin < (1u << 16) && !mbar_test(&sh.q_full, 0); ++spin) __nanosleep(64);
        for (int jt = max(0, issued - 2); jt < issued; ++jt) {
          uint64_t* kb = &sh.k_full[jt % Cfg::kKStages];
          uint64_t* vb = &sh.v_full[jt % Cfg::kVStages];
          const uint32_t kp = (jt / Cfg::kKStages) & 1, vp = (jt / Cfg::kVStages) & 1;
          for (unsigned spin = 0; spin < (1u << 16) && !(mbar_test(kb, kp) && mbar_test(vb, vp)); ++spin) __nanosleep(64);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_instr_desc_bf16(kQTile, kKTile, 0, 0);
      constexpr uint32_t idesc_pv = make_instr_desc_bf16(kQTile, HD, 0, 1);     // V is MN-major
      const uint32_t q_addr = smem_u32(q_smem), p_addr = smem_u32(p_smem);
      bool ok = mbar_wait(&sh.q_full, 0, abort);
      if (!ok) LLMIE_FAIL(kStatusTimeoutFull);
      auto issue_scores = [&](int jt) -> bool {
        const int ks = jt % Cfg::kKStages, b = jt % Cfg::kSBufs, use = jt / Cfg::kSBufs;
        if (!mbar_wait(&sh.k_full[ks], (jt / Cfg::kKStages) & 1, abort)) { LLMIE_FAIL(kStatusTimeoutFull); return false; }
        if (use >= 1 && !mbar_wait(&sh.s_free[b], (use - 1) & 1, abort)) { LLMIE_FAIL(kStatusTimeoutMma); return false; }
        tc_fence_after_sync();
        const uint32_t k_addr = smem_u32(k_smem + ks * Cfg::kKvBytes);
#pragma unroll
        for (int kk = 0; kk < HD / 16; ++kk) {
          const uint32_t off = (kk >> 2) * kSubTileBytes + (kk & 3) * 32;
          mma_bf16_ss(tmem + b * 128, make_smem_desc(q_addr + off, 16, 1024), make_smem_desc(k_addr + off, 16, 1024),
                      idesc_s, kk > 0 ? 1u : 0u);
        }
        mma_commit(&sh.s_full[b]);
        mma_commit(&sh.k_empty[ks]);             // this K tile is free once the scores are computed
        return true;
      };
      if (ok) ok = issue_scores(0);
      if (ok && n_tiles > 1) ok = issue_scores(1);
      for (int jt = 0; ok && jt < n_tiles; ++jt) {
        const int vs = jt % Cfg::kVStages;
        const uint32_t pv_col = Cfg::kPvAlias ? (uint32_t)(jt & 1) * 128 : (uint32_t)Cfg::kPvCol;
        if (!mbar_wait(&sh.p_ready, jt & 1, abort)) { LLMIE_FAIL(kStatusTimeoutMma); break; }
        if (!mbar_wait(&sh.v_full[vs], (jt / Cfg::kVStages) & 1, abort)) { LLMIE_FAIL(kStatusTimeoutFull); break; }
        tc_fence_after_sync();
        const uint32_t v_addr = smem_u32(v_smem + vs * Cfg::kKvBytes);
#pragma unroll
        for (int kk = 0; kk < kKTile / 16; ++kk) {
          // A = P, K-major: 16 keys = 32 bytes inside a 64-key sub-tile. B = V, MN-major: 16 keys = 16 rows.
          const uint64_t dp = make_smem_desc(p_addr + (kk >> 2) * kSubTileBytes + (kk & 3) * 32, 16, 1024);
          const uint64_t dv = make_smem_desc(v_addr + kk * 2048, kSubTileBytes, 1024);
          mma_bf16_ss(tmem + pv_col, dp, dv, idesc_pv, kk > 0 ? 1u : 0u);
        }
        mma_commit(&sh.pv_full);
        mma_commit(&sh.v_empty[vs]);
        // the scores two tiles ahead go into the buffer of this tile, once the softmax threads have let go of it
        if (jt + 2 < n_tiles && !issue_scores(jt + 2)) break;
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax, two threads per query row
    // Warps 2..5 take the first 64 key columns of a tile (and the first half of the head dimension of
    // the output), warps 6..9 the second; a warp reads the TMEM lanes of its quarter (warp % 4).
    const int quarter = warp & 3;
    const int half = (warp - 2) >> 2;
    const int r = quarter * 32 + lane;                   // row of the tile = TMEM lane
    const uint32_t lane_addr = tmem + ((uint32_t)(quarter * 32) << 16);
    const int qpos = start + t0 + r;                     // absolute position of this query
    const int lo = first_visible_key(qpos, window);
    const float sl2 = scale * 1.4426950408889634f;       // exp(x * scale) = exp2(x * scale * log2 e)
    const float sig_b = SIGMOID ? so.sigmoid_bias[head] * 1.4426950408889634f : 0.f;
    constexpr int kCols = kKTile / 2;                    // key columns of a tile this thread handles
    constexpr int kOut = HD / 2;                         // output columns this thread keeps
    float o[kOut];
#pragma unroll
    for (int d = 0; d < kOut; ++d) o[d] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;                // l_run: the sum over this thread's columns only
    bool ok = true;
    // hands `mine` to the row's other thread and takes its value; n counts the exchanges of this block
    int n_exchanges = 0;
    auto exchange = [&](float mine, float& theirs) -> bool {
      const int buf = n_exchanges & 1;
      sh.row_val[buf][half][r] = mine;
      mbar_arrive(&sh.pair_bar[quarter]);                // release: the value is written before the arrival counts
      const bool ok_ = mbar_wait(&sh.pair_bar[quarter], n_exchanges & 1, abort);
      theirs = sh.row_val[buf][half ^ 1][r];
      ++n_exchanges;
      return ok_;
    };
    // Adds the P.V tile of key tile j to the output, which is first brought to that tile's maximum by alpha_j.
    // The whole warp calls it together, after it has seen pv_full for this tile.
    auto add_pv = [&](int j, float alpha_j) {
      tc_fence_after_sync();
      const uint32_t col = Cfg::kPvAlias ? (uint32_t)(j & 1) * 128 : (uint32_t)Cfg::kPvCol;
      const uint64_t alpha_pair = pair_of(alpha_j, alpha_j);
#pragma unroll
      for (int c0 = 0; c0 < kOut; c0 += 32) {
        uint32_t v[32];
        tmem_ld_32x32(lane_addr + col + half * kOut + c0, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 2)
          fma_pair(o[c0 + i], o[c0 + i + 1], o[c0 + i], o[c0 + i + 1], alpha_pair,
                   pair_of(__uint_as_float(v[i]), __uint_as_float(v[i + 1])));
      }
      tc_fence_before_sync();                  // our TMEM reads are done before the arrival below counts
      if (Cfg::kPvAlias) mbar_arrive(&sh.s_free[j & 1]);     // the buffer may take the scores of tile j + 2
    };
    float alpha_prev = 1.f;                    // alpha of the tile whose P.V tile has not been added yet
    for (int jt = 0; jt < n_tiles; ++jt) {
      const int b = jt % Cfg::kSBufs;
      // every decision to give up is taken by the whole warp: the tensor-memory reads below are warp-wide
      // instructions, a warp must never reach them with some of its lanes gone
      if (!__all_sync(0xffffffffu, mbar_wait(&sh.s_full[b], (jt / Cfg::kSBufs) & 1, abort))) { LLMIE_FAIL(kStatusTimeoutMma); ok = false; break; }
      tc_fence_after_sync();
      const int tile = tile_of(jt);
      const int kbase = tile * kKTile + half * kCols;
      const bool edge = (tile * kKTile + kKTile - 1 > start + t0) ||
                        tile * kKTile < sh.last_lo;
      // pass 1: the row's maximum over the keys it may see
      // (four running maxima and, below, four running sums: one chain of 64 dependent operations would be
      // what a row's time consists of)
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      const int lo_rel = lo - kbase;
#pragma unroll
      for (int c0 = 0; c0 < kCols; c0 += 32) {
        if (SIGMOID && !edge) continue;           // nothing to mark, and no maximum is wanted
        uint32_t v[32];
        tmem_ld_32x32(lane_addr + b * 128 + half * kCols + c0, v);
        tmem_ld_wait();
        if (SCORED) {
          // The cap and the bias by distance change every score of every tile: they are applied here, once, and the
          // changed scores written back to tensor memory in the units the second pass expects (score / scale), with
          // -inf where this row may not look (as the branch below does for edge tiles).
          const unsigned span = (unsigned)(qpos - lo);
          const int kept_rel = min(keep_first, qpos + 1) - kbase;
          const float* brow = so.dist_bias ? so.dist_bias + (size_t)head * so.bias_len : nullptr;
          const float inv_cap = so.softcap > 0.f ? 1.f / so.softcap : 0.f;
          const float inv_scale = 1.f / scale;
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            float x = __uint_as_float(v[i]) * scale;
            if (so.softcap > 0.f) x = so.softcap * tanh_approx(x * inv_cap);
            if (brow) x += __ldg(brow + min(max(qpos - (kbase + c0 + i), 0), so.bias_len - 1));
            v[i] = __float_as_uint(x * inv_scale);
            if (edge && (unsigned)(c0 + i - lo_rel) > span && c0 + i >= kept_rel) v[i] = 0xff800000u;
            mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(v[i]));
          }
          tmem_st_32x32(lane_addr + b * 128 + half * kCols + c0, v);
        } else if (SIGMOID) {
          // no maximum is wanted: only what this row may not see is marked, in the tiles where there is any
          const unsigned span = (unsigned)(qpos - lo);
          const int kept_rel = min(keep_first, qpos + 1) - kbase;
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if ((unsigned)(c0 + i - lo_rel) > span && c0 + i >= kept_rel) v[i] = 0xff800000u;
          tmem_st_32x32(lane_addr + b * 128 + half * kCols + c0, v);
        } else if (edge) {
          // A tile that the causal line or the window's far end crosses: the scores this row may not see become
          // -inf here, in tensor memory too, so that the second pass is the same for every tile (2^-inf = 0).
          // Column c of this thread's half is seen if lo <= kbase + c <= qpos (one unsigned comparison), or if
          // it is one of the kept first keys: kbase + c < min(keep_first, qpos + 1).
          const unsigned span = (unsigned)(qpos - lo);
          const int kept_rel = min(keep_first, qpos + 1) - kbase;
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            if ((unsigned)(c0 + i - lo_rel) > span && c0 + i >= kept_rel) v[i] = 0xff800000u;
            mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(v[i]));
          }
          tmem_st_32x32(lane_addr + b * 128 + half * kCols + c0, v);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(v[i]));
        }
      }
      if (edge || SCORED) tmem_st_wait();
      float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      if (!SIGMOID) {
        float other;
        if (!__all_sync(0xffffffffu, exchange(m_tile, other))) { LLMIE_FAIL(kStatusTimeoutMma); ok = false; break; }
        m_tile = fmaxf(m_tile, other);
      }
      const float m_new = SIGMOID ? 0.f : fmaxf(m_run, m_tile);
      const float m_use = (m_new == -INFINITY) ? 0.f : m_new;      // a row that has seen no key yet
      const float alpha = SIGMOID ? 1.f : exp2_approx((m_run - m_use) * sl2);      // 0 while m_run is -inf
      const float m_scaled = m_use * sl2;
      // pass 2: probabilities, their sum, and P in bfloat16 into the swizzled operand tile
      uint64_t ls[2] = {0ull, 0ull};             // four running sums, as two pairs
      // sigmoid(x) = 1 / (1 + 2^(-x log2 e)): the pairs then hold -scale log2 e and -bias log2 e
      const uint64_t sl2_pair = SIGMOID ? pair_of(-sl2, -sl2) : pair_of(sl2, sl2);
      const uint64_t m_pair = SIGMOID ? pair_of(-sig_b, -sig_b) : pair_of(-m_scaled, -m_scaled);
      // 32 keys from column c0 of this thread's half: probabilities, summed and packed two to a word
      auto probabilities = [&](int c0, uint32_t (&w)[16]) {
        uint32_t v[32];
        tmem_ld_32x32(lane_addr + b * 128 + half * kCols + c0, v);
        tmem_ld_wait();
        float p[32];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float x0, x1;
          fma_pair(x0, x1, __uint_as_float(v[i]), __uint_as_float(v[i + 1]), sl2_pair, m_pair);
          p[i] = exp2_approx(x0);
          p[i + 1] = exp2_approx(x1);
          if (SIGMOID) {                       // a key that is not seen: 2^(+inf), and 1 / inf = 0
            p[i] = __fdividef(1.f, 1.f + p[i]);
            p[i + 1] = __fdividef(1.f, 1.f + p[i + 1]);
          }
        }
        if (!SIGMOID) {
#pragma unroll
          for (int i = 0; i < 32; i += 2) ls[(i >> 1) & 1] = add_pair(ls[(i >> 1) & 1], p[i], p[i + 1]);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) w[i] = pack_bf16(p[2 * i], p[2 * i + 1]);
      };
      auto store_p = [&](int c0, const uint32_t (&w)[16]) {
#pragma unroll
        for (int ch = 0; ch < 4; ++ch) {                 // four 16-byte chunks of 8 keys
          const int chunk = ((half * kCols + c0) >> 3) + ch;       // 0..15 within the 128 keys
          const uint4 q4 = make_uint4(w[ch * 4 + 0], w[ch * 4 + 1], w[ch * 4 + 2], w[ch * 4 + 3]);
          *reinterpret_cast<uint4*>(p_smem + (chunk >> 3) * kSubTileBytes + swizzle128_offset(r, chunk & 7)) = q4;
        }
      };
      static_assert(kCols == 64, "two chunks of 32 keys a thread");
      {
        // The first 32 probabilities are worked out while the tensor core may still be reading the previous P
        // for its P.V product; they go to shared memory once that product is done. Its tile is then added to
        // the output here, in the middle of this tile's work, where it is long complete: no thread waits for it.
        uint32_t w[16];
        probabilities(0, w);
        if (jt > 0 && !__all_sync(0xffffffffu, mbar_wait(&sh.pv_full, (jt - 1) & 1, abort))) { LLMIE_FAIL(kStatusTimeoutMma); ok = false; break; }
        store_p(0, w);
        if (jt > 0) add_pv(jt - 1, alpha_prev);
        probabilities(32, w);
        store_p(32, w);
      }
      tc_fence_before_sync();                  // our TMEM reads of S are done before the barriers are passed
      if (!Cfg::kPvAlias) mbar_arrive(&sh.s_free[b]);
      fence_proxy_async_smem();                // P is visible to the tensor core's reads
      mbar_arrive(&sh.p_ready);
      float l0, l1, l2, l3;
      split_pair(ls[0], l0, l1);
      split_pair(ls[1], l2, l3);
      l_run = fmaf(l_run, alpha, (l0 + l1) + (l2 + l3));
      m_run = m_new;
      alpha_prev = alpha;
    }
    if (ok) {
      if (__all_sync(0xffffffffu, mbar_wait(&sh.pv_full, (n_tiles - 1) & 1, abort))) add_pv(n_tiles - 1, alpha_prev);
      else { LLMIE_FAIL(kStatusTimeoutMma); ok = false; }
    }
    // the row's sum is the two halves' sums (both were kept relative to the same running maximum)
    if (ok && !SIGMOID) {
      float other;
      if (exchange(l_run, other)) l_run += other;
      else { LLMIE_FAIL(kStatusTimeoutMma); ok = false; }
    }
    if (ok && r < rows_here) {
      // the sink: one more term exp(0 - max) in the denominator (it has no value, the numerator stays);
      // a maximum far below zero makes the term infinite and the output zero, which is the limit
      if (sink && !SIGMOID) {
        const float sv = (SCORED && so.sink_vals) ? so.sink_vals[head] * 1.4426950408889634f : 0.f;
        l_run += exp2_approx(sv - m_run * sl2);
      }
      const float inv = SIGMOID ? 1.f : 1.f / l_run;
      const size_t row_off = ((size_t)(q_begin + t0 + r) * n_q + head) * HD + half * kOut;
      __nv_bfloat16* dst = out + row_off;
      const __nv_bfloat16* gr = gate ? gate + (size_t)(q_begin + t0 + r) * gate_ld + head * HD + half * kOut : nullptr;
#pragma unroll
      for (int d = 0; d < kOut; d += 8) {
        float v8[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v8[e] = o[d + e] * inv;
        if (gr) {
          float g8[8];
          load8(gr + d, g8);
#pragma unroll
          for (int e = 0; e < 8; ++e) v8[e] = __fdividef(v8[e], 1.f + __expf(-g8[e]));
        }
        store8(dst + d, v8);
      }
    }
  }
#undef LLMIE_FAIL
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, Cfg::kTmemCols);
  }
}

template <int HD, bool SCORED, bool SIGMOID = false>
static int launch_prefill(const void* q, const void* k_cache, const void* v_cache, void* out, const int* cu_q,
                          const int* seq_slot, const int* seq_start, const int* block_table, int max_pages,
                          int n_pages_total, int n_tokens, int n_seqs, int max_q_len, int n_q, int n_kv, float scale,
                          int window, int keep_first, int sink, const void* gate, int gate_ld, int* status,
                          const ScoreOptions so, cudaStream_t stream) {
  using Cfg = AttnCfg<HD>;
  CUtensorMap map_q, map_k, map_v;
  int rc = tc::make_tmap_bf16_2d(&map_q, q, (uint64_t)n_tokens, (uint64_t)n_q * HD, (uint64_t)n_q * HD, kQTile);
  if (rc != LLMIE_OK) return rc;
  const uint64_t kv_rows = (uint64_t)n_pages_total * n_kv * 64;
  rc = tc::make_tmap_bf16_2d(&map_k, k_cache, kv_rows, HD, HD, 64);
  if (rc != LLMIE_OK) return rc;
  rc = tc::make_tmap_bf16_2d(&map_v, v_cache, kv_rows, HD, HD, 64);
  if (rc != LLMIE_OK) return rc;
  cudaError_t e = cudaFuncSetAttribute(attention_prefill_tc_kernel<HD, SCORED, SIGMOID>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       Cfg::kSmem);
  if (e != cudaSuccess) return (int)e;
  dim3 grid(n_q, (max_q_len + kQTile - 1) / kQTile, n_seqs);
  attention_prefill_tc_kernel<HD, SCORED, SIGMOID><<<grid, kAttnThreads, Cfg::kSmem, stream>>>(
      map_q, map_k, map_v, (__nv_bfloat16*)out, cu_q, seq_slot, seq_start, block_table, max_pages, n_pages_total - 1,
      n_q, n_kv, scale, window, keep_first, sink, (const __nv_bfloat16*)gate, gate_ld, status, so);
  LLMIE_LAUNCH_CHECK();
  return LLMIE_OK;
}

}  // namespace llmie

using namespace llmie;

extern "C" int llmie_attention_prefill_tc_supported(int hd, int page_size) {
  return ((hd == 64 || hd == 128) && page_size == 64) ? 1 : 0;
}

// q, out: bfloat16 [n_tokens, n_q * hd], sequences packed one after another (cu_q [n_seqs + 1]).
// caches: bfloat16 [n_pages_total, n_kv, 64, hd]; the LAST page (n_pages_total - 1) is a scratch
// page that may be read for key positions nobody holds. seq_start[i]: tokens sequence i held
// before this step (its new keys are already in the cache). max_q_len: longest new run, for the grid.
// scale must be positive. window: 0, n > 0 a sliding window, -n < 0 chunks of n positions (first_visible_key). Options,
// each off at 0 / null: keep_first (with a window: the first keys of a sequence stay
// visible behind it), sink (one more softmax term of score 0 without a value), gate (bfloat16 rows of n_q * hd
// elements, gate_ld apart, 16-byte aligned: the output is multiplied by sigmoid(gate)).
static int prefill_tc_entry(const void* q, const void* k_cache, const void* v_cache, void* out, const int* cu_q,
                            const int* seq_slot, const int* seq_start, const int* block_table, int max_pages,
                            int n_pages_total, int n_tokens, int n_seqs, int max_q_len, int n_q, int n_kv, int hd,
                            float scale, int window, int keep_first, int sink, const void* gate, int gate_ld, int* status,
                            const ScoreOptions so, cudaStream_t stream) {
  if (n_tokens < 0 || n_seqs < 0 || n_q <= 0 || n_kv <= 0 || n_q % n_kv || max_pages <= 0 || n_pages_total <= 0)
    return LLMIE_ERR_BAD_ARG;
  if (keep_first < 0 || (window < 0 && keep_first) || (gate && (gate_ld < n_q * hd || gate_ld % 8 || !aligned16(gate)))) return LLMIE_ERR_BAD_ARG;
  if (!(scale > 0.f)) return LLMIE_ERR_BAD_ARG;   // the running maximum is taken before the scores are scaled
  if (so.softcap < 0.f || (so.dist_bias && so.bias_len <= 0) || (so.sink_vals && !sink)) return LLMIE_ERR_BAD_ARG;
  if (so.sigmoid_bias && (so.softcap > 0.f || so.dist_bias || so.sink_vals || sink)) return LLMIE_ERR_BAD_ARG;
  if (!aligned16(q) || !aligned16(out) || !aligned16(k_cache) || !aligned16(v_cache)) return LLMIE_ERR_ALIGNMENT;
  if (n_tokens == 0 || n_seqs == 0 || max_q_len <= 0) return LLMIE_OK;
  if (n_seqs > 65535 || n_q > 65535) return LLMIE_ERR_UNSUPPORTED_SIZE;
  const bool scored = so.softcap > 0.f || so.dist_bias || so.sink_vals;
#define LLMIE_PREFILL_ARGS                                                                                            \
  q, k_cache, v_cache, out, cu_q, seq_slot, seq_start, block_table, max_pages, n_pages_total, n_tokens, n_seqs,       \
      max_q_len, n_q, n_kv, scale, window, keep_first, sink, gate, gate_ld, status, so, stream
  if (so.sigmoid_bias && hd == 64) return launch_prefill<64, false, true>(LLMIE_PREFILL_ARGS);
  if (so.sigmoid_bias && hd == 128) return launch_prefill<128, false, true>(LLMIE_PREFILL_ARGS);
  if (hd == 64) return scored ? launch_prefill<64, true>(LLMIE_PREFILL_ARGS) : launch_prefill<64, false>(LLMIE_PREFILL_ARGS);
  if (hd == 128) return scored ? launch_prefill<128, true>(LLMIE_PREFILL_ARGS) : launch_prefill<128, false>(LLMIE_PREFILL_ARGS);
#undef LLMIE_PREFILL_ARGS
  return LLMIE_ERR_UNSUPPORTED_SIZE;
}

extern "C" int llmie_attention_prefill_tc(const void* q, const void* k_cache, const void* v_cache, void* out,
                                          const int* cu_q, const int* seq_slot, const int* seq_start,
                                          const int* block_table, int max_pages, int n_pages_total, int n_tokens,
                                          int n_seqs, int max_q_len, int n_q, int n_kv, int hd, float scale, int window,
                                          int keep_first, int sink, const void* gate, int gate_ld, int* status,
                                          cudaStream_t stream) {
  return prefill_tc_entry(q, k_cache, v_cache, out, cu_q, seq_slot, seq_start, block_table, max_pages, n_pages_total,
                          n_tokens, n_seqs, max_q_len, n_q, n_kv, hd, scale, window, keep_first, sink, gate, gate_ld,
                          status, ScoreOptions{0.f, nullptr, 0, nullptr, nullptr}, stream);
}

// The same with the options that change single scores (see ScoreOptions): a cap, a bias by distance, the sink's score
// per head.
extern "C" int llmie_attention_prefill_tc_scored(const void* q, const void* k_cache, const void* v_cache, void* out,
                                                 const int* cu_q, const int* seq_slot, const int* seq_start,
                                                 const int* block_table, int max_pages, int n_pages_total, int n_tokens,
                                                 int n_seqs, int max_q_len, int n_q, int n_kv, int hd, float scale,
                                                 int window, int keep_first, int sink, const void* gate, int gate_ld,
                                                 int* status, float softcap, const float* dist_bias, int bias_len,
                                                 const float* sink_vals, cudaStream_t stream) {
  return prefill_tc_entry(q, k_cache, v_cache, out, cu_q, seq_slot, seq_start, block_table, max_pages, n_pages_total,
                          n_tokens, n_seqs, max_q_len, n_q, n_kv, hd, scale, window, keep_first, sink, gate, gate_ld,
                          status, ScoreOptions{softcap, dist_bias, bias_len, sink_vals, nullptr}, stream);
}

// Attention without a softmax: the weight of a visible key is sigmoid(scaled score + sigmoid_bias[head]) (float32
// [n_q]), not normalised over the keys; window, kept first keys and gate as above.
extern "C" int llmie_attention_prefill_tc_sigmoid(const void* q, const void* k_cache, const void* v_cache, void* out,
                                                  const int* cu_q, const int* seq_slot, const int* seq_start,
                                                  const int* block_table, int max_pages, int n_pages_total,
                                                  int n_tokens, int n_seqs, int max_q_len, int n_q, int n_kv, int hd,
                                                  float scale, int window, int keep_first, const void* gate,
                                                  int gate_ld, int* status, const float* sigmoid_bias,
                                                  cudaStream_t stream) {
  if (!sigmoid_bias) return LLMIE_ERR_BAD_ARG;
  return prefill_tc_entry(q, k_cache, v_cache, out, cu_q, seq_slot, seq_start, block_table, max_pages, n_pages_total,
                          n_tokens, n_seqs, max_q_len, n_q, n_kv, hd, scale, window, keep_first, 0, gate, gate_ld,
                          status, ScoreOptions{0.f, nullptr, 0, nullptr, sigmoid_bias}, stream);
}
