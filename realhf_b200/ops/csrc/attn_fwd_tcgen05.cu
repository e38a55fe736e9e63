// Packed variable-length (causal) attention forward for sm_100a: TMA -> shared (128B swizzle) -> tcgen05.mma -> TMEM.
//
//   O[t, h, :] = softmax(scale * Q[t, h, :] K[seq(t), kv(h), :]^T  (+ causal mask)) V        bf16 / fp16, fp32 softmax
//
// Optional sliding window (causal only): query i sees keys (i - window, i].  Key tiles that lie wholly below the window of the
// CTA's first query row are never loaded (all three roles walk the same tile range [tile0, tile0 + n_kv)); inside the
// remaining tiles the lower edge is a per-row column mask like the diagonal.
//
// Reference: flash-attn's `flash_attn_varlen_func` called from `impl/model/modules/attn.py:240-262`.  One CTA owns a
// 128-row query tile of one (sequence, head) and walks the key / value tiles of that sequence (up to the diagonal).
//
// CTA = 6 warps.  warp 0: TMA producer (Q once, then K_j / V_j into two-stage rings; K and V have their own barriers so a K
// stage is recycled as soon as S_j = Q K_j^T retired, before P_j V_j even started).  warp 1: MMA issuer + TMEM allocator.
// warps 2-5: softmax, one thread per query row (thread <-> TMEM lane), no cross-thread reductions.
//
// Tensor memory (512 columns): S double buffer [0,128) [128,256) and a double buffer for the per-tile product
// T_j = P_j V_j at [256,256+D) [384,384+D).  The running output stays in registers: O <- O * alpha_j + T_j with
// alpha_j = exp2((m_{j-1} - m_j) * scale * log2 e); accumulating per tile in TMEM and folding in registers costs one
// tcgen05.ld of T_j but no TMEM read-modify-write of O when the row maximum moves.  Issue order on the tensor pipe is
// S_0, S_1, PV_0, S_2, PV_1, ...: S_{j+1} is in flight while the softmax warps work on S_j, and the fold of T_{j-1} happens
// after P_j has been handed to the MMA warp, so it overlaps PV_j.
//
// P_j is written by the softmax threads as bf16 straight into the canonical K-major SWIZZLE_128B layout (the same bytes a
// TMA load of a [128 x 64] box would produce), fenced into the async proxy and consumed as the A operand of PV_j; V_j is
// the MN-major B operand (keys are the K dimension, head-dim contiguous), exactly the wgrad operand form of the GEMM.
//
// Outputs: O [T, nq, D] and LSE [nq, T] (natural log, scale applied) in the layout flash-attn's backward consumes.
//
// kSink variant (`WindowAttentionConfig`, inference only, no LSE): score = s * scale * temp_h - slope_h * (i - j) with
// slope_h = 2^(-slope_base (h + 1) / nq) (formed per element in the log2 domain with one extra FMA in each pass), a sliding
// window that also keeps the first `keep` keys (the key tiles of [0, keep) that lie below the window's first tile are walked
// first by all three roles), a per-head sink logit that starts the running maximum with denominator 1, and the row's output
// times sigmoid(gate logit of its head, or of the output element).  `chunk` > 0 replaces the window: a query sees the keys of its own
// chunk of positions up to itself (the tiles below the first row's chunk are not walked, a later row's chunk start is its lower
// mask edge).  kSimple: no distance term, no temperature, no kept first keys and a positive scale: the row maximum is taken over the raw
// products and scaled once, a weight costs one FMA and one exp2, the mask one comparison.  kCap (kSimple only): score = softcap *
// tanh(s * scale / softcap); the cap is monotone, so the raw maximum is capped once, and only the pass that forms the weights
// evaluates tanh per element.  kBias: score = s * scale * temp_h + bias_h(i - j), a learned number per head and distance.  The head's
// table (times log2 e) is staged in shared memory with 127 entries in front (distances of masked columns) and its last value
// repeated behind: a row's column c then reads entry (distance of the row's first column) - c, i.e. one base address per row and tile
// and an immediate offset per column, and the 32 rows of a warp read 32 consecutive entries.  Tiles beyond the table start in its
// constant tail.  kShared: the values are the keys.  Only K tiles travel; the MN-major operand of P V is the K tile read in the other
// major-ness (its 64-wide chunks of the head lie kBKV rows apart), so a stage is recycled after P V instead of after S, and the
// shared memory that V would take holds two more stages.  Query / key size kD and value size kDV may differ.
#include "gemm_common.cuh"

namespace {

constexpr int kBQ = 128;   // query rows per CTA (= UMMA M)
constexpr int kBKV = 128;  // keys per tile (= UMMA N of S, K of PV)
constexpr int kAttnThreads = 192;

struct AttnParams {
  const int* cu_seqlens;  // [B + 1]
  void* out;              // [T, nq, D]
  float* lse;             // [nq, T]
  int64_t out_ld;         // elements between consecutive tokens of `out`
  int T, nq, nkv;
  float scale;
  int causal;
  int window;             // > 0 (with causal): a query at position i sees keys (i - window, i]
  // kSink variant only
  int keep;               // with a window: keys [0, keep) stay visible to every later query
  const void* temp;       // [nq] per-head factor on the scaled score, or null
  const void* sink;       // [nq] per-head sink logit, or null
  const void* gate;       // gate logits, element (t, h) at gate[t * gate_ld + h], or null
  int64_t gate_ld;
  float slope_base;       // < 0: no distance term
  int vshare = 1;         // consecutive key heads that read one value head (V has nkv / vshare heads)
  int gate_mode = 1;      // gate logits: 1 one per head, 2 one per output element (element (t, h, c) at gate[t * gate_ld + h * D + c])
  int chunk = 0;          // > 0 (window 0): a query sees the keys of its own chunk
  float softcap = 0.f;    // kCap variant
  const float* bias = nullptr;   // kBias variant: [nq, bias_ld], the first n_bias columns are used; distances beyond read the last one
  int n_bias = 0, bias_ld = 0;
};

template <int kD, int kDV, bool kShared> struct ACfg {
  static constexpr int kDBlocks = kD / 64, kDVBlocks = kDV / 64;   // 64-element (128 B) column blocks of Q / K and of V
  static constexpr int kQBytes = kBQ * kD * 2;
  static constexpr int kKBytes = kBKV * kD * 2, kVBytes = kBKV * kDV * 2;   // one K / V stage
  static constexpr int kKStages = kShared ? 4 : 2;
  static constexpr int kPBytes = kBQ * kBKV * 2;
  static constexpr int kBars = kQBytes + kKStages * kKBytes + (kShared ? 0 : 2 * kVBytes) + kPBytes;   // offset of the barriers
  static constexpr int kSmemBytes = kBars + 1024 /*align*/ + 256 /*barriers*/;
};
constexpr int kBiasFront = kBKV - 1, kBiasPad = 2 * kBKV + kBKV;   // table entries in front / in all beyond n_bias
constexpr int kMaxSmem = 227 * 1024;

enum Bar { Q_FULL = 0, K_FULL = 1, K_EMPTY = 3, V_FULL = 5, V_EMPTY = 7, S_FULL = 9, S_EMPTY = 11, P_FULL = 13, P_EMPTY = 14,
           O_FULL = 15, O_EMPTY = 17, NUM_BARS = 19 };

// Every wait is bounded: a wait that runs out sets the CTA's `dead` flag (all later waits of the CTA then return at once), and the
// kernel ends normally after a pause that lets its own copies land; `rb_attn_wait_error` tells the host.
__device__ int g_wait_error = 0;
constexpr int kWaitPolls = 1 << 20;

RB_DEVICE void bounded_wait(uint32_t bar, uint32_t parity, volatile uint32_t* dead) {
  for (int i = 0; !ptx::mbar_try_wait(bar, parity); ++i)
    if (i >= kWaitPolls || *dead) { *dead = 1; return; }
}

RB_DEVICE void st_shared_v4(uint32_t addr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}
template <typename T> RB_DEVICE uint32_t pack2(float lo, float hi);
template <> RB_DEVICE uint32_t pack2<__nv_bfloat16>(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
template <> RB_DEVICE uint32_t pack2<__half>(float lo, float hi) {
  __half2 v = __floats2half2_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// cap * tanh(s * scale / cap) + add in the log2 domain, tanh(x) = 1 - 2 / (1 + 2^(2 x log2 e)): c = 2 log2 e * scale / cap,
// k = cap log2 e, k_add = k + add.  Absolute error a few ulp of k; saturates to +-k.
RB_DEVICE float soft_cap2(float s, float c, float k, float k_add) {
  return fmaf(-2.f * k, __fdividef(1.f, 1.f + exp2f(fminf(s * c, 80.f))), k_add);
}

template <int kD, int kDV, typename T, int kFmt, bool kSink = false, bool kCap = false, bool kSimple = false, bool kBias = false, bool kShared = false>
__global__ void __launch_bounds__(kAttnThreads, 1) attn_fwd_kernel(const __grid_constant__ CUtensorMap tma_q,
                                                                   const __grid_constant__ CUtensorMap tma_k,
                                                                   const __grid_constant__ CUtensorMap tma_v, AttnParams p) {
  static_assert(!kShared || kD == kDV, "shared keys and values have one size");
  static_assert(!kBias || (kSink && !kSimple && !kCap), "kBias is a form of kSink");
  constexpr bool kOneMask = kSimple || kBias;      // no kept first keys: visible columns are one range
  using C = ACfg<kD, kDV, kShared>;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int qt = gridDim.x - 1 - blockIdx.x;  // long (late) query tiles first: they walk the most key tiles
  const int tok0 = p.cu_seqlens[seq];
  const int L = p.cu_seqlens[seq + 1] - tok0;
  const int q0 = qt * kBQ;
  if (q0 >= L) return;  // uniform for the CTA, before any barrier / TMEM allocation
  const int hk = head / (p.nq / p.nkv);
  const int kv_len = p.causal ? min(L, q0 + kBQ) : L;
  const int win = (p.causal && p.window > 0) ? p.window : 0;
  const int chunk = kSink ? p.chunk : 0;
  // first key tile any row of this CTA can see
  const int tile0 = (kSink && chunk > 0) ? (q0 / chunk * chunk) / kBKV : win > 0 ? max(0, q0 - win + 1) / kBKV : 0;
  // kSink: the tiles of the kept first keys that lie wholly below tile0 come first in every role's walk
  const int n_keep = (kSink && !kOneMask && win > 0) ? min(RB_CEIL_DIV(p.keep, kBKV), tile0) : 0;
  const int n_kv = n_keep + RB_CEIL_DIV(kv_len, kBKV) - tile0;    // >= 1: the diagonal tile is always visible
  auto tile_of = [&](int j) { return j < n_keep ? j : tile0 + j - n_keep; };

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t sQ = ptx::smem_u32(smem);
  const uint32_t sK = sQ + C::kQBytes;
  const uint32_t sV = sK + C::kKStages * C::kKBytes;
  const uint32_t sP = sV + (kShared ? 0 : 2 * C::kVBytes);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::kBars);
  float* tab = reinterpret_cast<float*>(smem + C::kBars + 256);      // kBias
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + NUM_BARS);
  volatile uint32_t* dead = tmem_ptr + 1;
  auto bar = [&](int i) { return ptx::smem_u32(&bars[i]); };
  // stage and barriers of key tile j (kShared: four stages, the last two on V's barriers)
  auto k_stage = [](int j) { return kShared ? j & 3 : j & 1; };
  auto k_par = [](int j) { return (uint32_t)(kShared ? j >> 2 : j >> 1) & 1u; };
  auto k_full = [](int st) { return st < 2 ? K_FULL + st : V_FULL + st - 2; };
  auto k_empty = [](int st) { return st < 2 ? K_EMPTY + st : V_EMPTY + st - 2; };
  if constexpr (kBias) {
    for (int i = threadIdx.x; i < p.n_bias + kBiasPad; i += kAttnThreads)
      tab[i] = p.bias[(int64_t)head * p.bias_ld + min(max(i - kBiasFront, 0), p.n_bias - 1)] * 1.4426950408889634f;
  }

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0 && lane == 0) {
    *dead = 0;
    ptx::prefetch_tensormap(&tma_q);
    ptx::prefetch_tensormap(&tma_k);
    ptx::prefetch_tensormap(&tma_v);
    for (int i = 0; i < NUM_BARS; ++i) {
      const bool softmax_side = (i == S_EMPTY || i == S_EMPTY + 1 || i == P_FULL || i == O_EMPTY || i == O_EMPTY + 1);
      ptx::mbar_init(bar(i), softmax_side ? 4 : 1);  // one arrival per softmax warp
    }
    ptx::fence_barrier_init();
  }
  if (warp == 1) {
    ptx::tmem_alloc(ptx::smem_u32(tmem_ptr), 512);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before();
  __syncthreads();
  ptx::tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  auto wait = [&](uint32_t b, uint32_t parity) { bounded_wait(b, parity, dead); };

  if (warp == 0) {
    // ===================================================== TMA producer
    if (lane == 0) {
      ptx::mbar_arrive_expect_tx(bar(Q_FULL), C::kQBytes);
#pragma unroll
      for (int kb = 0; kb < C::kDBlocks; ++kb)
        ptx::tma_load_2d(sQ + kb * (kBQ * 128), &tma_q, bar(Q_FULL), head * kD + kb * 64, tok0 + q0);
      for (int j = 0; j < n_kv; ++j) {
        const int row = tok0 + tile_of(j) * kBKV;
        const int ks = k_stage(j);
        wait(bar(k_empty(ks)), k_par(j) ^ 1);
        ptx::mbar_arrive_expect_tx(bar(k_full(ks)), C::kKBytes);
#pragma unroll
        for (int kb = 0; kb < C::kDBlocks; ++kb)
          ptx::tma_load_2d(sK + ks * C::kKBytes + kb * (kBKV * 128), &tma_k, bar(k_full(ks)), hk * kD + kb * 64, row);
        if constexpr (kShared) continue;
        const int st = j & 1;
        const uint32_t par = (uint32_t)(j >> 1) & 1u;
        wait(bar(V_EMPTY + st), par ^ 1);
        ptx::mbar_arrive_expect_tx(bar(V_FULL + st), C::kVBytes);
        // V is the MN-major B operand of P V: it is staged as two 64-key halves, each [d chunk][64 keys][128 B], i.e. exactly
        // the stage format (and the 8 KB chunk stride) of the GEMM's MN-major operands
#pragma unroll
        for (int half = 0; half < kBKV / 64; ++half)
#pragma unroll
          for (int kb = 0; kb < C::kDVBlocks; ++kb)
            ptx::tma_load_2d(sV + st * C::kVBytes + half * (64 * kDV * 2) + kb * (64 * 128), &tma_v, bar(V_FULL + st),
                             (hk / p.vshare) * kDV + kb * 64, row + half * 64);
      }
    }
  } else if (warp == 1) {
    // ===================================================== MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = ptx::make_idesc_f16(kFmt, kBQ, kBKV, 0, 0);  // Q, K both K-major (head-dim contiguous)
      constexpr uint32_t idesc_o = ptx::make_idesc_f16(kFmt, kBQ, kDV, 0, 1);    // P K-major, V MN-major
      auto issue_s = [&](int j) {
        const int st = j & 1, ks = k_stage(j);
        const uint32_t par = (uint32_t)(j >> 1) & 1u;
        wait(bar(k_full(ks)), k_par(j));
        wait(bar(S_EMPTY + st), par ^ 1);
        ptx::tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < kD / 16; ++kk) {
          const uint32_t off = (kk >> 2) * (kBQ * 128) + (kk & 3) * 32;
          ptx::tc_mma_f16(tmem_base + st * 128, ptx::make_smem_desc_sw128(sQ + off, 16, 1024),
                          ptx::make_smem_desc_sw128(sK + ks * C::kKBytes + off, 16, 1024), idesc_s, kk != 0 ? 1u : 0u);
        }
        if constexpr (!kShared) ptx::tc_commit(bar(k_empty(ks)));  // K stage reusable once S_j retired
        ptx::tc_commit(bar(S_FULL + st));
      };
      wait(bar(Q_FULL), 0);
      issue_s(0);
      for (int j = 0; j < n_kv; ++j) {
        if (j + 1 < n_kv) issue_s(j + 1);
        const int st = j & 1;
        const uint32_t par = (uint32_t)(j >> 1) & 1u;
        wait(bar(P_FULL), (uint32_t)j & 1u);
        if constexpr (!kShared) wait(bar(V_FULL + st), par);   // (kShared: the tile arrived before S_j was issued)
        wait(bar(O_EMPTY + st), par ^ 1);
        ptx::tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < kBKV / 16; ++kk) {
          // A: 16 keys = 32 B inside the 128 B row of key block kk/4; B: 16 key rows = 2048 B down every 64-wide d chunk of
          // key half kk/4 (kShared: of the whole K tile, whose chunks hold all kBKV keys)
          const uint32_t b_off = kShared ? sK + k_stage(j) * C::kKBytes + kk * 2048 : sV + st * C::kVBytes + (kk >> 2) * (64 * kDV * 2) + (kk & 3) * 2048;
          ptx::tc_mma_f16(tmem_base + 256 + st * 128,
                          ptx::make_smem_desc_sw128(sP + (kk >> 2) * (kBQ * 128) + (kk & 3) * 32, 16, 1024),
                          ptx::make_smem_desc_sw128(b_off, (kShared ? kBKV : 64) * 128, 1024), idesc_o, kk != 0 ? 1u : 0u);
        }
        ptx::tc_commit(bar(kShared ? k_empty(k_stage(j)) : V_EMPTY + st));
        ptx::tc_commit(bar(P_EMPTY));
        ptx::tc_commit(bar(O_FULL + st));
      }
    }
  } else {
    // ===================================================== softmax + output (4 warps; thread = query row = TMEM lane)
    const int quad = warp & 3;
    const int row = quad * 32 + lane;
    const int q_pos = q0 + row;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quad * 32) << 16);
    const float sl2 = p.scale * 1.4426950408889634f;
    const uint32_t p_row = sP + (uint32_t)(row >> 3) * 1024u + (uint32_t)(row & 7) * 128u;
    const uint32_t sw = (uint32_t)(row & 7);
    float m_run = -INFINITY, l_run = 0.f, alpha_prev = 0.f;
    const int row_lo = (kSink && chunk > 0) ? q_pos / chunk * chunk : win > 0 ? q_pos - win + 1 : 0;   // first visible key of the row
    const int last_lo = (kSink && chunk > 0) ? (q0 + kBQ - 1) / chunk * chunk : q0 + kBQ - win;      // of the tile's last row
    const bool bounded = win > 0 || (kSink && chunk > 0);
    const float cap_c = kCap ? 2.f * 1.4426950408889634f * p.scale / p.softcap : 0.f, cap_k = kCap ? p.softcap * 1.4426950408889634f : 0.f;
    // kSink: scores live in the log2 domain, t = s * c2 - slope2 * (q_pos - key_pos); the sink starts the maximum
    float c2 = 0.f, slope2 = 0.f;
    if constexpr (kSink) {
      c2 = sl2 * (p.temp ? rb::to_f(reinterpret_cast<const T*>(p.temp)[head]) : 1.f);
      if constexpr (!kSimple && !kBias) slope2 = p.slope_base >= 0.f ? exp2f(-p.slope_base * (float)(head + 1) / (float)p.nq) * 1.4426950408889634f : 0.f;
      if (p.sink) { m_run = rb::to_f(reinterpret_cast<const T*>(p.sink)[head]) * 1.4426950408889634f; l_run = 1.f; }
    }
    float O[kDV];
#pragma unroll
    for (int i = 0; i < kDV; ++i) O[i] = 0.f;

    auto fold = [&](int t, float a) {  // O <- O * a + T_t
      const int b = t & 1;
      wait(bar(O_FULL + b), (uint32_t)(t >> 1) & 1u);
      ptx::tc_fence_after();
#pragma unroll
      for (int c = 0; c < kDV / 32; ++c) {
        uint32_t r[32];
        ptx::tc_ld_32x32(lane_addr + 256 + b * 128 + c * 32, r);
        ptx::tc_wait_ld();
#pragma unroll
        for (int i = 0; i < 32; ++i) O[c * 32 + i] = fmaf(O[c * 32 + i], a, __uint_as_float(r[i]));
      }
      ptx::tc_fence_before();
      __syncwarp();
      if (lane == 0) ptx::mbar_arrive(bar(O_EMPTY + b));
    };

    for (int j = 0; j < n_kv; ++j) {
      const int b = j & 1;
      const int kv0 = tile_of(j) * kBKV;
      wait(bar(S_FULL + b), (uint32_t)(j >> 1) & 1u);
      ptx::tc_fence_after();
      // only the last tile of the sequence, the diagonal tile and the tiles the window's lower edge crosses need per-element
      // masks (uniform over the CTA)
      const bool need_mask = (kv0 + kBKV > L) || (p.causal && kv0 + kBKV - 1 > q0) || (bounded && last_lo > kv0);
      const int lim = (p.causal ? min(L, q_pos + 1) : L) - kv0;  // local key columns [lo, lim) are visible to this row
      const int lo = bounded ? row_lo - kv0 : 0;
      const int kept = kSink && !kOneMask ? p.keep - kv0 : 0;                 // kSink: local columns below `kept` stay visible under `lo`
      const uint32_t n_vis = (uint32_t)max(lim - lo, 0);
      auto hidden = [&](int col) {
        if constexpr (kOneMask) return (uint32_t)(col - lo) >= n_vis;
        return col >= lim || (col < lo && (!kSink || col >= kept));
      };
      const float base = kSink && !kBias ? slope2 * (float)(kv0 - q_pos) : 0.f;
      // kBias: entry of the row's column 0 (q0 - kv0 >= 0: the diagonal tile is the last one); beyond the table its constant tail
      const float* brow = kBias ? tab + min(q0 - kv0, p.n_bias - 1 + kBiasFront) + row + kBiasFront : nullptr;
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < kBKV / 32; ++c) {
        uint32_t r[32];
        ptx::tc_ld_32x32(lane_addr + b * 128 + c * 32, r);
        ptx::tc_wait_ld();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float s = __uint_as_float(r[i]);
          if constexpr (kBias) s = fmaf(s, c2, brow[-(c * 32 + i)]);
          else if constexpr (kSink && !kSimple) s = fmaf(s, c2, fmaf(slope2, (float)(c * 32 + i), base));
          if (need_mask && hidden(c * 32 + i)) s = -INFINITY;
          mx = fmaxf(mx, s);
        }
      }
      if constexpr (kSimple) {
        if (mx != -INFINITY) mx = kCap ? soft_cap2(mx, cap_c, cap_k, cap_k) : mx * c2;
      }
      const float m_new = fmaxf(m_run, mx);
      const float m_eff = (m_new == -INFINITY) ? 0.f : m_new;  // fully masked so far: keep exp2 arguments finite
      const float alpha = kSink ? exp2f(m_run - m_eff) : exp2f((m_run - m_eff) * sl2);
      const float neg_m = kSink ? -m_eff : -m_eff * sl2;
      if (j > 0) wait(bar(P_EMPTY), (uint32_t)(j - 1) & 1u);  // PV_{j-1} finished reading the P buffer
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < kBKV / 32; ++c) {
        uint32_t r[32];
        ptx::tc_ld_32x32(lane_addr + b * 128 + c * 32, r);
        ptx::tc_wait_ld();
        uint32_t w[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float e0, e1;
          if constexpr (kCap) {
            e0 = exp2f(soft_cap2(__uint_as_float(r[i]), cap_c, cap_k, cap_k + neg_m));
            e1 = exp2f(soft_cap2(__uint_as_float(r[i + 1]), cap_c, cap_k, cap_k + neg_m));
          } else if constexpr (kBias) {
            e0 = exp2f(fmaf(__uint_as_float(r[i]), c2, brow[-(c * 32 + i)]) + neg_m);
            e1 = exp2f(fmaf(__uint_as_float(r[i + 1]), c2, brow[-(c * 32 + i + 1)]) + neg_m);
          } else if constexpr (kSimple) {
            e0 = exp2f(fmaf(__uint_as_float(r[i]), c2, neg_m));
            e1 = exp2f(fmaf(__uint_as_float(r[i + 1]), c2, neg_m));
          } else if constexpr (kSink) {
            e0 = exp2f(fmaf(__uint_as_float(r[i]), c2, fmaf(slope2, (float)(c * 32 + i), base)) + neg_m);
            e1 = exp2f(fmaf(__uint_as_float(r[i + 1]), c2, fmaf(slope2, (float)(c * 32 + i + 1), base)) + neg_m);
          } else {
            e0 = exp2f(fmaf(__uint_as_float(r[i]), sl2, neg_m));
            e1 = exp2f(fmaf(__uint_as_float(r[i + 1]), sl2, neg_m));
          }
          if (need_mask) {
            if (hidden(c * 32 + i)) e0 = 0.f;
            if (hidden(c * 32 + i + 1)) e1 = 0.f;
          }
          sum += e0 + e1;
          w[i >> 1] = pack2<T>(e0, e1);
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const uint32_t piece = (uint32_t)(c * 4 + t);  // 16-byte piece (8 keys) of this row: key block piece/8, slot piece%8
          st_shared_v4(p_row + (piece >> 3) * (kBQ * 128) + (((piece & 7) ^ sw) << 4), w[4 * t], w[4 * t + 1], w[4 * t + 2],
                       w[4 * t + 3]);
        }
      }
      ptx::tc_fence_before();     // our tcgen05.ld of S_j are complete (wait::ld) before the MMA warp may overwrite the buffer
      ptx::fence_proxy_async();   // P_j (generic-proxy stores) visible to the tensor core's async-proxy reads
      __syncwarp();
      if (lane == 0) {
        ptx::mbar_arrive(bar(S_EMPTY + b));
        ptx::mbar_arrive(bar(P_FULL));
      }
      l_run = fmaf(l_run, alpha, sum);
      m_run = m_new;
      if (j > 0) fold(j - 1, alpha_prev);
      alpha_prev = alpha;
    }
    fold(n_kv - 1, alpha_prev);

    if (q_pos < L) {
      float inv = 1.f / l_run;
      if constexpr (kSink) {
        if (p.gate && p.gate_mode == 1)
          inv *= 1.f / (1.f + __expf(-rb::to_f(reinterpret_cast<const T*>(p.gate)[(int64_t)(tok0 + q_pos) * p.gate_ld + head])));
        if (p.gate && p.gate_mode == 2) {          // (rows of the gate are 16-byte aligned: checked by the host)
          const T* gr = reinterpret_cast<const T*>(p.gate) + (int64_t)(tok0 + q_pos) * p.gate_ld + (int64_t)head * kDV;
#pragma unroll
          for (int i = 0; i < kDV; i += 8) {
            const rb::Pack<T, 8> gv = *reinterpret_cast<const rb::Pack<T, 8>*>(gr + i);
#pragma unroll
            for (int j = 0; j < 8; ++j) O[i + j] *= __fdividef(1.f, 1.f + __expf(-rb::to_f(gv.v[j])));
          }
        }
      }
      T* dst = reinterpret_cast<T*>(p.out) + (int64_t)(tok0 + q_pos) * p.out_ld + (int64_t)head * kDV;
#pragma unroll
      for (int i = 0; i < kDV; i += 8) {
        uint4 v;
        v.x = pack2<T>(O[i] * inv, O[i + 1] * inv);
        v.y = pack2<T>(O[i + 2] * inv, O[i + 3] * inv);
        v.z = pack2<T>(O[i + 4] * inv, O[i + 5] * inv);
        v.w = pack2<T>(O[i + 6] * inv, O[i + 7] * inv);
        *reinterpret_cast<uint4*>(dst + i) = v;
      }
      if constexpr (!kSink) p.lse[(int64_t)head * p.T + tok0 + q_pos] = m_run * p.scale + __logf(l_run);
    }
  }

  ptx::tc_fence_before();
  __syncthreads();
  if (*dead) {
    if (threadIdx.x == 0) g_wait_error = 1;
    for (int i = 0; i < 1000; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    ptx::tc_fence_after();
    ptx::tmem_dealloc(tmem_base, 512);
  }
}

template <int kD, int kDV, typename T, int kFmt, bool kSink = false, bool kCap = false, bool kSimple = false, bool kBias = false, bool kShared = false>
int launch_attn_fwd(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const AttnParams& p, int B,
                    int max_seqlen, cudaStream_t s) {
  using C = ACfg<kD, kDV, kShared>;
  auto kern = attn_fwd_kernel<kD, kDV, T, kFmt, kSink, kCap, kSimple, kBias, kShared>;
  const int smem = C::kSmemBytes + (kBias ? (p.n_bias + kBiasPad) * 4 : 0);
  if (smem > kMaxSmem) return -32;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kBias ? kMaxSmem : C::kSmemBytes) != cudaSuccess) return -30;
    attr_set = true;
  }
  dim3 grid(RB_CEIL_DIV(max_seqlen, kBQ), p.nq, B);
  kern<<<grid, kAttnThreads, smem, s>>>(mq, mk, mv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -31;
}

}  // namespace

// 1 if a bounded wait of the kernel ran out since the last call (synchronises; for diagnostics)
extern "C" int rb_attn_wait_error() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, g_wait_error, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) cudaMemcpyToSymbol(g_wait_error, &zero, sizeof(int));
  return v;
}

// q / k / v: [T, heads, hd] views (unit stride over hd, `heads * hd` contiguous columns, row pitch *_ld elements) -- e.g. the
// three column ranges of the fused QKV projection.  out [T, nq, hd] with row pitch out_ld, lse [nq, T] fp32.
// dt: 1 = bf16, 2 = fp16.  Returns 0 or a negative code (unsupported shape / descriptor failure).
// window > 0 (causal only): sliding-window attention.
extern "C" int rb_attn_fwd_window(const void* q, const void* k, const void* v, void* out, float* lse, const int* cu_seqlens,
                                  int64_t q_ld, int64_t k_ld, int64_t v_ld, int64_t out_ld, int T, int B, int nq, int nkv, int hd,
                                  int max_seqlen, float scale, int causal, int window, int dt, cudaStream_t s) {
  if (hd != 128 && hd != 64) return -1;
  if (dt != 1 && dt != 2) return -2;
  if (nq % nkv != 0 || T <= 0 || B <= 0 || max_seqlen <= 0) return -3;
  if ((q_ld | k_ld | v_ld | out_ld) % 8 != 0) return -4;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)out) & 15) return -5;
  CUtensorMap mq, mk, mv;
  const int bf = dt == 1;
  if (!make_tmap(&mq, q, bf, T, (uint64_t)nq * hd, q_ld, 64, kBQ)) return -10;
  if (!make_tmap(&mk, k, bf, T, (uint64_t)nkv * hd, k_ld, 64, kBKV)) return -11;
  if (!make_tmap(&mv, v, bf, T, (uint64_t)nkv * hd, v_ld, 64, 64)) return -12;  // 64-key halves, see the producer
  if (window > 0 && !causal) return -6;
  AttnParams p{cu_seqlens, out, lse, out_ld, T, nq, nkv, scale, causal, window, 0, nullptr, nullptr, nullptr, 0, -1.f};
  if (hd == 128) {
    return bf ? launch_attn_fwd<128, 128, __nv_bfloat16, 1>(mq, mk, mv, p, B, max_seqlen, s)
              : launch_attn_fwd<128, 128, __half, 0>(mq, mk, mv, p, B, max_seqlen, s);
  }
  return bf ? launch_attn_fwd<64, 64, __nv_bfloat16, 1>(mq, mk, mv, p, B, max_seqlen, s)
            : launch_attn_fwd<64, 64, __half, 0>(mq, mk, mv, p, B, max_seqlen, s);
}

extern "C" int rb_attn_fwd(const void* q, const void* k, const void* v, void* out, float* lse, const int* cu_seqlens,
                           int64_t q_ld, int64_t k_ld, int64_t v_ld, int64_t out_ld, int T, int B, int nq, int nkv, int hd,
                           int max_seqlen, float scale, int causal, int dt, cudaStream_t s) {
  return rb_attn_fwd_window(q, k, v, out, lse, cu_seqlens, q_ld, k_ld, v_ld, out_ld, T, B, nq, nkv, hd, max_seqlen, scale, causal, 0, dt, s);
}

// Window attention with a sink on the tensor cores (see the kSink notes at the top): q / k [T, heads, hd], v [T, heads, vd] as for
// rb_attn_fwd (head sizes of 64 or 128), temp / sink [nq] in the operand type or null, gate logits at gate[t * gate_ld + h] (gate_mode
// 1) or gate[t * gate_ld + h * vd + c] (gate_mode 2) or null, window <= 0 = every earlier key, keep = first keys that stay visible,
// chunk > 0 = chunked instead of windowed, softcap > 0 = capped scores (kSimple cases only), slope_base < 0 = no distance term, bias
// [nq, n_bias] fp32 or null.  kv_shared: the values are the keys (v is not read).  hd != vd takes the kSimple cases; returns a negative
// code for what it does not take.
extern "C" int rb_attn_fwd_sink(const void* q, const void* k, const void* v, void* out, const int* cu_seqlens, int64_t q_ld, int64_t k_ld,
                                int64_t v_ld, int64_t out_ld, int T, int B, int nq, int nkv, int hd, int vd, int max_seqlen, float scale, int window,
                                int keep, const void* temp, const void* sink, const void* gate, int64_t gate_ld, int gate_mode, int chunk,
                                float softcap, float slope_base, const float* bias, int n_bias, int kv_shared, int dt, int vshare, cudaStream_t s) {
  if ((hd != 128 && hd != 64) || (vd != 128 && vd != 64)) return -1;
  if (dt != 1 && dt != 2) return -2;
  if (nq % nkv != 0 || T <= 0 || B <= 0 || max_seqlen <= 0 || vshare < 1 || nkv % vshare) return -3;
  if (kv_shared) { v = k; v_ld = k_ld; if (hd != vd || vshare != 1) return -3; }
  if ((q_ld | k_ld | v_ld | out_ld) % 8 != 0) return -4;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)out) & 15) return -5;
  if (gate != nullptr && gate_mode == 2 && (gate_ld % 8 != 0 || ((uintptr_t)gate & 15))) return -6;
  const bool plain_mask = slope_base < 0.f && (window <= 0 || keep == 0);
  const bool simple = plain_mask && temp == nullptr && scale > 0.f && bias == nullptr;
  if (softcap > 0.f && !simple) return -7;
  if (chunk > 0 && window > 0) return -8;
  if (bias != nullptr && (!plain_mask || n_bias < 1 || hd != vd)) return -9;
  if (hd != vd && (!simple || softcap > 0.f)) return -9;
  CUtensorMap mq, mk, mv;
  const int bf = dt == 1;
  if (!make_tmap(&mq, q, bf, T, (uint64_t)nq * hd, q_ld, 64, kBQ)) return -10;
  if (!make_tmap(&mk, k, bf, T, (uint64_t)nkv * hd, k_ld, 64, kBKV)) return -11;
  if (!make_tmap(&mv, v, bf, T, (uint64_t)(nkv / vshare) * vd, v_ld, 64, 64)) return -12;
  AttnParams p{cu_seqlens, out, nullptr, out_ld, T, nq, nkv, scale, 1, window > 0 ? window : 0, window > 0 ? keep : 0, temp, sink, gate, gate_ld,
               slope_base, vshare, gate_mode, chunk, softcap, bias, window > 0 && n_bias > window ? window : n_bias, n_bias};
#define RB_GO2(HD, VD, ...)                                                                                               \
  return bf ? launch_attn_fwd<HD, VD, __nv_bfloat16, 1, true, __VA_ARGS__>(mq, mk, mv, p, B, max_seqlen, s)              \
            : launch_attn_fwd<HD, VD, __half, 0, true, __VA_ARGS__>(mq, mk, mv, p, B, max_seqlen, s)
#define RB_GO(...)                                 \
  if (hd == 128) { RB_GO2(128, 128, __VA_ARGS__); } \
  RB_GO2(64, 64, __VA_ARGS__)
  if (hd != vd) {
    if (hd == 128) { RB_GO2(128, 64, false, true); }
    RB_GO2(64, 128, false, true);
  }
  if (bias != nullptr && kv_shared) { RB_GO(false, false, true, true); }
  if (bias != nullptr) { RB_GO(false, false, true); }
  if (softcap > 0.f) { RB_GO(true, true); }
  if (simple) { RB_GO(false, true); }
  RB_GO(false, false);
#undef RB_GO
#undef RB_GO2
}
