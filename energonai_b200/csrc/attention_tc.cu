// Prompt-pass attention on the 5th-generation tensor cores (tcgen05 + TMEM + TMA).
//
//   out[b,i,h,:] = softmax_j( scale * q[b,i,h,:].k[b,j,h,:] + mask[b,j] ; causal ) . v[b,j,h,:]
// (energonai/model/attention.py:105-124, without materialising the score tensor).
//
// One CTA owns 128 query rows of one (sequence, head) and walks the visible keys in tiles of
// 128.  Both products run on tcgen05.mma with fp32 accumulators in tensor memory:
//   S  = Q . K_tile^T    (128 x 128, K = head_dim)   TMEM columns [t*128, +128) for row tile t
//   O += P . V_tile      (128 x head_dim, K = 128)    TMEM columns [256 + t*128, +head_dim)
// Q, K and V tiles arrive by TMA (3-D maps over the [batch][row][head*dim] views, 128-byte
// swizzle, rows beyond the sequence read as zeros).  V is used as it lies in memory: for the
// second product the contraction index (keys) runs down the rows of the tile, which the shared-
// memory descriptor expresses as an N-major B operand, so nothing is transposed.
// A CTA serves two row tiles (256 query rows; with query heads of 192 one).  Warp roles (320 threads): warp 0 issues
// TMA, warp 1 issues the MMAs, warps 2-5 and 6-9 are the softmax of row tile 0 and 1: thread r
// owns query row r, reads its score row from TMEM (tcgen05.ld), keeps the running maximum / sum
// (fp32, log2 domain) and writes the probabilities as the 16-bit, swizzled A operand of the second
// product into shared memory.  The output row accumulates in TMEM across the key tiles (the
// second product adds to it).  Its scale is the maximum the row had when it was last rescaled:
// only when a new tile raises the row maximum by more than 2^8 do the softmax warps read the row
// back, multiply it and store it again (tcgen05.ld / st), so that in the common case they never
// wait for the second product and the probabilities stay below 2^8 (fine in fp16 and bf16, the
// sum is fp32).  The two row tiles alternate on the tensor core: while the softmax warps of one
// work on their scores, it serves the other.
//
// Query heads may share a key / value head in groups.  A biased form takes r1 ln(1 + r2 distance) off
// every score, read from a table per head (a row's 32 scores of a chunk are 32 consecutive entries, the
// lanes of a warp one entry apart: loads that coalesce, where a logarithm per score would double the
// work of the special-function unit), and may add one to the softmax denominator (a sink of score 0).
//
// A sliding window (row i sees only the `window` keys up to its own position) shortens the range of
// key tiles a row tile walks and hides the leading keys of its first tiles; nothing else changes.  Chunks
// (a row sees only its own chunk of so many positions, counted from the sequence's first row behind the
// padding) do the same with another lower bound, and a number per head may join the softmax as a
// score without a value.
//
// The capped form bounds scores by cap tanh(score / cap) and takes slope * distance off; a window may keep the
// first positions of a sequence visible, whose key tiles then come first in the walk of both row tiles (they
// are numbered as if they lay right in front of the window's first tile).  While no score of 32 keys is
// above 0.35 cap, tanh is its Taylor series (five terms leave 1e-7 of the argument); otherwise it takes an
// exponential and a reciprocal.  The output may be multiplied by the sigmoid of a gate.
//
// Every mbarrier wait is bounded; a wait that runs out is recorded, the CTA's roles leave (each
// decision made uniform over the warp first), copies in flight are given time to land, TMEM is
// freed and the kernel returns.
#include <type_traits>

#include "tc_ops.cuh"

namespace eb {
namespace {

// (kRows of tc_ops.cuh: query rows per row tile)
constexpr int kKeys = 128;                 // keys per tile
constexpr int kMaxTiles = 2;

// Shared-memory plan per head size.  With head_dim 128 everything but a second V stage fits, with 192 one row tile does.
template <int D, int DV> struct TcSmem {
  static constexpr int kTiles = D > 128 ? 1 : kMaxTiles;       // row tiles per CTA, each with its own four softmax warps
  static constexpr int kThreads = 64 + kTiles * 128;
  static constexpr uint32_t kQBytes = (D / 64) * kRows * 128, kKBytes = (D / 64) * kKeys * 128, kVBytes = (DV / 64) * kKeys * 128,
                            kPBytes = 2 * kRows * 128;
  static constexpr int kVStages = DV > 64 ? 1 : 2;
  static constexpr size_t kTotal = 1024 + 1024 + (size_t)kTiles * kQBytes + 2 * kKBytes + (size_t)kVStages * kVBytes + (size_t)kTiles * kPBytes;
};
constexpr float kLog2eTc = 1.4426950408889634f;
// From this distance on r1 log2(1 + r2 d) is interpolated between d, d - 16 and d - 32: the third derivative
// is at most 2 r1 / (ln 2 d^3), so the parabola is off by less than 1e-5 r1.
constexpr int kFarKeys = 512;
constexpr float kSmallTanh = 0.35f;        // below this argument the capped form takes the series
constexpr float kRescaleLog2 = 8.f;         // the accumulated row is rescaled when its maximum grows by more than 2^8

struct TcParams {
  int B, H, Sq, Sk, causal;
  int window;                              // > 0: row i sees keys j with i - j < window only (causal)
  int group;                               // query heads per key / value head
  const float *bias;                       // biased form: [H][bias_ld], r1 * log2(1 + r2 * distance)
  long long bias_ld;
  int sink;
  const float *sinks;                      // plain form: per head, a score without a value (null: none)
  int chunk;                               // > 0: row i sees only the keys of its chunk, counted from `first`
  const int *first;                        // [B] padding rows in front of each sequence (they see themselves), or null
  int keep;                                // capped form: so many positions from `first` on stay visible behind the window
  const float *slopes;                     // ... slopes[h] * distance is taken off, or null
  float cap_log2, cap_scale;               // ... cap * log2(e) and scale / cap (0: no cap)
  const void *gate;                        // output times sigmoid(gate), laid out like it with strides of its own, or null
  long long g_bs, g_rs;
  int mask_vec;                            // mask rows start on 16-byte boundaries
  float scale_log2;                        // scale * log2(e)
  const void *mask;                        // additive [B][>= Sk] in T, or null
  long long mask_bs;
  void *o;
  long long o_bs, o_rs;
};

// ---- the attention kernel ----------------------------------------------------------------------
// Shared memory (1024-aligned): [1 KB barriers, TMEM slot, abort flag][Q: 2 row tiles x D/64
// sub-tiles of 128 rows x 128 B][K ring: 2 x D/64 sub-tiles][V ring: kVStages x D/64 sub-tiles
// of 128 key rows x 128 B][P: 2 row tiles x 2 sub-tiles of 128 rows x 128 B].
enum { kFormPlain, kFormBias, kFormCapped };

// tanh(z) / z for |z| <= kSmallTanh, two at a time, w = z^2
__device__ __forceinline__ void tanh_series(float &p0, float &p1, float w0, float w1) {
  constexpr float c4 = 62.f / 2835.f, c3 = -17.f / 315.f, c2 = 2.f / 15.f, c1 = -1.f / 3.f;
  fma2(p0, p1, w0, w1, c4, c4, c3, c3);
  fma2(p0, p1, p0, p1, w0, w1, c2, c2);
  fma2(p0, p1, p0, p1, w0, w1, c1, c1);
  fma2(p0, p1, p0, p1, w0, w1, 1.f, 1.f);
}
__device__ __forceinline__ float tanh_exp(float z) { return 1.f - __fdividef(2.f, 1.f + ex2(z * (2.f * kLog2eTc))); }

template <typename T, int D, int DV, int FORM>
__global__ void __launch_bounds__(TcSmem<D, DV>::kThreads, 1)
attention_prefill_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                            const __grid_constant__ CUtensorMap tm_v, const TcParams p) {
  constexpr bool BIAS = FORM == kFormBias, CAPPED = FORM == kFormCapped;
  constexpr int kSub = D / 64, kSubV = DV / 64;                  // 64-column sub-tiles of Q / K and V
  using Smem = TcSmem<D, DV>;
  constexpr int kVStages = Smem::kVStages, kTiles = Smem::kTiles;
  constexpr uint32_t kQBytes = Smem::kQBytes, kKBytes = Smem::kKBytes, kVBytes = Smem::kVBytes, kPBytes = Smem::kPBytes;
  constexpr uint32_t kTmemCols = 512, kPvCol = 2 * kKeys;
  constexpr int kBf16 = std::is_same<T, __nv_bfloat16>::value ? 1 : 0;
  constexpr uint32_t kIdescS = tc_idesc(kKeys, kBf16), kIdescPV = tc_idesc(DV, kBf16) | (1u << 16);   // bit 16: B is N-major

  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = s32(smem_raw);
  uint8_t *smem = smem_raw + (((raw + 1023u) & ~1023u) - raw);
  uint64_t *bars = reinterpret_cast<uint64_t *>(smem);
  const uint32_t bar0 = s32(bars);
  // per-ring barriers are indexed by stage, per-row-tile barriers by tile (8 bytes apart)
  const uint32_t q_full = bar0, k_full = bar0 + 8, k_empty = bar0 + 24, v_full = bar0 + 40, v_empty = bar0 + 56,
                 s_full = bar0 + 72, p_full = bar0 + 88, pv_full = bar0 + 104;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + 256);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(smem + 264);
  const uint32_t q_addr = s32(smem) + 1024, k_addr = q_addr + kTiles * kQBytes, v_addr = k_addr + 2 * kKBytes,
                 p_addr = v_addr + kVStages * kVBytes;
  uint8_t *p_ptr = smem + 1024 + kTiles * kQBytes + 2 * kKBytes + kVStages * kVBytes;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qb = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, hk = h / p.group, b = blockIdx.z;   // longest (latest, under the causal mask) blocks first
  const int q0 = qb * (kTiles * kRows), shift = p.Sk - p.Sq;
  if (p.first) griddep_wait();
  const int first = p.first ? p.first[b] : 0;
  // first key that the row at position i sees
  auto seen_from = [&](int i) {
    if (!CAPPED && p.window > 0) return i - p.window + 1;
    const int f = min(first, max(i, 0));
    if (CAPPED) return p.window > 0 ? max(f, i - p.window + 1) : f;
    return p.chunk > 0 && i > f ? f + (i - f) / p.chunk * p.chunk : f;
  };
  // key tiles each row tile walks: all of them, or up to its last row's diagonal; none for a
  // row tile that lies wholly behind the end of the sequence
  // With a window a row tile starts at the first key its first row sees: tiles [ks[t], nt[t]) of
  // the CTA's [jmin, nmax).  (The ranges of the two row tiles rise together and leave no gap.)
  int nt[kTiles], ks[kTiles], nmax = 0, jmin = 0x7fffffff;
#pragma unroll
  for (int t = 0; t < kTiles; ++t) {
    const int qt0 = q0 + t * kRows;
    const int last_key = p.causal ? min(p.Sk - 1, qt0 + kRows - 1 + shift) : p.Sk - 1;
    nt[t] = (qt0 < p.Sq && last_key >= 0) ? last_key / kKeys + 1 : 0;
    ks[t] = max(0, seen_from(qt0 + shift)) / kKeys;
    if (nt[t] > 0) jmin = min(jmin, ks[t]);
    nmax = max(nmax, nt[t]);
  }
  if (jmin > nmax) jmin = nmax;
  // tiles with kept positions in front of the window, numbered [jmin, jwin)
  const int jwin = jmin, kept_tile = first / kKeys;
  if (CAPPED && p.keep > 0 && p.window > 0 && nmax > 0) {
    const int kept = min((min(first + p.keep, p.Sk) - 1) / kKeys + 1, jmin) - kept_tile;
    jmin -= max(kept, 0);
#pragma unroll
    for (int t = 0; t < kTiles; ++t) ks[t] = jmin;
  }
  auto tile_of = [&](int j) { return CAPPED && j < jwin ? kept_tile + j - jmin : j; };

  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_k) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_v) : "memory");
    bar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      bar_init(k_full + 8 * s, 1);
      bar_init(k_empty + 8 * s, 1);
      bar_init(v_full + 8 * s, 1);
      bar_init(v_empty + 8 * s, 1);
      bar_init(s_full + 8 * s, 1);
      bar_init(p_full + 8 * s, 4);
      bar_init(pv_full + 8 * s, 1);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    __syncwarp();
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(s32(tmem_slot)), "r"(kTmemCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  griddep_launch();
  griddep_wait();

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0 && nmax > 0) {
      bar_expect_tx(q_full, kTiles * kQBytes);
#pragma unroll
      for (int t = 0; t < kTiles; ++t)
#pragma unroll
        for (int kb = 0; kb < kSub; ++kb)
          tma_load_3d(q_addr + t * kQBytes + kb * kRows * 128, &tm_q, q_full, h * D + kb * 64, q0 + t * kRows, b);
      // K runs one tile ahead of V: its stage is released earlier (after the scores, not after
      // the value product), and the next scores are what the softmax warps wait for
      auto load_k = [&](int j) -> bool {
        const int i = j - jmin, st = i & 1;
        if (i >= 2 && !bar_wait(k_empty + 8 * st, ((i >> 1) - 1) & 1, abort_flag, 1)) return false;
        bar_expect_tx(k_full + 8 * st, kKBytes);
#pragma unroll
        for (int kb = 0; kb < kSub; ++kb)
          tma_load_3d(k_addr + st * kKBytes + kb * kKeys * 128, &tm_k, k_full + 8 * st, hk * D + kb * 64, tile_of(j) * kKeys, b);
        return true;
      };
      bool ok = load_k(jmin);
      for (int j = jmin; j < nmax && ok; ++j) {
        const int i = j - jmin, vs = i % kVStages, vu = i / kVStages;
        if (j + 1 < nmax && !load_k(j + 1)) break;
        if (i >= kVStages && !bar_wait(v_empty + 8 * vs, (vu - 1) & 1, abort_flag, 9)) break;
        bar_expect_tx(v_full + 8 * vs, kVBytes);
#pragma unroll
        for (int kb = 0; kb < kSubV; ++kb)
          tma_load_3d(v_addr + vs * kVBytes + kb * kKeys * 128, &tm_v, v_full + 8 * vs, hk * DV + kb * 64, tile_of(j) * kKeys, b);
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    // Per row tile the order is S(0), then for every key tile j, as soon as P(j) is written
    // (which also says that S(j) has been read): S(j+1) first, so the softmax warps get their
    // next scores as early as possible, then O += P(j) . V(j).
    if (lane == 0 && nmax > 0) {
      // (with a window, the second row tile joins at key tile ks[1]: its first scores are issued in
      // the round before, behind those of the first row tile)
      auto last_reader = [&](int j) { return (kTiles > 1 && j >= ks[kTiles - 1] && j < nt[kTiles - 1]) ? kTiles - 1 : 0; };
      auto issue_scores = [&](int t, int j) -> bool {
        const int st = (j - jmin) & 1;
        if (!bar_wait(k_full + 8 * st, ((j - jmin) >> 1) & 1, abort_flag, 3)) return false;
        tc_fence_after();
#pragma unroll
        for (int kb = 0; kb < kSub; ++kb) {
          const uint64_t a = tc_desc(q_addr + t * kQBytes + kb * kRows * 128), bd = tc_desc(k_addr + st * kKBytes + kb * kKeys * 128);
#pragma unroll
          for (int k = 0; k < 4; ++k) tc_mma(tmem + t * kKeys, a + 2 * k, bd + 2 * k, kIdescS, (kb > 0 || k > 0) ? 1u : 0u);
        }
        tc_commit(s_full + 8 * t);
        if (t == last_reader(j)) tc_commit(k_empty + 8 * st);
        return true;
      };
      bool ok = bar_wait(q_full, 0, abort_flag, 2);
      for (int t = 0; t < kTiles && ok; ++t)
        if (nt[t] > 0 && ks[t] == jmin) ok = issue_scores(t, jmin);
      for (int j = jmin; j < nmax && ok; ++j) {
        const int vs = (j - jmin) % kVStages, vu = (j - jmin) / kVStages;
        for (int t = 0; t < kTiles && ok; ++t) {
          if (nt[t] > 0 && ks[t] == j + 1) ok = issue_scores(t, j + 1);
          if (j < ks[t] || j >= nt[t]) continue;
          ok = ok && bar_wait(p_full + 8 * t, (j - ks[t]) & 1, abort_flag, 5);
          if (ok && j + 1 < nt[t]) ok = issue_scores(t, j + 1);
          ok = ok && bar_wait(v_full + 8 * vs, vu & 1, abort_flag, 10);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int a2 = 0; a2 < 2; ++a2) {
            const uint64_t a = tc_desc(p_addr + t * kPBytes + a2 * kRows * 128);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              // 16 keys per instruction: two 8-row groups (2048 bytes) down the V tile
              const uint64_t bd = tc_desc_nmajor(v_addr + vs * kVBytes + (a2 * 4 + k) * 2048, kKeys * 128);
              tc_mma(tmem + kPvCol + t * kKeys, a + 2 * k, bd, kIdescPV, (j > ks[t] || a2 > 0 || k > 0) ? 1u : 0u);
            }
          }
          tc_commit(pv_full + 8 * t);
          if (t == last_reader(j)) tc_commit(v_empty + 8 * vs);
        }
      }
    }
  } else {
    // ---------------- softmax warps: 4 per row tile, thread = query row ----------------
    const int t = (warp - 2) >> 2, quarter = warp & 3, row = quarter * 32 + lane, qi = q0 + t * kRows + row;
    const int ntiles = nt[t], first_tile = ks[t];
    const uint32_t t_s = tmem + ((uint32_t)(quarter * 32) << 16) + t * kKeys, t_pv = t_s + kPvCol;
    const uint32_t my_s_full = s_full + 8 * t, my_p_full = p_full + 8 * t, my_pv_full = pv_full + 8 * t;
    uint8_t *p_row = p_ptr + t * kPBytes + row * 128;
    const T *mrow = p.mask ? reinterpret_cast<const T *>(p.mask) + (long long)b * p.mask_bs : nullptr;
    const int vis_end = p.causal ? min(p.Sk, qi + shift + 1) : p.Sk;               // keys [0, vis_end) are visible to this row
    const int vis_begin = CAPPED ? max(first, seen_from(qi + shift)) : seen_from(qi + shift);      // ... from this key on
    const int kept_end = CAPPED ? first + p.keep : 0;                              // (capped: and [first, kept_end))
    // m_ref: the maximum the accumulated row and l_run are scaled by (a sink is a score of 0 seen already)
    const bool zero_sink = (BIAS || CAPPED) && p.sink;
    float m_ref = zero_sink ? 0.f : -1e30f, l_run = zero_sink ? 1.f : 0.f;
    if (!BIAS && p.sinks) {
      m_ref = p.sinks[h] * kLog2eTc;
      l_run = 1.f;
    }
    // A bias that only lowers scores need not enter the maximum: any reference that is not below the
    // largest score will do as long as the probabilities keep their precision, which bf16 does over its
    // whole range.  fp16 does not, and a negative r1 raises scores: there the maximum includes it.
    const float *bias = BIAS ? p.bias + (long long)h * p.bias_ld : nullptr;
    const bool bias_in_max = BIAS && (!kBf16 || bias[1] < 0.f);
    const float slope = CAPPED && p.slopes ? p.slopes[h] * kLog2eTc : 0.f;
    // capped score of a raw product without the bias, in the log2 domain
    auto capped = [&](float x) { return p.cap_scale > 0.f ? p.cap_log2 * tanh_exp(x * p.cap_scale) : x * p.scale_log2; };
    bool alive = ntiles > 0;
    for (int j = first_tile; j < ntiles && alive; ++j) {
      const int key0 = tile_of(j) * kKeys;
      // Work per chunk of 32 keys, decided for the warp as a whole (tensor-memory loads are
      // warp-wide): 0 = hidden from every row of the warp (behind the diagonal or the end of the
      // sequence): nothing to read, P = 0; 1 = visible to every row and no mask value set: one
      // multiply-add and one exponential per key, most chunks of a long prompt; 2 = per-key
      // work (the chunk the diagonal crosses, chunks with mask values).  Lane l keeps the mask
      // value of key l of each chunk, in the log2 domain.
      // (The biased form keeps its chunk loops rolled: unrolled, its body outgrew the instruction cache,
      // which was the largest stall.  So it packs the classes and reads mask values again.)
      int cls[kKeys / 32];
      float mval[kKeys / 32];
      uint32_t classes = 0, small = 0;              // (small: bit c, the series serves chunk c)
#pragma unroll
      for (int c = 0; c < kKeys / 32; ++c) {
        const int kb = key0 + c * 32;
        float mv = 0.f;
        if (mrow && kb + lane < p.Sk) mv = to_f32<T>(mrow[kb + lane]) * kLog2eTc;
        mval[c] = mv;
        const bool unkept = !CAPPED || kb >= kept_end || kb + 32 <= first, kept = CAPPED && kb >= first && kb + 32 <= min(kept_end, vis_end);
        const bool hidden = __all_sync(0xffffffffu, kb >= vis_end || (kb + 32 <= vis_begin && unkept));
        const bool simple = __all_sync(0xffffffffu, ((kb >= vis_begin && kb + 32 <= vis_end) || kept) && mv == 0.f);
        cls[c] = hidden ? 0 : (simple ? 1 : 2);
        if (BIAS || CAPPED) classes |= (uint32_t)cls[c] << (2 * c);
      }
      auto mask_value = [&](int c) { return mrow && key0 + c * 32 + lane < p.Sk ? to_f32<T>(mrow[key0 + c * 32 + lane]) * kLog2eTc : 0.f; };
      if (!__all_sync(0xffffffffu, bar_wait(my_s_full, (j - first_tile) & 1, abort_flag, 7))) { alive = false; break; }
      tc_fence_after();
      // pass 1: the row maximum of this tile (log2 domain, masks applied)
      float r0 = -INFINITY, r1 = -INFINITY, r2 = -INFINITY, r3 = -INFINITY, m_tile = -1e30f;
      auto maximum = [&](int c, int kind, float mv) {
        if (kind == 0) return;
        float x[32];
        tc_ld32(t_s + c * 32, x);
        const int gap = qi + shift - (key0 + c * 32);                 // distance to the chunk's first key
        if (kind == 1 && bias_in_max) {
#pragma unroll
          for (int e = 0; e < 32; ++e) m_tile = fmaxf(m_tile, fmaf(x[e], p.scale_log2, -__ldg(bias + gap - e)));
        } else if (kind == 1) {
#pragma unroll
          for (int e = 0; e < 32; e += 4) {
            r0 = fmaxf(r0, x[e]);
            r1 = fmaxf(r1, x[e + 1]);
            r2 = fmaxf(r2, x[e + 2]);
            r3 = fmaxf(r3, x[e + 3]);
          }
        } else {
          const int nvis = vis_end - (key0 + c * 32), n0 = vis_begin - (key0 + c * 32);
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            float v = fmaf(x[e], p.scale_log2, __shfl_sync(0xffffffffu, mv, e));
            if (bias_in_max) v -= __ldg(bias + max(0, gap - e));
            m_tile = fmaxf(m_tile, e < nvis && e >= n0 ? v : -INFINITY);
          }
        }
      };
      // the largest capped score of a chunk, less the bias of its nearest key: an upper bound that is at most 31 slopes
      // (or, with the series, twice its range) too high, which the range of bf16 and fp32 takes
      auto visible = [&](int key) { return key < vis_end && (key >= vis_begin || (key >= first && key < kept_end)); };
      auto bound = [&](int c, int kind) {
        if (kind == 0) return;
        float x[32], top = -INFINITY, big = 0.f;
        tc_ld32(t_s + c * 32, x);
        const int kb = key0 + c * 32;
        if (kind == 1) {
#pragma unroll
          for (int e = 0; e < 32; ++e) big = fmaxf(big, fabsf(x[e]));
          if (__all_sync(0xffffffffu, big * p.cap_scale <= kSmallTanh)) {
            small |= 1u << c;
            top = big;
          } else {
#pragma unroll
            for (int e = 0; e < 32; ++e) top = fmaxf(top, x[e]);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e) top = fmaxf(top, visible(kb + e) ? x[e] : -INFINITY);
        }
        if (kBf16) {
          if (top > -INFINITY) m_tile = fmaxf(m_tile, ((small >> c) & 1 ? top * p.scale_log2 : capped(top)) - slope * (float)max(0, qi + shift - kb - 31));
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (kind == 1 || visible(kb + e)) m_tile = fmaxf(m_tile, capped(x[e]) - slope * (float)(qi + shift - kb - e));
        }
      };
      if constexpr (CAPPED) {
#pragma unroll 1
        for (int c = 0; c < kKeys / 32; ++c) bound(c, (classes >> (2 * c)) & 3);
      } else if constexpr (BIAS) {
#pragma unroll 1
        for (int c = 0; c < kKeys / 32; ++c) maximum(c, (classes >> (2 * c)) & 3, mask_value(c));
      } else {
#pragma unroll
        for (int c = 0; c < kKeys / 32; ++c) maximum(c, cls[c], mval[c]);
      }
      r0 = fmaxf(fmaxf(r0, r1), fmaxf(r2, r3));
      if (r0 > -INFINITY) m_tile = fmaxf(m_tile, r0 * p.scale_log2);   // the scale is positive: the maximum commutes with it
      // The previous tile's value product must be complete before P is overwritten (it reads P)
      // and before the accumulated row is rescaled; it was issued right behind the scores just
      // read, so this wait is normally over already.
      if (j > first_tile && !__all_sync(0xffffffffu, bar_wait(my_pv_full, (j - 1 - first_tile) & 1, abort_flag, 8))) { alive = false; break; }
      // rescale only when some row of the warp gained more than 2^8 (the loads and stores of
      // tensor memory are warp-wide, so the warp decides together)
      if (__any_sync(0xffffffffu, m_tile > m_ref + kRescaleLog2)) {
        const float m_new = fmaxf(m_ref, m_tile);
        const float alpha = ex2(m_ref - m_new);
        m_ref = m_new;
        l_run *= alpha;
        if (j > first_tile) {
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < DV / 32; ++c) {
            float x[32];
            tc_ld32(t_pv + c * 32, x);
#pragma unroll
            for (int e = 0; e < 32; ++e) x[e] *= alpha;
            tc_st32(t_pv + c * 32, x);
          }
          tc_st_wait();
        }
      }
      // pass 2: probabilities -> the 16-bit A operand of the second product (swizzled rows of 128 bytes)
      float l0 = 0.f, l1 = 0.f;
      const float neg_m = -m_ref;
      auto weights = [&](int c, int kind, float mv) {
        uint8_t *dst = p_row + (c >> 1) * (kRows * 128);
        if (kind == 0) {
#pragma unroll
          for (int g = 0; g < 4; ++g) *reinterpret_cast<uint4 *>(dst + ((((c & 1) * 4 + g) ^ (row & 7)) << 4)) = make_uint4(0, 0, 0, 0);
          return;
        }
        float x[32];
        tc_ld32(t_s + c * 32, x);
        const int gap = qi + shift - (key0 + c * 32);
        if (CAPPED) {
          const int kb = key0 + c * 32;
          const float base = neg_m - slope * (float)(qi + shift - kb);
          if ((small >> c) & 1) {
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              float z0, z1, p0, p1, b0, b1;
              mul2(z0, z1, x[e], x[e + 1], p.cap_scale, p.cap_scale);
              mul2(z0, z1, z0, z1, z0, z1);
              tanh_series(p0, p1, z0, z1);
              mul2(x[e], x[e + 1], x[e], x[e + 1], p.scale_log2, p.scale_log2);
              fma2(b0, b1, (float)e, (float)(e + 1), slope, slope, base, base);
              fma2(x[e], x[e + 1], x[e], x[e + 1], p0, p1, b0, b1);
            }
#pragma unroll
            for (int e = 0; e < 32; ++e) x[e] = ex2(x[e]);
          } else {
#pragma unroll
            for (int e = 0; e < 32; ++e) {
              const float v = ex2(capped(x[e]) + fmaf((float)e, slope, base));
              x[e] = kind == 1 || visible(kb + e) ? v : 0.f;
            }
          }
        } else if (kind == 1 && BIAS) {
          // far from the diagonal the bias of a chunk's 32 keys is a parabola through three of them
          if (q0 + t * kRows + quarter * 32 + shift - (key0 + c * 32) - 32 >= kFarKeys) {
            const float b0 = __ldg(bias + gap), b1 = __ldg(bias + gap - 16), b2 = __ldg(bias + gap - 32);
            const float c0 = neg_m - b0, c1 = (3.f * b0 + b2 - 4.f * b1) * (1.f / 32.f), c2 = (2.f * b1 - b0 - b2) * (1.f / 512.f);
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              float s0, s1;
              fma2(s0, s1, (float)e, (float)(e + 1), c2, c2, c1, c1);
              fma2(s0, s1, s0, s1, (float)e, (float)(e + 1), c0, c0);
              fma2(x[e], x[e + 1], x[e], x[e + 1], p.scale_log2, p.scale_log2, s0, s1);
            }
          } else {
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              float s0, s1;
              add2(s0, s1, neg_m, neg_m, -__ldg(bias + gap - e), -__ldg(bias + gap - e - 1));
              fma2(x[e], x[e + 1], x[e], x[e + 1], p.scale_log2, p.scale_log2, s0, s1);
            }
          }
#pragma unroll
          for (int e = 0; e < 32; ++e) x[e] = ex2(x[e]);
        } else if (kind == 1) {
#pragma unroll
          for (int e = 0; e < 32; ++e) x[e] = ex2(fmaf(x[e], p.scale_log2, neg_m));
        } else {
          const int nvis = vis_end - (key0 + c * 32), n0 = vis_begin - (key0 + c * 32);
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            float v = fmaf(x[e], p.scale_log2, __shfl_sync(0xffffffffu, mv, e));
            if (BIAS) v -= __ldg(bias + max(0, gap - e));
            x[e] = e < nvis && e >= n0 ? ex2(v + neg_m) : 0.f;
          }
        }
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint4 w;
          w.x = pack2<T>(x[g * 8 + 0], x[g * 8 + 1]);
          w.y = pack2<T>(x[g * 8 + 2], x[g * 8 + 3]);
          w.z = pack2<T>(x[g * 8 + 4], x[g * 8 + 5]);
          w.w = pack2<T>(x[g * 8 + 6], x[g * 8 + 7]);
#pragma unroll
          for (int e = 0; e < 8; e += 2) {
            l0 += x[g * 8 + e];
            l1 += x[g * 8 + e + 1];
          }
          *reinterpret_cast<uint4 *>(dst + ((((c & 1) * 4 + g) ^ (row & 7)) << 4)) = w;
        }
      };
      if constexpr (BIAS || CAPPED) {
#pragma unroll 1
        for (int c = 0; c < kKeys / 32; ++c) weights(c, (classes >> (2 * c)) & 3, mask_value(c));
      } else {
#pragma unroll
        for (int c = 0; c < kKeys / 32; ++c) weights(c, cls[c], mval[c]);
      }
      l_run += l0 + l1;
      // P is complete for this warp's 32 rows: make it visible to the tensor core's reads.  The
      // same arrival tells the issuer that S has been read and that the row has been rescaled.
      tc_fence_before();
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) bar_arrive(my_p_full);
    }
    if (alive && !__all_sync(0xffffffffu, bar_wait(my_pv_full, (ntiles - 1 - first_tile) & 1, abort_flag, 11))) alive = false;
    if (alive) {
      tc_fence_after();
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      T *orow = reinterpret_cast<T *>(p.o) + (long long)b * p.o_bs + (long long)qi * p.o_rs + h * DV;
      const T *grow = p.gate ? reinterpret_cast<const T *>(p.gate) + (long long)b * p.g_bs + (long long)qi * p.g_rs + h * DV : nullptr;
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        float x[32];
        tc_ld32(t_pv + c * 32, x);                 // warp-wide: rows behind the end of the sequence read too, and store nothing
        if (qi < p.Sq) {
          if (grow) {
#pragma unroll
            for (int g = 0; g < 4; ++g) {
              Vec16<T> w;
              float f[8];
              w.load(grow + c * 32 + g * 8);
              w.unpack(f);
#pragma unroll
              for (int e = 0; e < 8; ++e) x[g * 8 + e] = __fdividef(x[g * 8 + e], 1.f + ex2(-f[e] * kLog2eTc));
            }
          }
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            uint4 w;
            w.x = pack2<T>(x[g * 8 + 0] * inv, x[g * 8 + 1] * inv);
            w.y = pack2<T>(x[g * 8 + 2] * inv, x[g * 8 + 3] * inv);
            w.z = pack2<T>(x[g * 8 + 4] * inv, x[g * 8 + 5] * inv);
            w.w = pack2<T>(x[g * 8 + 6] * inv, x[g * 8 + 7] * inv);
            *reinterpret_cast<uint4 *>(orow + c * 32 + g * 8) = w;
          }
        }
      }
    }
  }

  // ---------------- teardown ----------------
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    const unsigned long long t0 = gtimer();
    while (gtimer() - t0 < 2000000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols) : "memory");
  }
}

// ---- host side ---------------------------------------------------------------------------------
// out[h][d] = r1[h] * log2(1 + r2[h] * d)
__global__ void distance_bias_kernel(const float *r1, const float *r2, int len, float *out) {
  griddep_wait();
  griddep_launch();
  const int d = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y;
  if (d < len) out[(long long)h * len + d] = r1[h] * log2f(fmaf(r2[h], (float)d, 1.f));
}

template <typename T, int D, int DV, int FORM>
int launch_tc(const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mv, const TcParams &p, cudaStream_t st) {
  constexpr size_t smem = TcSmem<D, DV>::kTotal;
  constexpr int kTiles = TcSmem<D, DV>::kTiles;
  static_assert(smem <= 227 * 1024, "shared memory");
  auto kern = attention_prefill_tc_kernel<T, D, DV, FORM>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "attention_prefill: cannot reserve %zu bytes of shared memory", smem);
    }
    configured[dev] = true;
  }
  dim3 grid((p.Sq + kTiles * kRows - 1) / (kTiles * kRows), p.H, p.B);
  launch_pdl(kern, grid, dim3(TcSmem<D, DV>::kThreads), smem, st, mq, mk, mv, p);
  return check_launch("attention_prefill");
}

}  // namespace

// Status words of this file's kernels, for eb_device_status.
int attention_tc_status(int *out4, bool clear) { return tc_status(out4, clear); }

}  // namespace eb

using namespace eb;

struct TcCapped {
  int keep;
  const float *slopes;
  float cap;
};

static int prefill_tc_impl(const void *q, const void *k, const void *v, void *out, const void *mask,
                                       long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                                       long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                       long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                                       int heads, int q_len, int kv_len, int head_dim, int causal, int window, float scale,
                                       int dtype, void *stream, int kv_group = 1, const float *bias = nullptr, long long bias_ld = 0,
                                       int sink = 0, const float *sinks = nullptr, int chunk = 0, const int32_t *first = nullptr,
                                       int v_dim = 0, const TcCapped *capped = nullptr, const void *gate = nullptr, long long g_batch_stride = 0,
                                       long long g_row_stride = 0) {
  if (batch == 0 || heads == 0 || q_len == 0) return EB_OK;
  EB_REQUIRE(dtype == EB_F16 || dtype == EB_BF16, "attention_prefill: fp16 or bf16 only (dtype %d)", dtype);
  if (v_dim == 0) v_dim = head_dim;
  const bool large = head_dim == 192 && v_dim != 192 && !capped && !bias;             // (plain form, with smaller value heads)
  EB_REQUIRE(head_dim == 64 || head_dim == 128 || large, "attention_prefill: head_dim %d not supported (64 or 128)", head_dim);
  EB_REQUIRE(v_dim == head_dim || (v_dim == 64 && !bias) || (large && v_dim == 128), "attention_prefill: value heads of %d not supported", v_dim);
  EB_REQUIRE(batch > 0 && heads > 0 && q_len > 0 && kv_len > 0, "attention_prefill: negative or zero size");
  EB_REQUIRE(heads <= 65535 && batch <= 65535, "attention_prefill: batch and heads are limited to 65535");
  EB_REQUIRE(q && k && v && out, "attention_prefill: null pointer");
  EB_REQUIRE(aligned16(q) && aligned16(k) && aligned16(v) && aligned16(out), "attention_prefill: pointers must be 16-byte aligned");
  const long long strides[] = {q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                               o_batch_stride, o_row_stride};
  for (long long s : strides) EB_REQUIRE(s % 8 == 0, "attention_prefill: strides must be multiples of 8 elements");
  EB_REQUIRE(kv_len >= q_len || !causal, "attention_prefill: causal attention needs kv_len >= q_len");
  EB_REQUIRE(scale > 0.f, "attention_prefill: the scale must be positive");
  EB_REQUIRE(window >= 0 && (window == 0 || causal), "attention_prefill: a window needs the causal mask");
  EB_REQUIRE(!capped || (capped->keep >= 0 && capped->cap >= 0.f && !mask && !bias && !chunk), "attention_prefill: bad capped form");
  EB_REQUIRE(!gate || (aligned16(gate) && g_batch_stride % 8 == 0 && g_row_stride % 8 == 0), "attention_prefill: the gate's rows start on 16-byte boundaries");
  cudaStream_t st = as_stream(stream);
  const long long hd = (long long)heads * head_dim, hkd = hd / kv_group, hvd = (long long)heads / kv_group * v_dim;
  CUtensorMap mq, mk, mv;
  int rc;
  if ((rc = tc_map3(&mv, v, dtype, hvd, kv_len, batch, v_row_stride, v_batch_stride, kKeys))) return rc;
  if ((rc = tc_map3(&mq, q, dtype, hd, q_len, batch, q_row_stride, q_batch_stride, kRows))) return rc;
  if ((rc = tc_map3(&mk, k, dtype, hkd, kv_len, batch, k_row_stride, k_batch_stride, kKeys))) return rc;
  TcParams p{};
  p.B = batch; p.H = heads; p.Sq = q_len; p.Sk = kv_len; p.causal = causal; p.window = window;
  p.scale_log2 = scale * kLog2eTc;
  p.mask = mask; p.mask_bs = mask_batch_stride;
  p.mask_vec = mask && aligned16(mask) && mask_batch_stride % 8 == 0;
  p.o = out; p.o_bs = o_batch_stride; p.o_rs = o_row_stride;
  p.group = kv_group; p.bias = bias; p.bias_ld = bias_ld; p.sink = sink;
  p.sinks = sinks; p.chunk = chunk; p.first = first;
  p.gate = gate; p.g_bs = g_batch_stride; p.g_rs = g_row_stride;
  if (capped) {
    p.keep = capped->keep; p.slopes = capped->slopes;
    p.cap_log2 = capped->cap * kLog2eTc; p.cap_scale = capped->cap > 0.f ? scale / capped->cap : 0.f;
  }
#define EB_TC(T, D, DV) (capped ? launch_tc<T, D, DV, kFormCapped>(mq, mk, mv, p, st) : launch_tc<T, D, DV, kFormPlain>(mq, mk, mv, p, st))
#define EB_TC_B(T, D) (bias ? launch_tc<T, D, D, kFormBias>(mq, mk, mv, p, st) : EB_TC(T, D, D))
  if (large) {
    if (v_dim == 64) return dtype == EB_F16 ? launch_tc<__half, 192, 64, kFormPlain>(mq, mk, mv, p, st) : launch_tc<__nv_bfloat16, 192, 64, kFormPlain>(mq, mk, mv, p, st);
    return dtype == EB_F16 ? launch_tc<__half, 192, 128, kFormPlain>(mq, mk, mv, p, st) : launch_tc<__nv_bfloat16, 192, 128, kFormPlain>(mq, mk, mv, p, st);
  }
  if (v_dim != head_dim) return dtype == EB_F16 ? EB_TC(__half, 128, 64) : EB_TC(__nv_bfloat16, 128, 64);
  if (dtype == EB_F16) return head_dim == 64 ? EB_TC_B(__half, 64) : EB_TC_B(__half, 128);
  return head_dim == 64 ? EB_TC_B(__nv_bfloat16, 64) : EB_TC_B(__nv_bfloat16, 128);
#undef EB_TC_B
#undef EB_TC
}

extern "C" int eb_attention_prefill_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                                       long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                                       long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                       long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                                       int heads, int q_len, int kv_len, int head_dim, int causal, float scale, int dtype,
                                       void *stream) {
  return prefill_tc_impl(q, k, v, out, mask, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, mask_batch_stride, batch, heads, q_len, kv_len, head_dim, causal, 0, scale, dtype,
                         stream);
}

extern "C" int eb_attention_prefill_window_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                                       long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                                       long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                       long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                                       int heads, int q_len, int kv_len, int head_dim, int window, float scale, int dtype,
                                       void *stream) {
  return prefill_tc_impl(q, k, v, out, mask, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, mask_batch_stride, batch, heads, q_len, kv_len, head_dim, 1, window, scale, dtype,
                         stream);
}

extern "C" int eb_distance_bias(const float *r1, const float *r2, int heads, int len, float *table, void *stream) {
  if (heads == 0 || len == 0) return EB_OK;
  EB_REQUIRE(r1 && r2 && table && heads > 0 && heads <= 65535 && len > 0, "distance_bias: bad arguments");
  launch_pdl(distance_bias_kernel, dim3((len + 255) / 256, heads), dim3(256), 0, as_stream(stream), r1, r2, len, table);
  return check_launch("distance_bias");
}

extern "C" int eb_attention_prefill_biased_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                                       long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                                       long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                       long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                                       int heads, int kv_group, int q_len, int kv_len, int head_dim, int window, const float *bias_table,
                                       int bias_len, int sink, float scale, int dtype, void *stream) {
  EB_REQUIRE(kv_group > 0 && heads % kv_group == 0, "attention_prefill: %d heads do not share keys in groups of %d", heads, kv_group);
  EB_REQUIRE(bias_table && bias_len >= kv_len + kMaxTiles * kRows, "attention_prefill: the bias table needs %d distances, has %d",
             kv_len + kMaxTiles * kRows, bias_len);
  return prefill_tc_impl(q, k, v, out, mask, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, mask_batch_stride, batch, heads, q_len, kv_len, head_dim, 1, window, scale, dtype,
                         stream, kv_group, bias_table, bias_len, sink);
}

extern "C" int eb_attention_prefill_chunk_tc(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                                       long long q_row_stride, long long k_batch_stride, long long k_row_stride,
                                       long long v_batch_stride, long long v_row_stride, long long o_batch_stride,
                                       long long o_row_stride, int batch, int heads, int kv_group, int len, int head_dim, int chunk,
                                       const int32_t *first, const float *sinks, float scale, int dtype, void *stream) {
  EB_REQUIRE(kv_group > 0 && heads % kv_group == 0, "attention_prefill: %d heads do not share keys in groups of %d", heads, kv_group);
  EB_REQUIRE(chunk >= 0, "attention_prefill: a chunk of %d positions", chunk);
  return prefill_tc_impl(q, k, v, out, nullptr, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, 0, batch, heads, len, len, head_dim, 1, 0, scale, dtype, stream, kv_group, nullptr, 0, 0,
                         sinks, chunk, first);
}

extern "C" int eb_attention_prefill_gated_tc(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                                       long long q_row_stride, long long k_batch_stride, long long k_row_stride, long long v_batch_stride,
                                       long long v_row_stride, long long o_batch_stride, long long o_row_stride, long long g_batch_stride,
                                       long long g_row_stride, int batch, int heads, int kv_group, int len, int k_dim, int v_dim,
                                       const int32_t *first, const float *sinks, float scale, int dtype, void *stream) {
  EB_REQUIRE(kv_group > 0 && heads % kv_group == 0, "attention_prefill: %d heads do not share keys in groups of %d", heads, kv_group);
  return prefill_tc_impl(q, k, v, out, nullptr, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, 0, batch, heads, len, len, k_dim, 1, 0, scale, dtype, stream, kv_group, nullptr, 0, 0,
                         sinks, 0, first, v_dim, nullptr, gate, g_batch_stride, g_row_stride);
}

extern "C" int eb_attention_prefill_capped_tc(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                                       long long q_row_stride, long long k_batch_stride, long long k_row_stride, long long v_batch_stride,
                                       long long v_row_stride, long long o_batch_stride, long long o_row_stride, long long g_batch_stride,
                                       long long g_row_stride, int batch, int heads, int kv_group, int len, int k_dim, int v_dim, int window,
                                       int keep, const int32_t *first, const float *slopes, float cap, int sink, float scale, int dtype,
                                       void *stream) {
  EB_REQUIRE(kv_group > 0 && heads % kv_group == 0, "attention_prefill: %d heads do not share keys in groups of %d", heads, kv_group);
  const TcCapped capped{keep, slopes, cap};
  return prefill_tc_impl(q, k, v, out, nullptr, q_batch_stride, q_row_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride,
                         o_batch_stride, o_row_stride, 0, batch, heads, len, len, k_dim, 1, window, scale, dtype, stream, kv_group, nullptr, 0, sink,
                         nullptr, 0, first, v_dim, &capped, gate, g_batch_stride, g_row_stride);
}
