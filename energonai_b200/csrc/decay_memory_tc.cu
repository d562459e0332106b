// Decaying memories of a prompt on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), 128 tokens at a time.
// With L_t the running sum of the log decays inside a chunk that begins with state S, the recurrences of
// eb_ssm_scan and eb_gla_scan unroll to
//
//   y_t = sum_{s <= t} p_ts v_s + exp(L_t) S^T q_t,      S' = exp(L_end) S + sum_s exp(L_end - L_s) k_s v_s^T
//
//   state space    L is one number per head:  p_ts = exp(L_t - L_s) dt_s (q_t.k_s), + skip where s = t;  q = C, k = B,
//                  dt goes with the value;  the products q.k are common to the heads of a group
//   gated linear   L is one number per key channel:  p_ts = sum_d exp(L_td - L_sd) q_td k_sd
//
// (every exponent is <= 0).  A CTA owns 128 value columns, those of one head or (state space, heads of 64) of two
// neighbouring heads of a group, and walks the chunks in order.  Products are 128-row tcgen05.mma with fp32
// accumulators in tensor memory:
//   A = Q K^T        [t][s]      state space only; P = weighted A goes to tensor memory as an operand
//   O = Q S, P V     [t][v]      S as a bf16 operand in shared memory.  Gated linear: one accumulator, exp(L_t) is part
//                                of Q; state space: Q S is read out and scaled while P V is computed
//   S += K^T V       [d][v]      one factor as bf16 hi + lo parts, so that what enters the state keeps 16 bits of
//                                mantissa: the value times exp(L_end - L_s) dt_s (state space; two heads then share
//                                one product), the key times exp(L_end - L_s) (gated linear)
// The state's fp32 master stays in tensor memory from chunk to chunk (lane = key channel); between two chunks
// it is decayed there and copied out as the next operand.
//
// For gated linear attention everything that needs no state is done beforehand by gla_prepare, in parallel over the
// chunks: P, Q exp(L_t), both parts of K exp(L_end - L_s), exp(L_end).  Its scores are products of operands
// (in two bf16 parts each) that carry the decay relative to the start of their block of 16 tokens (exponents <= 0 for
// earlier blocks; inside a block exp(L_start - L_s) may grow, and a block in which it could overflow is summed
// directly instead).
//
// Warp roles (512 threads): 0 TMA, 1 MMA issue, 2-3 gates of the state-space heads; 4-11 thread = token, 64 value
// columns each: scores to weights, output (turned around in shared memory); 12-15 thread = key channel: the
// state between two chunks, and the weighted values.
//
// Every mbarrier wait is bounded, as in attention_tc.cu ("where" codes 400 and up).
#include "decay_gates.cuh"
#include "tc_ops.cuh"

namespace eb {
namespace {

constexpr int kChunk = kRows;              // tokens per chunk
constexpr int kCols = 128;                 // value columns per CTA
constexpr int kChunkThreads = 512;
constexpr float kLog2eDecay = 1.4426950408889634f;

struct ChunkParams {
  // state space
  const float *dt;
  long long ldt;
  const float *dt_bias, *a_log, *skip;
  int pair, group;             // heads per CTA (2: of 64 columns each), heads per B / C
  const int *first;
  // gated linear
  const float *decay;          // [batch][chunk][heads][DK]: exp(L_end)
  void *o;
  long long ldo;
  float *S;                    // [batch][heads][DK][dv]
  int seq, heads, dv, slices, chunks;
};

// Gate-derived values of a chunk and head, double-buffered (log2 domain).
struct SsmGates {
  float g2[kChunk];            // L_t
  float u2[kChunk];            // log2(dt_s) - L_s
  float wk[kChunk];            // exp(L at the end of its block of 32 tokens - L_s) dt_s
  float w[kChunk];             // exp(L_end - L_s) dt_s
  float end[kChunk / 32];      // L at the end of each block
  float decay, pad[3];         // exp(L_end)
};

template <int DK, bool SSM> struct ChunkSmem {
  static constexpr uint32_t kOp = (DK / 64) * kRows * 128, kWide = 2 * kRows * 128, kState = 2 * DK * 128;
  static constexpr uint32_t kHead = (256 + (SSM ? 4 * sizeof(SsmGates) : 0) + 1023) / 1024 * 1024;
  static constexpr uint32_t kQ = kHead, kK = kQ + kOp, kK2 = kK + kOp, kP = kK2 + (SSM ? 0 : kOp), kV = kP + (SSM ? 0 : kWide),
                            kV2 = kV + kWide, kV3 = kV2 + (SSM ? kWide : 0), kS = kV3 + (SSM ? kWide : 0), kStage = kS + kState,
                            kEnd = kStage + 8 * 32 * 64;
  static constexpr size_t kTotal = 1024 + kEnd;
  // (with DK = 64 the state's product reads a second 64-column atom behind K: other tiles' memory, whose rows are dropped)
};

template <int DK, bool SSM>
__global__ void __launch_bounds__(kChunkThreads, 1)
decay_chunk_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_k2,
                   const __grid_constant__ CUtensorMap tm_p, const __grid_constant__ CUtensorMap tm_v, const ChunkParams p) {
  using T = __nv_bfloat16;
  using L = ChunkSmem<DK, SSM>;
  constexpr int kSub = DK / 64;
  constexpr uint32_t kAtom = kRows * 128;                        // bytes of a [128][64] sub-tile
  constexpr uint32_t kTmemCols = 512, kColA = 0, kColP = 128, kColO = 256, kColS = 384;
  constexpr uint32_t kIdescA = tc_idesc(kChunk, 1), kIdescO = tc_idesc(kCols, 1) | (1u << 16), kIdescO64 = tc_idesc(64, 1) | (1u << 16),
                     kIdescS = tc_idesc(kCols, 1) | (1u << 15) | (1u << 16);           // bits 15 / 16: A / B run along M / N

  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = s32(smem_raw);
  uint8_t *smem = smem_raw + (((raw + 1023u) & ~1023u) - raw);
  const uint32_t bar0 = s32(smem);
  const uint32_t q_full = bar0, q_empty = bar0 + 8, k_full = bar0 + 16, k_empty = bar0 + 24, v_full = bar0 + 32, v_empty = bar0 + 40, s_full = bar0 + 48,
                 pw_full = bar0 + 56, vw_full = bar0 + 64, state_full = bar0 + 72, delta_full = bar0 + 80, qs_full = bar0 + 88, o1_read = bar0 + 96,
                 o_full = bar0 + 104, o_empty = bar0 + 112, g_full = bar0 + 120, g_empty = bar0 + 136;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + 192);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(smem + 200);
  SsmGates *gates = reinterpret_cast<SsmGates *>(smem + 256);     // [slot][head of the pair]
  const uint32_t q_addr = bar0 + L::kQ, k_addr = bar0 + L::kK, k2_addr = bar0 + L::kK2, p_addr = bar0 + L::kP, v_addr = bar0 + L::kV,
                 vhi_addr = bar0 + L::kV2, vlo_addr = bar0 + L::kV3, s_addr = bar0 + L::kS;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.x, b = blockIdx.y, nc = p.chunks;
  const bool two = SSM && p.pair == 2;
  const int h0 = two ? 2 * unit : unit / p.slices, slice = two ? 0 : unit % p.slices;
  const int col0 = two ? unit * kCols : h0 * p.dv + slice * kCols, live = two ? kCols : min(kCols, p.dv - slice * kCols);

  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_k) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_v) : "memory");
    if (!SSM) {
      asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_k2) : "memory");
      asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_p) : "memory");
    }
    const uint32_t once[] = {q_full, q_empty, k_full, k_empty, v_full, v_empty, s_full, delta_full, qs_full, o_full};
    for (uint32_t bar : once) bar_init(bar, 1);
    bar_init(pw_full, 8);
    bar_init(vw_full, 4);
    bar_init(state_full, DK / 32);
    bar_init(o1_read, 8);
    bar_init(o_empty, 8);
    for (int i = 0; i < 2; ++i) {
      bar_init(g_full + 8 * i, two ? 2 : 1);
      bar_init(g_empty + 8 * i, 12);
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
  const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_slot, 0);
  griddep_launch();
  griddep_wait();

  auto wait = [&](uint32_t bar, int parity, int where) { return __all_sync(0xffffffffu, bar_wait(bar, parity, abort_flag, where)) != 0; };

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      const int hk = SSM ? h0 / p.group : h0;
      auto tile = [&](uint32_t dst, const CUtensorMap *map, uint32_t bar, int x, int subs, int c) {
        for (int i = 0; i < subs; ++i) tma_load_3d(dst + i * kAtom, map, bar, x + i * 64, c * kChunk, b);
      };
      auto ahead = [&](const CUtensorMap *map, int x, int subs, int c) {
        for (int i = 0; i < subs; ++i) tma_prefetch_3d(map, x + i * 64, c * kChunk, b);
      };
      for (int c = 0; c < nc; ++c) {
        const int before = (c - 1) & 1;
        if (c > 0 && !bar_wait(k_empty, before, abort_flag, 1)) break;
        bar_expect_tx(k_full, SSM ? L::kOp + L::kWide : 2 * L::kOp);
        tile(k_addr, &tm_k, k_full, hk * DK, kSub, c);
        if (!SSM) tile(k2_addr, &tm_k2, k_full, hk * DK, kSub, c);
        if (SSM) {
          tile(vhi_addr, &tm_v, k_full, col0, 2, c);           // (the values that are weighted in place)
          if (c > 0 && !bar_wait(q_empty, before, abort_flag, 2)) break;
          bar_expect_tx(q_full, L::kOp);
          tile(q_addr, &tm_q, q_full, hk * DK, kSub, c);
        }
        if (c > 0 && !bar_wait(v_empty, before, abort_flag, 3)) break;
        bar_expect_tx(v_full, L::kWide);
        tile(v_addr, &tm_v, v_full, col0, 2, c);
        if (!SSM) {
          if (c > 0 && !bar_wait(q_empty, before, abort_flag, 4)) break;
          bar_expect_tx(q_full, L::kOp + L::kWide);
          tile(q_addr, &tm_q, q_full, hk * DK, kSub, c);
          tile(p_addr, &tm_p, q_full, hk * kChunk, 2, c);
        }
        // the stages are single: what can be had ahead is that the next chunk's rows wait in L2
        if (c + 1 < nc) {
          ahead(&tm_k, hk * DK, kSub, c + 1);
          ahead(&tm_q, hk * DK, kSub, c + 1);
          ahead(&tm_v, col0, 2, c + 1);
          if (!SSM) {
            ahead(&tm_k2, hk * DK, kSub, c + 1);
            ahead(&tm_p, hk * kChunk, 2, c + 1);
          }
        }
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer (the whole warp goes along, see tc_mma_warp) ----------------
    for (int c = 0; c < nc; ++c) {
      const int ph = c & 1, before = (c - 1) & 1;
      if (!wait(k_full, ph, 5)) break;
      if (SSM) {
        if (!wait(q_full, ph, 6)) break;
        if (c > 0 && !wait(pw_full, before, 7)) break;       // the last scores have been read
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          const uint32_t at = (k >> 2) * kAtom + (k & 3) * 32;
          tc_mma_warp(tmem + kColA, tc_desc(q_addr + at), tc_desc(k_addr + at), kIdescA, k > 0 ? 1u : 0u);
        }
        tc_commit_warp(s_full);
        if (!wait(vw_full, ph, 8)) break;
      } else if (!wait(v_full, ph, 9)) {
        break;
      }
      if (c > 0 && !wait(state_full, before, 10)) break;
      tc_fence_after();
#pragma unroll
      for (int k = 0; k < 2 * kChunk / 16; ++k) {              // 16 tokens per instruction: two 8-row groups of K and of V
        const uint32_t at = (k % (kChunk / 16)) * 2048;
        const bool lo = k >= kChunk / 16;
        const uint32_t ka = SSM ? k_addr : (lo ? k2_addr : k_addr), va = SSM ? (lo ? vlo_addr : vhi_addr) : v_addr;
        tc_mma_warp(tmem + kColS, tc_desc_nmajor(ka + at, kAtom), tc_desc_nmajor(va + at, kAtom), kIdescS, (c > 0 || k > 0) ? 1u : 0u);
      }
      tc_commit_warp(delta_full);
      tc_commit_warp(k_empty);
      if (!SSM && !wait(q_full, ph, 11)) break;
      if (c > 0) {
        if (!wait(o_empty, before, 12)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < DK / 16; ++k)
          tc_mma_warp(tmem + kColO, tc_desc(q_addr + (k >> 2) * kAtom + (k & 3) * 32), tc_desc_nmajor(s_addr + k * 2048, DK * 128), kIdescO, k > 0 ? 1u : 0u);
      }
      if (SSM) {
        tc_commit_warp(q_empty);
        tc_commit_warp(qs_full);
        if (!wait(pw_full, ph, 13) || !wait(v_full, ph, 14)) break;
        if (c > 0 && !wait(o1_read, before, 15)) break;
        tc_fence_after();
        if (two) {
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int k = 0; k < kChunk / 16; ++k)              // 8 columns of P per instruction
              tc_mma_ts_warp(tmem + kColO + 64 * j, tmem + kColP + 64 * j + 8 * k, tc_desc_nmajor(v_addr + j * kAtom + k * 2048, kAtom), kIdescO64, k > 0 ? 1u : 0u);
        } else {
#pragma unroll
          for (int k = 0; k < kChunk / 16; ++k)
            tc_mma_ts_warp(tmem + kColO, tmem + kColP + 8 * k, tc_desc_nmajor(v_addr + k * 2048, kAtom), kIdescO, k > 0 ? 1u : 0u);
        }
      } else {
#pragma unroll
        for (int k = 0; k < kChunk / 16; ++k)
          tc_mma_warp(tmem + kColO, tc_desc(p_addr + (k >> 2) * kAtom + (k & 3) * 32), tc_desc_nmajor(v_addr + k * 2048, kAtom), kIdescO,
                      (c > 0 || k > 0) ? 1u : 0u);
        tc_commit_warp(q_empty);
        tc_commit_warp(qs_full);
      }
      tc_commit_warp(o_full);
      tc_commit_warp(v_empty);
    }
  } else if (warp < 4) {
    // ---------------- gates of a state-space head: 32 tokens at a time ----------------
    const int j = warp - 2;
    if (SSM && (j == 0 || two)) {
      const int h = h0 + j;
      const float bias = p.dt_bias[h], a_log = p.a_log[h];
      const int t_first = p.first ? p.first[b] : 0;
      float raw_dt;
      auto fetch = [&](int t) { raw_dt = p.dt[((long long)b * p.seq + min(t, p.seq - 1)) * p.ldt + h]; };
      fetch(lane);
      for (int c = 0; c < nc; ++c) {
        const int slot = c & 1;
        if (c >= 2 && !wait(g_empty + 8 * slot, ((c >> 1) - 1) & 1, 16)) break;
        SsmGates &g = gates[slot * 2 + j];
        float end = 0.f;                               // of the tokens so far
#pragma unroll 1
        for (int i = 0; i < kChunk; i += 32) {
          const int t = c * kChunk + i + lane;
          const bool alive = t >= t_first && t < p.seq;        // padding, or behind the end: adds nothing, forgets nothing
          const float dt = alive ? softplus(raw_dt + bias) : 0.f;
          float x = alive ? log_decay_ssm(a_log, dt) * kLog2eDecay : 0.f;
          fetch(t + 32);
#pragma unroll
          for (int o = 1; o < 32; o <<= 1) {
            const float y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
          }
          x += end;
          end = __shfl_sync(0xffffffffu, x, 31);
          g.g2[i + lane] = x;
          g.u2[i + lane] = log2f(dt) - x;
          g.wk[i + lane] = dt * ex2(end - x);
          if (lane == 0) g.end[i / 32] = end;
        }
        __syncwarp();
#pragma unroll 1
        for (int i = lane; i < kChunk; i += 32) g.w[i] = g.wk[i] * ex2(end - g.end[i / 32]);
        if (lane == 0) g.decay = ex2(end);
        __syncwarp();
        if (lane == 0) bar_arrive(g_full + 8 * slot);
      }
    }
  } else if (warp < 12) {
    // ---------------- weights and output: thread = token, columns [64 j, 64 j + 64) ----------------
    const int j = (warp - 4) >> 2, quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t t_lane = tmem + ((uint32_t)(quarter * 32) << 16);
    uint8_t *stage = smem + L::kStage + (warp - 4) * (32 * 64);
    const float skip = SSM ? p.skip[two ? h0 + j : h0] : 0.f;
    for (int c = 0; c < nc; ++c) {
      const int ph = c & 1, slot = c & 1;
      float y[64];
      if constexpr (SSM) {
        if (!wait(g_full + 8 * slot, (c >> 1) & 1, 17)) break;
        const SsmGates &g = gates[slot * 2 + (two ? j : 0)];
        const float g2 = g.g2[row];
        if (!wait(s_full, ph, 18)) break;
        tc_fence_after();
        // two heads: each set of warps weights all scores for its own; one: each takes half of the keys
        const int cc0 = two ? 0 : 2 * j, cc1 = two ? 4 : 2 * j + 2;
        const uint32_t t_p = t_lane + kColP + (two ? 64 * j : 0);
#pragma unroll 1
        for (int cc = cc0; cc < cc1; ++cc) {
          uint32_t packed[16];
          if (cc > quarter) {                          // behind the diagonal for every row of the warp
#pragma unroll
            for (int e = 0; e < 16; ++e) packed[e] = 0u;
          } else {
            float x[32];
            tc_ld32(t_lane + kColA + cc * 32, x);
            if (cc < quarter) {                        // the row's part of the decay times the key's
              const float from_end = ex2(g2 - g.end[cc]);
#pragma unroll
              for (int e = 0; e < 32; e += 4) {
                float4 u = *reinterpret_cast<const float4 *>(g.wk + cc * 32 + e);
                mul2(u.x, u.y, u.x, u.y, from_end, from_end);
                mul2(u.z, u.w, u.z, u.w, from_end, from_end);
                mul2(x[e], x[e + 1], x[e], x[e + 1], u.x, u.y);
                mul2(x[e + 2], x[e + 3], x[e + 2], x[e + 3], u.z, u.w);
              }
            } else {
#pragma unroll
              for (int e = 0; e < 32; e += 4) {
                float4 u = *reinterpret_cast<const float4 *>(g.u2 + cc * 32 + e);
                add2(u.x, u.y, u.x, u.y, g2, g2);
                add2(u.z, u.w, u.z, u.w, g2, g2);
                mul2(x[e], x[e + 1], x[e], x[e + 1], ex2(u.x), ex2(u.y));
                mul2(x[e + 2], x[e + 3], x[e + 2], x[e + 3], ex2(u.z), ex2(u.w));
              }
#pragma unroll
              for (int e = 0; e < 32; ++e) x[e] = e < lane ? x[e] : (e == lane ? x[e] + skip : 0.f);
            }
#pragma unroll
            for (int e = 0; e < 32; e += 2) packed[e / 2] = pack2<T>(x[e], x[e + 1]);
          }
          tc_st16(t_p + cc * 16, packed);
        }
        tc_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) bar_arrive(pw_full);
        if (c > 0) {
          // what the chunk's first state gives
          if (!wait(qs_full, ph, 19)) break;
          tc_fence_after();
          const float inter = ex2(g2);
          tc_ld32(t_lane + kColO + 64 * j, y);
          tc_ld32(t_lane + kColO + 64 * j + 32, y + 32);
#pragma unroll
          for (int e = 0; e < 64; e += 2) mul2(y[e], y[e + 1], y[e], y[e + 1], inter, inter);
          tc_fence_before();
          __syncwarp();
          if (lane == 0) bar_arrive(o1_read);
        } else {
#pragma unroll
          for (int e = 0; e < 64; ++e) y[e] = 0.f;
        }
        __syncwarp();
        if (lane == 0) bar_arrive(g_empty + 8 * slot);
      }
      if (!wait(o_full, ph, 20)) break;
      tc_fence_after();
      const int rows = p.seq - c * kChunk - quarter * 32;
      T *ob = reinterpret_cast<T *>(p.o) + ((long long)b * p.seq + c * kChunk + quarter * 32) * p.ldo + col0 + 64 * j;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float *yh = y + 32 * half;
        if constexpr (SSM) {
          float x[32];
          tc_ld32(t_lane + kColO + 64 * j + 32 * half, x);
#pragma unroll
          for (int e = 0; e < 32; e += 2) add2(yh[e], yh[e + 1], yh[e], yh[e + 1], x[e], x[e + 1]);
        } else {
          tc_ld32(t_lane + kColO + 64 * j + 32 * half, yh);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) bar_arrive(o_empty);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
#pragma unroll
        for (int g = 0; g < 4; ++g)
          *reinterpret_cast<uint4 *>(stage + lane * 64 + ((g ^ ((lane >> 1) & 3)) << 4)) =
              make_uint4(pack2<T>(y[32 * half + 8 * g], y[32 * half + 8 * g + 1]), pack2<T>(y[32 * half + 8 * g + 2], y[32 * half + 8 * g + 3]),
                         pack2<T>(y[32 * half + 8 * g + 4], y[32 * half + 8 * g + 5]), pack2<T>(y[32 * half + 8 * g + 6], y[32 * half + 8 * g + 7]));
        __syncwarp();
        // 32 columns of the warp's 32 rows: 4 lanes store a row
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int r = i * 8 + (lane >> 2), col = 32 * half + (lane & 3) * 8;
          const uint4 w = *reinterpret_cast<const uint4 *>(stage + r * 64 + (((lane & 3) ^ ((r >> 1) & 3)) << 4));
          if (r < rows && 64 * j + col < live) *reinterpret_cast<uint4 *>(ob + (long long)r * p.ldo + col) = w;
        }
        __syncwarp();
      }
    }
  } else {
    // ---------------- state between two chunks (thread = key channel), weighted values ----------------
    const int quarter = warp & 3, d = quarter * 32 + lane, tid = threadIdx.x - 12 * 32;
    const uint32_t t_state = tmem + ((uint32_t)(quarter * 32) << 16) + kColS;
    const bool mine = quarter * 32 < DK;
    uint8_t *s_ptr = smem + L::kS;
    bool alive = SSM || mine;
    for (int c = 0; c < nc && alive; ++c) {          // (warps without a key channel have the weighted values to do, or nothing)
      const int ph = c & 1, before = (c - 1) & 1, slot = c & 1;
      float decay0 = 1.f, decay1 = 1.f;
      if constexpr (!SSM) {
        if (c > 0 && mine) decay0 = decay1 = p.decay[(((long long)b * nc + c) * p.heads + h0) * DK + d];
      } else {
        if (!wait(g_full + 8 * slot, (c >> 1) & 1, 21)) { alive = false; break; }
        decay0 = gates[slot * 2].decay;
        decay1 = two ? gates[slot * 2 + 1].decay : decay0;
      }
      if (c > 0) {
        // the state this chunk begins with: operand copy for Q S (the last one has been read), and the master
        // decayed for what is added to it
        if (!wait(delta_full, before, 22) || !wait(qs_full, before, 23)) { alive = false; break; }
        if (mine) {
          tc_fence_after();
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) {
            float x[32];
            tc_ld32(t_state + cc * 32, x);
            uint8_t *dst = s_ptr + (cc >> 1) * (DK * 128) + d * 128;
#pragma unroll
            for (int g = 0; g < 4; ++g)
              *reinterpret_cast<uint4 *>(dst + ((((cc & 1) * 4 + g) ^ (d & 7)) << 4)) =
                  make_uint4(pack2<T>(x[g * 8], x[g * 8 + 1]), pack2<T>(x[g * 8 + 2], x[g * 8 + 3]), pack2<T>(x[g * 8 + 4], x[g * 8 + 5]),
                             pack2<T>(x[g * 8 + 6], x[g * 8 + 7]));
            const float dc = cc < 2 ? decay0 : decay1;
#pragma unroll
            for (int e = 0; e < 32; e += 2) mul2(x[e], x[e + 1], x[e], x[e + 1], dc, dc);
            tc_st32(t_state + cc * 32, x);
          }
          tc_st_wait();
          tc_fence_before();
          asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
          __syncwarp();
          if (lane == 0) bar_arrive(state_full);
        }
      }
      if constexpr (SSM) {
        if (!wait(k_full, ph, 24)) { alive = false; break; }
        uint8_t *hi_ptr = smem + L::kV2, *lo_ptr = smem + L::kV3;
        // thread = 8 columns of every 8th row, in place; the rows of a batch are read before any of them is written
        const int piece = tid & 15, r0 = tid >> 4;
        const float *w = gates[slot * 2 + (two ? piece >> 3 : 0)].w;
        const uint32_t off = (uint32_t)(piece >> 3) * kAtom;
#pragma unroll 1
        for (int i0 = 0; i0 < kChunk / 8; i0 += 8) {
          uint4 v[8];
          float ws[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int r = r0 + 8 * (i0 + i);
            v[i] = *reinterpret_cast<const uint4 *>(hi_ptr + off + r * 128 + (((piece & 7) ^ (r & 7)) << 4));
            ws[i] = w[r];
          }
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int r = r0 + 8 * (i0 + i);
            const uint32_t at = off + r * 128 + (((piece & 7) ^ (r & 7)) << 4), vv[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float2 f = unpack2<T>(vv[e]);
              mul2(f.x, f.y, f.x, f.y, ws[i], ws[i]);
              hi[e] = pack2<T>(f.x, f.y);
              const float2 x = unpack2<T>(hi[e]);
              add2(f.x, f.y, f.x, f.y, -x.x, -x.y);
              lo[e] = pack2<T>(f.x, f.y);
            }
            *reinterpret_cast<uint4 *>(hi_ptr + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4 *>(lo_ptr + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        __syncwarp();
        if (lane == 0) {
          bar_arrive(vw_full);
          bar_arrive(g_empty + 8 * slot);
        }
      }
    }
    if (alive && mine && wait(delta_full, (nc - 1) & 1, 25)) {
      tc_fence_after();
#pragma unroll 1
      for (int cc = 0; cc < 4; ++cc) {
        float x[32];
        tc_ld32(t_state + cc * 32, x);
        const int h = two ? h0 + (cc >> 1) : h0, v0 = two ? (cc & 1) * 32 : slice * kCols + cc * 32;
        float *S = p.S + (((long long)b * p.heads + h) * DK + d) * p.dv + v0;
#pragma unroll
        for (int e = 0; e < 32; e += 8)
          if (v0 + e < p.dv) {                         // (dv is a multiple of 8)
            *reinterpret_cast<float4 *>(S + e) = make_float4(x[e], x[e + 1], x[e + 2], x[e + 3]);
            *reinterpret_cast<float4 *>(S + e + 4) = make_float4(x[e + 4], x[e + 5], x[e + 6], x[e + 7]);
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

template <int DK, bool SSM>
int launch_chunks(const char *name, const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mk2, const CUtensorMap &mp, const CUtensorMap &mv,
                  const ChunkParams &p, int B, cudaStream_t st) {
  constexpr size_t smem = ChunkSmem<DK, SSM>::kTotal;
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  auto kern = decay_chunk_kernel<DK, SSM>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "%s: cannot reserve %zu bytes of shared memory", name, smem);
    }
    configured[dev] = true;
  }
  const int units = SSM && p.pair == 2 ? p.heads / 2 : p.heads * p.slices;
  launch_pdl(kern, dim3(units, B), dim3(kChunkThreads), smem, st, mq, mk, mk2, mp, mv, p);
  return check_launch(name);
}

// ---- gated linear attention: what needs no state -----------------------------------------------------------
constexpr int kPrepThreads = 256;
constexpr float kSafeLog2 = 100.f;         // inside a block of 16 tokens exp(L_start - L_s) stays below 2^100, or the block is summed directly

struct PrepParams {
  const void *q, *k;           // rows ldp apart, heads of DK
  long long ldp;
  const float *z;              // [row][heads*DK]
  long long ldz;
  float inv_tau, scale;
  const int *first;
  void *qt, *khi, *klo;        // [row][heads*DK]
  void *pm;                    // [row][heads*128]
  float *decay;                // [batch][chunk][heads][DK]
  int seq, heads, chunks;
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Two numbers as bf16 parts: what a product with both loses is 2^-16 of it.
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
  hi = pack2<__nv_bfloat16>(x, y);
  const float2 b = unpack2<__nv_bfloat16>(hi);
  lo = pack2<__nv_bfloat16>(x - b.x, y - b.y);
}

template <int DK> struct PrepSmem {
  static constexpr int kLd = DK + 8;       // row strides without bank conflicts
  static constexpr size_t kTotal = (size_t)kChunk * kLd * (4 + 2) + kPrepThreads * 4;
};

template <int DK>
__global__ void __launch_bounds__(kPrepThreads, 2) gla_prepare_kernel(const PrepParams p) {
  using T = __nv_bfloat16;
  constexpr int kLd = PrepSmem<DK>::kLd, kParts = kPrepThreads / DK, kTokens = kChunk / kParts, kPacks = DK / 8;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  float *Lm = reinterpret_cast<float *>(smem_raw);                         // [128][kLd]: L_t in log2 units
  T *ks = reinterpret_cast<T *>(smem_raw + (size_t)kChunk * kLd * 4);      // [128][kLd]
  float *ends = reinterpret_cast<float *>(smem_raw + (size_t)kChunk * kLd * 6);
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = c * kChunk, n = min(kChunk, p.seq - t0), first = (p.first ? p.first[b] : 0) - t0;
  const long long row0 = (long long)b * p.seq + t0;
  const T *q = reinterpret_cast<const T *>(p.q) + row0 * p.ldp + h * DK, *k = reinterpret_cast<const T *>(p.k) + row0 * p.ldp + h * DK;

  // keys (zero for padding and behind the end) on their way to shared memory, queries to registers
  constexpr int kIters = kChunk * kPacks / kPrepThreads, kRowStep = kPrepThreads / kPacks;
  const int r_of = tid / kPacks, x_of = (tid % kPacks) * 8;
  uint4 qv[kIters];
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int r = r_of + i * kRowStep;
    const bool ok = r >= first && r < n;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s32(ks + r * kLd + x_of)), "l"(ok ? k + (long long)r * p.ldp + x_of : k), "r"(ok ? 16 : 0) : "memory");
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
  for (int i = 0; i < kIters; ++i) qv[i] = *reinterpret_cast<const uint4 *>(q + (long long)min(r_of + i * kRowStep, n - 1) * p.ldp + x_of);
  // log decays and their running sums
  {
    constexpr int kBatch = 32;
    const int d = tid % DK, part = tid / DK;
    const float *z = p.z + row0 * p.ldz + h * DK + d;
    float run = 0.f;
#pragma unroll 1
    for (int i0 = 0; i0 < kTokens; i0 += kBatch) {
      float zz[kBatch];
#pragma unroll
      for (int i = 0; i < kBatch; ++i) zz[i] = z[(long long)min(part * kTokens + i0 + i, n - 1) * p.ldz];
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
        const int r = part * kTokens + i0 + i;
        const float l = log_decay_gla(zz[i], p.inv_tau) * kLog2eDecay;
        run += r >= first && r < n ? l : 0.f;
        Lm[r * kLd + d] = run;
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    ends[tid] = run;
    __syncthreads();
    float before = 0.f;
    for (int i = 0; i < part; ++i) before += ends[i * DK + d];
    if (part > 0)
      for (int i = 0; i < kTokens; ++i) Lm[(part * kTokens + i) * kLd + d] += before;
    if (part == kParts - 1) p.decay[(((long long)b * p.chunks + c) * p.heads + h) * DK + d] = ex2(before + run);
  }
  __syncthreads();

  // Q exp(L_t) and K exp(L_end - L_s)
  T *qt = reinterpret_cast<T *>(p.qt) + row0 * p.heads * DK + h * DK, *khi = reinterpret_cast<T *>(p.khi) + row0 * p.heads * DK + h * DK,
    *klo = reinterpret_cast<T *>(p.klo) + row0 * p.heads * DK + h * DK;
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int r = r_of + i * kRowStep, x = x_of;
    if (r >= n) break;
    const uint4 kv = *reinterpret_cast<const uint4 *>(ks + r * kLd + x);
    const uint32_t qw[4] = {qv[i].x, qv[i].y, qv[i].z, qv[i].w}, kw[4] = {kv.x, kv.y, kv.z, kv.w};
    uint32_t a[4], hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 l = *reinterpret_cast<const float2 *>(Lm + r * kLd + x + 2 * e), end = *reinterpret_cast<const float2 *>(Lm + (kChunk - 1) * kLd + x + 2 * e);
      const float2 qf = unpack2<T>(qw[e]), kf = unpack2<T>(kw[e]);
      a[e] = pack2<T>(qf.x * p.scale * ex2(l.x), qf.y * p.scale * ex2(l.y));
      split2(kf.x * ex2(end.x - l.x), kf.y * ex2(end.y - l.y), hi[e], lo[e]);
    }
    const long long at = (long long)r * p.heads * DK + x;
    *reinterpret_cast<uint4 *>(qt + at) = make_uint4(a[0], a[1], a[2], a[3]);
    *reinterpret_cast<uint4 *>(khi + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4 *>(klo + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }

  // P: blocks of 16 rows against tiles of 8 keys; lane (g, t): rows g and g + 8, columns 2 t and 2 t + 1 of a tile.  Block
  // w has 2 w + 2 tiles; the warps of blocks w and 7 - w share theirs, 9 each.
  const int g = lane >> 2, t = lane & 3, low = min(warp, 7 - warp);
  T *pm = reinterpret_cast<T *>(p.pm) + row0 * p.heads * kChunk + h * kChunk;
  auto block = [&](int w, int tile0, int tile1) {
    const int m0 = w * 16;
    if (m0 >= n) return;
    const float *base = Lm + (m0 - 1) * kLd;                     // L in front of the block (0 for the first)
    auto before = [&](int x) { return m0 > 0 ? *reinterpret_cast<const float2 *>(base + x) : make_float2(0.f, 0.f); };
    float spread = 0.f;
    for (int d = lane; d < DK; d += 32) spread = fmaxf(spread, (m0 > 0 ? base[d] : 0.f) - Lm[(m0 + 15) * kLd + d]);
    const bool direct = warp_max(spread) > kSafeLog2;
    uint32_t a[DK / 16][4], a_lo[DK / 16][4];
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = m0 + g + 8 * (i & 1), x = kk * 16 + 2 * t + (i < 2 ? 0 : 8);
        const float2 bb = before(x), l = *reinterpret_cast<const float2 *>(Lm + r * kLd + x);
        const float2 f = r < n ? unpack2<T>(*reinterpret_cast<const uint32_t *>(q + (long long)r * p.ldp + x)) : make_float2(0.f, 0.f);
        split2(f.x * p.scale * ex2(l.x - bb.x), f.y * p.scale * ex2(l.y - bb.y), a[kk][i], a_lo[kk][i]);
      }
#pragma unroll 1
    for (int i = tile0; i < tile1; ++i) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      if (direct && i >= 2 * w) {
#pragma unroll 1
        for (int e = 0; e < 4; ++e) {
          const int r = m0 + g + 8 * (e >> 1), s = i * 8 + 2 * t + (e & 1);
          float sum = 0.f;
          if (s <= r && r < n)
            for (int d = 0; d < DK; ++d)
              sum = fmaf(to_f32<T>(q[(long long)r * p.ldp + d]) * p.scale * ex2(Lm[r * kLd + d] - Lm[s * kLd + d]), to_f32<T>(ks[s * kLd + d]), sum);
          if (e == 0) acc[0] = sum;
          else if (e == 1) acc[1] = sum;
          else if (e == 2) acc[2] = sum;
          else acc[3] = sum;
        }
      } else {
        const int s = i * 8 + g;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const int x0 = kk * 16 + 2 * t, x1 = x0 + 8;
          const float2 b0 = before(x0), b1 = before(x1);
          const float2 l0 = *reinterpret_cast<const float2 *>(Lm + s * kLd + x0), l1 = *reinterpret_cast<const float2 *>(Lm + s * kLd + x1);
          const float2 f0 = unpack2<T>(*reinterpret_cast<const uint32_t *>(ks + s * kLd + x0)), f1 = unpack2<T>(*reinterpret_cast<const uint32_t *>(ks + s * kLd + x1));
          uint32_t k0, k0_lo, k1, k1_lo;
          split2(f0.x * ex2(b0.x - l0.x), f0.y * ex2(b0.y - l0.y), k0, k0_lo);
          split2(f1.x * ex2(b1.x - l1.x), f1.y * ex2(b1.y - l1.y), k1, k1_lo);
          mma_bf16(acc, a[kk], k0, k1);
          mma_bf16(acc, a_lo[kk], k0, k1);
          mma_bf16(acc, a[kk], k0_lo, k1_lo);
        }
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = m0 + g + 8 * e, s = i * 8 + 2 * t;
        if (r < n)
          *reinterpret_cast<uint32_t *>(pm + (long long)r * p.heads * kChunk + s) = pack2<T>(s <= r ? acc[2 * e] : 0.f, s + 1 <= r ? acc[2 * e + 1] : 0.f);
      }
    }
  };
  // keys behind a block are hidden from it
  for (int i = tid; i < n * (kChunk / 8); i += kPrepThreads) {
    const int r = i / (kChunk / 8), s = i % (kChunk / 8);
    if (s >= 2 * (r / 16) + 2) *reinterpret_cast<uint4 *>(pm + (long long)r * p.heads * kChunk + s * 8) = make_uint4(0, 0, 0, 0);
  }
  // (tile 7 - 2 low on of the larger block is its own warp's)
#pragma unroll 1
  for (int turn = 0; turn < 2; ++turn) {
    if (warp < 4) block(turn == 0 ? low : 7 - low, 0, turn == 0 ? 2 * low + 2 : 7 - 2 * low);
    else if (turn == 0) block(warp, 7 - 2 * low, 2 * warp + 2);
  }
}

template <int DK> int launch_prepare(const PrepParams &p, int B, cudaStream_t st) {
  constexpr size_t smem = PrepSmem<DK>::kTotal;
  auto kern = gla_prepare_kernel<DK>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "gla_prepare: cannot reserve %zu bytes of shared memory", smem);
    }
    configured[dev] = true;
  }
  launch_pdl(kern, dim3(p.chunks, p.heads, B), dim3(kPrepThreads), smem, st, p);
  return check_launch("gla_prepare");
}

int check_chunks(const char *name, int batch, int seq, int heads, int dk, int dv, int dtype) {
  if (dtype != EB_BF16) return fail(EB_EINVAL, "%s: bf16 only (dtype %d)", name, dtype);
  if (dk != 64 && dk != 128) return fail(EB_EINVAL, "%s: key head size %d not supported (64 or 128)", name, dk);
  if (batch <= 0 || batch > 65535 || seq <= 0 || heads <= 0 || heads > 65535 || dv <= 0 || dv % 8 != 0 || dv > (1 << 20)) return fail(EB_EINVAL, "%s: bad sizes", name);
  return EB_OK;
}

}  // namespace

int decay_tc_status(int *out4, bool clear) { return tc_status(out4, clear); }

}  // namespace eb

using namespace eb;

extern "C" int eb_ssm_chunks(const void *xbc, long long ldx, const float *dt, long long ldt, const float *dt_bias, const float *a_log, const float *skip,
                             const int32_t *first, void *y, long long ldy, float *S, int batch, int seq, int heads, int groups, int dk, int dv, int dtype,
                             void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  if (int rc = check_chunks("ssm_chunks", batch, seq, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(xbc && dt && dt_bias && a_log && skip && y && S, "ssm_chunks: null pointer");
  EB_REQUIRE(groups > 0 && heads % groups == 0, "ssm_chunks: %d heads do not share %d groups", heads, groups);
  EB_REQUIRE(ldx >= (long long)heads * dv + 2ll * groups * dk && ldx % 8 == 0 && ldt >= heads && ldy >= (long long)heads * dv && ldy % 8 == 0,
             "ssm_chunks: row strides must be multiples of 8 and hold a row");
  EB_REQUIRE(aligned16(xbc) && aligned16(y) && aligned16(S), "ssm_chunks: pointers must be 16-byte aligned");
  const char *x = reinterpret_cast<const char *>(xbc), *k = x + (size_t)heads * dv * 2, *q = k + (size_t)groups * dk * 2;
  CUtensorMap mq, mk, mv;
  int rc;
  if ((rc = tc_map3(&mq, q, dtype, (long long)groups * dk, seq, batch, ldx, ldx * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mk, k, dtype, (long long)groups * dk, seq, batch, ldx, ldx * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mv, x, dtype, (long long)heads * dv, seq, batch, ldx, ldx * seq, kChunk))) return rc;
  ChunkParams p{};
  p.dt = dt; p.ldt = ldt; p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.group = heads / groups;
  p.pair = dv == 64 && p.group % 2 == 0 ? 2 : 1;
  p.first = first; p.o = y; p.ldo = ldy; p.S = S; p.seq = seq; p.heads = heads; p.dv = dv; p.slices = (dv + kCols - 1) / kCols;
  p.chunks = (seq + kChunk - 1) / kChunk;
  cudaStream_t st = as_stream(stream);
  return dk == 64 ? launch_chunks<64, true>("ssm_chunks", mq, mk, mk, mv, mv, p, batch, st)
                  : launch_chunks<128, true>("ssm_chunks", mq, mk, mk, mv, mv, p, batch, st);
}

extern "C" size_t eb_gla_chunks_workspace_bytes(int batch, int seq, int heads, int dk) {
  if (batch <= 0 || seq <= 0 || heads <= 0 || dk <= 0) return 0;
  const size_t rows = (size_t)batch * seq, chunks = ((size_t)seq + kChunk - 1) / kChunk;
  return rows * heads * ((size_t)3 * dk + kChunk) * 2 + (size_t)batch * chunks * heads * dk * 4 + 16;
}

extern "C" int eb_gla_chunks(const void *q, const void *k, const void *v, long long ldp, const float *z, long long ldz, float tau, float scale,
                             const int32_t *first, void *o, long long ldo, float *S, int batch, int seq, int heads, int dk, int dv, int dtype,
                             void *workspace, size_t workspace_bytes, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  if (int rc = check_chunks("gla_chunks", batch, seq, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(q && k && v && z && o && S, "gla_chunks: null pointer");
  EB_REQUIRE(tau > 0.f && ldp % 8 == 0 && ldo % 8 == 0 && ldz >= (long long)heads * dk && ldo >= (long long)heads * dv,
             "gla_chunks: tau must be positive, row strides multiples of 8 that hold a row");
  EB_REQUIRE(aligned16(q) && aligned16(k) && aligned16(v) && aligned16(o) && aligned16(S), "gla_chunks: pointers must be 16-byte aligned");
  const size_t need = eb_gla_chunks_workspace_bytes(batch, seq, heads, dk);
  EB_REQUIRE(workspace && workspace_bytes >= need && aligned16(workspace), "gla_chunks: needs a workspace of %zu bytes", need);
  const size_t rows = (size_t)batch * seq, op = rows * heads * dk * 2;
  char *w = reinterpret_cast<char *>(workspace), *qt = w, *khi = qt + op, *klo = khi + op, *pm = klo + op, *dc = pm + rows * heads * kChunk * 2;
  const int chunks = (seq + kChunk - 1) / kChunk;
  PrepParams a{};
  a.q = q; a.k = k; a.ldp = ldp; a.z = z; a.ldz = ldz; a.inv_tau = 1.f / tau; a.scale = scale; a.first = first; a.qt = qt; a.khi = khi; a.klo = klo;
  a.pm = pm; a.decay = reinterpret_cast<float *>(dc); a.seq = seq; a.heads = heads; a.chunks = chunks;
  cudaStream_t st = as_stream(stream);
  if (int rc = dk == 64 ? launch_prepare<64>(a, batch, st) : launch_prepare<128>(a, batch, st)) return rc;
  CUtensorMap mq, mk, mk2, mp, mv;
  const long long lw = (long long)heads * dk, lp = (long long)heads * kChunk;
  int rc;
  if ((rc = tc_map3(&mq, qt, dtype, lw, seq, batch, lw, lw * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mk, khi, dtype, lw, seq, batch, lw, lw * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mk2, klo, dtype, lw, seq, batch, lw, lw * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mp, pm, dtype, lp, seq, batch, lp, lp * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mv, v, dtype, (long long)heads * dv, seq, batch, ldp, ldp * seq, kChunk))) return rc;
  ChunkParams p{};
  p.decay = a.decay; p.pair = 1; p.group = 1; p.o = o; p.ldo = ldo; p.S = S; p.seq = seq; p.heads = heads; p.dv = dv; p.slices = (dv + kCols - 1) / kCols;
  p.chunks = chunks;
  return dk == 64 ? launch_chunks<64, false>("gla_chunks", mq, mk, mk2, mp, mv, p, batch, st)
                  : launch_chunks<128, false>("gla_chunks", mq, mk, mk2, mp, mv, p, batch, st);
}
