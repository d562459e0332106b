// Matrix memory of a prompt on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), 128 tokens at a
// time.  Inside a chunk that begins with state (S, n, m), with F_t the running sum of the log forget
// gates, u_s = i_s - F_s and M_t = max(m, max_{s <= t} u_s), the recurrence of eb_memory_scan unrolls to
//
//   o_t  ~ sum_{s <= t} exp(u_s - M_t) (q_t.k_s) v_s + exp(m - M_t) S^T q_t
//   S'   = exp(m - M_end) S + sum_s exp(u_s - M_end) k_s v_s^T,   n' likewise,   m' = M_end + F_end
//
// (the running maximum of the recurrence is m_t = M_t + F_t; every exponent here is <= 0).
//
// A CTA owns 128 value columns of one (sequence, head) and walks the chunks in order.  All products
// are 128-row tcgen05.mma with fp32 accumulators in tensor memory:
//   A = Q K^T                 [t][s]       Q, K as they come by TMA
//   O1 = Q S                  [t][v]       S as bf16 hi + lo operands in shared memory
//   O2 = P V                  [t][v]       P = weighted scores, written over A in tensor memory
//   S^T += V^T (w K)          [v][d]       w K as bf16 hi + lo, in place over K
// The state is kept transposed, value column = lane: its fp32 master stays in tensor memory across the
// chunks.  What enters or leaves the recurrent state is split into two bf16 parts (hi + lo), so that it
// keeps 16 bits of mantissa where a single operand would have 8; a weighted score is rounded once, as
// attention weights are.
//
// Warp roles (512 threads): 0 TMA, 1 MMA issue, 2 the gates (one chunk ahead: gate functions, running
// sums and maxima, 32 tokens at a time), 3 idle; 4-7 thread = token: weights the scores, forms the
// denominator, stores the output (turned around in shared memory: rows of 128 bytes); 8-11 q.n for the
// denominator; 12-15 thread = value column: decays the state and writes its operand copies; then 8-15
// together weight the keys and sum them into n (thread = 8 columns of every 8th or 16th row).
//
// The chain from chunk to chunk is: keys arrive, A, keys weighted, state updated.  So the state's product
// is issued before those of the output, which fill the tensor core while the next keys arrive.
//
// Every mbarrier wait is bounded, as in attention_tc.cu ("where" codes 300 and up).
#include <type_traits>

#include "memory_gates.cuh"
#include "tc_ops.cuh"

namespace eb {
namespace {

constexpr int kChunk = kRows;              // tokens per chunk
constexpr int kCols = 128;                 // value columns per CTA
constexpr int kMemThreads = 512;
constexpr float kLog2eMem = 1.4426950408889634f;

struct MemTcParams {
  const float *gates;
  long long ldg;
  const float *bias_i, *bias_f;
  float cap, scale;
  const int *first;
  void *o;
  long long ldo;
  float *S, *n, *m;
  int seq, heads, dv, chunks;
};

// Gate-derived values of a chunk, double-buffered.
struct GateBuf {
  float u2[kChunk];            // u log2(e)
  float M2[kChunk];            // M log2(e)
  float inter[kChunk];         // exp(m - M_t)
  float floor_[kChunk];        // exp(-m_t)
  float w[kChunk];             // exp(u_s - M_end)
  float decay, pad[3];         // exp(m - M_end)
};

template <int DK> struct MemSmem {
  static constexpr uint32_t kOp = (DK / 64) * kRows * 128, kV = 2 * kRows * 128;          // a [128][DK] operand, a [128][128] one
  static constexpr uint32_t kGates = 256, kN = kGates + 2 * sizeof(GateBuf), kQn = kN + 2 * DK * 4, kRed = kQn + 2 * kChunk * 4,
                            kHead = (kRed + 2 * 8 * DK * 4 + 1023) / 1024 * 1024, kStage = 4 * 32 * 128;
  static constexpr size_t kTotal = 1024 + kHead + 5 * (size_t)kOp + kV + kStage;
};

template <int DK>
__global__ void __launch_bounds__(kMemThreads, 1)
memory_chunk_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                    const MemTcParams p) {
  using T = __nv_bfloat16;
  using L = MemSmem<DK>;
  constexpr int kSub = DK / 64;
  constexpr uint32_t kAtom = kRows * 128;                        // bytes of a [128][64] sub-tile
  constexpr uint32_t kTmemCols = 512, kColA = 0, kColO1 = 128, kColO2 = 256, kColS = 384;
  constexpr uint32_t kIdescA = tc_idesc(kChunk, 1), kIdescO = tc_idesc(kCols, 1), kIdescPV = kIdescO | (1u << 16),
                     kIdescS = tc_idesc(DK, 1) | (1u << 15) | (1u << 16);          // bits 15 / 16: A / B run along M / N

  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = s32(smem_raw);
  uint8_t *smem = smem_raw + (((raw + 1023u) & ~1023u) - raw);
  const uint32_t bar0 = s32(smem);
  const uint32_t q_full = bar0, q_empty = bar0 + 8, k_full = bar0 + 16, v_full = bar0 + 24, k_empty = bar0 + 32, s_full = bar0 + 40, p_full = bar0 + 48,
                 o_full = bar0 + 56, o_empty = bar0 + 64, state_full = bar0 + 72, kw_full = bar0 + 80, delta_full = bar0 + 88, g_full = bar0 + 96,
                 g_empty = bar0 + 112, red_full = bar0 + 128, v_empty = bar0 + 136, qs_full = bar0 + 144, qn_full = bar0 + 152, n_full = bar0 + 160;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + 224);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(smem + 232);
  GateBuf *gate_buf = reinterpret_cast<GateBuf *>(smem + L::kGates);
  float *n_buf = reinterpret_cast<float *>(smem + L::kN), *qn_buf = reinterpret_cast<float *>(smem + L::kQn), *red = reinterpret_cast<float *>(smem + L::kRed);
  uint8_t *q_ptr = smem + L::kHead, *k_ptr = q_ptr + L::kOp, *lo_ptr = k_ptr + L::kOp, *shi_ptr = lo_ptr + L::kOp, *slo_ptr = shi_ptr + L::kOp,
          *v_ptr = slo_ptr + L::kOp, *stage_ptr = v_ptr + L::kV;
  const uint32_t q_addr = s32(q_ptr), k_addr = s32(k_ptr), lo_addr = s32(lo_ptr), shi_addr = s32(shi_ptr), slo_addr = s32(slo_ptr), v_addr = s32(v_ptr);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slice = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int nc = p.chunks;

  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_k) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_v) : "memory");
    bar_init(q_full, 1);
    bar_init(q_empty, 1 + 4);                // the products' commit, and the warps that read q for the denominator
    bar_init(k_full, 1);
    bar_init(v_full, 1);
    bar_init(k_empty, 1);
    bar_init(v_empty, 1);
    bar_init(s_full, 1);
    bar_init(p_full, 4);
    bar_init(o_full, 1);
    bar_init(o_empty, 4);
    bar_init(state_full, 4);
    bar_init(kw_full, 8);
    bar_init(delta_full, 1);
    bar_init(red_full, 8);
    bar_init(qs_full, 1);
    bar_init(qn_full, 4);
    bar_init(n_full, 4);
    for (int i = 0; i < 2; ++i) {
      bar_init(g_full + 8 * i, 1);
      bar_init(g_empty + 8 * i, 12);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (threadIdx.x < DK) n_buf[threadIdx.x] = 0.f;
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

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      for (int c = 0; c < nc; ++c) {
        if (c > 0 && !bar_wait(q_empty, (c - 1) & 1, abort_flag, 1)) break;
        bar_expect_tx(q_full, L::kOp);
#pragma unroll
        for (int i = 0; i < kSub; ++i) tma_load_3d(q_addr + i * kAtom, &tm_q, q_full, h * DK + i * 64, c * kChunk, b);
        if (c > 0 && !bar_wait(k_empty, (c - 1) & 1, abort_flag, 2)) break;
        bar_expect_tx(k_full, L::kOp);
#pragma unroll
        for (int i = 0; i < kSub; ++i) tma_load_3d(k_addr + i * kAtom, &tm_k, k_full, h * DK + i * 64, c * kChunk, b);
        if (c > 0 && !bar_wait(v_empty, (c - 1) & 1, abort_flag, 24)) break;
        bar_expect_tx(v_full, L::kV);
#pragma unroll
        for (int i = 0; i < 2; ++i) tma_load_3d(v_addr + i * kAtom, &tm_v, v_full, h * p.dv + slice * kCols + i * 64, c * kChunk, b);
        // the stages are single: what can be had ahead is that the next chunk's rows wait in L2
        if (c + 1 < nc) {
#pragma unroll
          for (int i = 0; i < kSub; ++i) {
            tma_prefetch_3d(&tm_q, h * DK + i * 64, (c + 1) * kChunk, b);
            tma_prefetch_3d(&tm_k, h * DK + i * 64, (c + 1) * kChunk, b);
          }
#pragma unroll
          for (int i = 0; i < 2; ++i) tma_prefetch_3d(&tm_v, h * p.dv + slice * kCols + i * 64, (c + 1) * kChunk, b);
        }
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    // (the whole warp goes along, see tc_mma_warp)
    {
      auto wait = [&](uint32_t bar, int parity, int where) { return __all_sync(0xffffffffu, bar_wait(bar, parity, abort_flag, where)); };
      for (int c = 0; c < nc; ++c) {
        const int ph = c & 1, before = (c - 1) & 1;
        if (!wait(q_full, ph, 3) || !wait(k_full, ph, 4)) break;
        if (c > 0 && !wait(o_full, before, 5)) break;          // the weighted scores of the last chunk lie where A goes
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          const uint32_t at = (k >> 2) * kAtom + (k & 3) * 32;
          tc_mma_warp(tmem + kColA, tc_desc(q_addr + at), tc_desc(k_addr + at), kIdescA, k > 0 ? 1u : 0u);
        }
        tc_commit_warp(s_full);
        if (!wait(v_full, ph, 8) || !wait(kw_full, ph, 10)) break;
        if (c > 0 && !wait(state_full, before, 6)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 2 * kChunk / 16; ++k) {    // 16 tokens per instruction: two 8-row groups of V and of w K
          const uint32_t at = (k % (kChunk / 16)) * 2048;
          tc_mma_warp(tmem + kColS, tc_desc_nmajor(v_addr + at, kAtom), tc_desc_nmajor((k < kChunk / 16 ? k_addr : lo_addr) + at, kAtom), kIdescS,
                      (c > 0 || k > 0) ? 1u : 0u);
        }
        tc_commit_warp(delta_full);
        tc_commit_warp(k_empty);
        if (c > 0) {
          if (!wait(o_empty, before, 7)) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 2 * DK / 16; ++k) {
            const uint32_t at = ((k >> 2) % kSub) * kAtom + (k & 3) * 32;
            tc_mma_warp(tmem + kColO1, tc_desc(q_addr + at), tc_desc((k < DK / 16 ? shi_addr : slo_addr) + at), kIdescO, k > 0 ? 1u : 0u);
          }
        }
        tc_commit_warp(q_empty);
        tc_commit_warp(qs_full);
        if (!wait(p_full, ph, 9)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < kChunk / 16; ++k)          // 8 columns of P per instruction
          tc_mma_ts_warp(tmem + kColO2, tmem + kColA + 8 * k, tc_desc_nmajor(v_addr + k * 2048, kAtom), kIdescPV, k > 0 ? 1u : 0u);
        tc_commit_warp(o_full);
        tc_commit_warp(v_empty);
      }
    }
  } else if (warp == 2) {
    // ---------------- gates: 4 consecutive tokens per lane ----------------
    const float bi = p.bias_i[h], bf = p.bias_f[h];
    const int t_first = p.first ? p.first[b] : 0;
    float m = 0.f;
    // pre-activations are requested 32 tokens ahead
    float ai, af;
    auto fetch = [&](int t) {
      const float *g = p.gates + ((long long)b * p.seq + min(t, p.seq - 1)) * p.ldg;
      ai = g[h];
      af = g[p.heads + h];
    };
    fetch(lane);
    bool alive = true;
    for (int c = 0; c < nc && alive; ++c) {
      const int slot = c & 1;
      if (c >= 2 && !__all_sync(0xffffffffu, bar_wait(g_empty + 8 * slot, ((c >> 1) - 1) & 1, abort_flag, 11))) { alive = false; break; }
      GateBuf &gb = gate_buf[slot];
      float F_end = 0.f, M_end = m;                    // of the tokens so far
#pragma unroll 1
      for (int j = 0; j < kChunk; j += 32) {
        const int t = c * kChunk + j + lane;
        const bool live = t >= t_first && t < p.seq;   // padding, or behind the end: adds nothing, forgets nothing
        const float li = live ? log_input_gate(ai, bi, p.cap) : -INFINITY;
        float F = live ? log_forget_gate(af, bf, p.cap) : 0.f;
        fetch(t + 32);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, F, o);
          if (lane >= o) F += x;
        }
        F += F_end;
        F_end = __shfl_sync(0xffffffffu, F, 31);
        const float u = li - F;
        float M = u;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, M, o);
          if (lane >= o) M = fmaxf(M, x);
        }
        M = fmaxf(M, M_end);
        M_end = __shfl_sync(0xffffffffu, M, 31);
        gb.u2[j + lane] = u * kLog2eMem;
        gb.M2[j + lane] = M * kLog2eMem;
        gb.inter[j + lane] = ex2((m - M) * kLog2eMem);
        gb.floor_[j + lane] = ex2(-(M + F) * kLog2eMem);
      }
#pragma unroll 1
      for (int j = lane; j < kChunk; j += 32) gb.w[j] = ex2(gb.u2[j] - M_end * kLog2eMem);   // (this lane's own entries)
      if (lane == 0) gb.decay = ex2((m - M_end) * kLog2eMem);
      m = M_end + F_end;
      __syncwarp();
      if (lane == 0) bar_arrive(g_full + 8 * slot);
    }
    if (slice == 0 && lane == 0) p.m[(long long)b * p.heads + h] = m;
  } else if (warp >= 4 && warp < 8) {
    // ---------------- scores and output: thread = token ----------------
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t t_lane = tmem + ((uint32_t)(quarter * 32) << 16);
    uint8_t *stage = stage_ptr + quarter * (32 * 128);
    bool alive = true;
    for (int c = 0; c < nc && alive; ++c) {
      const int ph = c & 1, slot = c & 1;
      if (!__all_sync(0xffffffffu, bar_wait(g_full + 8 * slot, (c >> 1) & 1, abort_flag, 12))) { alive = false; break; }
      const GateBuf &gb = gate_buf[slot];
      const float M2 = gb.M2[row], inter = gb.inter[row], floor_ = gb.floor_[row];
      if (!__all_sync(0xffffffffu, bar_wait(s_full, ph, abort_flag, 13))) { alive = false; break; }
      tc_fence_after();
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll 1
      for (int cc = 0; cc < kChunk / 32; ++cc) {
        uint32_t packed[16];
        if (cc > quarter) {                            // behind the diagonal for every row of the warp
#pragma unroll
          for (int e = 0; e < 16; ++e) packed[e] = 0u;
        } else {
          float x[32];
          tc_ld32(t_lane + kColA + cc * 32, x);
#pragma unroll
          for (int e = 0; e < 32; e += 4) {
            float4 u = *reinterpret_cast<const float4 *>(gb.u2 + cc * 32 + e);
            add2(u.x, u.y, u.x, u.y, -M2, -M2);
            add2(u.z, u.w, u.z, u.w, -M2, -M2);
            mul2(x[e], x[e + 1], x[e], x[e + 1], ex2(u.x), ex2(u.y));
            mul2(x[e + 2], x[e + 3], x[e + 2], x[e + 3], ex2(u.z), ex2(u.w));
          }
          if (cc == quarter) {
#pragma unroll
            for (int e = 0; e < 32; ++e) x[e] = e <= lane ? x[e] : 0.f;
          }
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            add2(sum0, sum1, sum0, sum1, x[e], x[e + 1]);
            packed[e / 2] = pack2<T>(x[e], x[e + 1]);
          }
        }
        tc_st16(t_lane + kColA + cc * 16, packed);     // over scores of this row that have been read
      }
      tc_st_wait();
      // the part of the chunk's first state in the denominator
      if (!__all_sync(0xffffffffu, bar_wait(qn_full, ph, abort_flag, 14))) { alive = false; break; }
      const float qn = qn_buf[slot * kChunk + row];
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        bar_arrive(p_full);
        bar_arrive(g_empty + 8 * slot);
      }
      const float den = fmaxf(fabsf(p.scale * fmaf(inter, qn, sum0 + sum1)), floor_) + kMemoryDenomEps;
      const float f2 = p.scale / den, f1 = f2 * inter;
      if (!__all_sync(0xffffffffu, bar_wait(o_full, ph, abort_flag, 16))) { alive = false; break; }
      tc_fence_after();
      T *ob = reinterpret_cast<T *>(p.o) + ((long long)b * p.seq + c * kChunk + quarter * 32) * p.ldo + h * p.dv + slice * kCols;
      const int left = p.dv - slice * kCols;           // value columns of this slice that exist (a multiple of 8)
      const int rows = p.seq - c * kChunk - quarter * 32;
#pragma unroll 1
      for (int cc = 0; cc < kCols / 32; ++cc) {
        uint32_t xr[32], yr[32];
        float x[32];
        tc_ld32_issue(t_lane + kColO2 + cc * 32, xr);
        tc_ld32_issue(t_lane + kColO1 + cc * 32, yr);
        tc_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e += 2) mul2(x[e], x[e + 1], __uint_as_float(xr[e]), __uint_as_float(xr[e + 1]), f2, f2);
        if (c > 0) {                                   // (the first chunk begins with nothing; O1 is not defined)
#pragma unroll
          for (int e = 0; e < 32; e += 2)
            fma2(x[e], x[e + 1], __uint_as_float(yr[e]), __uint_as_float(yr[e + 1]), f1, f1, x[e], x[e + 1]);
        }
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint4 w;
          w.x = pack2<T>(x[g * 8 + 0], x[g * 8 + 1]);
          w.y = pack2<T>(x[g * 8 + 2], x[g * 8 + 3]);
          w.z = pack2<T>(x[g * 8 + 4], x[g * 8 + 5]);
          w.w = pack2<T>(x[g * 8 + 6], x[g * 8 + 7]);
          *reinterpret_cast<uint4 *>(stage + lane * 128 + ((((cc & 1) * 4 + g) ^ (lane & 7)) << 4)) = w;
        }
        if ((cc & 1) == 0) continue;
        // 64 columns of the warp's 32 rows: 8 lanes store a row
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int r = i * 4 + (lane >> 3), col = (cc >> 1) * 64 + (lane & 7) * 8;
          const uint4 w = *reinterpret_cast<const uint4 *>(stage + r * 128 + (((lane & 7) ^ (r & 7)) << 4));
          if (r < rows && col < left) *reinterpret_cast<uint4 *>(ob + (long long)r * p.ldo + col) = w;
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) bar_arrive(o_empty);
    }
  } else if (warp >= 8) {
    // ---------------- q.n (warps 8-11), state (12-15), weighted keys (all) ----------------
    const int half = (warp - 8) >> 2, tid = threadIdx.x - 256 - half * 128, quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t t_state = tmem + ((uint32_t)(quarter * 32) << 16) + kColS;
    constexpr int kPieces = DK / 8, kRowStep = 128 / kPieces;                   // 16-byte pieces of a row; rows a pass of 128 threads covers
    const int piece = tid % kPieces, r0 = half * (kChunk / 2) + tid / kPieces;  // each half of the warps takes half of the rows
    const uint32_t piece_off = (uint32_t)(piece >> 3) * kAtom;
    bool alive = true;
    for (int c = 0; c < nc && alive; ++c) {
      const int ph = c & 1, before = (c - 1) & 1, slot = c & 1;
      auto wait = [&](uint32_t bar, int parity, int where) { return __all_sync(0xffffffffu, bar_wait(bar, parity, abort_flag, where)) != 0; };
      if (!wait(g_full + 8 * slot, (c >> 1) & 1, 17)) { alive = false; break; }
      const GateBuf &gb = gate_buf[slot];
      const float decay = gb.decay;
      if (half == 0) {
        // (p_full of the chunk before: the last q.n has been read)
        if ((c > 0 && (!wait(p_full, before, 18) || !wait(n_full, before, 19))) || !wait(q_full, ph, 20)) { alive = false; break; }
        const uint8_t *q_row = q_ptr + row * 128;
        const float *n = n_buf + slot * DK;
        float qn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int i = 0; i < DK / 8; ++i) {
          const uint4 w = *reinterpret_cast<const uint4 *>(q_row + (i >> 3) * kAtom + (((i & 7) ^ (row & 7)) << 4));
          const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
          const float4 n0 = *reinterpret_cast<const float4 *>(n + i * 8), n1 = *reinterpret_cast<const float4 *>(n + i * 8 + 4);
          const float nn[8] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = unpack2<T>(ww[e]);
            fma2(qn[(e & 1) * 2], qn[(e & 1) * 2 + 1], f.x, f.y, nn[2 * e], nn[2 * e + 1], qn[(e & 1) * 2], qn[(e & 1) * 2 + 1]);
          }
        }
        qn_buf[slot * kChunk + row] = (qn[0] + qn[1]) + (qn[2] + qn[3]);
        __syncwarp();
        if (lane == 0) {
          bar_arrive(qn_full);
          bar_arrive(q_empty);
        }
      } else if (c > 0) {
        // the state this chunk begins with: operand copies for Q S (the last ones have been read), and the
        // master decayed for what is added to it
        if (!wait(delta_full, before, 21) || !wait(qs_full, before, 22)) { alive = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int cc = 0; cc < DK / 32; ++cc) {
          float x[32];
          tc_ld32(t_state + cc * 32, x);
          const uint32_t off = (uint32_t)(cc >> 1) * kAtom + row * 128;
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float a = x[g * 8 + 2 * e], d = x[g * 8 + 2 * e + 1];
              hi[e] = pack2<T>(a, d);
              const float2 r = unpack2<T>(hi[e]);
              add2(a, d, a, d, -r.x, -r.y);
              lo[e] = pack2<T>(a, d);
            }
            const uint32_t at = off + ((((cc & 1) * 4 + g) ^ (row & 7)) << 4);
            *reinterpret_cast<uint4 *>(shi_ptr + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4 *>(slo_ptr + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
#pragma unroll
          for (int e = 0; e < 32; e += 2) mul2(x[e], x[e + 1], x[e], x[e + 1], decay, decay);
          tc_st32(t_state + cc * 32, x);
        }
        tc_st_wait();
        tc_fence_before();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        __syncwarp();
        if (lane == 0) bar_arrive(state_full);
      }
      if (!wait(k_full, ph, 23) || !wait(s_full, ph, 24)) { alive = false; break; }
      float acc[8] = {};
#pragma unroll 1
      for (int i0 = 0; i0 < kChunk / 2 / kRowStep; i0 += 4) {
        uint4 kv[4];
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {                  // the rows of a batch are read before any of them is written
          const int r = r0 + (i0 + i) * kRowStep;
          kv[i] = *reinterpret_cast<const uint4 *>(k_ptr + piece_off + r * 128 + (((piece & 7) ^ (r & 7)) << 4));
          w[i] = gb.w[r];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int r = r0 + (i0 + i) * kRowStep;
          const uint32_t kk[4] = {kv[i].x, kv[i].y, kv[i].z, kv[i].w};
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float2 f = unpack2<T>(kk[e]);
            mul2(f.x, f.y, f.x, f.y, w[i], w[i]);
            add2(acc[2 * e], acc[2 * e + 1], acc[2 * e], acc[2 * e + 1], f.x, f.y);
            hi[e] = pack2<T>(f.x, f.y);
            const float2 x = unpack2<T>(hi[e]);
            add2(f.x, f.y, f.x, f.y, -x.x, -x.y);
            lo[e] = pack2<T>(f.x, f.y);
          }
          const uint32_t at = piece_off + r * 128 + (((piece & 7) ^ (r & 7)) << 4);
          *reinterpret_cast<uint4 *>(k_ptr + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4 *>(lo_ptr + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) bar_arrive(kw_full);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
#pragma unroll
        for (int o = kPieces; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
      }
      if (lane < kPieces) {
#pragma unroll
        for (int e = 0; e < 8; ++e) red[(slot * 8 + warp - 8) * DK + piece * 8 + e] = acc[e];
      }
      __syncwarp();
      if (lane == 0) bar_arrive(red_full);
      if (half == 0) {
        if (!wait(red_full, ph, 25)) { alive = false; break; }
        if (tid < DK) {
          float sum = 0.f;
#pragma unroll
          for (int i = 0; i < 8; ++i) sum += red[(slot * 8 + i) * DK + tid];
          n_buf[(slot ^ 1) * DK + tid] = fmaf(decay, n_buf[slot * DK + tid], sum);
        }
        __syncwarp();
        if (lane == 0) bar_arrive(n_full);
      }
      __syncwarp();
      if (lane == 0) bar_arrive(g_empty + 8 * slot);
    }
    if (half == 0) {
      if (alive && slice == 0 && tid < DK) p.n[((long long)b * p.heads + h) * DK + tid] = n_buf[(nc & 1) * DK + tid];
      alive = false;                                   // (the state is the other half's)
    }
    if (alive && !__all_sync(0xffffffffu, bar_wait(delta_full, (nc - 1) & 1, abort_flag, 26))) alive = false;
    if (alive) {
      tc_fence_after();
      const long long bh = (long long)b * p.heads + h;
      const int v = slice * kCols + row;
#pragma unroll 1
      for (int cc = 0; cc < DK / 32; ++cc) {
        float x[32];
        tc_ld32(t_state + cc * 32, x);
        if (v < p.dv) {
          float *S = p.S + (bh * DK + cc * 32) * p.dv + v;
#pragma unroll
          for (int e = 0; e < 32; ++e) S[(long long)e * p.dv] = x[e];
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

template <int DK> int launch_chunks(const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mv, const MemTcParams &p, int B, cudaStream_t st) {
  constexpr size_t smem = MemSmem<DK>::kTotal;
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  auto kern = memory_chunk_kernel<DK>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "memory_chunks: cannot reserve %zu bytes of shared memory", smem);
    }
    configured[dev] = true;
  }
  launch_pdl(kern, dim3((p.dv + kCols - 1) / kCols, p.heads, B), dim3(kMemThreads), smem, st, mq, mk, mv, p);
  return check_launch("memory_chunks");
}

}  // namespace

int memory_tc_status(int *out4, bool clear) { return tc_status(out4, clear); }

}  // namespace eb

using namespace eb;

extern "C" int eb_memory_chunks(const void *q, const void *k, const void *v, long long ldp, const float *gates, long long ldg, const float *bias_i,
                                const float *bias_f, float cap, float scale, const int32_t *first, void *o, long long ldo, float *S, float *n,
                                float *m, int batch, int seq, int heads, int dk, int dv, int dtype, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  EB_REQUIRE(dtype == EB_BF16, "memory_chunks: bf16 only (dtype %d)", dtype);
  EB_REQUIRE(dk == 64 || dk == 128, "memory_chunks: key head size %d not supported (64 or 128)", dk);
  EB_REQUIRE(q && k && v && gates && bias_i && bias_f && o && S && n && m, "memory_chunks: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && seq > 0 && heads > 0 && heads <= 65535 && dv > 0 && dv % 8 == 0, "memory_chunks: bad sizes");
  EB_REQUIRE(ldp % 8 == 0 && ldo % 8 == 0 && ldg >= 2 * heads && ldo >= (long long)heads * dv, "memory_chunks: row strides must be multiples of 8 and hold a row");
  EB_REQUIRE(cap > 0.f, "memory_chunks: the gates' cap must be positive");
  EB_REQUIRE(aligned16(q) && aligned16(k) && aligned16(v) && aligned16(o), "memory_chunks: pointers must be 16-byte aligned");
  CUtensorMap mq, mk, mv;
  int rc;
  if ((rc = tc_map3(&mq, q, dtype, (long long)heads * dk, seq, batch, ldp, ldp * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mk, k, dtype, (long long)heads * dk, seq, batch, ldp, ldp * seq, kChunk))) return rc;
  if ((rc = tc_map3(&mv, v, dtype, (long long)heads * dv, seq, batch, ldp, ldp * seq, kChunk))) return rc;
  MemTcParams p{};
  p.gates = gates; p.ldg = ldg; p.bias_i = bias_i; p.bias_f = bias_f; p.cap = cap; p.scale = scale; p.first = first;
  p.o = o; p.ldo = ldo; p.S = S; p.n = n; p.m = m; p.seq = seq; p.heads = heads; p.dv = dv; p.chunks = (seq + kChunk - 1) / kChunk;
  cudaStream_t st = as_stream(stream);
  return dk == 64 ? launch_chunks<64>(mq, mk, mv, p, batch, st) : launch_chunks<128>(mq, mk, mv, p, batch, st);
}
