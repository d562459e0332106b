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
// Warp roles (384 threads): 0 TMA, 1 MMA issue, 2 the gates (one chunk ahead: gate functions, running
// sums and maxima, 4 tokens per lane), 3 idle, 4-7 thread = token: weights the scores, forms the
// denominator, stores the output, 8-11 weight the keys and sum them into n (thread = 8 columns of every
// 8th or 16th row), then thread = value column: decays the state and writes its operand copies.
//
// Every mbarrier wait is bounded, as in attention_tc.cu ("where" codes 300 and up).
#include <type_traits>

#include "memory_gates.cuh"
#include "tc_ops.cuh"

namespace eb {
namespace {

constexpr int kChunk = kRows;              // tokens per chunk
constexpr int kCols = 128;                 // value columns per CTA
constexpr int kMemThreads = 384;
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
  float decay, m_next, pad[2]; // exp(m - M_end), M_end + F_end
};

template <int DK> struct MemSmem {
  static constexpr uint32_t kOp = (DK / 64) * kRows * 128, kV = 2 * kRows * 128;          // a [128][DK] operand, a [128][128] one
  static constexpr uint32_t kGates = 256, kN = kGates + 2 * sizeof(GateBuf), kRed = kN + 2 * DK * 4, kHead = (kRed + 4 * DK * 4 + 1023) / 1024 * 1024;
  static constexpr size_t kTotal = 1024 + kHead + 5 * (size_t)kOp + kV;
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
  const uint32_t q_full = bar0, q_empty = bar0 + 8, k_full = bar0 + 16, v_full = bar0 + 24, kv_empty = bar0 + 32, s_full = bar0 + 40, p_full = bar0 + 48,
                 o_full = bar0 + 56, o_empty = bar0 + 64, state_full = bar0 + 72, kw_full = bar0 + 80, delta_full = bar0 + 88, g_full = bar0 + 96,
                 g_empty = bar0 + 112, red_full = bar0 + 128;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(smem + 192);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(smem + 200);
  GateBuf *gate_buf = reinterpret_cast<GateBuf *>(smem + L::kGates);
  float *n_buf = reinterpret_cast<float *>(smem + L::kN), *red = reinterpret_cast<float *>(smem + L::kRed);
  uint8_t *q_ptr = smem + L::kHead, *k_ptr = q_ptr + L::kOp, *lo_ptr = k_ptr + L::kOp, *shi_ptr = lo_ptr + L::kOp, *slo_ptr = shi_ptr + L::kOp,
          *v_ptr = slo_ptr + L::kOp;
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
    bar_init(kv_empty, 1);
    bar_init(s_full, 1);
    bar_init(p_full, 4);
    bar_init(o_full, 1);
    bar_init(o_empty, 4);
    bar_init(state_full, 4);
    bar_init(kw_full, 4);
    bar_init(delta_full, 1);
    bar_init(red_full, 4);
    for (int i = 0; i < 2; ++i) {
      bar_init(g_full + 8 * i, 1);
      bar_init(g_empty + 8 * i, 8);
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
  const uint32_t tmem = *tmem_slot;
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
        if (c > 0 && !bar_wait(kv_empty, (c - 1) & 1, abort_flag, 2)) break;
        bar_expect_tx(k_full, L::kOp);
#pragma unroll
        for (int i = 0; i < kSub; ++i) tma_load_3d(k_addr + i * kAtom, &tm_k, k_full, h * DK + i * 64, c * kChunk, b);
        bar_expect_tx(v_full, L::kV);
#pragma unroll
        for (int i = 0; i < 2; ++i) tma_load_3d(v_addr + i * kAtom, &tm_v, v_full, h * p.dv + slice * kCols + i * 64, c * kChunk, b);
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      for (int c = 0; c < nc; ++c) {
        const int ph = c & 1, before = (c - 1) & 1;
        if (!bar_wait(q_full, ph, abort_flag, 3) || !bar_wait(k_full, ph, abort_flag, 4)) break;
        if (c > 0 && !bar_wait(o_full, before, abort_flag, 5)) break;          // the weighted scores of the last chunk lie where A goes
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < kSub; ++i) {
          const uint64_t a = tc_desc(q_addr + i * kAtom), bd = tc_desc(k_addr + i * kAtom);
#pragma unroll
          for (int k = 0; k < 4; ++k) tc_mma(tmem + kColA, a + 2 * k, bd + 2 * k, kIdescA, (i > 0 || k > 0) ? 1u : 0u);
        }
        tc_commit(s_full);
        if (c > 0) {
          if (!bar_wait(state_full, before, abort_flag, 6) || !bar_wait(o_empty, before, abort_flag, 7)) break;
          tc_fence_after();
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int i = 0; i < kSub; ++i) {
              const uint64_t a = tc_desc(q_addr + i * kAtom), bd = tc_desc((part ? slo_addr : shi_addr) + i * kAtom);
#pragma unroll
              for (int k = 0; k < 4; ++k) tc_mma(tmem + kColO1, a + 2 * k, bd + 2 * k, kIdescO, (part > 0 || i > 0 || k > 0) ? 1u : 0u);
            }
        }
        tc_commit(q_empty);
        if (!bar_wait(v_full, ph, abort_flag, 8) || !bar_wait(p_full, ph, abort_flag, 9)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < kChunk / 16; ++k)          // 16 tokens per instruction: 8 columns of P, two 8-row groups of V
          tc_mma_ts(tmem + kColO2, tmem + kColA + 8 * k, tc_desc_nmajor(v_addr + k * 2048, kAtom), kIdescPV, k > 0 ? 1u : 0u);
        tc_commit(o_full);
        if (!bar_wait(kw_full, ph, abort_flag, 10)) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < kChunk / 16; ++k)
            tc_mma(tmem + kColS, tc_desc_nmajor(v_addr + k * 2048, kAtom), tc_desc_nmajor((part ? lo_addr : k_addr) + k * 2048, kAtom), kIdescS,
                   (c > 0 || part > 0 || k > 0) ? 1u : 0u);
        tc_commit(delta_full);
        tc_commit(kv_empty);
      }
    }
  } else if (warp == 2) {
    // ---------------- gates: 4 consecutive tokens per lane ----------------
    const float bi = p.bias_i[h], bf = p.bias_f[h];
    const int t_first = p.first ? p.first[b] : 0;
    float m = 0.f;
    for (int c = 0; c < nc; ++c) {
      const int slot = c & 1;
      float li[4], F[4];
      float run = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = c * kChunk + lane * 4 + j;
        li[j] = -INFINITY;                             // padding, or behind the end: adds nothing, forgets nothing
        if (t >= t_first && t < p.seq) {
          const float *g = p.gates + ((long long)b * p.seq + t) * p.ldg;
          li[j] = log_input_gate(g[h], bi, p.cap);
          run += log_forget_gate(g[p.heads + h], bf, p.cap);
        }
        F[j] = run;
      }
      float base = run;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, base, o);
        if (lane >= o) base += x;
      }
      const float F_end = __shfl_sync(0xffffffffu, base, 31);
      base -= run;
      float u[4], top = -INFINITY;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        F[j] += base;
        u[j] = li[j] - F[j];
        top = fmaxf(top, u[j]);
      }
      float upto = top;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, upto, o);
        if (lane >= o) upto = fmaxf(upto, x);
      }
      const float M_end = fmaxf(m, __shfl_sync(0xffffffffu, upto, 31));
      float prev = __shfl_up_sync(0xffffffffu, upto, 1);
      float M = lane == 0 ? m : fmaxf(m, prev);
      if (c >= 2 && !__all_sync(0xffffffffu, bar_wait(g_empty + 8 * slot, ((c >> 1) - 1) & 1, abort_flag, 11))) break;
      GateBuf &gb = gate_buf[slot];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = lane * 4 + j;
        M = fmaxf(M, u[j]);
        gb.u2[t] = u[j] * kLog2eMem;
        gb.M2[t] = M * kLog2eMem;
        gb.inter[t] = expf(m - M);
        gb.floor_[t] = expf(-(M + F[j]));
        gb.w[t] = expf(u[j] - M_end);
      }
      if (lane == 0) {
        gb.decay = expf(m - M_end);
        gb.m_next = M_end + F_end;
      }
      m = M_end + F_end;
      __syncwarp();
      if (lane == 0) bar_arrive(g_full + 8 * slot);
    }
    if (slice == 0 && lane == 0) p.m[(long long)b * p.heads + h] = m;
  } else if (warp >= 4 && warp < 8) {
    // ---------------- scores and output: thread = token ----------------
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t t_lane = tmem + ((uint32_t)(quarter * 32) << 16);
    const uint8_t *q_row = q_ptr + row * 128;
    bool alive = true;
    for (int c = 0; c < nc && alive; ++c) {
      const int ph = c & 1, before = (c - 1) & 1, slot = c & 1;
      if (!__all_sync(0xffffffffu, bar_wait(g_full + 8 * slot, (c >> 1) & 1, abort_flag, 12))) { alive = false; break; }
      const GateBuf &gb = gate_buf[slot];
      const float M2 = gb.M2[row], inter = gb.inter[row], floor_ = gb.floor_[row];
      if (!__all_sync(0xffffffffu, bar_wait(s_full, ph, abort_flag, 13))) { alive = false; break; }
      tc_fence_after();
      float sum = 0.f;
#pragma unroll
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
            const float4 u = *reinterpret_cast<const float4 *>(gb.u2 + cc * 32 + e);
            x[e] *= ex2(u.x - M2); x[e + 1] *= ex2(u.y - M2); x[e + 2] *= ex2(u.z - M2); x[e + 3] *= ex2(u.w - M2);
          }
          if (cc == quarter) {
#pragma unroll
            for (int e = 0; e < 32; ++e) x[e] = e <= lane ? x[e] : 0.f;
          }
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            sum += x[e] + x[e + 1];
            packed[e / 2] = pack2<T>(x[e], x[e + 1]);
          }
        }
        tc_st16(t_lane + kColA + cc * 16, packed);     // over scores of this row that have been read
      }
      tc_st_wait();
      // the chunk's first state: its part of the denominator is q . n
      float qn = 0.f;
      if (c > 0) {
        if (!__all_sync(0xffffffffu, bar_wait(state_full, before, abort_flag, 14)) || !__all_sync(0xffffffffu, bar_wait(q_full, ph, abort_flag, 15))) {
          alive = false;
          break;
        }
        const float *n = n_buf + slot * DK;
#pragma unroll
        for (int i = 0; i < DK / 8; ++i) {
          const uint4 w = *reinterpret_cast<const uint4 *>(q_row + (i >> 3) * kAtom + (((i & 7) ^ (row & 7)) << 4));
          const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
          const float4 n0 = *reinterpret_cast<const float4 *>(n + i * 8), n1 = *reinterpret_cast<const float4 *>(n + i * 8 + 4);
          const float nn[8] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = unpack2<T>(ww[e]);
            qn = fmaf(f.x, nn[2 * e], qn);
            qn = fmaf(f.y, nn[2 * e + 1], qn);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        bar_arrive(p_full);
        bar_arrive(q_empty);
        bar_arrive(g_empty + 8 * slot);
      }
      const float den = fmaxf(fabsf(p.scale * fmaf(inter, qn, sum)), floor_) + kMemoryDenomEps;
      const float f2 = p.scale / den, f1 = f2 * inter;
      if (!__all_sync(0xffffffffu, bar_wait(o_full, ph, abort_flag, 16))) { alive = false; break; }
      tc_fence_after();
      const int t = c * kChunk + row;
      T *orow = reinterpret_cast<T *>(p.o) + ((long long)b * p.seq + t) * p.ldo + h * p.dv + slice * kCols;
      const int left = p.dv - slice * kCols;           // value columns of this slice that exist (a multiple of 8)
#pragma unroll 1
      for (int cc = 0; cc < kCols / 32; ++cc) {
        float x[32];
        tc_ld32(t_lane + kColO2 + cc * 32, x);
#pragma unroll
        for (int e = 0; e < 32; ++e) x[e] *= f2;
        if (c > 0) {
          float y[32];
          tc_ld32(t_lane + kColO1 + cc * 32, y);
#pragma unroll
          for (int e = 0; e < 32; ++e) x[e] = fmaf(y[e], f1, x[e]);
        }
        if (t < p.seq) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            if (cc * 32 + g * 8 >= left) break;
            uint4 w;
            w.x = pack2<T>(x[g * 8 + 0], x[g * 8 + 1]);
            w.y = pack2<T>(x[g * 8 + 2], x[g * 8 + 3]);
            w.z = pack2<T>(x[g * 8 + 4], x[g * 8 + 5]);
            w.w = pack2<T>(x[g * 8 + 6], x[g * 8 + 7]);
            *reinterpret_cast<uint4 *>(orow + cc * 32 + g * 8) = w;
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) bar_arrive(o_empty);
    }
  } else if (warp >= 8) {
    // ---------------- keys and state ----------------
    const int tid = threadIdx.x - 256, quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t t_state = tmem + ((uint32_t)(quarter * 32) << 16) + kColS;
    constexpr int kPieces = DK / 8, kRowStep = 128 / kPieces;                   // 16-byte pieces of a row; rows a pass covers
    const int piece = tid % kPieces, r0 = tid / kPieces;
    const uint32_t piece_off = (uint32_t)(piece >> 3) * kAtom;
    bool alive = true;
    for (int c = 0; c < nc && alive; ++c) {
      const int ph = c & 1, before = (c - 1) & 1, slot = c & 1;
      if (!__all_sync(0xffffffffu, bar_wait(g_full + 8 * slot, (c >> 1) & 1, abort_flag, 17))) { alive = false; break; }
      const GateBuf &gb = gate_buf[slot];
      const float decay = gb.decay;
      if (c > 0) {
        // the state this chunk begins with: operand copies for Q S, and the master decayed for what is added to it
        if (!__all_sync(0xffffffffu, bar_wait(delta_full, before, abort_flag, 18))) { alive = false; break; }
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
              const float a = x[g * 8 + 2 * e], d = x[g * 8 + 2 * e + 1];
              hi[e] = pack2<T>(a, d);
              const float2 r = unpack2<T>(hi[e]);
              lo[e] = pack2<T>(a - r.x, d - r.y);
            }
            const uint32_t at = off + ((((cc & 1) * 4 + g) ^ (row & 7)) << 4);
            *reinterpret_cast<uint4 *>(shi_ptr + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4 *>(slo_ptr + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
#pragma unroll
          for (int e = 0; e < 32; ++e) x[e] *= decay;
          tc_st32(t_state + cc * 32, x);
        }
        tc_st_wait();
        tc_fence_before();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        __syncwarp();
        if (lane == 0) bar_arrive(state_full);
      }
      if (!__all_sync(0xffffffffu, bar_wait(k_full, ph, abort_flag, 19)) || !__all_sync(0xffffffffu, bar_wait(s_full, ph, abort_flag, 20))) {
        alive = false;
        break;
      }
      float acc[8] = {};
#pragma unroll
      for (int i = 0; i < kChunk / kRowStep; ++i) {
        const int r = r0 + i * kRowStep;
        const uint32_t at = piece_off + r * 128 + (((piece & 7) ^ (r & 7)) << 4);
        const uint4 kv = *reinterpret_cast<const uint4 *>(k_ptr + at);
        const uint32_t kk[4] = {kv.x, kv.y, kv.z, kv.w};
        const float w = gb.w[r];
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = unpack2<T>(kk[e]);
          const float a = w * f.x, d = w * f.y;
          acc[2 * e] += a;
          acc[2 * e + 1] += d;
          hi[e] = pack2<T>(a, d);
          const float2 x = unpack2<T>(hi[e]);
          lo[e] = pack2<T>(a - x.x, d - x.y);
        }
        *reinterpret_cast<uint4 *>(k_ptr + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4 *>(lo_ptr + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
#pragma unroll
      for (int e = 0; e < 8; ++e) {
#pragma unroll
        for (int o = kPieces; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
      }
      if (lane < kPieces) {
#pragma unroll
        for (int e = 0; e < 8; ++e) red[quarter * DK + piece * 8 + e] = acc[e];
      }
      __syncwarp();
      if (lane == 0) bar_arrive(red_full);
      if (!__all_sync(0xffffffffu, bar_wait(red_full, ph, abort_flag, 22))) { alive = false; break; }
      if (tid < DK)
        n_buf[(slot ^ 1) * DK + tid] = fmaf(decay, n_buf[slot * DK + tid], red[tid] + red[DK + tid] + red[2 * DK + tid] + red[3 * DK + tid]);
      __syncwarp();
      if (lane == 0) {
        bar_arrive(kw_full);
        bar_arrive(g_empty + 8 * slot);
      }
    }
    if (alive && !__all_sync(0xffffffffu, bar_wait(delta_full, (nc - 1) & 1, abort_flag, 21))) alive = false;
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
      if (slice == 0 && tid < DK) p.n[bh * DK + tid] = n_buf[(nc & 1) * DK + tid];
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
