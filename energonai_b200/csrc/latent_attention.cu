// Attention over a latent cache, and the plain windowed attention behind it.
//
//   latent_decode    one new position per sequence with the key and value projections absorbed into
//                    the query and the output: every head of a sequence reads the SAME cached row
//                    c_j (its key and its value), so the kernel is a pass over the visible part of
//                    the cache shared by 16 or 32 heads of a CTA:
//                       s[h][j] = scale * qa[h] . c_j,   o[h] = sum_j softmax_j(s[h]) c_j
//                    on mma.sync with fp32 scores, statistics and accumulators, cache tiles by TMA.
//                    The key range is split over the CTAs of a cluster, which merge their parts
//                    through distributed shared memory (or over more CTAs and a merge kernel).
//   attention_plain  any head sizes, fp32 or 16 bit, one warp per query row: the path of models run
//                    in 32-bit and of head sizes the tensor-core kernels do not have.
//
// Keys are addressed by position: the cache row of position j is j mod ring_rows (a cache that holds
// no more than a window), or j.  Position i of a sequence sees the positions
//   max(first[b], i - window + 1) .. i.
#include <cuda.h>

#include "common.cuh"

namespace eb {
namespace {

constexpr float kLog2eLat = 1.4426950408889634f;

__device__ __forceinline__ uint32_t lat_s32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lat_ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lat_ldm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
template <typename T> __device__ __forceinline__ void lat_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1);
template <> __device__ __forceinline__ void lat_mma<__half>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <> __device__ __forceinline__ void lat_mma<__nv_bfloat16>(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LatentParams {
  const void *q;               // [B][heads * R]
  long long q_bs;
  const void *c;               // cache [B][ring_rows][>= R]
  long long c_bs, c_ld;
  int ring_rows;
  void *o;                     // [B][heads * R]
  long long o_bs;
  int heads, window, nsplit;
  const int *pos_dev;          // position of the query, the same for every sequence
  const int *first;            // [B] first position of each sequence, or null
  float scale_log2;
  const float *sinks;          // per head: exp of it joins the softmax denominator, or null
  float *part_o;               // [B][heads][nsplit][R]; null: the splits are a cluster
  float *part_ml;              // [B][heads][nsplit][2]
};

constexpr int kLatKeys = 64, kLatThreads = 256, kLatWarps = 8;
constexpr int kSubBytes = kLatKeys * 128;          // 64 cache rows x 64 columns, 128-byte swizzled rows
constexpr unsigned long long kLatWaitNs = 1000ull * 1000ull * 1000ull;
constexpr int kLatHead = 1024;                     // barriers, abort flag, merge factors

__device__ int g_lat_status[4];                    // [0] code, [1] where, [2] block, [3] detail

__device__ __forceinline__ unsigned long long lat_timer() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ bool lat_try(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok != 0;
}
// Bounded wait; false when it ran out (recorded) or another thread's did.
__device__ __noinline__ bool lat_wait_slow(uint32_t bar, uint32_t parity, volatile int *abort_flag) {
  const unsigned long long t0 = lat_timer();
  for (unsigned it = 1;; ++it) {
    if (lat_try(bar, parity)) return true;
    if ((it & 63u) == 0) {
      if (*abort_flag) return false;
      if (lat_timer() - t0 > kLatWaitNs) {
        *abort_flag = 1;
        if (atomicCAS(&g_lat_status[0], 0, EB_ETIMEDOUT) == 0) {
          g_lat_status[1] = 1;
          g_lat_status[2] = blockIdx.x;
          g_lat_status[3] = (int)parity;
        }
        return false;
      }
    }
  }
}
// Byte offset of 16-byte chunk `ch` of row `row` in a tile of 64-column sub-tiles as TMA writes them.
__device__ __forceinline__ uint32_t lat_tile_off(int row, int ch, int sub_bytes) {
  return (uint32_t)((ch >> 3) * sub_bytes + row * 128 + (((ch & 7) ^ (row & 7)) << 4));
}
// The same inside a tile of `bytes` per row (P: 64 keys, 128 bytes).
__device__ __forceinline__ uint32_t lat_off(int row, int ch, int bytes) { return (uint32_t)(row * bytes + ((ch ^ (row & 7)) << 4)); }
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t cluster_addr(uint32_t local, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local), "r"(rank));
  return r;
}
__device__ __forceinline__ float cluster_ld(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr));
  return v;
}
__device__ __forceinline__ float4 cluster_ld4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr));
  return v;
}

// R: latent width (multiple of 64, at most 576); MT: 16-head tiles per CTA (1 or 2).
//
// The visible positions lie in a cyclic range of cache rows; the CTA walks its share of the 64-row
// tiles of that range in ROW order (a softmax does not care about order), so a tile is one
// TMA copy whether or not the ring has wrapped, and rows that are not visible are
// masked by their distance to the query's row.  Three tiles are in flight; a stage is free once
// every warp has passed the barrier behind its last read, so thread 0 refills it right there.
// The scores of tile i + 1 and the value product of tile i are independent and issued together.
//
// Splits up to 8 form a cluster: every CTA leaves its partial output in shared memory and adds up a
// slice of the columns of all of them (distributed shared memory).  More splits go through global
// memory and latent_merge_kernel.
//
// Shared memory: [head][3 stages of R/64 sub-tiles][P: MT*16 x 64][row maxima, row sums]; the queries
// pass through stage 2 on their way to registers, the partial output through stage 0.
template <int R, int MT> struct LatSmem {
  static constexpr int kStage = (R / 64) * kSubBytes;
  static constexpr int kP = MT * 16 * kLatKeys * 2;
  static constexpr size_t kTotal = 1024 + kLatHead + 3 * (size_t)kStage + kP + 2 * (size_t)kLatWarps * 16 * MT * sizeof(float);
  static_assert(MT * 16 * R * 2 <= kStage && MT * 16 * R * 4 <= 2 * kStage, "the queries and the partial output fit the stages they pass through");
  static_assert(kTotal <= 227 * 1024, "shared memory");
};

template <typename T, int R, int MT>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_c, const LatentParams p) {
  constexpr int kStage = LatSmem<R, MT>::kStage;
  constexpr int kNT = MT;                          // 8-key tiles per warp in the score product
  constexpr int kChains = 4 / kNT;                 // independent accumulators per key tile
  constexpr int kWarpCols = R / kLatWarps;         // output columns per warp: 8..64
  constexpr int kON = kWarpCols / 8;               // 8-column tiles per warp
  extern __shared__ uint8_t lat_raw[];
  uint8_t *sm = lat_raw + (((lat_s32(lat_raw) + 1023u) & ~1023u) - lat_s32(lat_raw));
  const uint32_t base = lat_s32(sm), s_c = base + kLatHead, s_p = s_c + 3 * kStage;
  uint8_t *p_ptr = sm + kLatHead + 3 * kStage;
  float *s_max = reinterpret_cast<float *>(p_ptr + LatSmem<R, MT>::kP), *s_sum = s_max + kLatWarps * 16 * MT;
  volatile int *abort_flag = reinterpret_cast<volatile int *>(sm + 32);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int split = blockIdx.x, h0 = blockIdx.y * 16 * MT, b = blockIdx.z;
  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tm_c) : "memory");
    for (int s = 0; s < 3; ++s) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(base + 8 * s) : "memory");
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  griddep_wait();
  griddep_launch();

  // visible range, as cache rows: n_keys rows that end with the query's row pr
  const int pos = *p.pos_dev, cap = p.ring_rows;
  int lo = p.first ? p.first[b] : 0;
  if (p.window > 0) lo = max(lo, pos - p.window + 1);
  lo = max(max(lo, pos - cap + 1), 0);
  const int n_keys = max(0, pos + 1 - lo);
  const int pr = pos % cap, row_lo = lo % cap;
  int tile_a = row_lo / kLatKeys, tiles_all = (cap + kLatKeys - 1) / kLatKeys, ntiles = 0;
  if (n_keys > 0) {
    if (row_lo + n_keys <= cap) ntiles = (row_lo + n_keys - 1) / kLatKeys - tile_a + 1;
    else {                                          // the range wraps: up to the last tile, then from row 0 on
      const int c = (row_lo + n_keys - cap - 1) / kLatKeys;
      ntiles = tiles_all - tile_a + (c == tile_a ? c : c + 1);
    }
  }
  const int t0 = (int)((long long)ntiles * split / p.nsplit), t1 = (int)((long long)ntiles * (split + 1) / p.nsplit);
  auto tile_row = [&](int i) {
    const int t = tile_a + i;
    return (t >= tiles_all ? t - tiles_all : t) * kLatKeys;
  };
  auto load = [&](int i) {                          // thread 0
    const int st = (i - t0) % 3;
    const uint32_t bar = base + 8 * st, dst = s_c + st * kStage;
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(kStage) : "memory");
    const int row = tile_row(i);
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];"
                 ::"r"(dst), "l"(&tm_c), "r"(0), "r"(row), "r"(0), "r"(b), "r"(bar) : "memory");
  };
  if (threadIdx.x == 0) {
    if (t0 < t1) load(t0);
    if (t0 + 1 < t1) load(t0 + 1);
  }

  // queries (rows beyond the heads are zero) -> stage 2 -> registers
  const T *qb = reinterpret_cast<const T *>(p.q) + (long long)b * p.q_bs;
  for (int i = threadIdx.x; i < MT * 16 * (R / 8); i += kLatThreads) {
    const int r = i / (R / 8), ch = i % (R / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h0 + r < p.heads) v = *reinterpret_cast<const uint4 *>(qb + (long long)(h0 + r) * R + ch * 8);
    *reinterpret_cast<uint4 *>(sm + kLatHead + 2 * kStage + lat_tile_off(r, ch, MT * 16 * 128)) = v;
  }
  __syncthreads();
  // warp -> (16-head tile, key group) of the score product
  const int mt = MT == 1 ? 0 : warp >> 2, kg = MT == 1 ? warp : warp & 3;
  uint32_t qf[R / 16][4];
#pragma unroll
  for (int k = 0; k < R / 16; ++k)
    lat_ldm4(qf[k], s_c + 2 * kStage + lat_tile_off(mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, k * 2 + (lane >> 4), MT * 16 * 128));
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // stage 2 was written by threads, TMA writes it next
  __syncthreads();
  if (threadIdx.x == 0 && t0 + 2 < t1) load(t0 + 2);

  float acc[MT][kON][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < kON; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  // running maximum of head rows g and g + 8 of every 16-head tile (all warps keep the same
  // values), this warp's share of the row sums of its own tile
  float m_run[MT][2], l_run[2] = {0.f, 0.f};
#pragma unroll
  for (int m = 0; m < MT; ++m) m_run[m][0] = m_run[m][1] = -1e30f;
  if (p.sinks && split == 0) {                      // a score that every head has seen already; one thread per row counts it
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int h = h0 + m * 16 + g + e * 8;
        if (h < p.heads) {
          m_run[m][e] = p.sinks[h] * kLog2eLat;
          if (m == mt && kg == 0 && tq == 0) l_run[e] = 1.f;
        }
      }
  }
  const int key_w = kg * 8 * kNT;
  // A wait that ran out is not acted on before the end: the barriers below stay matched, the
  // remaining waits are skipped, the result is unspecified and the status word says so.
  bool dead = false;
  float s[kNT][4];
  // scores of this warp's keys of tile i (in flight or landed), scaled, hidden keys at -inf
  auto scores = [&](int i) {
    const int st = (i - t0) % 3;
    const uint32_t bar = base + 8 * st, cs = s_c + st * kStage, parity = ((i - t0) / 3) & 1;
    if (!dead && !lat_try(bar, parity)) dead = !lat_wait_slow(bar, parity, abort_flag);
    dead = __any_sync(0xffffffffu, dead);
    float c[kNT][kChains][4];
#pragma unroll
    for (int n = 0; n < kNT; ++n)
#pragma unroll
      for (int j = 0; j < kChains; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) c[n][j][e] = 0.f;
#pragma unroll
    for (int k = 0; k < R / 32; ++k)
#pragma unroll
      for (int n = 0; n < kNT; ++n) {
        uint32_t bf[4];                            // 8 keys x 32 columns
        lat_ldm4(bf, cs + lat_tile_off(key_w + n * 8 + (lane & 7), k * 4 + (lane >> 3), kSubBytes));
        lat_mma<T>(c[n][(2 * k) % kChains], qf[2 * k], bf[0], bf[1]);
        lat_mma<T>(c[n][(2 * k + 1) % kChains], qf[2 * k + 1], bf[2], bf[3]);
      }
    const int row = tile_row(i) + key_w;
#pragma unroll
    for (int n = 0; n < kNT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = c[n][0][e];
#pragma unroll
        for (int j = 1; j < kChains; ++j) v += c[n][j][e];
        const int r = row + n * 8 + tq * 2 + (e & 1);
        const int d = pr - r, back = d < 0 ? d + cap : d;               // positions before the query
        s[n][e] = (r < cap && back < n_keys) ? v * p.scale_log2 : -INFINITY;
      }
  };
  if (t0 < t1) scores(t0);
#pragma unroll 1
  for (int i = t0; i < t1; ++i) {
    const uint32_t cs = s_c + ((i - t0) % 3) * kStage;
    float mx0 = -1e30f, mx1 = -1e30f;
#pragma unroll
    for (int n = 0; n < kNT; ++n) {
      mx0 = fmaxf(mx0, fmaxf(s[n][0], s[n][1]));
      mx1 = fmaxf(mx1, fmaxf(s[n][2], s[n][3]));
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, o));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, o));
    }
    if (tq == 0) {
      s_max[(mt * 8 + kg) * 16 + g] = mx0;
      s_max[(mt * 8 + kg) * 16 + g + 8] = mx1;
    }
    __syncthreads();
    // every warp is through with tile i - 1: its stage takes tile i + 2 (the first two are requested above)
    if (threadIdx.x == 0 && i > t0 && i + 2 < t1) load(i + 2);
    float alpha[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float v = m_run[m][e];
#pragma unroll
        for (int w = 0; w < kLatWarps / MT; ++w) v = fmaxf(v, s_max[(m * 8 + w) * 16 + g + e * 8]);
        alpha[m][e] = exp2f(m_run[m][e] - v);
        m_run[m][e] = v;
      }
    // probabilities of this warp's keys -> shared memory (operand type); sums in fp32
    const float m0 = MT == 1 ? m_run[0][0] : (mt ? m_run[MT - 1][0] : m_run[0][0]);
    const float m1 = MT == 1 ? m_run[0][1] : (mt ? m_run[MT - 1][1] : m_run[0][1]);
    l_run[0] *= MT == 1 ? alpha[0][0] : (mt ? alpha[MT - 1][0] : alpha[0][0]);
    l_run[1] *= MT == 1 ? alpha[0][1] : (mt ? alpha[MT - 1][1] : alpha[0][1]);
#pragma unroll
    for (int n = 0; n < kNT; ++n) {
      const float p0 = exp2f(s[n][0] - m0), p1 = exp2f(s[n][1] - m0), p2 = exp2f(s[n][2] - m1), p3 = exp2f(s[n][3] - m1);
      l_run[0] += p0 + p1;
      l_run[1] += p2 + p3;
      const int col = key_w + n * 8 + tq * 2, r0 = mt * 16 + g, r1 = r0 + 8;
      *reinterpret_cast<uint32_t *>(p_ptr + lat_off(r0, col >> 3, 128) + (col & 7) * 2) = pack2<T>(p0, p1);
      *reinterpret_cast<uint32_t *>(p_ptr + lat_off(r1, col >> 3, 128) + (col & 7) * 2) = pack2<T>(p2, p3);
    }
    __syncthreads();
    // O = alpha * O + P . C over this warp's columns, beside the scores of the next tile
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < kON; ++n) {
        acc[m][n][0] *= alpha[m][0];
        acc[m][n][1] *= alpha[m][0];
        acc[m][n][2] *= alpha[m][1];
        acc[m][n][3] *= alpha[m][1];
      }
#pragma unroll
    for (int k = 0; k < kLatKeys / 16; ++k) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        lat_ldm4(pf[m], s_p + lat_off(m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, k * 2 + (lane >> 4), 128));
#pragma unroll
      for (int n = 0; n < kON; n += 2) {
        uint32_t vf[4];
        // 16 keys x 16 columns: matrices (keys 0-7, cols 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15);
        // for the last of an odd number of 8-column tiles the upper half of the lanes repeats the lower's rows
        const int ch = kON >= 2 ? warp * kON + min(n + (lane >> 4), kON - 1) : warp;
        lat_ldm4t(vf, cs + lat_tile_off(k * 16 + (lane & 15), ch, kSubBytes));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          lat_mma<T>(acc[m][n], pf[m], vf[0], vf[1]);
          if (n + 1 < kON) lat_mma<T>(acc[m][n + 1 < kON ? n + 1 : n], pf[m], vf[2], vf[3]);
        }
      }
    }
    if (i + 1 < t1) scores(i + 1);
  }

  // ---- row sums over the key groups ----
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    if (tq == 0) s_sum[(mt * 8 + kg) * 16 + g + e * 8] = l_run[e];
  }
  __syncthreads();
  const bool clustered = p.nsplit > 1 && !p.part_o;
  float *part = reinterpret_cast<float *>(sm + kLatHead);               // [MT*16][R] over the stages
  float *f_m = reinterpret_cast<float *>(sm + 64), *f_l = f_m + 16 * MT;  // this CTA's maxima and sums, for its cluster
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = m * 16 + g + e * 8, h = h0 + r, col = warp * kWarpCols + tq * 2;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < kLatWarps / MT; ++w) l += s_sum[(m * 8 + w) * 16 + g + e * 8];
      if (clustered) {
#pragma unroll
        for (int n = 0; n < kON; ++n) *reinterpret_cast<float2 *>(part + r * R + col + n * 8) = make_float2(acc[m][n][e * 2], acc[m][n][e * 2 + 1]);
        if (warp == 0 && tq == 0) { f_m[r] = m_run[m][e]; f_l[r] = l; }
      } else if (h < p.heads && p.nsplit == 1) {
        const float inv = l > 0.f ? 1.f / l : 0.f;
        T *o = reinterpret_cast<T *>(p.o) + (long long)b * p.o_bs + (long long)h * R + col;
#pragma unroll
        for (int n = 0; n < kON; ++n) *reinterpret_cast<uint32_t *>(o + n * 8) = pack2<T>(acc[m][n][e * 2] * inv, acc[m][n][e * 2 + 1] * inv);
      } else if (h < p.heads) {
        const long long at = ((long long)b * p.heads + h) * p.nsplit + split;
        float *o = p.part_o + at * R + col;
#pragma unroll
        for (int n = 0; n < kON; ++n) *reinterpret_cast<float2 *>(o + n * 8) = make_float2(acc[m][n][e * 2], acc[m][n][e * 2 + 1]);
        if (warp == 0 && tq == 0) {
          p.part_ml[at * 2] = m_run[m][e];
          p.part_ml[at * 2 + 1] = l;
        }
      }
    }
  if (clustered) {
    float *f_scale = s_max;                                            // [nsplit][16 * MT]
    cluster_sync_all();
    if (threadIdx.x < 16 * MT) {
      const int r = threadIdx.x;
      float pm[8], pl[8], M = -1e30f, L = 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < p.nsplit) {
          pm[c] = cluster_ld(cluster_addr(lat_s32(f_m + r), c));
          pl[c] = cluster_ld(cluster_addr(lat_s32(f_l + r), c));
          M = fmaxf(M, pm[c]);
        }
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < p.nsplit) L += exp2f(pm[c] - M) * pl[c];
      const float inv = L > 0.f ? 1.f / L : 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < p.nsplit) f_scale[c * 16 * MT + r] = exp2f(pm[c] - M) * inv;
    }
    __syncthreads();
    // this CTA's columns of every head: R / nsplit of them, four at a time
    const int cols4 = R / p.nsplit / 4, c_first = split * (R / p.nsplit);
    for (int i = threadIdx.x; i < 16 * MT * cols4; i += kLatThreads) {
      const int r = i / cols4, col = c_first + (i - r * cols4) * 4;
      if (h0 + r >= p.heads) continue;
      const uint32_t at = lat_s32(part + r * R + col);
      float4 v[8];
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < p.nsplit) v[c] = cluster_ld4(cluster_addr(at, c));
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < p.nsplit) {
          const float f = f_scale[c * 16 * MT + r];
          o.x = fmaf(f, v[c].x, o.x); o.y = fmaf(f, v[c].y, o.y); o.z = fmaf(f, v[c].z, o.z); o.w = fmaf(f, v[c].w, o.w);
        }
      T *dst = reinterpret_cast<T *>(p.o) + (long long)b * p.o_bs + (long long)(h0 + r) * R + col;
      *reinterpret_cast<uint2 *>(dst) = make_uint2(pack2<T>(o.x, o.y), pack2<T>(o.z, o.w));
    }
    cluster_sync_all();                                                // nobody leaves while a peer still reads
  }
  if (__syncthreads_or(dead)) {
    // grace period for copies that may still be in flight to this CTA's shared memory
    const unsigned long long w0 = lat_timer();
    while (lat_timer() - w0 < 2000000ull) __nanosleep(1000);
  }
}

// o[b][h] = sum_split 2^(m - M) o_split / sum_split 2^(m - M) l_split
template <typename T>
__global__ void latent_merge_kernel(const LatentParams p, int R) {
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x, b = blockIdx.y;
  const long long part0 = ((long long)b * p.heads + h) * p.nsplit;
  extern __shared__ float f_scale[];               // [nsplit] factors 2^(m - M) / L
  if (threadIdx.x < 32) {
    const float2 *ml = reinterpret_cast<const float2 *>(p.part_ml) + part0;
    float M = -1e30f, L = 0.f;
    for (int i = threadIdx.x; i < p.nsplit; i += 32) M = fmaxf(M, ml[i].x);
    M = warp_max(M);
    for (int i = threadIdx.x; i < p.nsplit; i += 32) {
      const float f = exp2f(ml[i].x - M);
      f_scale[i] = f;
      L += f * ml[i].y;
    }
    L = warp_sum(L);
    const float inv = L > 0.f ? 1.f / L : 0.f;
    for (int i = threadIdx.x; i < p.nsplit; i += 32) f_scale[i] *= inv;
  }
  // the parts are requested before the factors are known
  const int d = threadIdx.x * 4;
  const float4 *src = reinterpret_cast<const float4 *>(p.part_o + part0 * R + d);
  float4 v[8], o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int i0 = 0; i0 < p.nsplit; i0 += 8) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i0 + i < p.nsplit && d < R) v[i] = src[(long long)(i0 + i) * (R / 4)];
    if (i0 == 0) __syncthreads();                  // (every thread comes here)
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i0 + i < p.nsplit) {
        const float f = f_scale[i0 + i];
        o.x = fmaf(f, v[i].x, o.x); o.y = fmaf(f, v[i].y, o.y); o.z = fmaf(f, v[i].z, o.z); o.w = fmaf(f, v[i].w, o.w);
      }
  }
  if (d >= R) return;
  T *dst = reinterpret_cast<T *>(p.o) + (long long)b * p.o_bs + (long long)h * R + d;
  *reinterpret_cast<uint2 *>(dst) = make_uint2(pack2<T>(o.x, o.y), pack2<T>(o.z, o.w));
}

typedef CUresult (*LatEncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// 4-D map (column in a block of 64, row, column block, batch) over the cache; one box holds 64 rows of
// all column blocks, each written as a sub-tile of 128-byte swizzled rows.  Rows behind the last one
// read as zeros.
int latent_map(CUtensorMap *map, const void *cache, int dtype, int R, int rows, int batch, long long row_stride, long long batch_stride) {
  static LatEncodeFn fn = nullptr;
  if (!fn) {
    void *sym = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<LatEncodeFn>(sym);
  }
  if (!fn) return fail(EB_ECUDA, "latent_decode: cuTensorMapEncodeTiled is not available from the driver");
  cuuint64_t dims[4] = {64, (cuuint64_t)rows, (cuuint64_t)(R / 64), (cuuint64_t)batch};
  cuuint64_t strides[3] = {(cuuint64_t)row_stride * 2, 128, (cuuint64_t)batch_stride * 2};
  cuuint32_t box[4] = {64, (cuuint32_t)kLatKeys, (cuuint32_t)(R / 64), 1}, estr[4] = {1, 1, 1, 1};
  CUresult r = fn(map, dtype == EB_BF16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 4, const_cast<void *>(cache), dims,
                  strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(EB_ECUDA, "latent_decode: cuTensorMapEncodeTiled failed with CUresult %d", (int)r);
  return EB_OK;
}

// Splits that are a power of two up to 8 form a cluster and need no scratch.
bool latent_clustered(int nsplit) { return nsplit == 2 || nsplit == 4 || nsplit == 8; }

template <typename T, int R, int MT>
int launch_latent(const CUtensorMap &map, const LatentParams &p, int B, cudaStream_t st) {
  constexpr size_t smem = LatSmem<R, MT>::kTotal;
  auto kern = latent_decode_kernel<T, R, MT>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "latent_decode: cannot reserve %zu bytes of shared memory", smem);
    }
    configured[dev] = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.nsplit, (p.heads + 16 * MT - 1) / (16 * MT), B);
  cfg.blockDim = dim3(kLatThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = p.part_o ? 1 : p.nsplit;
  attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  cudaLaunchKernelEx(&cfg, kern, map, p);
  if (int rc = check_launch("latent_decode")) return rc;
  if (p.part_o) {
    launch_pdl(latent_merge_kernel<T>, dim3(p.heads, B), dim3(R < 128 ? 32 : R / 4), p.nsplit * sizeof(float), st, p, R);
    return check_launch("latent_merge");
  }
  return EB_OK;
}

template <typename T, int R> int launch_latent_mt(const CUtensorMap &map, const LatentParams &p, int B, cudaStream_t st) {
  return p.heads > 16 ? launch_latent<T, R, 2>(map, p, B, st) : launch_latent<T, R, 1>(map, p, B, st);
}

template <typename T> int launch_latent_r(const CUtensorMap &map, const LatentParams &p, int B, int R, cudaStream_t st) {
  switch (R) {
    case 64: return launch_latent_mt<T, 64>(map, p, B, st);
    case 128: return launch_latent_mt<T, 128>(map, p, B, st);
    case 192: return launch_latent_mt<T, 192>(map, p, B, st);
    case 256: return launch_latent_mt<T, 256>(map, p, B, st);
    case 320: return launch_latent_mt<T, 320>(map, p, B, st);
    case 384: return launch_latent_mt<T, 384>(map, p, B, st);
    case 512: return launch_latent_mt<T, 512>(map, p, B, st);
    default: return launch_latent_mt<T, 576>(map, p, B, st);
  }
}

// ---- plain attention -------------------------------------------------------------------------------
struct PlainParams {
  const void *q, *k, *v;
  void *o;
  long long q_bs, q_rs, q_hs, k_bs, k_rs, k_hs, v_bs, v_rs, v_hs, o_bs, o_rs, o_hs;
  int heads, q_len, dk, dv, window, ring_rows;
  const int *pos_dev;          // position of query row 0, or null (0)
  const int *first;
  float scale_log2;
  int group;                   // query heads per key / value head
  const float *r1, *r2;        // per head: r1 * ln(1 + r2 * distance) is taken off the score, or null
  int sink;                    // one is added to the softmax denominator
  const float *sinks;          // per head: exp of it is (instead of one)
  int chunk;                   // > 0: a position sees only its own chunk of so many, counted from first
  int keep, kept_rows;         // the first `keep` positions stay visible; cache rows in front of the ring that hold them
  const float *slopes;         // per head: slope * distance is taken off the score, or null
  float cap_log2, inv_cap;     // score <- cap tanh(score / cap), or inv_cap 0
};

// tanh of a score over its cap: of 32-bit models by the library (not the approximation that fast math puts in its
// place, whose error the cap would multiply)
template <typename T> __device__ __forceinline__ float capped_tanh(float x) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * x)); }
template <> __device__ __forceinline__ float capped_tanh<float>(float x) {
  const float a = fabsf(x), e = expm1f(-2.f * a);
  return copysignf(__fdiv_rn(-e, 2.f + e), x);
}

template <typename T>
__global__ void attention_plain_kernel(const PlainParams p) {
  extern __shared__ float pl_smem[];
  griddep_wait();
  griddep_launch();
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int i = blockIdx.x * warps + warp, h = blockIdx.y, b = blockIdx.z;
  if (i >= p.q_len) return;
  float *sq = pl_smem + (long long)warp * (p.dk + p.dv), *so = sq + p.dk;
  const T *q = reinterpret_cast<const T *>(p.q) + b * p.q_bs + i * p.q_rs + h * p.q_hs;
  for (int d = lane; d < p.dk; d += 32) sq[d] = to_f32<T>(q[d]);
  for (int d = lane; d < p.dv; d += 32) so[d] = 0.f;
  __syncwarp();
  const int pos = (p.pos_dev ? *p.pos_dev : 0) + i;
  int lo = p.first ? p.first[b] : 0;
  if (p.window > 0) lo = max(lo, pos - p.window + 1);
  if (p.chunk > 0 && pos > lo) lo += (pos - lo) / p.chunk * p.chunk;
  lo = max(lo, max(0, pos - p.ring_rows + 1));
  const int start = p.first ? min(p.first[b], lo) : 0, kept = min(p.keep, lo - start), count = kept + pos + 1 - lo;
  // entry n of what is visible: its position, and its row
  auto position = [&](int n) { return n < kept ? start + n : lo + n - kept; };
  auto row_of = [&](int n) {
    if (n < kept && p.kept_rows > 0) return (long long)n;
    return (long long)(p.kept_rows + position(n) % p.ring_rows);
  };
  const T *K = reinterpret_cast<const T *>(p.k) + b * p.k_bs + h / p.group * p.k_hs, *V = reinterpret_cast<const T *>(p.v) + b * p.v_bs + h / p.group * p.v_hs;
  const float r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f, slope = p.slopes ? p.slopes[h] * kLog2eLat : 0.f;
  float m = p.sinks ? p.sinks[h] * kLog2eLat : p.sink ? 0.f : -1e30f, l = p.sinks || p.sink ? 1.f : 0.f;      // the sink: a score without a value
  for (int n0 = 0; n0 < count; n0 += 32) {
    float s = -INFINITY;
    if (n0 + lane < count) {
      const int j = position(n0 + lane);
      const T *kr = K + row_of(n0 + lane) * p.k_rs;
      float a = 0.f;
      for (int d = 0; d < p.dk; ++d) a = fmaf(sq[d], to_f32<T>(kr[d]), a);
      s = a * p.scale_log2;
      if (p.inv_cap > 0.f) s = p.cap_log2 * capped_tanh<T>(a * p.inv_cap);
      if (p.r1) s -= r1 * log2f(fmaf(r2, (float)(pos - j), 1.f));
      s -= slope * (float)(pos - j);
    }
    const float mn = fmaxf(m, warp_max(s)), alpha = exp2f(m - mn), pj = exp2f(s - mn);
    m = mn;
    l = l * alpha + warp_sum(pj);
    const int n = min(32, count - n0);
    for (int d = lane; d - lane < p.dv; d += 32) {
      float a = d < p.dv ? so[d] * alpha : 0.f;
      for (int jj = 0; jj < n; ++jj) {
        const float w = __shfl_sync(0xffffffffu, pj, jj);
        if (d < p.dv) a = fmaf(w, to_f32<T>(V[row_of(n0 + jj) * p.v_rs + d]), a);
      }
      if (d < p.dv) so[d] = a;
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T *o = reinterpret_cast<T *>(p.o) + b * p.o_bs + i * p.o_rs + h * p.o_hs;
  for (int d = lane; d < p.dv; d += 32) o[d] = from_f32<T>(so[d] * inv);
}

template <typename T> int launch_plain(const PlainParams &p, int B, cudaStream_t st) {
  int warps = 4;
  const size_t per = (size_t)(p.dk + p.dv) * sizeof(float);
  while (warps > 1 && warps * per > 48 * 1024) warps >>= 1;
  if (warps * per > 48 * 1024)
    return fail(EB_EUNSUPPORTED, "attention_plain: head sizes %d / %d are too large", p.dk, p.dv);
  launch_pdl(attention_plain_kernel<T>, dim3((p.q_len + warps - 1) / warps, p.heads, B), dim3(warps * 32), warps * per, st, p);
  return check_launch("attention_plain");
}

}  // namespace

// Status words of this file's kernels, for eb_device_status.
int latent_status(int *out4, bool clear) {
  int host[4] = {0, 0, 0, 0};
  if (cudaMemcpyFromSymbol(host, g_lat_status, sizeof(host)) != cudaSuccess) {
    cudaGetLastError();
    return EB_ECUDA;
  }
  for (int i = 0; i < 4; ++i) out4[i] = host[i];
  if (clear && host[0] != 0) {
    int zero[4] = {0, 0, 0, 0};
    cudaMemcpyToSymbol(g_lat_status, zero, sizeof(zero));
  }
  return EB_OK;
}

}  // namespace eb

using namespace eb;

extern "C" size_t eb_latent_decode_scratch_bytes(int batch, int heads, int rank, int nsplit) {
  if (batch <= 0 || heads <= 0 || rank <= 0 || nsplit <= 1 || latent_clustered(nsplit)) return 0;
  return (size_t)batch * heads * nsplit * (rank + 2) * sizeof(float);
}

extern "C" int eb_latent_decode(const void *q, long long q_batch_stride, const void *cache, long long cache_batch_stride,
                                long long cache_row_stride, int ring_rows, void *out, long long out_batch_stride, int batch, int heads,
                                int rank, int window, const int32_t *pos_device, const int32_t *first, float scale, int dtype,
                                int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  return eb_latent_decode_sink(q, q_batch_stride, cache, cache_batch_stride, cache_row_stride, ring_rows, out, out_batch_stride, batch, heads, rank, window,
                               pos_device, first, nullptr, scale, dtype, nsplit, scratch, scratch_bytes, stream);
}

extern "C" int eb_latent_decode_sink(const void *q, long long q_batch_stride, const void *cache, long long cache_batch_stride,
                                long long cache_row_stride, int ring_rows, void *out, long long out_batch_stride, int batch, int heads,
                                int rank, int window, const int32_t *pos_device, const int32_t *first, const float *sinks, float scale, int dtype,
                                int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  if (batch == 0 || heads == 0) return EB_OK;
  EB_REQUIRE(dtype == EB_F16 || dtype == EB_BF16, "latent_decode: fp16 or bf16 only (dtype %d)", dtype);
  EB_REQUIRE(rank == 64 || rank == 128 || rank == 192 || rank == 256 || rank == 320 || rank == 384 || rank == 512 || rank == 576,
             "latent_decode: latent width %d not supported (64, 128, 192, 256, 320, 384, 512 or 576)", rank);
  EB_REQUIRE(batch > 0 && batch <= 65535 && heads > 0 && ring_rows > 0 && window >= 0 && nsplit >= 1 && nsplit <= 1024, "latent_decode: bad sizes");
  EB_REQUIRE(q && cache && out && pos_device, "latent_decode: null pointer");
  EB_REQUIRE(aligned16(q) && aligned16(cache) && aligned16(out), "latent_decode: pointers must be 16-byte aligned");
  EB_REQUIRE(q_batch_stride % 8 == 0 && cache_batch_stride % 8 == 0 && cache_row_stride % 8 == 0 && cache_row_stride >= rank &&
                 out_batch_stride % 8 == 0, "latent_decode: strides must be multiples of 8 elements");
  LatentParams p{};
  p.q = q; p.q_bs = q_batch_stride; p.c = cache; p.c_bs = cache_batch_stride; p.c_ld = cache_row_stride; p.ring_rows = ring_rows;
  p.o = out; p.o_bs = out_batch_stride; p.heads = heads; p.window = window; p.nsplit = nsplit;
  p.pos_dev = pos_device; p.first = first; p.sinks = sinks; p.scale_log2 = scale * kLog2eLat;
  if (nsplit > 1 && !latent_clustered(nsplit)) {
    const size_t need = eb_latent_decode_scratch_bytes(batch, heads, rank, nsplit);
    EB_REQUIRE(scratch && scratch_bytes >= need && aligned16(scratch), "latent_decode: %d splits need a scratch of %zu bytes", nsplit, need);
    p.part_o = reinterpret_cast<float *>(scratch);
    p.part_ml = p.part_o + (size_t)batch * heads * nsplit * rank;
  }
  cudaStream_t st = as_stream(stream);
  CUtensorMap map;
  if (int rc = latent_map(&map, cache, dtype, rank, ring_rows, batch, cache_row_stride, cache_batch_stride)) return rc;
  return dtype == EB_F16 ? launch_latent_r<__half>(map, p, batch, rank, st) : launch_latent_r<__nv_bfloat16>(map, p, batch, rank, st);
}

static int plain_impl(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                                  long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                                  long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                                  long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                                  int v_dim, int window, int ring_rows, const int32_t *pos_device, const int32_t *first, const float *bias_r1,
                                  const float *bias_r2, int sink, const float *sinks, int chunk, float scale, int dtype, void *stream,
                                  int keep = 0, int kept_rows = 0, const float *slopes = nullptr, float cap = 0.f) {
  if (batch == 0 || heads == 0 || q_len == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "attention_plain: bad dtype %d", dtype);
  EB_REQUIRE(q && k && v && out, "attention_plain: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && heads > 0 && heads <= 65535 && q_len > 0 && k_dim > 0 && v_dim > 0 && window >= 0 && ring_rows > 0,
             "attention_plain: bad sizes");
  EB_REQUIRE(kv_group > 0 && heads % kv_group == 0, "attention_plain: %d heads do not share keys in groups of %d", heads, kv_group);
  EB_REQUIRE((bias_r1 == nullptr) == (bias_r2 == nullptr), "attention_plain: the distance bias has two numbers per head");
  PlainParams p{};
  EB_REQUIRE(keep >= 0 && (kept_rows == 0 || kept_rows == keep) && cap >= 0.f, "attention_plain: a cache keeps all %d first positions or none", keep);
  p.group = kv_group; p.r1 = bias_r1; p.r2 = bias_r2; p.sink = sink; p.sinks = sinks; p.chunk = chunk;
  p.keep = keep; p.kept_rows = kept_rows; p.slopes = slopes;
  if (cap > 0.f) { p.cap_log2 = cap * kLog2eLat; p.inv_cap = scale / cap; }
  p.q = q; p.k = k; p.v = v; p.o = out;
  p.q_bs = q_batch_stride; p.q_rs = q_row_stride; p.q_hs = q_head_stride;
  p.k_bs = k_batch_stride; p.k_rs = k_row_stride; p.k_hs = k_head_stride;
  p.v_bs = v_batch_stride; p.v_rs = v_row_stride; p.v_hs = v_head_stride;
  p.o_bs = o_batch_stride; p.o_rs = o_row_stride; p.o_hs = o_head_stride;
  p.heads = heads; p.q_len = q_len; p.dk = k_dim; p.dv = v_dim; p.window = window; p.ring_rows = ring_rows;
  p.pos_dev = pos_device; p.first = first; p.scale_log2 = scale * kLog2eLat;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_plain<float>(p, batch, st);
  if (dtype == EB_F16) return launch_plain<__half>(p, batch, st);
  return launch_plain<__nv_bfloat16>(p, batch, st);
}

extern "C" int eb_attention_plain(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                                  long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                                  long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                                  long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                                  int v_dim, int window, int ring_rows, const int32_t *pos_device, const int32_t *first, const float *bias_r1,
                                  const float *bias_r2, int sink, float scale, int dtype, void *stream) {
  return plain_impl(q, k, v, out, q_batch_stride, q_row_stride, q_head_stride, k_batch_stride, k_row_stride, k_head_stride, v_batch_stride,
                    v_row_stride, v_head_stride, o_batch_stride, o_row_stride, o_head_stride, batch, heads, kv_group, q_len, k_dim, v_dim, window,
                    ring_rows, pos_device, first, bias_r1, bias_r2, sink, nullptr, 0, scale, dtype, stream);
}

extern "C" int eb_attention_plain_chunk(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                                  long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                                  long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                                  long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                                  int v_dim, int chunk, int ring_rows, const int32_t *pos_device, const int32_t *first,
                                  const float *sinks, float scale, int dtype, void *stream) {
  EB_REQUIRE(chunk >= 0, "attention_plain: a chunk of %d positions", chunk);
  return plain_impl(q, k, v, out, q_batch_stride, q_row_stride, q_head_stride, k_batch_stride, k_row_stride, k_head_stride, v_batch_stride,
                    v_row_stride, v_head_stride, o_batch_stride, o_row_stride, o_head_stride, batch, heads, kv_group, q_len, k_dim, v_dim, 0,
                    ring_rows, pos_device, first, nullptr, nullptr, 0, sinks, chunk, scale, dtype, stream);
}

extern "C" int eb_attention_plain_capped(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                                  long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                                  long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                                  long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                                  int v_dim, int window, int keep, int kept_rows, int ring_rows, const int32_t *pos_device, const int32_t *first,
                                  const float *slopes, float cap, int sink, float scale, int dtype, void *stream) {
  return plain_impl(q, k, v, out, q_batch_stride, q_row_stride, q_head_stride, k_batch_stride, k_row_stride, k_head_stride, v_batch_stride,
                    v_row_stride, v_head_stride, o_batch_stride, o_row_stride, o_head_stride, batch, heads, kv_group, q_len, k_dim, v_dim, window,
                    ring_rows, pos_device, first, nullptr, nullptr, sink, nullptr, 0, scale, dtype, stream, keep, kept_rows, slopes, cap);
}
