// Attention over a latent cache, and the plain windowed attention behind it.
//
//   latent_decode    one new position per sequence with the key and value projections absorbed into
//                    the query and the output: every head of a sequence reads the SAME cached row
//                    c_j (its key and its value), so the kernel is a pass over the visible part of
//                    the cache shared by 16 or 32 heads of a CTA:
//                       s[h][j] = scale * qa[h] . c_j,   o[h] = sum_j softmax_j(s[h]) c_j
//                    on mma.sync with fp32 scores, statistics and accumulators.  The key range is
//                    split over CTAs; a second small kernel merges the parts.
//   attention_plain  any head sizes, fp32 or 16 bit, one warp per query row: the path of models run
//                    in 32-bit and of head sizes the tensor-core kernels do not have.
//
// Keys are addressed by position: the cache row of position j is j mod ring_rows (a cache that holds
// no more than a window), or j.  Position i of a sequence sees the positions
//   max(first[b], i - window + 1) .. i.
#include "common.cuh"

namespace eb {
namespace {

constexpr float kLog2eLat = 1.4426950408889634f;

__device__ __forceinline__ uint32_t lat_s32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lat_cp16(uint32_t dst, const void *src, bool valid) {
  const int bytes = valid ? 16 : 0;   // source size 0 zero-fills the destination
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void lat_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void lat_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
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
  float *part_o;               // [B][heads][nsplit][R]
  float *part_ml;              // [B][heads][nsplit][2]
};

constexpr int kLatKeys = 64, kLatThreads = 256, kLatWarps = 8;

// Byte offset of 16-byte chunk `chunk` of row `row` in a tile of `bytes` per row, chunks XOR-ed with
// the row (conflict-free cp.async and ldmatrix; bytes is a multiple of 128).
__device__ __forceinline__ uint32_t lat_off(int row, int chunk, int bytes) { return (uint32_t)(row * bytes + ((chunk ^ (row & 7)) << 4)); }

// R: latent width (multiple of 64, at most 512); MT: 16-head tiles per CTA (1 or 2).
// Shared memory: [2 stages of 64 rows x R][queries MT*16 x R][P: MT*16 x 64][row maxima, row sums].
template <typename T, int R, int MT>
__global__ void __launch_bounds__(kLatThreads, 1) latent_decode_kernel(const LatentParams p) {
  constexpr int kRowB = R * 2, kChunks = R / 8;
  constexpr int kStage = kLatKeys * kRowB;
  constexpr int kNT = MT;                          // 8-key tiles per warp in the score product
  constexpr int kWarpCols = R / kLatWarps;         // output columns per warp: 8..64
  constexpr int kON = kWarpCols / 8;               // 8-column tiles per warp
  extern __shared__ __align__(128) uint8_t lat_smem[];
  const uint32_t s_c = lat_s32(lat_smem), s_q = s_c + 2 * kStage, s_p = s_q + MT * 16 * kRowB;
  float *s_max = reinterpret_cast<float *>(lat_smem + 2 * kStage + MT * 16 * kRowB + MT * 16 * kLatKeys * 2);   // [8 key groups][MT*16]
  float *s_sum = s_max + kLatWarps * 16 * MT;

  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int split = blockIdx.x, hg = blockIdx.y, b = blockIdx.z;
  const int h0 = hg * 16 * MT;
  const int pos = *p.pos_dev;
  int lo = p.first ? p.first[b] : 0;
  if (p.window > 0) lo = max(lo, pos - p.window + 1);
  // (a position outside the cache would be a caller's error; the range is clamped to what exists)
  lo = max(lo, pos - p.ring_rows + 1);
  lo = max(lo, 0);
  const int n_keys = max(0, pos + 1 - lo);
  const int ntiles = (n_keys + kLatKeys - 1) / kLatKeys;
  const int t0 = (int)((long long)ntiles * split / p.nsplit), t1 = (int)((long long)ntiles * (split + 1) / p.nsplit);

  const T *cb = reinterpret_cast<const T *>(p.c) + (long long)b * p.c_bs;
  const int ring0 = lo % p.ring_rows;
  auto load = [&](int tile, int stage) {
    for (int i = threadIdx.x; i < kLatKeys * kChunks; i += kLatThreads) {
      const int r = i / kChunks, ch = i % kChunks, k = tile * kLatKeys + r;
      int row = ring0 + k;
      if (row >= p.ring_rows) row -= p.ring_rows;
      const bool ok = k < n_keys;
      lat_cp16(s_c + stage * kStage + lat_off(r, ch, kRowB), cb + (ok ? (long long)row * p.c_ld + ch * 8 : 0), ok);
    }
    lat_commit();
  };

  // queries of this head group (rows beyond the heads are zero)
  const T *qb = reinterpret_cast<const T *>(p.q) + (long long)b * p.q_bs;
  for (int i = threadIdx.x; i < MT * 16 * kChunks; i += kLatThreads) {
    const int r = i / kChunks, ch = i % kChunks;
    const bool ok = h0 + r < p.heads;
    lat_cp16(s_q + lat_off(r, ch, kRowB), qb + (ok ? (long long)(h0 + r) * R + ch * 8 : 0), ok);
  }
  lat_commit();
  if (t0 < t1) load(t0, 0);
  lat_wait<0>();
  __syncthreads();

  // warp -> (16-head tile, key group) of the score product; its queries stay in registers
  const int mt = MT == 1 ? 0 : warp >> 2, kg = MT == 1 ? warp : warp & 3;
  uint32_t qf[R / 16][4];
#pragma unroll
  for (int k = 0; k < R / 16; ++k) {
    const int r = mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ch = k * 2 + (lane >> 4);
    lat_ldm4(qf[k], s_q + lat_off(r, ch, kRowB));
  }
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

  for (int t = t0; t < t1; ++t) {
    const int stage = (t - t0) & 1;
    const uint32_t cs = s_c + stage * kStage;
    if (t + 1 < t1) load(t + 1, stage ^ 1);        // the other stage was released by the barrier at the end of the last round
    // ---- scores of this warp's keys ----
    float s[kNT][4];
#pragma unroll
    for (int n = 0; n < kNT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
    const int key_w = kg * 8 * kNT;
#pragma unroll
    for (int k = 0; k < R / 32; ++k) {
#pragma unroll
      for (int n = 0; n < kNT; ++n) {
        uint32_t bf[4];                            // 8 keys x 32 columns
        lat_ldm4(bf, cs + lat_off(key_w + n * 8 + (lane & 7), k * 4 + (lane >> 3), kRowB));
        lat_mma<T>(s[n], qf[2 * k], bf[0], bf[1]);
        lat_mma<T>(s[n], qf[2 * k + 1], bf[2], bf[3]);
      }
    }
    float mx0 = -1e30f, mx1 = -1e30f;
#pragma unroll
    for (int n = 0; n < kNT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = t * kLatKeys + key_w + n * 8 + tq * 2 + (e & 1);
        s[n][e] = key < n_keys ? s[n][e] * p.scale_log2 : -INFINITY;
        if (e < 2) mx0 = fmaxf(mx0, s[n][e]);
        else mx1 = fmaxf(mx1, s[n][e]);
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
    // ---- new maxima, rescale factors ----
    constexpr int kGroups = kLatWarps / MT;
    float alpha[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float v = m_run[m][e];
#pragma unroll
        for (int w = 0; w < kGroups; ++w) v = fmaxf(v, s_max[(m * 8 + w) * 16 + g + e * 8]);
        alpha[m][e] = exp2f(m_run[m][e] - v);
        m_run[m][e] = v;
      }
    // ---- probabilities of this warp's keys -> shared memory (operand type) ----
    l_run[0] *= alpha[mt][0];
    l_run[1] *= alpha[mt][1];
#pragma unroll
    for (int n = 0; n < kNT; ++n) {
      const float p0 = exp2f(s[n][0] - m_run[mt][0]), p1 = exp2f(s[n][1] - m_run[mt][0]);
      const float p2 = exp2f(s[n][2] - m_run[mt][1]), p3 = exp2f(s[n][3] - m_run[mt][1]);
      l_run[0] += p0 + p1;
      l_run[1] += p2 + p3;
      const int col = key_w + n * 8 + tq * 2;
      const int r0 = mt * 16 + g, r1 = r0 + 8;
      *reinterpret_cast<uint32_t *>(lat_smem + (s_p - s_c) + lat_off(r0, col >> 3, 128) + (col & 7) * 2) = pack2<T>(p0, p1);
      *reinterpret_cast<uint32_t *>(lat_smem + (s_p - s_c) + lat_off(r1, col >> 3, 128) + (col & 7) * 2) = pack2<T>(p2, p3);
    }
    __syncthreads();
    // ---- O = alpha * O + P . C over this warp's columns ----
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
        if (kON >= 2) {
          // 16 keys x 16 columns: matrices (keys 0-7, cols 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
          lat_ldm4t(vf, cs + lat_off(k * 16 + (lane & 15), warp * (kWarpCols / 8) + n + (lane >> 4), kRowB));
        } else {
          // one 8-column tile per warp: the upper half of the lanes repeats the lower's rows
          lat_ldm4t(vf, cs + lat_off(k * 16 + (lane & 15), warp, kRowB));
        }
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          lat_mma<T>(acc[m][n], pf[m], vf[0], vf[1]);
          if (kON >= 2) lat_mma<T>(acc[m][n + (kON >= 2 ? 1 : 0)], pf[m], vf[2], vf[3]);
        }
      }
    }
    lat_wait<0>();
    __syncthreads();
  }

  // ---- row sums over the key groups ----
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    if (tq == 0) s_sum[(mt * 8 + kg) * 16 + g + e * 8] = l_run[e];
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = h0 + m * 16 + g + e * 8;
      if (h >= p.heads) continue;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < kLatWarps / MT; ++w) l += s_sum[(m * 8 + w) * 16 + g + e * 8];
      if (p.nsplit == 1) {
        const float inv = l > 0.f ? 1.f / l : 0.f;
        T *o = reinterpret_cast<T *>(p.o) + (long long)b * p.o_bs + (long long)h * R + warp * kWarpCols + tq * 2;
#pragma unroll
        for (int n = 0; n < kON; ++n)
          *reinterpret_cast<uint32_t *>(o + n * 8) = pack2<T>(acc[m][n][e * 2] * inv, acc[m][n][e * 2 + 1] * inv);
      } else {
        const long long part = ((long long)b * p.heads + h) * p.nsplit + split;
        float *o = p.part_o + part * R + warp * kWarpCols + tq * 2;
#pragma unroll
        for (int n = 0; n < kON; ++n) *reinterpret_cast<float2 *>(o + n * 8) = make_float2(acc[m][n][e * 2], acc[m][n][e * 2 + 1]);
        if (warp == 0 && tq == 0) {
          p.part_ml[part * 2] = m_run[m][e];
          p.part_ml[part * 2 + 1] = l;
        }
      }
    }
}

// o[b][h] = sum_split 2^(m - M) o_split / sum_split 2^(m - M) l_split
template <typename T>
__global__ void latent_merge_kernel(const LatentParams p, int R) {
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x, b = blockIdx.y;
  const long long part0 = ((long long)b * p.heads + h) * p.nsplit;
  const float *ml = p.part_ml + part0 * 2;
  float M = -1e30f, L = 0.f;
  for (int i = 0; i < p.nsplit; ++i) M = fmaxf(M, ml[2 * i]);
  for (int i = 0; i < p.nsplit; ++i) L += exp2f(ml[2 * i] - M) * ml[2 * i + 1];
  const float inv = L > 0.f ? 1.f / L : 0.f;
  for (int d = threadIdx.x; d < R; d += blockDim.x) {
    float v = 0.f;
#pragma unroll 4
    for (int i = 0; i < p.nsplit; ++i) v = fmaf(exp2f(ml[2 * i] - M), p.part_o[(part0 + i) * R + d], v);
    reinterpret_cast<T *>(p.o)[(long long)b * p.o_bs + (long long)h * R + d] = from_f32<T>(v * inv);
  }
}

template <typename T, int R, int MT>
int launch_latent(const LatentParams &p, int B, cudaStream_t st) {
  constexpr size_t smem = 2 * (size_t)kLatKeys * R * 2 + (size_t)MT * 16 * R * 2 + (size_t)MT * 16 * kLatKeys * 2 +
                          2 * (size_t)kLatWarps * 16 * MT * sizeof(float);
  static_assert(smem <= 227 * 1024, "shared memory");
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
  launch_pdl(kern, dim3(p.nsplit, (p.heads + 16 * MT - 1) / (16 * MT), B), dim3(kLatThreads), smem, st, p);
  if (int rc = check_launch("latent_decode")) return rc;
  if (p.nsplit > 1) {
    launch_pdl(latent_merge_kernel<T>, dim3(p.heads, B), dim3(R < 256 ? R : 256), 0, st, p, R);
    return check_launch("latent_merge");
  }
  return EB_OK;
}

template <typename T, int R> int launch_latent_mt(const LatentParams &p, int B, cudaStream_t st) {
  return p.heads > 16 ? launch_latent<T, R, 2>(p, B, st) : launch_latent<T, R, 1>(p, B, st);
}

template <typename T> int launch_latent_r(const LatentParams &p, int B, int R, cudaStream_t st) {
  switch (R) {
    case 64: return launch_latent_mt<T, 64>(p, B, st);
    case 128: return launch_latent_mt<T, 128>(p, B, st);
    case 256: return launch_latent_mt<T, 256>(p, B, st);
    case 384: return launch_latent_mt<T, 384>(p, B, st);
    default: return launch_latent_mt<T, 512>(p, B, st);
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
};

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
  lo = max(lo, max(0, pos - p.ring_rows + 1));
  const T *K = reinterpret_cast<const T *>(p.k) + b * p.k_bs + h * p.k_hs, *V = reinterpret_cast<const T *>(p.v) + b * p.v_bs + h * p.v_hs;
  float m = -1e30f, l = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    if (j <= pos) {
      const T *kr = K + (long long)(j % p.ring_rows) * p.k_rs;
      float a = 0.f;
      for (int d = 0; d < p.dk; ++d) a = fmaf(sq[d], to_f32<T>(kr[d]), a);
      s = a * p.scale_log2;
    }
    const float mn = fmaxf(m, warp_max(s)), alpha = exp2f(m - mn), pj = exp2f(s - mn);
    m = mn;
    l = l * alpha + warp_sum(pj);
    const int n = min(32, pos + 1 - j0);
    for (int d = lane; d - lane < p.dv; d += 32) {
      float a = d < p.dv ? so[d] * alpha : 0.f;
      for (int jj = 0; jj < n; ++jj) {
        const float w = __shfl_sync(0xffffffffu, pj, jj);
        if (d < p.dv) a = fmaf(w, to_f32<T>(V[(long long)((j0 + jj) % p.ring_rows) * p.v_rs + d]), a);
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
}  // namespace eb

using namespace eb;

extern "C" size_t eb_latent_decode_scratch_bytes(int batch, int heads, int rank, int nsplit) {
  if (batch <= 0 || heads <= 0 || rank <= 0 || nsplit <= 1) return 0;
  return (size_t)batch * heads * nsplit * (rank + 2) * sizeof(float);
}

extern "C" int eb_latent_decode(const void *q, long long q_batch_stride, const void *cache, long long cache_batch_stride,
                                long long cache_row_stride, int ring_rows, void *out, long long out_batch_stride, int batch, int heads,
                                int rank, int window, const int32_t *pos_device, const int32_t *first, float scale, int dtype,
                                int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  if (batch == 0 || heads == 0) return EB_OK;
  EB_REQUIRE(dtype == EB_F16 || dtype == EB_BF16, "latent_decode: fp16 or bf16 only (dtype %d)", dtype);
  EB_REQUIRE(rank == 64 || rank == 128 || rank == 256 || rank == 384 || rank == 512,
             "latent_decode: latent width %d not supported (64, 128, 256, 384 or 512)", rank);
  EB_REQUIRE(batch > 0 && batch <= 65535 && heads > 0 && ring_rows > 0 && window >= 0 && nsplit >= 1 && nsplit <= 1024, "latent_decode: bad sizes");
  EB_REQUIRE(q && cache && out && pos_device, "latent_decode: null pointer");
  EB_REQUIRE(aligned16(q) && aligned16(cache) && aligned16(out), "latent_decode: pointers must be 16-byte aligned");
  EB_REQUIRE(q_batch_stride % 8 == 0 && cache_batch_stride % 8 == 0 && cache_row_stride % 8 == 0 && cache_row_stride >= rank &&
                 out_batch_stride % 8 == 0, "latent_decode: strides must be multiples of 8 elements");
  LatentParams p{};
  p.q = q; p.q_bs = q_batch_stride; p.c = cache; p.c_bs = cache_batch_stride; p.c_ld = cache_row_stride; p.ring_rows = ring_rows;
  p.o = out; p.o_bs = out_batch_stride; p.heads = heads; p.window = window; p.nsplit = nsplit;
  p.pos_dev = pos_device; p.first = first; p.scale_log2 = scale * kLog2eLat;
  if (nsplit > 1) {
    const size_t need = eb_latent_decode_scratch_bytes(batch, heads, rank, nsplit);
    EB_REQUIRE(scratch && scratch_bytes >= need && aligned16(scratch), "latent_decode: %d splits need a scratch of %zu bytes", nsplit, need);
    p.part_o = reinterpret_cast<float *>(scratch);
    p.part_ml = p.part_o + (size_t)batch * heads * nsplit * rank;
  }
  cudaStream_t st = as_stream(stream);
  return dtype == EB_F16 ? launch_latent_r<__half>(p, batch, rank, st) : launch_latent_r<__nv_bfloat16>(p, batch, rank, st);
}

extern "C" int eb_attention_plain(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                                  long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                                  long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                                  long long o_row_stride, long long o_head_stride, int batch, int heads, int q_len, int k_dim, int v_dim,
                                  int window, int ring_rows, const int32_t *pos_device, const int32_t *first, float scale, int dtype,
                                  void *stream) {
  if (batch == 0 || heads == 0 || q_len == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "attention_plain: bad dtype %d", dtype);
  EB_REQUIRE(q && k && v && out, "attention_plain: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && heads > 0 && heads <= 65535 && q_len > 0 && k_dim > 0 && v_dim > 0 && window >= 0 && ring_rows > 0,
             "attention_plain: bad sizes");
  PlainParams p{};
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
