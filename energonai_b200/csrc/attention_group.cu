// Generation-step attention for query heads in groups that share a key / value head: one pass over the
// cached keys and values per group (HBM-bound).  The query heads of a group are the rows of the
// mma.sync tile, so a key fragment is read once for up to 16 heads.  Each warp takes 16 keys of every
// 64-key tile and loads, waits for and consumes only those; two tiles are in flight per CTA.  The
// position range of a (sequence, group) may be split over CTAs, merged by the last to arrive.
//
// A chunk mask (a position sees only its own chunk of so many positions, counted from the sequence's first)
// goes with a ring cache: position p in row p mod rows.
//
// A window may keep the first positions visible; the cache then has rows for them in front of its ring.  With it go
// capped scores, cap tanh(score / cap), and a bias linear in the distance.  The output may be multiplied by the
// sigmoid of a gate.
//
// Scores: scale q.k - r1 ln(1 + r2 distance), optionally a sink (one more in the denominator, or exp of a
// number per head), all fp32;
// an attention weight is rounded once, as an operand of the value product.
#include "attention_mma.cuh"

namespace eb {
namespace {

constexpr int kTile = 64, kGroupThreads = 128, kRowsPerCta = 16, kStages = 2;
constexpr float kLog2eGroup = 1.4426950408889634f;
constexpr int kCounterSlots = 16384;

struct GroupParams {
  const void *q, *k, *v;
  void *o;
  long long q_bs, k_bs, k_rs, v_bs, v_rs, o_bs;
  const float *sinks;                               // per head, or null (with sink: 0)
  int chunk;                                        // RING: positions of a chunk
  int group, blocks, cache_rows, nsplit, sink;      // blocks: CTAs of up to 16 heads per group
  const int *pos_dev, *first;
  const float *r1, *r2;
  int window, keep;                                 // window form: of which the first `keep` cache rows hold the first positions
  const float *slopes;                              // ... per head, slope * distance is taken off, or null
  float cap_log2, cap_scale;                        // ... cap * log2(e) and scale / cap, or 0
  const void *gate;                                 // [B][heads * D] or null
  long long g_bs;
  float scale_log2;
  float *scratch;                                   // [unit][nsplit][16][D + 2]
  int *counters;
};

enum { kAll, kChunk, kWindow };                       // what of the past is visible

// tanh by an exponential and a reciprocal: the error of the special function for tanh would be multiplied by the cap
__device__ __forceinline__ float tanh_exp(float z) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * z)); }
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// WIDE: groups of more than 8 heads; else the second half of the tile's rows is not looked at.
template <typename T, int D, bool WIDE, int FORM>
__global__ void __launch_bounds__(kGroupThreads) attention_group_decode_kernel(const GroupParams p) {
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr bool RING = FORM == kChunk, WINDOW = FORM == kWindow;
  constexpr int kTileBytes = kTile * D * 2, kLd = D + 2, kHalves = WIDE ? 2 : 1;
  const uint32_t k_s = (uint32_t)__cvta_generic_to_shared(smem), v_s = k_s + kStages * kTileBytes;
  float *red = reinterpret_cast<float *>(smem);     // after the key loop: [4 warps][16][D + 2]
  __shared__ int s_last;
  static_assert(4 * kRowsPerCta * kLd * 4 <= 2 * kStages * kTileBytes, "the warps' partial rows reuse the tiles' memory");

  griddep_wait();
  griddep_launch();
  const int split = blockIdx.x, hk = blockIdx.y / p.blocks, hb = blockIdx.y % p.blocks, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int h0 = hk * p.group + hb * kRowsPerCta, nh = min(kRowsPerCta, p.group - hb * kRowsPerCta);
  const int pos = RING || WINDOW ? max(*p.pos_dev, 0) : min(max(*p.pos_dev, 0), p.cache_rows - 1);
  int lo = p.first ? min(max(p.first[b], 0), pos) : 0;
  const int start = lo;
  if (WINDOW) lo = max(p.window > 0 ? max(lo, pos - p.window + 1) : lo, pos - p.cache_rows + 1);
  // window form: entries are counted, first the kept positions in front of the window, then those of the window
  const int kept = WINDOW ? min(p.keep, lo - start) : 0, Sk = WINDOW ? kept + pos + 1 - lo : pos + 1;
  if (RING) lo = max(lo + (pos - lo) / p.chunk * p.chunk, pos - p.cache_rows + 1);
  // tile n holds the positions from base + 64 n on
  const int base = WINDOW ? 0 : RING ? lo : lo / kTile * kTile, tiles = (Sk - base + kTile - 1) / kTile, per = (tiles + p.nsplit - 1) / p.nsplit;
  const int tile0 = split * per, tile1 = min(tiles, tile0 + per);
  const int r0 = RING ? base % p.cache_rows : WINDOW ? lo % p.cache_rows : 0;

  const T *qb = reinterpret_cast<const T *>(p.q) + b * p.q_bs + (long long)h0 * D;
  const T *kb = reinterpret_cast<const T *>(p.k) + b * p.k_bs + hk * D;
  const T *vb = reinterpret_cast<const T *>(p.v) + b * p.v_bs + hk * D;
  auto load_kv = [&](int n, int buf) {
    if (RING) {
      load_warp_ring<T, D>(k_s + buf * kTileBytes, kb, p.k_rs, n * kTile, Sk - base, r0, p.cache_rows, warp, lane);
      load_warp_ring<T, D>(v_s + buf * kTileBytes, vb, p.v_rs, n * kTile, Sk - base, r0, p.cache_rows, warp, lane);
      return;
    }
    if (WINDOW) {
      load_warp_kept<T, D>(k_s + buf * kTileBytes, kb, p.k_rs, n * kTile, Sk, kept, p.keep, r0, p.cache_rows, warp, lane);
      load_warp_kept<T, D>(v_s + buf * kTileBytes, vb, p.v_rs, n * kTile, Sk, kept, p.keep, r0, p.cache_rows, warp, lane);
      return;
    }
    load_warp_rows<T, D>(k_s + buf * kTileBytes, kb, p.k_rs, base + n * kTile, Sk, warp, lane);
    load_warp_rows<T, D>(v_s + buf * kTileBytes, vb, p.v_rs, base + n * kTile, Sk, warp, lane);
  };
  for (int i = 0; i < kStages - 1; ++i) {
    if (tile0 + i < tile1) load_kv(tile0 + i, i);
    cp_async_commit();
  }
  uint32_t qf[D / 16][4];
  const bool row_ok[2] = {g < nh, WIDE && g + 8 < nh};
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const T *qr = qb + (g + 8 * r) * D + kk * 16 + 2 * t;
      qf[kk][r] = row_ok[r] ? *reinterpret_cast<const uint32_t *>(qr) : 0u;
      qf[kk][2 + r] = row_ok[r] ? *reinterpret_cast<const uint32_t *>(qr + 8) : 0u;
    }
  float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
  if (p.r1) {
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if (row_ok[r]) { r1[r] = p.r1[h0 + g + 8 * r]; r2[r] = p.r2[h0 + g + 8 * r]; }
  }
  if (WINDOW && p.slopes) {
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if (row_ok[r]) r1[r] = p.slopes[h0 + g + 8 * r] * kLog2eGroup;
  }
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  for (int n = tile0; n < tile1; ++n) {
    const int buf = (n - tile0) % kStages;
    if (n + kStages - 1 < tile1) load_kv(n + kStages - 1, (buf + kStages - 1) % kStages);
    cp_async_commit();
    cp_async_wait<kStages - 1>();
    __syncwarp();
    const uint32_t kt = k_s + buf * kTileBytes, vt = v_s + buf * kTileBytes;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t kf[4];
      ldmatrix_x4(kf, kt + tile_off<D>(warp * 16 + (lane & 7) + 8 * (lane >> 4), kk * 2 + ((lane >> 3) & 1)));
      mma16816<T>(s[0], qf[kk], kf[0], kf[1]);
      mma16816<T>(s[1], qf[kk], kf[2], kf[3]);
    }
    float corr[2] = {1.f, 1.f};
#pragma unroll
    for (int r = 0; r < kHalves; ++r) {
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = base + n * kTile + warp * 16 + i * 8 + 2 * t + e;
          float x = s[i][2 * r + e] * p.scale_log2;
          if (WINDOW) {
            if (p.cap_scale > 0.f) x = p.cap_log2 * tanh_exp(s[i][2 * r + e] * p.cap_scale);
            x -= r1[r] * (float)(pos - (j < kept ? start + j : lo + j - kept));
            if (j >= Sk || !row_ok[r]) x = -INFINITY;
          } else {
            x -= r1[r] * log2f(fmaf(r2[r], (float)max(pos - j, 0), 1.f));
            if (j > pos || j < lo || !row_ok[r]) x = -INFINITY;
          }
          s[i][2 * r + e] = x;
          mx = fmaxf(mx, x);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m_run[r], mx), m_use = m_new == -INFINITY ? 0.f : m_new;
      corr[r] = exp2f(m_run[r] - m_use);
      m_run[r] = m_new;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[i][2 * r + e] = exp2f(s[i][2 * r + e] - m_use);
          sum += s[i][2 * r + e];
        }
      l_run[r] = l_run[r] * corr[r] + sum;
    }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < D / 8; ++i) {
        o[i][0] *= corr[0]; o[i][1] *= corr[0];
        if (WIDE) { o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
      }
    }
    const uint32_t pf[4] = {eb::pack2<T>(s[0][0], s[0][1]), WIDE ? eb::pack2<T>(s[0][2], s[0][3]) : 0u, eb::pack2<T>(s[1][0], s[1][1]),
                            WIDE ? eb::pack2<T>(s[1][2], s[1][3]) : 0u};
#pragma unroll
    for (int db = 0; db < D / 16; ++db) {
      uint32_t vf[4];
      ldmatrix_x4_trans(vf, vt + tile_off<D>(warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1), db * 2 + (lane >> 4)));
      mma16816<T>(o[2 * db], pf, vf[0], vf[1]);
      mma16816<T>(o[2 * db + 1], pf, vf[2], vf[3]);
    }
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();                                  // all tiles are consumed: their memory takes the partial rows
#pragma unroll
  for (int r = 0; r < kHalves; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    float *mine = red + (warp * kRowsPerCta + g + 8 * r) * kLd;
#pragma unroll
    for (int i = 0; i < D / 8; ++i) *reinterpret_cast<float2 *>(mine + i * 8 + 2 * t) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
    if (t == 0) { mine[D] = m_run[r]; mine[D + 1] = l; }
  }
  __syncthreads();
  // row by row: the parts of the warps, or of the splits, in one scale; the sink joins the last merge
  auto sink_score = [&](int row) { return !p.sink ? -INFINITY : p.sinks ? p.sinks[h0 + row] * kLog2eGroup : 0.f; };
  auto merge = [&](const float *parts, int count, long long stride, int row, int d, bool sink, float &m_out, float &l_out) {
    const float sc = sink ? sink_score(row) : -INFINITY;
    float m = sc;
    for (int i = 0; i < count; ++i) m = fmaxf(m, __ldcg(parts + i * stride + row * kLd + D));
    const float ref = m == -INFINITY ? 0.f : m;
    float l = exp2f(sc - ref), acc = 0.f;
    for (int i = 0; i < count; ++i) {
      const float w = exp2f(__ldcg(parts + i * stride + row * kLd + D) - ref);
      l = fmaf(__ldcg(parts + i * stride + row * kLd + D + 1), w, l);
      acc = fmaf(__ldcg(parts + i * stride + row * kLd + d), w, acc);
    }
    m_out = m;
    l_out = l;
    return acc;
  };
  const T *gate = p.gate ? reinterpret_cast<const T *>(p.gate) + b * p.g_bs + (long long)h0 * D : nullptr;
  auto result = [&](float acc, float l, int i) {
    const float y = l > 0.f ? acc / l : 0.f;
    return from_f32<T>(gate ? y * sigmoid_fast(to_f32<T>(gate[i])) : y);
  };
  T *out = reinterpret_cast<T *>(p.o) + b * p.o_bs + (long long)h0 * D;
  const int unit = b * gridDim.y + blockIdx.y;
  float *slot = p.nsplit > 1 ? p.scratch + ((size_t)unit * p.nsplit + split) * (kRowsPerCta * kLd) : nullptr;
  for (int i = threadIdx.x; i < nh * D; i += kGroupThreads) {
    const int row = i / D, d = i % D;
    // (shared memory: plain loads)
    const float sc = p.nsplit == 1 ? sink_score(row) : -INFINITY;
    float m = sc;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, red[(w * kRowsPerCta + row) * kLd + D]);
    const float ref = m == -INFINITY ? 0.f : m;
    float l = exp2f(sc - ref), acc = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float *part = red + (w * kRowsPerCta + row) * kLd;
      const float f = exp2f(part[D] - ref);
      l = fmaf(part[D + 1], f, l);
      acc = fmaf(part[d], f, acc);
    }
    if (!slot) {
      out[row * D + d] = result(acc, l, i);
    } else {
      slot[row * kLd + d] = acc;
      if (d == 0) { slot[row * kLd + D] = m; slot[row * kLd + D + 1] = l; }
    }
  }
  if (!slot) return;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    s_last = atomicAdd(p.counters + unit, 1) == p.nsplit - 1;
    if (s_last) p.counters[unit] = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  const float *all = p.scratch + (size_t)unit * p.nsplit * (kRowsPerCta * kLd);
  for (int i = threadIdx.x; i < nh * D; i += kGroupThreads) {
    float m, l;
    const float acc = merge(all, p.nsplit, kRowsPerCta * kLd, i / D, i % D, p.sink != 0, m, l);
    out[i] = result(acc, l, i);
  }
}

template <typename T, int D, bool WIDE, int FORM> int launch_group_as(const GroupParams &p, int kv_heads, int B, cudaStream_t st) {
  constexpr size_t smem = 2 * kStages * (size_t)kTile * D * 2;
  auto kern = attention_group_decode_kernel<T, D, WIDE, FORM>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "attention_group_decode: cannot reserve %zu bytes of shared memory", smem);
    }
    configured[dev] = true;
  }
  launch_pdl(kern, dim3(p.nsplit, kv_heads * p.blocks, B), dim3(kGroupThreads), smem, st, p);
  return check_launch("attention_group_decode");
}

template <typename T, int D> int launch_group(const GroupParams &p, int form, int kv_heads, int B, cudaStream_t st) {
#define EB_GROUP(FORM) (p.group > 8 ? launch_group_as<T, D, true, FORM>(p, kv_heads, B, st) : launch_group_as<T, D, false, FORM>(p, kv_heads, B, st))
  return form == kWindow ? EB_GROUP(kWindow) : form == kChunk ? EB_GROUP(kChunk) : EB_GROUP(kAll);
#undef EB_GROUP
}

inline int head_blocks(int heads, int kv_heads) { return (heads / kv_heads + kRowsPerCta - 1) / kRowsPerCta; }

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" size_t eb_attention_group_decode_scratch_bytes(int batch, int heads, int kv_heads, int head_dim, int nsplit) {
  if (batch <= 0 || heads <= 0 || kv_heads <= 0 || nsplit <= 1) return 0;
  return kCounterSlots * sizeof(int) + (size_t)batch * kv_heads * head_blocks(heads, kv_heads) * nsplit * kRowsPerCta * (head_dim + 2) * sizeof(float);
}

struct GroupWindow {
  int window, keep;
  const float *slopes;
  float cap;
  const void *gate;
  long long gate_batch_stride;
};

static int group_decode_impl(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                                         long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                         long long out_batch_stride, int batch, int heads, int kv_heads, int head_dim, int cache_rows,
                                         const int32_t *pos_device, const int32_t *first, const float *bias_r1, const float *bias_r2, int sink,
                                         const float *sinks, int chunk, float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes,
                                         void *stream, const GroupWindow *win = nullptr) {
  if (batch == 0) return EB_OK;
  EB_REQUIRE(dtype == EB_F16 || dtype == EB_BF16, "attention_group_decode: fp16 or bf16 only (dtype %d)", dtype);
  EB_REQUIRE(head_dim == 64 || head_dim == 128, "attention_group_decode: head_dim %d not supported (64 or 128)", head_dim);
  EB_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0, "attention_group_decode: %d heads do not share %d key / value heads", heads, kv_heads);
  EB_REQUIRE(batch > 0 && batch <= 65535 && cache_rows > 0 && nsplit >= 1 && nsplit <= 1024, "attention_group_decode: bad sizes");
  EB_REQUIRE(q && k && v && out && pos_device, "attention_group_decode: null pointer");
  EB_REQUIRE((bias_r1 == nullptr) == (bias_r2 == nullptr), "attention_group_decode: the distance bias has two numbers per head");
  EB_REQUIRE(aligned16(q) && aligned16(k) && aligned16(v) && aligned16(out), "attention_group_decode: pointers must be 16-byte aligned");
  const long long strides[] = {q_batch_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride, out_batch_stride};
  for (long long s : strides) EB_REQUIRE(s % 8 == 0, "attention_group_decode: strides must be multiples of 8 elements");
  GroupParams p{};
  p.q = q; p.k = k; p.v = v; p.o = out; p.q_bs = q_batch_stride; p.k_bs = k_batch_stride; p.k_rs = k_row_stride; p.v_bs = v_batch_stride;
  p.v_rs = v_row_stride; p.o_bs = out_batch_stride; p.group = heads / kv_heads; p.blocks = head_blocks(heads, kv_heads);
  p.cache_rows = cache_rows; p.nsplit = nsplit; p.sink = sink; p.sinks = sinks; p.chunk = chunk; p.pos_dev = pos_device; p.first = first; p.r1 = bias_r1; p.r2 = bias_r2;
  p.scale_log2 = scale * kLog2eGroup;
  if (win) {
    EB_REQUIRE(win->window >= 0 && win->keep >= 0 && win->cap >= 0.f && (!win->gate || win->gate_batch_stride % 8 == 0), "attention_group_decode: bad window form");
    p.window = win->window; p.keep = win->keep; p.slopes = win->slopes; p.gate = win->gate; p.g_bs = win->gate_batch_stride;
    if (win->cap > 0.f) { p.cap_log2 = win->cap * kLog2eGroup; p.cap_scale = scale / win->cap; }
  }
  const int form = win ? kWindow : chunk > 0 ? kChunk : kAll;
  EB_REQUIRE((long long)kv_heads * p.blocks <= 65535, "attention_group_decode: too many heads");
  if (nsplit > 1) {
    const size_t need = eb_attention_group_decode_scratch_bytes(batch, heads, kv_heads, head_dim, nsplit);
    EB_REQUIRE((long long)batch * kv_heads * p.blocks <= kCounterSlots, "attention_group_decode: more than %d (sequence, group) pairs cannot be split", kCounterSlots);
    EB_REQUIRE(scratch && scratch_bytes >= need && aligned16(scratch), "attention_group_decode: nsplit=%d needs a scratch of %zu bytes, zero-filled once", nsplit, need);
    p.counters = reinterpret_cast<int *>(scratch);
    p.scratch = reinterpret_cast<float *>(reinterpret_cast<char *>(scratch) + kCounterSlots * sizeof(int));
  }
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F16) return head_dim == 64 ? launch_group<__half, 64>(p, form, kv_heads, batch, st) : launch_group<__half, 128>(p, form, kv_heads, batch, st);
  return head_dim == 64 ? launch_group<__nv_bfloat16, 64>(p, form, kv_heads, batch, st) : launch_group<__nv_bfloat16, 128>(p, form, kv_heads, batch, st);
}

extern "C" int eb_attention_group_decode(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                                         long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                         long long out_batch_stride, int batch, int heads, int kv_heads, int head_dim, int cache_rows,
                                         const int32_t *pos_device, const int32_t *first, const float *bias_r1, const float *bias_r2, int sink,
                                         float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  return group_decode_impl(q, k, v, out, q_batch_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride, out_batch_stride, batch, heads,
                           kv_heads, head_dim, cache_rows, pos_device, first, bias_r1, bias_r2, sink, nullptr, 0, scale, dtype, nsplit, scratch,
                           scratch_bytes, stream);
}

extern "C" int eb_attention_group_decode_chunk(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                                         long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                         long long out_batch_stride, int batch, int heads, int kv_heads, int head_dim, int ring_rows, int chunk,
                                         const int32_t *pos_device, const int32_t *first, const float *sinks, float scale, int dtype,
                                         int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  EB_REQUIRE(chunk >= 0, "attention_group_decode: a chunk of %d positions", chunk);
  return group_decode_impl(q, k, v, out, q_batch_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride, out_batch_stride, batch, heads,
                           kv_heads, head_dim, ring_rows, pos_device, first, nullptr, nullptr, sinks ? 1 : 0, sinks, chunk, scale, dtype, nsplit, scratch,
                           scratch_bytes, stream);
}

extern "C" int eb_attention_group_decode_capped(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                                         long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                         long long out_batch_stride, long long gate_batch_stride, int batch, int heads, int kv_heads, int head_dim,
                                         int keep, int ring_rows, int window, const int32_t *pos_device, const int32_t *first, const float *slopes,
                                         float cap, int sink, float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes, void *stream) {
  const GroupWindow win{window, keep, slopes, cap, gate, gate_batch_stride};
  return group_decode_impl(q, k, v, out, q_batch_stride, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride, out_batch_stride, batch, heads,
                           kv_heads, head_dim, ring_rows, pos_device, first, nullptr, nullptr, sink, nullptr, 0, scale, dtype, nsplit, scratch,
                           scratch_bytes, stream, &win);
}
