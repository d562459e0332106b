// The residual step of blocks whose two sublayers read the same stream side by side, each through a norm and a
// short causal convolution of the normed rows over time:
//
//   x = src  (or x as it was) + y;   u = x / sqrt(mean(x^2) + eps)
//   h1_t = w1 (u_t + sum_j c1_j u_(t - taps + 1 + j)),   h2_t likewise with w2 and c2
//
// Both norms share u, so a sequence's state is one ring of the last rows u, and norm weight and taps are one
// fp32 table k[j] = w (c_j + [j is the current token]) per sublayer.  Stream, sums and taps are fp32; u is
// rounded only where it goes to the ring.
//
// Prompt: a CTA walks a strip of a sequence's tokens, a thread owning 4 columns (or several packs of 4); the last
// rows u stay in its registers.  The rows in front of the strip are recomputed (so x is written to
// another buffer than it is read from); a group of tokens shares one reduction.  Step: one CTA per sequence,
// the rows in front from the ring.
#include "common.cuh"

namespace eb {
namespace {

struct StreamConvParams {
  const void *src;                                 // embedding rows (T) or null
  long long lds;
  const float *x_in;
  long long ldx;
  const void *y;                                   // T or null
  long long ldy;
  float *x_out;
  const float *k1, *k2;                            // [taps][n2]
  void *h1, *h2;                                   // T; h2 null: one sublayer
  long long ldh;
  void *ring;                                      // T [batch][ring_rows][n2]
  long long ring_bs, ring_ld;
  int ring_rows, seq, n2, strip;
  const int *first, *pos_dev;
  float inv_count, eps;
};

template <typename T> __device__ __forceinline__ void ld4(const T *p, float (&f)[4]) {
  const uint2 w = *reinterpret_cast<const uint2 *>(p);
  const float2 a = unpack2<T>(w.x), b = unpack2<T>(w.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
template <> __device__ __forceinline__ void ld4<float>(const float *p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4 *>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
template <typename T> __device__ __forceinline__ void st4(T *p, const float (&f)[4]) {
  *reinterpret_cast<uint2 *>(p) = make_uint2(pack2<T>(f[0], f[1]), pack2<T>(f[2], f[3]));
}
template <> __device__ __forceinline__ void st4<float>(float *p, const float (&f)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]); }

// Sums of four values over a warp with six shuffles: lanes 8 q .. 8 q + 7 hold the sum of v[q].
__device__ __forceinline__ float sum4(const float (&v)[4], int lane) {
  const bool hi = lane & 16, mid = lane & 8;
  float a = hi ? v[2] : v[0], b = hi ? v[3] : v[1];
  a += __shfl_xor_sync(0xffffffffu, hi ? v[0] : v[2], 16);
  b += __shfl_xor_sync(0xffffffffu, hi ? v[1] : v[3], 16);
  float s = mid ? b : a;
  s += __shfl_xor_sync(0xffffffffu, mid ? a : b, 8);
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  return s;
}

__device__ __forceinline__ void copy_async(void *dst, const void *src, int bytes, bool live) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  const int n = live ? bytes : 0;                  // the rest is filled with zeros
  if (bytes == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}

// The sums of part[0 .. warps) over all warps, in every thread.
__device__ __forceinline__ void total4(const float4 *part, int warps, int lane, float (&total)[4]) {
  const float4 q = lane < warps ? part[lane] : make_float4(0.f, 0.f, 0.f, 0.f);
  const float v[4] = {q.x, q.y, q.z, q.w}, s = sum4(v, lane);
#pragma unroll
  for (int i = 0; i < 4; ++i) total[i] = __shfl_sync(0xffffffffu, s, 8 * i);
}

// A prompt.  Every thread copies the columns of the next group of tokens that it will need itself into shared memory
// while it works on this one; rows are read from there twice, for the sums and for the norm.  PACKS: packs of 4
// columns per thread, G: tokens per group.
template <typename T, int TAPS, int PACKS, int G>
__global__ void __launch_bounds__(1024) stream_conv_kernel(const StreamConvParams p) {
  constexpr int kBack = TAPS - 1, kLead = (kBack + G - 1) / G * G;
  constexpr bool kKeep = TAPS <= 4 && PACKS == 1;                // the tap tables stay in registers
  __shared__ float4 part[2][32];
  extern __shared__ __align__(16) uint8_t sm[];
  griddep_wait();
  griddep_launch();
  const int b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = blockDim.x;
  const int first = p.first ? p.first[b] : 0, t0 = blockIdx.x * p.strip, t1 = min(p.seq, t0 + p.strip);
  const long long row0 = (long long)b * p.seq;
  float *sx = reinterpret_cast<float *>(sm);                     // [2][G][PACKS][n] packs of x, or of src
  T *sy = reinterpret_cast<T *>(sm + (size_t)2 * G * PACKS * n * 16);
  auto slot = [&](int st, int i, int k) { return (((st * G + i) * PACKS + k) * n + tid) * 4; };
  int col[PACKS];
  bool on[PACKS];
#pragma unroll
  for (int k = 0; k < PACKS; ++k) {
    col[k] = (tid + k * n) * 4;
    on[k] = col[k] < p.n2;
  }
  auto live = [&](int t) { return t >= t0 - kBack && t >= 0 && t < t1; };
  auto fetch = [&](int g0, int st) {
#pragma unroll
    for (int i = 0; i < G; ++i) {
      const int t = g0 + i;
#pragma unroll
      for (int k = 0; k < PACKS; ++k) {
        const bool ok = live(t) && on[k];
        const long long at = ok ? row0 + t : row0;
        const int c = on[k] ? col[k] : 0;
        if (p.src) copy_async(sx + slot(st, i, k), reinterpret_cast<const T *>(p.src) + at * p.lds + c, 4 * sizeof(T), ok);
        else copy_async(sx + slot(st, i, k), p.x_in + at * p.ldx + c, 16, ok);
        if (p.y) copy_async(sy + slot(st, i, k), reinterpret_cast<const T *>(p.y) + at * p.ldy + c, 4 * sizeof(T), ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto row = [&](int st, int i, int k, float (&x)[4]) {
    if (p.src) ld4<T>(reinterpret_cast<const T *>(sx + slot(st, i, k)), x);
    else ld4<float>(sx + slot(st, i, k), x);
    if (p.y) {
      float y[4];
      ld4<T>(sy + slot(st, i, k), y);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] += y[e];
    }
  };
  T *ring = reinterpret_cast<T *>(p.ring) + b * p.ring_bs;
  float c1[kKeep ? TAPS : 1][4], c2[kKeep ? TAPS : 1][4];
  if constexpr (kKeep) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      if (on[0]) {
        ld4<float>(p.k1 + (long long)j * p.n2 + col[0], c1[j]);
        if (p.h2) ld4<float>(p.k2 + (long long)j * p.n2 + col[0], c2[j]);
      }
  }
  float u[PACKS][TAPS][4];                           // the last rows; u[.][kBack]: the current one
#pragma unroll
  for (int k = 0; k < PACKS; ++k)
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) u[k][j][e] = 0.f;
  int st = 0;
  fetch(t0 - kLead, 0);
#pragma unroll 1
  for (int g0 = t0 - kLead; g0 < t1; g0 += G, st ^= 1) {
    if (g0 + G < t1) fetch(g0 + G, st ^ 1);
    else asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    float sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < G; ++i)
#pragma unroll
      for (int k = 0; k < PACKS; ++k) {
        float x[4];
        row(st, i, k, x);
        if (g0 + i >= t0 && g0 + i < t1 && on[k]) st4<float>(p.x_out + (row0 + g0 + i) * p.ldx + col[k], x);
#pragma unroll
        for (int e = 0; e < 4; ++e) sq[i] = fmaf(x[e], x[e], sq[i]);
      }
    const float s = sum4(sq, lane);
    if ((lane & 7) == 0) reinterpret_cast<float *>(&part[st][warp])[lane >> 3] = s;
    __syncthreads();
    float total[4];
    total4(part[st], n >> 5, lane, total);
#pragma unroll
    for (int i = 0; i < G; ++i) {
      const int t = g0 + i;
      const float r = t >= first ? rsqrtf(total[i] * p.inv_count + p.eps) : 0.f;     // (in front of a sequence nothing lies)
      const bool out = t >= t0 && t < t1;
#pragma unroll
      for (int k = 0; k < PACKS; ++k) {
#pragma unroll
        for (int j = 0; j < kBack; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) u[k][j][e] = u[k][j + 1][e];
        row(st, i, k, u[k][kBack]);
#pragma unroll
        for (int e = 0; e < 4; ++e) u[k][kBack][e] *= r;
        if (!out || !on[k]) continue;
        auto conv = [&](const float *table, const float (&kept)[kKeep ? TAPS : 1][4], void *h) {
          float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            float w[4];
            if constexpr (!kKeep) ld4<float>(table + (long long)j * p.n2 + col[k], w);
#pragma unroll
            for (int e = 0; e < 4; ++e) a[e] = fmaf(kKeep ? kept[kKeep ? j : 0][e] : w[e], u[k][j][e], a[e]);
          }
          st4<T>(reinterpret_cast<T *>(h) + (row0 + t) * p.ldh + col[k], a);
        };
        conv(p.k1, c1, p.h1);
        if (p.h2) conv(p.k2, c2, p.h2);
        if (p.seq - t <= p.ring_rows) st4<T>(ring + (long long)(t % p.ring_rows) * p.ring_ld + col[k], u[k][kBack]);
      }
    }
  }
}

// One token per sequence.
template <typename T, int PACKS>
__global__ void __launch_bounds__(1024) stream_conv_step_kernel(const StreamConvParams p, int taps) {
  __shared__ float4 part[32];
  griddep_wait();
  griddep_launch();
  const int b = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first = p.first ? p.first[b] : 0, pos = max(*p.pos_dev, 0);
  T *ring = reinterpret_cast<T *>(p.ring) + b * p.ring_bs;
  float x[PACKS][4], sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int k = 0; k < PACKS; ++k) {
    const int col = (tid + k * blockDim.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[k][e] = 0.f;
    if (col >= p.n2) continue;
    if (p.src) ld4<T>(reinterpret_cast<const T *>(p.src) + b * p.lds + col, x[k]);
    else ld4<float>(p.x_in + b * p.ldx + col, x[k]);
    if (p.y) {
      float y[4];
      ld4<T>(reinterpret_cast<const T *>(p.y) + b * p.ldy + col, y);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[k][e] += y[e];
    }
    st4<float>(p.x_out + b * p.ldx + col, x[k]);
#pragma unroll
    for (int e = 0; e < 4; ++e) sq[0] = fmaf(x[k][e], x[k][e], sq[0]);
  }
  // what the ring gives is added up before the sum is known
  float a1[PACKS][4], a2[PACKS][4];
#pragma unroll
  for (int k = 0; k < PACKS; ++k) {
    const int col = (tid + k * blockDim.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) a1[k][e] = a2[k][e] = 0.f;
    if (col >= p.n2) continue;
#pragma unroll 4
    for (int j = 0; j < taps - 1; ++j) {
      const int t = pos - (taps - 1) + j;
      if (t < first) continue;
      float u[4], w1[4], w2[4];
      ld4<T>(ring + (long long)(t % p.ring_rows) * p.ring_ld + col, u);
      ld4<float>(p.k1 + (long long)j * p.n2 + col, w1);
      if (p.h2) ld4<float>(p.k2 + (long long)j * p.n2 + col, w2);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        a1[k][e] = fmaf(w1[e], u[e], a1[k][e]);
        if (p.h2) a2[k][e] = fmaf(w2[e], u[e], a2[k][e]);
      }
    }
  }
  const float s = warp_sum(sq[0]);
  if (lane == 0) part[warp].x = s;
  __syncthreads();
  const float r = rsqrtf(warp_sum(lane < (blockDim.x >> 5) ? part[lane].x : 0.f) * p.inv_count + p.eps);
#pragma unroll
  for (int k = 0; k < PACKS; ++k) {
    const int col = (tid + k * blockDim.x) * 4;
    if (col >= p.n2) continue;
    float w[4];
    ld4<float>(p.k1 + (long long)(taps - 1) * p.n2 + col, w);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[k][e] *= r;
      a1[k][e] = fmaf(w[e], x[k][e], a1[k][e]);
    }
    st4<T>(reinterpret_cast<T *>(p.h1) + b * p.ldh + col, a1[k]);
    if (p.h2) {
      ld4<float>(p.k2 + (long long)(taps - 1) * p.n2 + col, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) a2[k][e] = fmaf(w[e], x[k][e], a2[k][e]);
      st4<T>(reinterpret_cast<T *>(p.h2) + b * p.ldh + col, a2[k]);
    }
    st4<T>(ring + (long long)(pos % p.ring_rows) * p.ring_ld + col, x[k]);
  }
}

template <typename T, int TAPS, int PACKS, int G> int launch_prompt(StreamConvParams p, int batch, cudaStream_t st) {
  const int threads = ((p.n2 / 4 + PACKS - 1) / PACKS + 31) / 32 * 32;
  const size_t smem = (size_t)2 * G * PACKS * threads * (16 + 4 * sizeof(T));
  auto kern = stream_conv_kernel<T, TAPS, PACKS, G>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return fail(EB_ECUDA, "stream_conv: cannot reserve %zu bytes of shared memory", smem);
  }
  // one strip per CTA the machine holds, of 8 to 64 tokens
  const int fit = (int)((220 * 1024) / (smem + 2048)), regs = 1024 / threads, per_sm = fit < regs ? (fit < 1 ? 1 : fit) : regs;
  const long long slots = (long long)per_sm * sm_count(), want = ((long long)batch * p.seq + slots - 1) / slots;
  p.strip = (int)((want < 8 ? 8 : want > 64 ? 64 : want) + G - 1) / G * G;
  launch_pdl(kern, dim3((p.seq + p.strip - 1) / p.strip, batch), dim3(threads), smem, st, p);
  return check_launch("stream_conv");
}

template <typename T> int launch_step(const StreamConvParams &p, int taps, int batch, cudaStream_t st) {
  auto go = [&](auto kern, int packs) {
    const int threads = ((p.n2 / 4 + packs - 1) / packs + 31) / 32 * 32;
    launch_pdl(kern, dim3(batch), dim3(threads), 0, st, p, taps);
    return check_launch("stream_conv");
  };
  return p.n2 <= 4096 ? go(stream_conv_step_kernel<T, 1>, 1) : go(stream_conv_step_kernel<T, 4>, 4);
}

template <typename T, int TAPS> int launch_taps(const StreamConvParams &p, int batch, cudaStream_t st) {
  if (p.n2 <= 4096) return launch_prompt<T, TAPS, 1, sizeof(T) == 2 ? 4 : 2>(p, batch, st);
  return launch_prompt<T, TAPS, 4, 1>(p, batch, st);
}

template <typename T> int launch_stream_conv(const StreamConvParams &p, int taps, int batch, bool step, cudaStream_t st) {
  if (step) return launch_step<T>(p, taps, batch, st);
  switch (taps) {
    case 2: return launch_taps<T, 2>(p, batch, st);
    case 3: return launch_taps<T, 3>(p, batch, st);
    case 4: return launch_taps<T, 4>(p, batch, st);
    case 8: return launch_taps<T, 8>(p, batch, st);
    default: return launch_taps<T, 16>(p, batch, st);
  }
}

constexpr int kMaxConvWidth = 16384;

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_stream_conv(const void *src, long long lds, const float *x_in, long long ldx, const void *y, long long ldy, float *x_out,
                              const float *k1, const float *k2, int taps, void *h1, void *h2, long long ldh, void *ring,
                              long long ring_batch_stride, long long ring_ld, int ring_rows, int batch, int seq, int n2, int count, float eps,
                              const int32_t *first, const int32_t *pos_device, int dtype, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "stream_conv: bad dtype %d", dtype);
  EB_REQUIRE((src || x_in) && x_out && k1 && h1 && ring && (!h2 || k2), "stream_conv: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && seq > 0 && (!pos_device || seq == 1), "stream_conv: bad row counts (a step has one row per sequence)");
  EB_REQUIRE(n2 > 0 && n2 % 8 == 0 && n2 <= kMaxConvWidth && count > 0 && count <= n2, "stream_conv: width %d must be a multiple of 8, at most %d", n2, kMaxConvWidth);
  EB_REQUIRE(taps == 2 || taps == 3 || taps == 4 || taps == 8 || taps == 16, "stream_conv: tables of 2, 3, 4, 8 or 16 taps (got %d)", taps);
  EB_REQUIRE(pos_device || x_in != x_out || src, "stream_conv: the rows of a prompt are read again by their neighbours and cannot be updated in place");
  EB_REQUIRE(ring_rows > 0 && ring_ld >= n2 && ring_ld % 8 == 0 && ring_batch_stride % 8 == 0, "stream_conv: the ring holds whole rows, strides multiples of 8");
  const long long lds_[] = {src ? lds : n2, ldx, y ? ldy : n2, ldh};
  for (long long l : lds_) EB_REQUIRE(l >= n2 && l % 8 == 0, "stream_conv: row strides must be multiples of 8 and >= n2");
  const void *ptrs[] = {src, x_in, y, x_out, k1, k2, h1, h2, ring};
  for (const void *q : ptrs) EB_REQUIRE(aligned16(q), "stream_conv: pointers must be 16-byte aligned");
  StreamConvParams p{};
  p.src = src; p.lds = lds; p.x_in = x_in; p.ldx = ldx; p.y = y; p.ldy = ldy; p.x_out = x_out; p.k1 = k1; p.k2 = k2; p.h1 = h1; p.h2 = h2; p.ldh = ldh;
  p.ring = ring; p.ring_bs = ring_batch_stride; p.ring_ld = ring_ld; p.ring_rows = ring_rows; p.seq = seq; p.n2 = n2;
  p.first = first; p.pos_dev = pos_device; p.inv_count = 1.f / (float)count; p.eps = eps;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_stream_conv<float>(p, taps, batch, pos_device != nullptr, st);
  if (dtype == EB_F16) return launch_stream_conv<__half>(p, taps, batch, pos_device != nullptr, st);
  return launch_stream_conv<__nv_bfloat16>(p, taps, batch, pos_device != nullptr, st);
}
