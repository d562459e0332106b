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
// Prompt: a CTA walks kStrip tokens of a sequence, a thread owning 4 columns (or several packs of 4); the last
// taps - 1 rows u stay in its registers.  The rows in front of the strip are recomputed (so x is written to
// another buffer than it is read from); four tokens share one reduction.  Step: one CTA per sequence, the
// rows in front from the ring.
#include "common.cuh"

namespace eb {
namespace {

constexpr int kGroup = 4;                          // tokens per reduction

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

// PACKS: packs of 4 columns per thread.
template <typename T, int TAPS, int PACKS, bool STEP>
__global__ void __launch_bounds__(1024) stream_conv_kernel(const StreamConvParams p) {
  constexpr int kBack = TAPS - 1;
  constexpr bool kKeep = TAPS <= 4 && PACKS == 1 && !STEP;       // the tap tables stay in registers
  __shared__ float4 part[2][32];
  griddep_wait();
  griddep_launch();
  const int b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int pos = STEP ? max(*p.pos_dev, 0) : 0;
  const int first = p.first ? p.first[b] : 0;
  const int t0 = STEP ? pos : blockIdx.x * p.strip, t1 = STEP ? pos + 1 : min(p.seq, t0 + p.strip);
  const long long row0 = STEP ? (long long)b - pos : (long long)b * p.seq;          // row of token t: row0 + t
  int col[PACKS];
  bool on[PACKS];
#pragma unroll
  for (int k = 0; k < PACKS; ++k) {
    col[k] = (threadIdx.x + k * blockDim.x) * 4;
    on[k] = col[k] < p.n2;
  }
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
  constexpr int G = STEP ? 1 : kGroup;
  float u[PACKS][kBack + G][4];                      // u[.][kBack + i]: token i of the group
#pragma unroll
  for (int k = 0; k < PACKS; ++k)
#pragma unroll
    for (int j = 0; j < kBack; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) u[k][j][e] = 0.f;
      const int t = pos - kBack + j;
      if (STEP && on[k] && t >= first) ld4<T>(ring + (long long)(t % p.ring_rows) * p.ring_ld + col[k], u[k][j]);
    }
  int buf = 0;
  constexpr int kLead = STEP ? 0 : (kBack + kGroup - 1) / kGroup * kGroup;
#pragma unroll 1
  for (int g0 = t0 - kLead; g0 < t1; g0 += G) {
    float sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < G; ++i) {
      const int t = g0 + i;
      const bool live = t >= t0 - kBack && t >= 0 && t < t1;
#pragma unroll
      for (int k = 0; k < PACKS; ++k) {
        float (&x)[4] = u[k][kBack + i];
#pragma unroll
        for (int e = 0; e < 4; ++e) x[e] = 0.f;
        if (!live || !on[k]) continue;
        if (p.src) ld4<T>(reinterpret_cast<const T *>(p.src) + (row0 + t) * p.lds + col[k], x);
        else ld4<float>(p.x_in + (row0 + t) * p.ldx + col[k], x);
        if (p.y) {
          float y[4];
          ld4<T>(reinterpret_cast<const T *>(p.y) + (row0 + t) * p.ldy + col[k], y);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] += y[e];
        }
        if (t >= t0 && (p.src || p.y || p.x_in != p.x_out)) st4<float>(p.x_out + (row0 + t) * p.ldx + col[k], x);
#pragma unroll
        for (int e = 0; e < 4; ++e) sq[i] = fmaf(x[e], x[e], sq[i]);
      }
    }
    const float s = sum4(sq, lane);
    if ((lane & 7) == 0) reinterpret_cast<float *>(&part[buf][warp])[lane >> 3] = s;
    __syncthreads();
    float4 tot = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < warps; ++w) {
      const float4 q = part[buf][w];
      tot.x += q.x; tot.y += q.y; tot.z += q.z; tot.w += q.w;
    }
    buf ^= 1;
    const float total[4] = {tot.x, tot.y, tot.z, tot.w};
#pragma unroll
    for (int i = 0; i < G; ++i) {
      const int t = g0 + i;
      const float r = t >= first ? rsqrtf(total[i] * p.inv_count + p.eps) : 0.f;     // (in front of a sequence nothing lies)
      const bool out = t >= t0 && t < t1;
#pragma unroll
      for (int k = 0; k < PACKS; ++k) {
#pragma unroll
        for (int e = 0; e < 4; ++e) u[k][kBack + i][e] *= r;
        if (!out || !on[k]) continue;
        float a1[4] = {0.f, 0.f, 0.f, 0.f}, a2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          float w[4];
          if constexpr (!kKeep) ld4<float>(p.k1 + (long long)j * p.n2 + col[k], w);
#pragma unroll
          for (int e = 0; e < 4; ++e) a1[e] = fmaf(kKeep ? c1[kKeep ? j : 0][e] : w[e], u[k][i + j][e], a1[e]);
        }
        st4<T>(reinterpret_cast<T *>(p.h1) + (row0 + t) * p.ldh + col[k], a1);
        if (p.h2) {
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            float w[4];
            if constexpr (!kKeep) ld4<float>(p.k2 + (long long)j * p.n2 + col[k], w);
#pragma unroll
            for (int e = 0; e < 4; ++e) a2[e] = fmaf(kKeep ? c2[kKeep ? j : 0][e] : w[e], u[k][i + j][e], a2[e]);
          }
          st4<T>(reinterpret_cast<T *>(p.h2) + (row0 + t) * p.ldh + col[k], a2);
        }
        if (STEP || p.seq - t <= p.ring_rows) st4<T>(ring + (long long)(t % p.ring_rows) * p.ring_ld + col[k], u[k][kBack + i]);
      }
    }
#pragma unroll
    for (int k = 0; k < PACKS; ++k)
#pragma unroll
      for (int j = 0; j < kBack; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[k][j][e] = u[k][G + j][e];
  }
}

template <typename T, int TAPS, int PACKS> int launch_packs(StreamConvParams p, int batch, bool step, cudaStream_t st) {
  const int threads = ((p.n2 / 4 + PACKS - 1) / PACKS + 31) / 32 * 32;
  if (step) {
    launch_pdl(stream_conv_kernel<T, TAPS, PACKS, true>, dim3(1, batch), dim3(threads), 0, st, p);
    return check_launch("stream_conv");
  }
  // strips as long as leaves about three CTAs of 512 threads per SM
  p.strip = 4 * kGroup;
  while (p.strip < 32 && (long long)batch * ((p.seq + p.strip - 1) / p.strip) > 6ll * sm_count()) p.strip *= 2;
  while (p.strip > kGroup && (long long)batch * ((p.seq + p.strip - 1) / p.strip) < 2ll * sm_count()) p.strip /= 2;
  launch_pdl(stream_conv_kernel<T, TAPS, PACKS, false>, dim3((p.seq + p.strip - 1) / p.strip, batch), dim3(threads), 0, st, p);
  return check_launch("stream_conv");
}

template <typename T, int TAPS> int launch_taps(const StreamConvParams &p, int batch, bool step, cudaStream_t st) {
  if (p.n2 <= 4096) return launch_packs<T, TAPS, 1>(p, batch, step, st);
  return launch_packs<T, TAPS, 4>(p, batch, step, st);
}

template <typename T> int launch_stream_conv(const StreamConvParams &p, int taps, int batch, bool step, cudaStream_t st) {
  switch (taps) {
    case 2: return launch_taps<T, 2>(p, batch, step, st);
    case 3: return launch_taps<T, 3>(p, batch, step, st);
    case 4: return launch_taps<T, 4>(p, batch, step, st);
    case 8: return launch_taps<T, 8>(p, batch, step, st);
    default: return launch_taps<T, 16>(p, batch, step, st);
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
