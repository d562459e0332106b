// Recurrent layers whose fp32 state per head is a matrix that decays, S = diag(a) S + k v^T, y = S^T q:
//
//   state space (ssm)   a = exp(-exp(A) dt), one number per head; k = dt B, q = C, shared by a group of
//                       heads; y gains D x.  x, B and C come out of a causal convolution per channel
//                       with SiLU, whose last inputs are kept in a ring.
//   gated linear (gla)  a = sigmoid(z)^(1/tau), one number per row of S; z is a low-rank projection.
//
//   short_conv          the convolution of a prompt
//   decay_scan          a whole prompt, token by token: the path of 32-bit models and of head sizes that
//                       the chunked tensor-core kernels (decay_memory_tc.cu) do not have
//   ssm_step, gla_step  one token per sequence, a pass over the state (state_pass.cuh); what lies between
//                       the projection and the state is in the same launch, and for gla the norm and
//                       the gate behind it
//   gate_group_norm     the gate and the norm (in equal parts of the row) behind the state-space layer
#include "decay_gates.cuh"
#include "state_pass.cuh"

namespace eb {
namespace {

__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

template <typename T> __device__ __forceinline__ void load_pack(const T *p, float (&f)[8]) {
  constexpr int N = Vec16<T>::N;
#pragma unroll
  for (int i = 0; i < 8 / N; ++i) {
    Vec16<T> v;
    float t[N];
    v.load(p + i * N);
    v.unpack(t);
#pragma unroll
    for (int e = 0; e < N; ++e) f[i * N + e] = t[e];
  }
}
template <typename T> __device__ __forceinline__ void store_pack(T *p, const float (&f)[8]) {
  constexpr int N = Vec16<T>::N;
#pragma unroll
  for (int i = 0; i < 8 / N; ++i) {
    Vec16<T> v;
    float t[N];
#pragma unroll
    for (int e = 0; e < N; ++e) t[e] = f[i * N + e];
    v.pack(t);
    v.store(p + i * N);
  }
}

// ---- convolution of a prompt ---------------------------------------------------------------------------
constexpr int kConvThreads = 128, kConvStrip = 32;

struct ConvParams {
  const void *x;
  long long ldx;
  const void *w, *b;           // [taps][C] (the last row is the current token's), [C]
  void *out;
  long long ldo;
  int C, taps, seq;
  const int *first;            // inputs in front of it are zero
  void *ring;                  // [batch][ring_rows][C]: position p in row p mod ring_rows
  long long ring_bs, ring_ld;
  int ring_rows;
};

// silu of what becomes a 16-bit operand, and of 32-bit models
template <typename T> __device__ __forceinline__ float conv_silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <> __device__ __forceinline__ float conv_silu<float>(float x) { return silu(x); }

// Four channels as 32-bit numbers
template <typename T> __device__ __forceinline__ void load4(const T *p, float (&f)[4]) {
  const uint2 w = *reinterpret_cast<const uint2 *>(p);
  const float2 a = unpack2<T>(w.x), b = unpack2<T>(w.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
template <> __device__ __forceinline__ void load4<float>(const float *p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4 *>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
template <typename T> __device__ __forceinline__ void store4(T *p, const float (&f)[4]) {
  *reinterpret_cast<uint2 *>(p) = make_uint2(pack2<T>(f[0], f[1]), pack2<T>(f[2], f[3]));
}
template <> __device__ __forceinline__ void store4<float>(float *p, const float (&f)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]); }

// Thread = 4 channels of kConvStrip tokens; TAPS > 0: the window in registers, else read again per token.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) short_conv_kernel(const ConvParams p) {
  griddep_wait();
  griddep_launch();
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * 4, b = blockIdx.z, t0 = blockIdx.y * kConvStrip;
  if (c >= p.C) return;
  const int first = p.first ? p.first[b] : 0, taps = TAPS > 0 ? TAPS : p.taps;
  const T *x = reinterpret_cast<const T *>(p.x) + (long long)b * p.seq * p.ldx + c;
  T *out = reinterpret_cast<T *>(p.out) + (long long)b * p.seq * p.ldo + c;
  T *ring = reinterpret_cast<T *>(p.ring) + b * p.ring_bs + c;
  const T *w = reinterpret_cast<const T *>(p.w) + c;
  auto input = [&](int t, float (&f)[4]) {
    if (t >= first && t < p.seq) {
      load4<T>(x + (long long)t * p.ldx, f);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) f[e] = 0.f;
    }
  };
  float bias[4];
  load4<T>(reinterpret_cast<const T *>(p.b) + c, bias);
  auto finish = [&](int t, const float (&cur)[4], float (&acc)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[e] = conv_silu<T>(acc[e]);
    store4<T>(out + (long long)t * p.ldo, acc);
    if (p.seq - t <= p.ring_rows) store4<T>(ring + (long long)(t % p.ring_rows) * p.ring_ld, cur);
  };
  if constexpr (TAPS > 0) {
    constexpr int kGroup = 8;                        // tokens whose inputs are in flight together
    float wv[TAPS][4], in[TAPS - 1 + kGroup][4];     // in[TAPS - 1 + i]: token i of the group
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load4<T>(w + (long long)j * p.C, wv[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(t0 - (TAPS - 1) + j, in[j]);
#pragma unroll 1
    for (int i0 = 0; i0 < kConvStrip; i0 += kGroup) {
#pragma unroll
      for (int i = 0; i < kGroup; ++i) input(t0 + i0 + i, in[TAPS - 1 + i]);
#pragma unroll
      for (int i = 0; i < kGroup; ++i) {
        float acc[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          acc[e] = bias[e];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(wv[j][e], in[i + j][e], acc[e]);
        }
        if (t0 + i0 + i < p.seq) finish(t0 + i0 + i, in[TAPS - 1 + i], acc);
      }
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) in[j][e] = in[kGroup + j][e];
    }
  } else {
    for (int t = t0; t < min(p.seq, t0 + kConvStrip); ++t) {
      float acc[4], f[4], wv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] = bias[e];
      for (int j = 0; j < taps; ++j) {
        input(t - (taps - 1) + j, f);
        load4<T>(w + (long long)j * p.C, wv);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(wv[e], f[e], acc[e]);
      }
      finish(t, f, acc);
    }
  }
}

template <typename T> int launch_conv(const ConvParams &p, int B, cudaStream_t st) {
  const dim3 g((p.C / 4 + kConvThreads - 1) / kConvThreads, (p.seq + kConvStrip - 1) / kConvStrip, B), b(kConvThreads);
  switch (p.taps) {
    case 2: launch_pdl(short_conv_kernel<T, 2>, g, b, 0, st, p); break;
    case 3: launch_pdl(short_conv_kernel<T, 3>, g, b, 0, st, p); break;
    case 4: launch_pdl(short_conv_kernel<T, 4>, g, b, 0, st, p); break;
    default: launch_pdl(short_conv_kernel<T, 0>, g, b, 0, st, p);
  }
  return check_launch("short_conv");
}

// ---- prompt, token by token ------------------------------------------------------------------------------
constexpr int kScanCols = 32, kScanThreads = 256, kScanWarps = kScanThreads / 32;

struct ScanParams {
  const void *q, *k, *v;       // rows ld apart; key / value heads of dk / dv, q and k shared by `group` heads
  long long ldq, ldk, ldv;
  int group;
  const float *gates;          // ssm: [row][heads] dt before bias and softplus; gla: [row][heads*dk] z
  long long ldg;
  const float *dt_bias, *a_log, *skip;
  float scale, inv_tau;
  const int *first;
  void *o;
  long long ldo;
  float *S;
  int seq, heads, dk, dv;
};

template <typename T, bool GLA>
__global__ void __launch_bounds__(kScanThreads) decay_scan_kernel(const ScanParams p) {
  extern __shared__ float sm[];
  float *S = sm, *as = S + p.dk * kScanCols, *qs = as + p.dk, *ks = qs + p.dk;
  __shared__ float red[kScanWarps][kScanCols + 1];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, b = blockIdx.z, hk = h / p.group;
  const int col = blockIdx.x * kScanCols + lane;
  const bool has = col < p.dv;
  for (int i = threadIdx.x; i < p.dk * kScanCols; i += kScanThreads) S[i] = 0.f;
  const int t0 = p.first ? min(max(p.first[b], 0), p.seq) : 0;
  const long long row0 = (long long)b * p.seq;
  T *o = reinterpret_cast<T *>(p.o) + h * p.dv + col;
  if (warp == 0 && has)
    for (int t = 0; t < t0; ++t) o[(row0 + t) * p.ldo] = from_f32<T>(0.f);
  const float a_log = GLA ? 0.f : p.a_log[h], bias = GLA ? 0.f : p.dt_bias[h], skip = GLA ? 0.f : p.skip[h];
  for (int t = t0; t < p.seq; ++t) {
    const long long row = row0 + t;
    const T *q = reinterpret_cast<const T *>(p.q) + row * p.ldq + hk * p.dk, *k = reinterpret_cast<const T *>(p.k) + row * p.ldk + hk * p.dk;
    const float v = has ? to_f32<T>(reinterpret_cast<const T *>(p.v)[row * p.ldv + h * p.dv + col]) : 0.f;
    float a = 0.f, w = 1.f;
    if (!GLA) {
      w = softplus(p.gates[row * p.ldg + h] + bias);
      a = expf(log_decay_ssm(a_log, w));
    }
    for (int d = threadIdx.x; d < p.dk; d += kScanThreads) {
      if (GLA) as[d] = expf(log_decay_gla(p.gates[row * p.ldg + h * p.dk + d], p.inv_tau));
      qs[d] = to_f32<T>(q[d]) * p.scale;
      ks[d] = to_f32<T>(k[d]) * w;
    }
    __syncthreads();
    float acc = 0.f;
    for (int d = warp; d < p.dk; d += kScanWarps) {
      const float s = fmaf(GLA ? as[d] : a, S[d * kScanCols + lane], ks[d] * v);
      S[d * kScanCols + lane] = s;
      acc = fmaf(s, qs[d], acc);
    }
    red[warp][lane] = acc;
    __syncthreads();
    if (warp == 0) {
      float y = skip * v;
#pragma unroll
      for (int i = 0; i < kScanWarps; ++i) y += red[i][lane];
      if (has) o[row * p.ldo] = from_f32<T>(y);
    }
  }
  if (has)
    for (int d = warp; d < p.dk; d += kScanWarps) p.S[(((long long)b * p.heads + h) * p.dk + d) * p.dv + col] = S[d * kScanCols + lane];
}

template <typename T, bool GLA> int launch_scan(const ScanParams &p, int B, cudaStream_t st) {
  const size_t smem = (size_t)p.dk * (kScanCols + 3) * sizeof(float);
  auto kern = decay_scan_kernel<T, GLA>;
  if (smem > 200 * 1024) return fail(EB_EUNSUPPORTED, "decay_scan: head size %d is too large", p.dk);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return fail(EB_ECUDA, "decay_scan: cannot reserve %zu bytes of shared memory", smem);
  }
  launch_pdl(kern, dim3((p.dv + kScanCols - 1) / kScanCols, p.heads, B), dim3(kScanThreads), smem, st, p);
  return check_launch("decay_scan");
}

// ---- one token per sequence: state space -------------------------------------------------------------------
struct SsmStepParams {
  const void *xbc;             // rows [x: heads*dv | B: groups*dk | C: groups*dk] before the convolution
  long long ldx;
  const void *conv_w, *conv_b;
  int taps, channels;
  void *ring;
  long long ring_bs, ring_ld;
  int ring_rows;
  const int *pos_dev, *first;
  const float *dt;
  long long ldt;
  const float *dt_bias, *a_log, *skip;
  void *out;
  long long ldo;
  float *S;
  int heads, groups, dk, dv, cols;
};

template <typename T>
__global__ void __launch_bounds__(kStepThreads, 4) ssm_step_kernel(const SsmStepParams p) {
  extern __shared__ float sm[];
  float *qs = sm, *ks = qs + p.dk, *vs = ks + p.dk, *red = vs + p.cols;         // red: [row groups][cols]
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, g = h / (p.heads / p.groups);
  const int c0 = blockIdx.x * p.cols, width = min(p.cols, p.dv - c0);
  StatePass pass(p.S + ((long long)b * p.heads + h) * p.dk * p.dv + c0, p.dk, p.dv, p.cols, width);
  pass.begin();
  const int pos = *p.pos_dev, first = p.first ? p.first[b] : 0;
  const float dt = softplus(p.dt[b * p.ldt + h] + p.dt_bias[h]), a = expf(log_decay_ssm(p.a_log[h], dt));
  // one channel of the convolution; `keep`: this CTA also puts its input into the ring
  const T *x = reinterpret_cast<const T *>(p.xbc) + b * p.ldx, *w = reinterpret_cast<const T *>(p.conv_w);
  T *ring = reinterpret_cast<T *>(p.ring) + b * p.ring_bs;
  auto conv = [&](int ch, bool keep) {
    const T cur = x[ch];
    float acc = fmaf(to_f32<T>(w[(long long)(p.taps - 1) * p.channels + ch]), to_f32<T>(cur), to_f32<T>(reinterpret_cast<const T *>(p.conv_b)[ch]));
    for (int j = 1; j < p.taps; ++j) {
      const int col = pos - j;
      if (col >= first && col >= 0)
        acc = fmaf(to_f32<T>(w[(long long)(p.taps - 1 - j) * p.channels + ch]), to_f32<T>(ring[(long long)(col % p.ring_rows) * p.ring_ld + ch]), acc);
    }
    // (the row of this position is none of the rows that are read)
    if (keep) ring[(long long)(pos % p.ring_rows) * p.ring_ld + ch] = cur;
    // what the projection and the convolution give is an operand: rounded as a prompt's is
    return to_f32<T>(from_f32<T>(conv_silu<T>(acc)));
  };
  const bool lead = blockIdx.x == 0 && h % (p.heads / p.groups) == 0;
  const int b0 = p.heads * p.dv + g * p.dk, c1 = b0 + p.groups * p.dk;
  for (int i = tid; i < 2 * p.dk; i += kStepThreads) {
    if (i < p.dk) ks[i] = conv(b0 + i, lead) * dt;
    else qs[i - p.dk] = conv(c1 + i - p.dk, lead);
  }
  // (from the last thread down: the first ones have the keys)
  for (int c = kStepThreads - 1 - tid; c < width; c += kStepThreads) vs[c] = conv(h * p.dv + c0 + c, true);
  __syncthreads();
  pass.run([a](int) { return a; }, ks, qs, vs, red);
  __syncthreads();
  T *out = reinterpret_cast<T *>(p.out) + b * p.ldo + h * p.dv + c0;
  const float skip = p.skip[h];
  for (int c = tid; c < width; c += kStepThreads) {
    float y = skip * vs[c];
    for (int r = 0; r < pass.R; ++r) y += red[r * p.cols + c];
    out[c] = from_f32<T>(y);
  }
}

// ---- one token per sequence: gated linear attention ---------------------------------------------------------
struct GlaStepParams {
  const void *q, *k, *v, *g, *low;      // column ranges of one row layout; low [rank]: the inner projection of the decay
  long long ldp;
  const void *w2, *b2;                  // [heads*dk][rank], [heads*dk]
  int rank;
  float inv_tau, scale;
  const void *norm;                     // [heads*dv]
  float inv_count, eps;
  void *out;
  long long ldo;
  float *S;
  int heads, dk, dv, cols;
};

template <typename T>
__global__ void __launch_bounds__(kStepThreads, 4) gla_step_kernel(const GlaStepParams p) {
  extern __shared__ float sm[];
  float *as = sm, *qs = as + p.dk, *ks = qs + p.dk, *vs = ks + p.dk, *red = vs + p.cols;
  __shared__ float scratch[kStepThreads / 32];
  __shared__ __align__(8) ClusterSum head_sum;
  const int peers = gridDim.x;
  cluster_sum_begin(head_sum, peers);
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int c0 = blockIdx.x * p.cols, width = min(p.cols, p.dv - c0);
  const T *q = reinterpret_cast<const T *>(p.q) + b * p.ldp + h * p.dk, *k = reinterpret_cast<const T *>(p.k) + b * p.ldp + h * p.dk,
          *v = reinterpret_cast<const T *>(p.v) + b * p.ldp + h * p.dv + c0, *g = reinterpret_cast<const T *>(p.g) + b * p.ldp + h * p.dv + c0,
          *low = reinterpret_cast<const T *>(p.low) + b * p.ldp;
  StatePass pass(p.S + ((long long)b * p.heads + h) * p.dk * p.dv + c0, p.dk, p.dv, p.cols, width);
  pass.begin();
  for (int d = tid; d < p.dk; d += kStepThreads) {
    const T *w = reinterpret_cast<const T *>(p.w2) + (long long)(h * p.dk + d) * p.rank;
    float z = 0.f;
    for (int r = 0; r < p.rank; r += 8) {
      float wf[8], lf[8];
      load_pack<T>(w + r, wf);
      load_pack<T>(low + r, lf);
#pragma unroll
      for (int e = 0; e < 8; ++e) z = fmaf(wf[e], lf[e], z);
    }
    z += to_f32<T>(reinterpret_cast<const T *>(p.b2)[h * p.dk + d]);
    as[d] = expf(log_decay_gla(z, p.inv_tau));
    qs[d] = to_f32<T>(q[d]) * p.scale;
    ks[d] = to_f32<T>(k[d]);
  }
  for (int c = tid; c < width; c += kStepThreads) vs[c] = to_f32<T>(v[c]);
  __syncthreads();
  pass.run([as](int d) { return as[d]; }, ks, qs, vs, red);
  __syncthreads();
  float sq = 0.f;
  for (int c = tid; c < width; c += kStepThreads) {
    float x = 0.f;
    for (int r = 0; r < pass.R; ++r) x += red[r * p.cols + c];
    red[c] = x;                                     // (row group 0: only this thread has read column c of it)
    sq = fmaf(x, x, sq);
  }
  sq = block_sum<kStepThreads>(sq, scratch);
  sq = cluster_sum(head_sum, peers, sq);
  const float rs = rsqrtf(sq * p.inv_count + p.eps);
  T *out = reinterpret_cast<T *>(p.out) + b * p.ldo + h * p.dv + c0;
  const T *norm = reinterpret_cast<const T *>(p.norm) + h * p.dv + c0;
  for (int c = tid; c < width; c += kStepThreads) out[c] = from_f32<T>(red[c] * rs * to_f32<T>(norm[c]) * silu(to_f32<T>(g[c])));
}

// ---- gate and norm behind the state-space layer ------------------------------------------------------------
constexpr int kGroupThreads = 256, kGroupKeep = 4;

struct GroupNormParams {
  const void *y, *z, *norm;
  long long ldy, ldz, ldo;
  void *out;
  float eps;
  int rows, parts, len;        // equal parts of len real columns
  int dv, pad;                 // real and padded columns of a head
};

// A warp (THREADS 32) or a CTA per (row, part); VEC elements at a time, which lie in one head and one part.
template <typename T, int VEC, int THREADS>
__global__ void __launch_bounds__(kGroupThreads) gate_group_norm_kernel(const GroupNormParams p) {
  __shared__ float scratch[kGroupThreads / 32];
  griddep_wait();
  griddep_launch();
  const int tid = THREADS == 32 ? threadIdx.x & 31 : threadIdx.x;
  const long long unit = THREADS == 32 ? (long long)blockIdx.x * (kGroupThreads / 32) + (threadIdx.x >> 5) : blockIdx.x;
  if (unit >= (long long)p.rows * p.parts) return;
  const long long row = unit / p.parts;
  const int part = (int)(unit - row * p.parts), n = p.len / VEC;
  const T *y = reinterpret_cast<const T *>(p.y) + row * p.ldy, *z = reinterpret_cast<const T *>(p.z) + row * p.ldz,
          *norm = reinterpret_cast<const T *>(p.norm);
  T *out = reinterpret_cast<T *>(p.out) + row * p.ldo;
  auto column = [&](int i) {                       // padded column of the part's i-th vector
    const int r = part * p.len + i * VEC;
    return p.dv == p.pad ? r : r / p.dv * p.pad + r % p.dv;
  };
  auto gated = [&](int c, float (&f)[VEC]) {
    float g[VEC];
    if constexpr (VEC == 8) {
      load_pack<T>(y + c, f);
      load_pack<T>(z + c, g);
    } else {
      f[0] = to_f32<T>(y[c]);
      g[0] = to_f32<T>(z[c]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] *= __fdividef(g[e], 1.f + __expf(-g[e]));
  };
  float keep[kGroupKeep][VEC], sq = 0.f;           // the first vectors per thread stay in registers
#pragma unroll
  for (int i = 0; i < kGroupKeep; ++i) {
    if (tid + i * THREADS >= n) break;
    gated(column(tid + i * THREADS), keep[i]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sq = fmaf(keep[i][e], keep[i][e], sq);
  }
  for (int i = tid + kGroupKeep * THREADS; i < n; i += THREADS) {
    float f[VEC];
    gated(column(i), f);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sq = fmaf(f[e], f[e], sq);
  }
  const float rs = rsqrtf(block_sum<THREADS>(sq, scratch) / (float)p.len + p.eps);
  auto finish = [&](int c, float (&f)[VEC]) {
    if constexpr (VEC == 8) {
      float w[8];
      load_pack<T>(norm + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= rs * w[e];
      store_pack<T>(out + c, f);
    } else {
      out[c] = from_f32<T>(f[0] * rs * to_f32<T>(norm[c]));
    }
  };
#pragma unroll
  for (int i = 0; i < kGroupKeep; ++i) {
    if (tid + i * THREADS >= n) break;
    finish(column(tid + i * THREADS), keep[i]);
  }
  for (int i = tid + kGroupKeep * THREADS; i < n; i += THREADS) {
    float f[VEC];
    gated(column(i), f);
    finish(column(i), f);
  }
}

template <typename T> int launch_group_norm(const GroupNormParams &p, cudaStream_t st) {
  const long long units = (long long)p.rows * p.parts;
  const bool vec = p.dv % 8 == 0 && p.len % 8 == 0, warp = p.len <= 1024 && units >= 2ll * sm_count();
  const dim3 g((unsigned)(warp ? (units + 7) / 8 : units)), b(kGroupThreads);
  if (vec && warp) launch_pdl(gate_group_norm_kernel<T, 8, 32>, g, b, 0, st, p);
  else if (vec) launch_pdl(gate_group_norm_kernel<T, 8, kGroupThreads>, g, b, 0, st, p);
  else if (warp) launch_pdl(gate_group_norm_kernel<T, 1, 32>, g, b, 0, st, p);
  else launch_pdl(gate_group_norm_kernel<T, 1, kGroupThreads>, g, b, 0, st, p);
  return check_launch("gate_group_norm");
}

#define EB_BY_TYPE(dtype, call)                    \
  do {                                             \
    if ((dtype) == EB_F32) { using T = float; return call; }            \
    if ((dtype) == EB_F16) { using T = __half; return call; }           \
    { using T = __nv_bfloat16; return call; }                           \
  } while (0)

int check_heads(const char *name, int batch, int heads, int dk, int dv, int dtype) {
  if (!dtype_ok(dtype)) return fail(EB_EINVAL, "%s: bad dtype %d", name, dtype);
  if (batch < 0 || batch > 65535 || heads <= 0 || heads > 65535 || dk <= 0 || dv <= 0) return fail(EB_EINVAL, "%s: bad sizes", name);
  if (dk % 8 != 0 || dv % 8 != 0) return fail(EB_EINVAL, "%s: head sizes must be multiples of 8 (%d, %d)", name, dk, dv);
  return EB_OK;
}

// Columns per CTA and shared memory of a step kernel with `vectors` numbers per key row; 0 if it does not fit.
size_t step_smem(int split, int dk, int dv, int vectors, int *cols) {
  *cols = ((dv + split - 1) / split + 3) / 4 * 4;
  if (*cols > 4 * kStepThreads) return 0;
  const size_t smem = (size_t)(vectors * dk + *cols + kStepThreads / (*cols / 4) * *cols) * sizeof(float);
  return smem > 48 * 1024 ? 0 : smem;
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_short_conv(const void *x, long long ldx, const void *w, const void *b, void *out, long long ldo, int batch, int seq, int channels,
                             int taps, const int32_t *first, void *ring, long long ring_batch_stride, long long ring_ld, int ring_rows, int dtype,
                             void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "short_conv: bad dtype %d", dtype);
  EB_REQUIRE(x && w && b && out && ring, "short_conv: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && seq > 0 && (seq + kConvStrip - 1) / kConvStrip <= 65535 && channels > 0 && channels % 8 == 0 && taps > 0 && ring_rows > 0,
             "short_conv: bad sizes (%d channels, %d taps)", channels, taps);
  EB_REQUIRE(ldx >= channels && ldo >= channels && ring_ld >= channels && ldx % 8 == 0 && ldo % 8 == 0 && ring_ld % 8 == 0 && ring_batch_stride % 8 == 0,
             "short_conv: strides must be multiples of 8 and hold a row");
  EB_REQUIRE(aligned16(x) && aligned16(w) && aligned16(b) && aligned16(out) && aligned16(ring), "short_conv: pointers must be 16-byte aligned");
  ConvParams p{};
  p.x = x; p.ldx = ldx; p.w = w; p.b = b; p.out = out; p.ldo = ldo; p.C = channels; p.taps = taps; p.seq = seq; p.first = first;
  p.ring = ring; p.ring_bs = ring_batch_stride; p.ring_ld = ring_ld; p.ring_rows = ring_rows;
  EB_BY_TYPE(dtype, launch_conv<T>(p, batch, as_stream(stream)));
}

extern "C" int eb_ssm_scan(const void *xbc, long long ldx, const float *dt, long long ldt, const float *dt_bias, const float *a_log, const float *skip,
                           const int32_t *first, void *y, long long ldy, float *S, int batch, int seq, int heads, int groups, int dk, int dv, int dtype,
                           void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  if (int rc = check_heads("ssm_scan", batch, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(xbc && dt && dt_bias && a_log && skip && y && S, "ssm_scan: null pointer");
  EB_REQUIRE(seq > 0 && groups > 0 && heads % groups == 0, "ssm_scan: %d heads do not share %d groups", heads, groups);
  EB_REQUIRE(ldx >= (long long)heads * dv + 2ll * groups * dk && ldt >= heads && ldy >= (long long)heads * dv, "ssm_scan: row strides smaller than the rows they hold");
  const size_t es = dtype_size(dtype);
  ScanParams p{};
  p.v = xbc; p.k = reinterpret_cast<const char *>(xbc) + (size_t)heads * dv * es; p.q = reinterpret_cast<const char *>(p.k) + (size_t)groups * dk * es;
  p.ldq = p.ldk = p.ldv = ldx; p.group = heads / groups; p.gates = dt; p.ldg = ldt; p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip;
  p.scale = 1.f; p.first = first; p.o = y; p.ldo = ldy; p.S = S; p.seq = seq; p.heads = heads; p.dk = dk; p.dv = dv;
  EB_BY_TYPE(dtype, (launch_scan<T, false>(p, batch, as_stream(stream))));
}

extern "C" int eb_gla_scan(const void *q, const void *k, const void *v, long long ldp, const float *z, long long ldz, float tau, float scale,
                           const int32_t *first, void *o, long long ldo, float *S, int batch, int seq, int heads, int dk, int dv, int dtype, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  if (int rc = check_heads("gla_scan", batch, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(q && k && v && z && o && S, "gla_scan: null pointer");
  EB_REQUIRE(seq > 0 && tau > 0.f, "gla_scan: bad sizes, or tau is not positive");
  EB_REQUIRE(ldz >= (long long)heads * dk && ldo >= (long long)heads * dv, "gla_scan: row strides smaller than the rows they hold");
  ScanParams p{};
  p.q = q; p.k = k; p.v = v; p.ldq = p.ldk = p.ldv = ldp; p.group = 1; p.gates = z; p.ldg = ldz; p.scale = scale; p.inv_tau = 1.f / tau;
  p.first = first; p.o = o; p.ldo = ldo; p.S = S; p.seq = seq; p.heads = heads; p.dk = dk; p.dv = dv;
  EB_BY_TYPE(dtype, (launch_scan<T, true>(p, batch, as_stream(stream))));
}

extern "C" int eb_ssm_step(const void *xbc, long long ldx, const void *conv_w, const void *conv_b, int taps, void *ring, long long ring_batch_stride,
                           long long ring_ld, int ring_rows, const int32_t *pos_device, const int32_t *first, const float *dt, long long ldt,
                           const float *dt_bias, const float *a_log, const float *skip, void *y, long long ldy, float *S, int batch, int heads,
                           int groups, int dk, int dv, int dtype, void *stream) {
  if (batch == 0) return EB_OK;
  if (int rc = check_heads("ssm_step", batch, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(xbc && conv_w && conv_b && ring && pos_device && dt && dt_bias && a_log && skip && y && S, "ssm_step: null pointer");
  EB_REQUIRE(groups > 0 && heads % groups == 0, "ssm_step: %d heads do not share %d groups", heads, groups);
  const long long channels = (long long)heads * dv + 2ll * groups * dk;
  EB_REQUIRE(taps > 0 && ring_rows > 0 && channels < (1 << 30) && ldx >= channels && ring_ld >= channels && ldt >= heads && ldy >= (long long)heads * dv,
             "ssm_step: row strides smaller than the rows they hold");
  EB_REQUIRE(aligned16(S), "ssm_step: the state must be 16-byte aligned");
  SsmStepParams p{};
  p.xbc = xbc; p.ldx = ldx; p.conv_w = conv_w; p.conv_b = conv_b; p.taps = taps; p.channels = (int)channels; p.ring = ring; p.ring_bs = ring_batch_stride;
  p.ring_ld = ring_ld; p.ring_rows = ring_rows; p.pos_dev = pos_device; p.first = first; p.dt = dt; p.ldt = ldt; p.dt_bias = dt_bias; p.a_log = a_log;
  p.skip = skip; p.out = y; p.ldo = ldy; p.S = S; p.heads = heads; p.groups = groups; p.dk = dk; p.dv = dv;
  const int split = state_split((long long)batch * heads, dv);
  const size_t smem = step_smem(split, dk, dv, 2, &p.cols);
  if (!smem) return fail(EB_EUNSUPPORTED, "ssm_step: head sizes %d / %d are too large", dk, dv);
  const dim3 grid(split, heads, batch);
  EB_BY_TYPE(dtype, (launch_pdl(ssm_step_kernel<T>, grid, dim3(kStepThreads), smem, as_stream(stream), p), check_launch("ssm_step")));
}

extern "C" int eb_gla_step(const void *q, const void *k, const void *v, const void *g, const void *low, long long ldp, const void *w2, const void *b2,
                           int rank, float tau, float scale, const void *norm, int dv_count, float eps, void *out, long long ldo, float *S, int batch,
                           int heads, int dk, int dv, int dtype, void *stream) {
  if (batch == 0) return EB_OK;
  if (int rc = check_heads("gla_step", batch, heads, dk, dv, dtype)) return rc;
  EB_REQUIRE(q && k && v && g && low && w2 && b2 && norm && out && S, "gla_step: null pointer");
  EB_REQUIRE(rank > 0 && rank % 8 == 0 && tau > 0.f && ldp % 8 == 0 && ldo >= (long long)heads * dv, "gla_step: the rank must be a multiple of 8, tau positive");
  EB_REQUIRE(dv_count > 0 && dv_count <= dv, "gla_step: the mean is over 1..dv elements");
  EB_REQUIRE(aligned16(S) && aligned16(low) && aligned16(w2), "gla_step: pointers must be 16-byte aligned");
  GlaStepParams p{};
  p.q = q; p.k = k; p.v = v; p.g = g; p.low = low; p.ldp = ldp; p.w2 = w2; p.b2 = b2; p.rank = rank; p.inv_tau = 1.f / tau; p.scale = scale;
  p.norm = norm; p.inv_count = 1.f / (float)dv_count; p.eps = eps; p.out = out; p.ldo = ldo; p.S = S; p.heads = heads; p.dk = dk; p.dv = dv;
  const int split = state_split((long long)batch * heads, dv);
  const size_t smem = step_smem(split, dk, dv, 3, &p.cols);
  if (!smem) return fail(EB_EUNSUPPORTED, "gla_step: head sizes %d / %d are too large", dk, dv);
  const dim3 grid(split, heads, batch);
  EB_BY_TYPE(dtype, (launch_state_step("gla_step", gla_step_kernel<T>, p, grid, split, smem, as_stream(stream))));
}

extern "C" int eb_gate_group_norm(const void *y, long long ldy, const void *z, long long ldz, const void *norm, float eps, void *out, long long ldo,
                                  int rows, int heads, int dv, int dv_padded, int parts, int dtype, void *stream) {
  if (rows == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "gate_group_norm: bad dtype %d", dtype);
  EB_REQUIRE(y && z && norm && out, "gate_group_norm: null pointer");
  EB_REQUIRE(rows > 0 && heads > 0 && dv > 0 && dv_padded >= dv && dv_padded % 8 == 0 && (long long)heads * dv_padded < (1 << 30), "gate_group_norm: bad sizes");
  EB_REQUIRE(parts > 0 && (long long)heads * dv % parts == 0, "gate_group_norm: %lld columns in %d equal parts", (long long)heads * dv, parts);
  const long long width = (long long)heads * dv_padded;
  EB_REQUIRE(ldy >= width && ldz >= width && ldo >= width && ldy % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0, "gate_group_norm: row strides must be multiples of 8 and hold a row");
  EB_REQUIRE(aligned16(y) && aligned16(z) && aligned16(norm) && aligned16(out), "gate_group_norm: pointers must be 16-byte aligned");
  EB_REQUIRE((long long)rows * parts < (1ll << 31), "gate_group_norm: too many rows");
  GroupNormParams p{};
  p.y = y; p.z = z; p.norm = norm; p.ldy = ldy; p.ldz = ldz; p.ldo = ldo; p.out = out; p.eps = eps; p.rows = rows; p.parts = parts;
  p.len = (int)((long long)heads * dv / parts); p.dv = dv; p.pad = dv_padded;
  EB_BY_TYPE(dtype, launch_group_norm<T>(p, as_stream(stream)));
}
