// Selective state space with a state per channel (Mamba): behind a short convolution, for channel c and state n
//
//   dt = softplus(z_c + bias_c);   S[c][n] = exp(-exp(a_log[c][n]) dt) S[c][n] + dt x_c B_n;   y_c = sum_n S[c][n] C_n + skip_c x_c
//   out_c = y_c silu(gate_c)
//
// B and C are common to all channels of a token.  Every state element has a decay of its own per token, so there is
// no product to put on the tensor cores: the exponentials set the pace (one per channel, state and token on
// the special-function units).
//
//   scan          a prompt: a channel's states over the lanes of a group, a few per lane in registers, up to 32
//                 tokens at a time through shared memory; steps, products dt x and the gate are formed by the whole
//                 CTA around each chunk, the sums over a group's lanes are taken for four tokens together.
//   scan_step     one token per sequence: the step's projection (dt_rank numbers per channel), the pass over the
//                 state and the gate in one launch; a CTA keeps its channels for several sequences, so that
//                 their projection is read once.
//   conv_step     the convolution of one token per sequence on its ring.
//
// State, steps, decays, B and C are fp32.  (Compiled without fast math: decays add up over a sequence.)
#include "common.cuh"
#include "decay_gates.cuh"
#include "packed_math.cuh"

namespace eb {
namespace {

constexpr float kLog2eScan = 1.4426950408889634f;

__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float gate_silu(float x) { return silu_fast(x); }
template <> __device__ __forceinline__ float gate_silu<float>(float x) { return x / (1.f + expf(-x)); }

// log(1 + exp(x)); 16-bit models take the special-function unit's exponential (2^-22 of the result)
template <typename T> __device__ __forceinline__ float step_size(float x) { return fmaxf(x, 0.f) + log1p_unit(ex2(-fabsf(x) * kLog2eScan)); }
template <> __device__ __forceinline__ float step_size<float>(float x) { return softplus(x); }

// One element's step, S' = exp(dt rate) S + in.  16-bit models: a power of two (rates times log2 e).  32-bit models form
// exp - 1: a slow decay is close to one, and the rounding of one, always to the same side, adds up over a sequence.
template <typename T> struct Decay {
  static constexpr float kScale = kLog2eScan;
  static __device__ __forceinline__ float step(float S, float e, float in) { return fmaf(ex2(e), S, in); }
};
template <> struct Decay<float> {
  static constexpr float kScale = 1.f;
  static __device__ __forceinline__ float step(float S, float e, float in) { return fmaf(expm1f(e), S, S + in); }
};

template <typename T> struct Two;
template <> struct Two<float> {
  using R = float2;
  static __device__ __forceinline__ float2 get(R r) { return r; }
  static __device__ __forceinline__ R put(float a, float b) { return make_float2(a, b); }
  static __device__ __forceinline__ R zero() { return make_float2(0.f, 0.f); }
};
template <typename T> struct Two {
  using R = uint32_t;
  static __device__ __forceinline__ float2 get(R r) { return unpack2<T>(r); }
  static __device__ __forceinline__ R put(float a, float b) { return pack2<T>(a, b); }
  static __device__ __forceinline__ R zero() { return 0u; }
};

struct SelScanParams {
  const void *x, *gate;        // rows of the convolved input and of the gate
  long long ldx, ldg;
  const float *z;              // prompt: rows of the steps' projection; step: not used
  long long ldz;
  const float *bc;             // rows [B: states | C: states]
  long long ldbc;
  const float *bias, *a_log, *skip;      // [inner], [inner][states], [inner]
  const void *low, *w;         // step: rows of the low-rank part, [inner][rank]
  long long ldl;
  int rank;
  const int *first;
  void *out;
  long long ldo;
  float *S;                    // [batch][inner][states]
  int batch, seq, inner, states, per_cta;
};

// Sums over the LPC lanes of a group of four values each (one per token).  The lane that ends with token i's sum is
// in group position (i * LPC / 4) or after it; LPC 1 and 2 hold several.
template <int LPC, typename F> __device__ __forceinline__ void group_sum4(float (&v)[4], int sub, F store) {
  if constexpr (LPC == 1) {
#pragma unroll
    for (int i = 0; i < 4; ++i) store(i, v[i]);
  } else {
    const bool hi = sub & (LPC / 2);
    float a = hi ? v[2] : v[0], b = hi ? v[3] : v[1];
    a += __shfl_xor_sync(0xffffffffu, hi ? v[0] : v[2], LPC / 2);
    b += __shfl_xor_sync(0xffffffffu, hi ? v[1] : v[3], LPC / 2);
    if constexpr (LPC == 2) {
      store(hi ? 2 : 0, a);
      store(hi ? 3 : 1, b);
    } else {
      const bool mid = sub & (LPC / 4);
      float s = mid ? b : a;
      s += __shfl_xor_sync(0xffffffffu, mid ? a : b, LPC / 4);
#pragma unroll
      for (int o = LPC / 8; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if ((sub & (LPC / 4 - 1)) == 0) store((hi ? 2 : 0) + (mid ? 1 : 0), s);
    }
  }
}

// NS: states per lane; LPC: lanes per channel, or per pair of them (CPT 2); NS * LPC >= states
template <int LPC, int CPT> constexpr int scan_threads = LPC * 8 / CPT > 128 ? LPC * 8 / CPT : 128;

template <typename T, int NS, int LPC, int CPT>
__global__ void __launch_bounds__(scan_threads<LPC, CPT>) selective_scan_kernel(const SelScanParams p) {
  using W = Two<T>;
  using R = typename W::R;
  constexpr int kThreads = scan_threads<LPC, CPT>, CH = CPT * kThreads / LPC, NP = NS * LPC;        // channels of this CTA, states with padding
  constexpr int kTokens = CH * CPT >= 128 ? 8 : CH >= 64 ? 16 : NP <= 32 ? 32 : NP <= 64 ? 16 : 8;
  constexpr int kPairs = CH / 2, kRowsPass = kThreads / kPairs;   // elementwise: thread = two channels of a token,
  constexpr int kPasses = kTokens > kRowsPass ? kTokens / kRowsPass : 1;                                  // this often per chunk
  constexpr int kBcVec = kTokens * 2 * NP / 4, kBcIters = (kBcVec + kThreads - 1) / kThreads;
  static_assert(kPasses == 1 || kRowsPass * kPasses == kTokens, "a chunk is whole passes");
  __shared__ __align__(16) float4 s_dt[2][kTokens][kPairs];       // of two channels: step, step * input
  __shared__ __align__(16) float s_bc[2][kTokens][2 * NP];
  __shared__ __align__(8) float s_y[2][kTokens][CH + 2];

  griddep_wait();
  griddep_launch();
  const int tid = threadIdx.x, c0 = blockIdx.x * CH, b = blockIdx.y;
  const int first = p.first ? p.first[b] : 0;
  const long long row0 = (long long)b * p.seq;
  // elementwise role: channels c0 + 2 * pc and the next, tokens pr + kRowsPass * i of a chunk
  const int pc = tid % kPairs, pr = tid / kPairs, ec = c0 + 2 * pc;
  const bool has_e = ec < p.inner && pr < kTokens;                // (inner is even)
  const float2 bias = has_e ? *reinterpret_cast<const float2 *>(p.bias + ec) : make_float2(0.f, 0.f);
  const float2 skip = has_e ? *reinterpret_cast<const float2 *>(p.skip + ec) : make_float2(0.f, 0.f);
  R xr[kPasses], gr[kPasses];
  float2 zr[kPasses];
  float4 bcr[kBcIters];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < kPasses; ++i) {
      const int t = t0 + pr + kRowsPass * i;
      xr[i] = gr[i] = W::zero();
      zr[i] = make_float2(0.f, 0.f);
      if (t < p.seq && has_e) {
        xr[i] = *reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.x) + (row0 + t) * p.ldx + ec);
        gr[i] = *reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.gate) + (row0 + t) * p.ldg + ec);
        zr[i] = *reinterpret_cast<const float2 *>(p.z + (row0 + t) * p.ldz + ec);
      }
    }
#pragma unroll
    for (int i = 0; i < kBcIters; ++i) {
      const int v = tid + i * kThreads, t = t0 + v / (2 * NP / 4), n = v % (2 * NP / 4) * 4;        // n: column of the padded row
      const int half = n >= NP, at = n - half * NP;
      bcr[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (v < kBcVec && t < p.seq && at < p.states) bcr[i] = *reinterpret_cast<const float4 *>(p.bc + (row0 + t) * p.ldbc + half * p.states + at);
    }
  };
  auto prepare = [&](int t0, int buf) {
#pragma unroll
    for (int i = 0; i < kPasses; ++i) {
      const int r = pr + kRowsPass * i, t = t0 + r;
      if (r >= kTokens) continue;
      const bool live = t >= first && t < p.seq;
      const float2 x = W::get(xr[i]);
      const float d0 = live ? step_size<T>(zr[i].x + bias.x) : 0.f, d1 = live ? step_size<T>(zr[i].y + bias.y) : 0.f;
      s_dt[buf][r][pc] = make_float4(d0, live ? d0 * x.x : 0.f, d1, live ? d1 * x.y : 0.f);
    }
#pragma unroll
    for (int i = 0; i < kBcIters; ++i) {
      const int v = tid + i * kThreads;
      if (v < kBcVec) *reinterpret_cast<float4 *>(&s_bc[buf][v / (2 * NP / 4)][v % (2 * NP / 4) * 4]) = bcr[i];
    }
  };

  // scan role: CPT channels from c on, states sub * NS ..
  const int cp = tid / LPC, sub = tid % LPC, c = c0 + CPT * cp;
  float A[CPT][NS], S[CPT][NS];
#pragma unroll
  for (int k = 0; k < CPT; ++k)
#pragma unroll
    for (int n = 0; n < NS; ++n) {
      const int s = sub * NS + n;
      A[k][n] = c < p.inner && s < p.states ? -expf(p.a_log[(long long)(c + k) * p.states + s]) * Decay<T>::kScale : 0.f;
      S[k][n] = 0.f;
    }
  fetch(0);
  prepare(0, 0);
  __syncthreads();
  const int chunks = (p.seq + kTokens - 1) / kTokens;
  for (int j = 0; j < chunks; ++j) {
    const int buf = j & 1, t0 = j * kTokens;
    R xk[kPasses], gk[kPasses];
#pragma unroll
    for (int i = 0; i < kPasses; ++i) { xk[i] = xr[i]; gk[i] = gr[i]; }
    const bool more = j + 1 < chunks;
    if (more) fetch(t0 + kTokens);
#pragma unroll 2
    for (int t = 0; t < kTokens; t += 4) {
      float y[CPT][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float d[2 * CPT];                            // (step, step * input) of the channels
        if constexpr (CPT == 2) {
          const float4 v = s_dt[buf][t + i][cp];
          d[0] = v.x; d[1] = v.y; d[2] = v.z; d[3] = v.w;
        } else {
          const float2 v = reinterpret_cast<const float2 *>(s_dt[buf][t + i])[cp];
          d[0] = v.x; d[1] = v.y;
        }
        const float *B = &s_bc[buf][t + i][sub * NS], *C = B + NP;
        float acc[CPT][2] = {}, bb[4], cc[4];
#pragma unroll
        for (int n = 0; n < NS; n += 2) {
          float2 bv, cv;
          if (NS % 4 == 0 && n % 4 == 0) {
            const float4 b4 = *reinterpret_cast<const float4 *>(B + n), c4 = *reinterpret_cast<const float4 *>(C + n);
            bb[0] = b4.x; bb[1] = b4.y; bb[2] = b4.z; bb[3] = b4.w;
            cc[0] = c4.x; cc[1] = c4.y; cc[2] = c4.z; cc[3] = c4.w;
          }
          if (NS % 4 == 0) {
            bv = make_float2(bb[n % 4], bb[n % 4 + 1]);
            cv = make_float2(cc[n % 4], cc[n % 4 + 1]);
          } else {
            bv = *reinterpret_cast<const float2 *>(B + n);
            cv = *reinterpret_cast<const float2 *>(C + n);
          }
#pragma unroll
          for (int k = 0; k < CPT; ++k) {
            float *s = S[k] + n, e0, e1, b0, b1;
            mul2(e0, e1, d[2 * k], d[2 * k], A[k][n], A[k][n + 1]);
            mul2(b0, b1, d[2 * k + 1], d[2 * k + 1], bv.x, bv.y);
            if constexpr (sizeof(T) == 2) {
              fma2(s[0], s[1], ex2(e0), ex2(e1), s[0], s[1], b0, b1);
            } else {
              s[0] = Decay<T>::step(s[0], e0, b0);
              s[1] = Decay<T>::step(s[1], e1, b1);
            }
            fma2(acc[k][0], acc[k][1], s[0], s[1], cv.x, cv.y, acc[k][0], acc[k][1]);
          }
        }
#pragma unroll
        for (int k = 0; k < CPT; ++k) y[k][i] = acc[k][0] + acc[k][1];
      }
#pragma unroll
      for (int k = 0; k < CPT; ++k) group_sum4<LPC>(y[k], sub, [&](int i, float v) { s_y[buf][t + i][CPT * cp + k] = v; });
    }
    if (more) prepare(t0 + kTokens, buf ^ 1);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kPasses; ++i) {
      const int r = pr + kRowsPass * i, t = t0 + r;
      if (t >= p.seq || !has_e || r >= kTokens) continue;
      const float2 x = W::get(xk[i]), g = W::get(gk[i]), y = *reinterpret_cast<const float2 *>(&s_y[buf][r][2 * pc]);
      *reinterpret_cast<R *>(reinterpret_cast<T *>(p.out) + (row0 + t) * p.ldo + ec) =
          W::put(fmaf(skip.x, x.x, y.x) * gate_silu<T>(g.x), fmaf(skip.y, x.y, y.y) * gate_silu<T>(g.y));
    }
  }
  if (c < p.inner) {
#pragma unroll
    for (int k = 0; k < CPT; ++k) {
      float *dst = p.S + ((long long)b * p.inner + c + k) * p.states + sub * NS;
#pragma unroll
      for (int n = 0; n < NS; n += 2)
        if (sub * NS + n < p.states) *reinterpret_cast<float2 *>(dst + n) = make_float2(S[k][n], S[k][n + 1]);
    }
  }
}

template <typename T> __device__ __forceinline__ float dot8(const T *a, const T *b, float acc) {
  constexpr int N = Vec16<T>::N;
#pragma unroll
  for (int i = 0; i < 8 / N; ++i) {
    Vec16<T> va, vb;
    float fa[N], fb[N];
    va.load(a + i * N);
    vb.load(b + i * N);
    va.unpack(fa);
    vb.unpack(fb);
#pragma unroll
    for (int e = 0; e < N; ++e) acc = fmaf(fa[e], fb[e], acc);
  }
  return acc;
}

constexpr int kSelStepThreads = 256;

template <typename T, int NS, int LPC>
__global__ void __launch_bounds__(kSelStepThreads) selective_step_kernel(const SelScanParams p) {
  constexpr int CH = kSelStepThreads / LPC;
  const int ch = threadIdx.x / LPC, sub = threadIdx.x % LPC, c = min(blockIdx.x * CH + ch, p.inner - 1);
  const bool mine = blockIdx.x * CH + ch < p.inner;
  float A[NS];
#pragma unroll
  for (int n = 0; n < NS; ++n) A[n] = sub * NS + n < p.states ? -expf(p.a_log[(long long)c * p.states + sub * NS + n]) * Decay<T>::kScale : 0.f;
  const float bias = p.bias[c], skip = p.skip[c];
  const T *w = reinterpret_cast<const T *>(p.w) + (long long)c * p.rank;
  griddep_wait();
  griddep_launch();
  const int b1 = min(p.batch, (int)(blockIdx.y + 1) * p.per_cta);
  for (int b = blockIdx.y * p.per_cta; b < b1; ++b) {
    float *Sp = p.S + ((long long)b * p.inner + c) * p.states + sub * NS;
    const float *B = p.bc + (long long)b * p.ldbc + sub * NS, *C = B + p.states;
    float4 S4[NS / 4], B4[NS / 4], C4[NS / 4];
#pragma unroll
    for (int n = 0; n < NS / 4; ++n) {
      S4[n] = B4[n] = C4[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (sub * NS + 4 * n < p.states) {
        S4[n] = *reinterpret_cast<const float4 *>(Sp + 4 * n);
        B4[n] = *reinterpret_cast<const float4 *>(B + 4 * n);
        C4[n] = *reinterpret_cast<const float4 *>(C + 4 * n);
      }
    }
    const float x = to_f32<T>(reinterpret_cast<const T *>(p.x)[b * p.ldx + c]), g = to_f32<T>(reinterpret_cast<const T *>(p.gate)[b * p.ldg + c]);
    const T *low = reinterpret_cast<const T *>(p.low) + b * p.ldl;
    float z = 0.f;
    for (int r = sub * 8; r < p.rank; r += LPC * 8) z = dot8<T>(w + r, low + r, z);
#pragma unroll
    for (int o = LPC / 2; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    const float dt = step_size<T>(z + bias), dx = dt * x;
    float y = 0.f;
#pragma unroll
    for (int n = 0; n < NS / 4; ++n) {
      S4[n].x = Decay<T>::step(S4[n].x, dt * A[4 * n], dx * B4[n].x);
      S4[n].y = Decay<T>::step(S4[n].y, dt * A[4 * n + 1], dx * B4[n].y);
      S4[n].z = Decay<T>::step(S4[n].z, dt * A[4 * n + 2], dx * B4[n].z);
      S4[n].w = Decay<T>::step(S4[n].w, dt * A[4 * n + 3], dx * B4[n].w);
      y = fmaf(S4[n].x, C4[n].x, fmaf(S4[n].y, C4[n].y, fmaf(S4[n].z, C4[n].z, fmaf(S4[n].w, C4[n].w, y))));
      if (mine && sub * NS + 4 * n < p.states) *reinterpret_cast<float4 *>(Sp + 4 * n) = S4[n];
    }
#pragma unroll
    for (int o = LPC / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (mine && sub == 0) reinterpret_cast<T *>(p.out)[b * p.ldo + c] = from_f32<T>(fmaf(skip, x, y) * gate_silu<T>(g));
  }
}

// ---- convolution of one token per sequence ----
struct ConvStepParams {
  const void *x;
  long long ldx;
  const void *w, *b;           // [taps][C], [C]
  void *out;
  long long ldo;
  int C, taps;
  const int *pos_dev, *first;
  void *ring;
  long long ring_bs, ring_ld;
  int ring_rows;
};

// Thread = two channels
template <typename T>
__global__ void __launch_bounds__(128) conv_step_kernel(const ConvStepParams p) {
  using W = Two<T>;
  using R = typename W::R;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 2, b = blockIdx.y;
  if (c >= p.C) return;
  griddep_wait();
  griddep_launch();
  const int pos = max(*p.pos_dev, 0), first = p.first ? p.first[b] : 0;
  T *ring = reinterpret_cast<T *>(p.ring) + b * p.ring_bs + c;
  const R cur = *reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.x) + b * p.ldx + c);
  float2 acc = W::get(*reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.b) + c));
  for (int j = 0; j < p.taps; ++j) {
    const int t = pos - (p.taps - 1) + j;
    if (t < first) continue;
    const float2 f = W::get(t == pos ? cur : *reinterpret_cast<const R *>(ring + (long long)(t % p.ring_rows) * p.ring_ld));
    const float2 w = W::get(*reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.w) + (long long)j * p.C + c));
    acc.x = fmaf(w.x, f.x, acc.x);
    acc.y = fmaf(w.y, f.y, acc.y);
  }
  *reinterpret_cast<R *>(ring + (long long)(pos % p.ring_rows) * p.ring_ld) = cur;
  *reinterpret_cast<R *>(reinterpret_cast<T *>(p.out) + b * p.ldo + c) = W::put(gate_silu<T>(acc.x), gate_silu<T>(acc.y));
}

template <typename T, int NS, int LPC, int CPT> int launch_scan(const SelScanParams &p, cudaStream_t st) {
  constexpr int kThreads = scan_threads<LPC, CPT>, CH = CPT * kThreads / LPC;
  launch_pdl(selective_scan_kernel<T, NS, LPC, CPT>, dim3((p.inner + CH - 1) / CH, p.batch), dim3(kThreads), 0, st, p);
  return check_launch("selective_scan");
}

template <typename T, int NS, int LPC> int launch_step(SelScanParams p, cudaStream_t st) {
  constexpr int CH = kSelStepThreads / LPC;
  const int tiles = (p.inner + CH - 1) / CH;
  p.per_cta = 1;
  while (p.per_cta < 8 && (long long)tiles * ((p.batch + 2 * p.per_cta - 1) / (2 * p.per_cta)) >= 4ll * sm_count()) p.per_cta *= 2;
  launch_pdl(selective_step_kernel<T, NS, LPC>, dim3(tiles, (p.batch + p.per_cta - 1) / p.per_cta), dim3(kSelStepThreads), 0, st, p);
  return check_launch("selective_step");
}

// 16 states: with few warps the machine wants many short chains, with plenty fewer loads of B and C per state
template <typename T> int launch_scan16(const SelScanParams &p, cudaStream_t st) {
  const double warps = (double)p.batch * p.inner * 16 / 128 / (4.0 * sm_count());      // per scheduler, four states per thread
  if (warps < 1.5) return launch_scan<T, 2, 8, 1>(p, st);
  return warps < 8.0 ? launch_scan<T, 2, 8, 2>(p, st) : launch_scan<T, 4, 4, 2>(p, st);
}

template <typename T> int launch_sel(const SelScanParams &p, bool step, cudaStream_t st) {
  if (p.states <= 4) return step ? launch_step<T, 4, 1>(p, st) : launch_scan<T, 4, 1, 1>(p, st);
  if (p.states <= 8) return step ? launch_step<T, 4, 2>(p, st) : launch_scan<T, 2, 4, 1>(p, st);
  if (p.states <= 16) return step ? launch_step<T, 4, 4>(p, st) : launch_scan16<T>(p, st);
  if (p.states <= 32) return step ? launch_step<T, 4, 8>(p, st) : launch_scan<T, 4, 8, 1>(p, st);
  if (p.states <= 64) return step ? launch_step<T, 8, 8>(p, st) : launch_scan<T, 4, 16, 1>(p, st);
  if (p.states <= 128) return step ? launch_step<T, 8, 16>(p, st) : launch_scan<T, 8, 16, 1>(p, st);
  return step ? launch_step<T, 8, 32>(p, st) : launch_scan<T, 8, 32, 1>(p, st);
}

int check_scan(const char *what, const SelScanParams &p) {
  EB_REQUIRE(p.x && p.gate && p.bc && p.bias && p.a_log && p.skip && p.out && p.S, "%s: null pointer", what);
  EB_REQUIRE(p.batch > 0 && p.batch <= 65535 && p.seq > 0 && p.inner > 0 && p.inner % 8 == 0, "%s: the channels are a multiple of 8 (got %d)", what, p.inner);
  EB_REQUIRE(p.states > 0 && p.states % 4 == 0 && p.states <= 256, "%s: the states are a multiple of 4, at most 256 (got %d)", what, p.states);
  EB_REQUIRE(p.ldx >= p.inner && p.ldg >= p.inner && p.ldo >= p.inner && p.ldbc >= 2 * p.states && p.ldx % 2 == 0 && p.ldg % 2 == 0 && p.ldo % 2 == 0 && p.ldbc % 4 == 0,
             "%s: row strides are too small or odd", what);
  EB_REQUIRE(aligned16(p.x) && aligned16(p.gate) && aligned16(p.bc) && aligned16(p.bias) && aligned16(p.a_log) && aligned16(p.skip) && aligned16(p.out) && aligned16(p.S),
             "%s: pointers must be 16-byte aligned", what);
  return EB_OK;
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_selective_scan(const void *x, long long ldx, const void *gate, long long ldg, const float *z, long long ldz, const float *bc,
                                 long long ldbc, const float *bias, const float *a_log, const float *skip, const int32_t *first, void *out,
                                 long long ldo, float *S, int batch, int seq, int inner, int states, int dtype, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "selective_scan: bad dtype %d", dtype);
  SelScanParams p{};
  p.x = x; p.ldx = ldx; p.gate = gate; p.ldg = ldg; p.z = z; p.ldz = ldz; p.bc = bc; p.ldbc = ldbc; p.bias = bias; p.a_log = a_log; p.skip = skip;
  p.first = first; p.out = out; p.ldo = ldo; p.S = S; p.batch = batch; p.seq = seq; p.inner = inner; p.states = states;
  if (int rc = check_scan("selective_scan", p)) return rc;
  EB_REQUIRE(z && aligned16(z) && ldz >= inner && ldz % 2 == 0, "selective_scan: the steps' projection has a row per token");
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_sel<float>(p, false, st);
  if (dtype == EB_F16) return launch_sel<__half>(p, false, st);
  return launch_sel<__nv_bfloat16>(p, false, st);
}

extern "C" int eb_selective_step(const void *x, long long ldx, const void *gate, long long ldg, const void *low, long long ldl, const void *w,
                                 int rank, const float *bc, long long ldbc, const float *bias, const float *a_log, const float *skip, void *out,
                                 long long ldo, float *S, int batch, int inner, int states, int dtype, void *stream) {
  if (batch == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "selective_step: bad dtype %d", dtype);
  SelScanParams p{};
  p.x = x; p.ldx = ldx; p.gate = gate; p.ldg = ldg; p.low = low; p.ldl = ldl; p.w = w; p.rank = rank; p.bc = bc; p.ldbc = ldbc; p.bias = bias;
  p.a_log = a_log; p.skip = skip; p.out = out; p.ldo = ldo; p.S = S; p.batch = batch; p.seq = 1; p.inner = inner; p.states = states;
  if (int rc = check_scan("selective_step", p)) return rc;
  EB_REQUIRE(low && w && aligned16(low) && aligned16(w) && rank > 0 && rank % 8 == 0 && ldl >= rank && ldl % 8 == 0, "selective_step: the rank is a multiple of 8 (got %d)", rank);
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_sel<float>(p, true, st);
  if (dtype == EB_F16) return launch_sel<__half>(p, true, st);
  return launch_sel<__nv_bfloat16>(p, true, st);
}

extern "C" int eb_short_conv_step(const void *x, long long ldx, const void *w, const void *b, void *out, long long ldo, int batch, int channels,
                                  int taps, const int32_t *pos_device, const int32_t *first, void *ring, long long ring_batch_stride,
                                  long long ring_ld, int ring_rows, int dtype, void *stream) {
  if (batch == 0 || channels == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "short_conv_step: bad dtype %d", dtype);
  EB_REQUIRE(x && w && b && out && ring && pos_device, "short_conv_step: null pointer");
  EB_REQUIRE(batch > 0 && batch <= 65535 && channels > 0 && channels % 8 == 0 && taps > 0 && ring_rows > 0, "short_conv_step: bad sizes");
  EB_REQUIRE(ldx >= channels && ldo >= channels && ring_ld >= channels && ldx % 2 == 0 && ldo % 2 == 0 && ring_ld % 2 == 0 && ring_batch_stride % 2 == 0,
             "short_conv_step: row strides are too small or odd");
  EB_REQUIRE(aligned16(x) && aligned16(w) && aligned16(b) && aligned16(out) && aligned16(ring), "short_conv_step: pointers must be 16-byte aligned");
  ConvStepParams p{};
  p.x = x; p.ldx = ldx; p.w = w; p.b = b; p.out = out; p.ldo = ldo; p.C = channels; p.taps = taps; p.pos_dev = pos_device; p.first = first;
  p.ring = ring; p.ring_bs = ring_batch_stride; p.ring_ld = ring_ld; p.ring_rows = ring_rows;
  cudaStream_t st = as_stream(stream);
  const dim3 g((channels / 2 + 127) / 128, batch), t(128);
  if (dtype == EB_F32) launch_pdl(conv_step_kernel<float>, g, t, 0, st, p);
  else if (dtype == EB_F16) launch_pdl(conv_step_kernel<__half>, g, t, 0, st, p);
  else launch_pdl(conv_step_kernel<__nv_bfloat16>, g, t, 0, st, p);
  return check_launch("short_conv_step");
}
