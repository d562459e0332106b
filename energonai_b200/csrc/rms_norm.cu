// RMS norm and what surrounds it in a decoder whose residual stream is kept in fp32:
//
//   rms_norm          y = x / sqrt(mean(x^2) + eps) * (w_offset + w), rows optionally written a
//                     second time into a ring cache (row of position p = p mod capacity)
//   rms_residual      x += norm(y), x fp32 in place, plus a copy of the new x in the operand type
//                     for the products that read it.  y is a plain row, or the weighted sum of the
//                     rows a mixture of experts produced for the token.  Optionally the router of
//                     the mixture that follows is evaluated on the new row in the same launch
//                     (generation steps: the row is already in registers, and one launch less
//                     lies on the critical path).
//   stream_update     the residual step of blocks that normalise in front of AND behind a
//                     sublayer: x += norm(y * sigmoid(gate)) * w_out, then h = norm(x) * w_next for
//                     the sublayer that follows.  With `src` it starts the stream: x = scale * src.
//   stream_add        the residual step of blocks that normalise in front of a sublayer only:
//                     x += scale * Y, then h = norm(x) * w_next.  Y is a row, the sum of two rows
//                     normalised each by itself (mixers side by side), or what a mixture of experts
//                     with identity experts and a gated shared expert produced for the token.
//                     Optionally the router of the mixture that follows is evaluated on h.
//
// One CTA per row, the row register-resident in packs of 8; statistics, weights and the residual
// are fp32 throughout.
#include "common.cuh"
#include "router.cuh"

namespace eb {
namespace {

constexpr int kNormThreads = 256;

template <typename T> __device__ __forceinline__ void load8(const T *p, float (&f)[8]);
template <> __device__ __forceinline__ void load8<float>(const float *p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__half>(const __half *p, float (&f)[8]) {
  Vec16<__half> v;
  v.load(p);
  v.unpack(f);
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16 *p, float (&f)[8]) {
  Vec16<__nv_bfloat16> v;
  v.load(p);
  v.unpack(f);
}
template <typename T> __device__ __forceinline__ void store8(T *p, const float (&f)[8]);
template <> __device__ __forceinline__ void store8<float>(float *p, const float (&f)[8]) {
  *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4 *>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
template <> __device__ __forceinline__ void store8<__half>(__half *p, const float (&f)[8]) {
  Vec16<__half> v;
  v.pack(f);
  v.store(p);
}
template <> __device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16 *p, const float (&f)[8]) {
  Vec16<__nv_bfloat16> v;
  v.pack(f);
  v.store(p);
}

struct RmsParams {
  const void *x;               // rows ldx apart
  long long ldx;
  const void *w;               // [n2] in the output type
  float w_offset, eps, inv_count;
  void *y;                     // rows ldy apart, or null
  long long ldy;
  int n1, n2;
  // ring cache: row (b, s) of the n1 = batch * rows_per_batch rows holds position pos0 + s of
  // sequence b; the last `ring_rows` positions are kept at ring + b*ring_bs + (position mod ring_rows)*ring_ld
  void *ring;
  long long ring_bs, ring_ld;
  int ring_rows, rows_per_batch;
  const int *pos_dev;          // device scalar with pos0, or null (pos0 = 0)
};

// THREADS per row: the CTA, or (rows of at most 1024 elements) one of its warps.
template <typename TI, typename TO, int PACKS, int THREADS>
__global__ void __launch_bounds__(kNormThreads) rms_norm_kernel(const RmsParams p) {
  __shared__ float scratch[kNormThreads / 32];
  griddep_wait();
  griddep_launch();
  const int tid = THREADS == 32 ? threadIdx.x & 31 : threadIdx.x;
  const long long row = THREADS == 32 ? (long long)blockIdx.x * (kNormThreads / 32) + (threadIdx.x >> 5) : blockIdx.x;
  if (row >= p.n1) return;                         // (a whole warp, and only where a warp is a row)
  const TI *x = reinterpret_cast<const TI *>(p.x) + row * p.ldx;
  const TO *w = reinterpret_cast<const TO *>(p.w);
  const int packs = p.n2 / 8;
  float v[PACKS][8];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = tid + i * THREADS;
    if (c >= packs) break;
    load8<TI>(x + c * 8, v[i]);
#pragma unroll
    for (int e = 0; e < 8; ++e) sq = fmaf(v[i][e], v[i][e], sq);
  }
  const float r = rsqrtf(block_sum<THREADS>(sq, scratch) * p.inv_count + p.eps);
  TO *ring = nullptr;
  if (p.ring) {
    const long long b = row / p.rows_per_batch;
    const int s = (int)(row - b * p.rows_per_batch);
    const int pos = (p.pos_dev ? *p.pos_dev : 0) + s;
    if (p.rows_per_batch - s <= p.ring_rows && pos >= 0)
      ring = reinterpret_cast<TO *>(p.ring) + b * p.ring_bs + (long long)(pos % p.ring_rows) * p.ring_ld;
  }
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = tid + i * THREADS;
    if (c >= packs) break;
    float wv[8];
    load8<TO>(w + c * 8, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) wv[e] = v[i][e] * r * (p.w_offset + wv[e]);
    if (p.y) store8<TO>(reinterpret_cast<TO *>(p.y) + row * p.ldy + c * 8, wv);
    if (ring) store8<TO>(ring + c * 8, wv);
  }
}

struct ResidualParams {
  const void *y;               // rows ldy apart (T)
  long long ldy;
  // combine: row t of the sublayer's output = sum_k weights[t*top+k] * y[rows ? rows[t*top+k] : t*top+k],
  // entries with idx < 0 left out
  const int *idx, *rows;
  const float *weights;
  int top;
  const void *w;               // [n2] T
  float w_offset, eps, inv_count;
  float *x;                    // fp32 residual stream, rows ldx apart, updated in place
  long long ldx;
  void *xt;                    // the new rows in T, rows ldt apart (null: not written)
  long long ldt;
  int n2;
  // router of the mixture that follows (null: none)
  const void *router;          // [experts][n2] T
  int experts, r_top;
  int *r_idx;
  float *r_weights;
};

// THREADS: 256, or 1024 with a router (few rows then, and the router's weights to read per row)
template <typename T, int PACKS, bool COMBINE, int THREADS>
__global__ void __launch_bounds__(THREADS) rms_residual_kernel(const ResidualParams p) {
  __shared__ float scratch[THREADS / 32];
  extern __shared__ float dyn[];                   // router: [n2] row, [experts] logits
  const long long row = blockIdx.x;
  const T *w = reinterpret_cast<const T *>(p.w);
  const int packs = p.n2 / 8;
  griddep_wait();
  griddep_launch();
  float v[PACKS][8];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    if (COMBINE) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] = 0.f;
      for (int k = 0; k < p.top; ++k) {
        const long long a = row * p.top + k;
        if (p.idx[a] < 0) continue;
        const long long src = p.rows ? p.rows[a] : a;
        const float s = p.weights[a];
        float f[8];
        load8<T>(reinterpret_cast<const T *>(p.y) + src * p.ldy + c * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = fmaf(s, f[e], v[i][e]);
      }
    } else {
      load8<T>(reinterpret_cast<const T *>(p.y) + row * p.ldy + c * 8, v[i]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) sq = fmaf(v[i][e], v[i][e], sq);
  }
  const float r = rsqrtf(block_sum<THREADS>(sq, scratch) * p.inv_count + p.eps);
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    float wv[8], xv[8];
    load8<T>(w + c * 8, wv);
    load8<float>(p.x + row * p.ldx + c * 8, xv);
#pragma unroll
    for (int e = 0; e < 8; ++e) xv[e] = fmaf(v[i][e] * r, p.w_offset + wv[e], xv[e]);
    store8<float>(p.x + row * p.ldx + c * 8, xv);
    if (p.xt) store8<T>(reinterpret_cast<T *>(p.xt) + row * p.ldt + c * 8, xv);
    if (p.router) {
      // the router reads the row as the products do: rounded to the operand type
#pragma unroll
      for (int e = 0; e < 8; ++e) dyn[c * 8 + e] = to_f32<T>(from_f32<T>(xv[e]));
    }
  }
  if (!p.router) return;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float *z = dyn + p.n2;
  for (int e = warp; e < p.experts; e += THREADS / 32) {
    const T *wr = reinterpret_cast<const T *>(p.router) + (long long)e * p.n2;
    float acc = 0.f;
#pragma unroll 4
    for (int c = lane; c < packs; c += 32) {
      float f[8];
      load8<T>(wr + c * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc = fmaf(f[j], dyn[c * 8 + j], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) z[e] = acc;
  }
  __syncthreads();
  if (warp == 0) route_warp(z, p.experts, p.r_top, p.r_idx + row * p.r_top, p.r_weights + row * p.r_top, nullptr, nullptr);
}

struct StreamParams {
  const void *src;             // T rows lds apart: x = src_scale * src instead of x as it is (null: x as it is)
  long long lds;
  float src_scale;
  const void *y, *gate;        // T rows; y null: nothing is added; gate null: no gate
  long long ldy, ldg;
  const float *w_out;          // [n2]
  float *x;                    // fp32 stream, rows ldx apart
  long long ldx;
  const void *w_next;          // [n2] T, or null: no h
  void *h;
  long long ldh;
  float eps, inv_count;
  int n2;
};

struct AddParams {
  const void *src, *src2;      // T rows: x = src + src2 instead of x as it is (null: x as it is; src2 may be null)
  long long lds, lds2;
  const void *y, *y2;          // T rows (y: expert rows with a mixture)
  long long ldy, ldy2;
  const float *w, *w2;         // [n2]: y and y2 are normalised and multiplied by these
  // mixture: sum_k weights[t*top+k] * (idx < experts ? y[rows ? rows[...] : t*top+k] : ident[t]) + gate[t] * shared[t]
  const int *idx, *rows;
  const float *weights, *gate;
  int top, experts;
  const void *ident, *shared;
  long long ldi, ldsh;
  float scale;
  float *x;
  long long ldx;
  const void *w_next;
  float next_scale;
  void *h;
  long long ldh;
  float eps, inv_count;
  int n2;
  // router on h (null: none): [choices (+ 1 with r_gate)][n2] T
  const void *router;
  int choices, r_top;
  RouterRule rule;
  int *r_idx;
  float *r_weights, *r_gate;
};

enum { kAddRow = 0, kAddTwo = 1, kAddMix = 2, kAddMixFew = 3 };      // kAddMixFew: few rows, several choices' rows in flight per thread

template <typename T, int PACKS, int FORM, int THREADS>
__global__ void __launch_bounds__(THREADS) stream_add_kernel(const AddParams p) {
  __shared__ float2 scratch[THREADS / 32];
  extern __shared__ float dyn[];                   // router: [n2] row, [choices + 1] logits, the rule's own
  const long long row = blockIdx.x;
  const int packs = p.n2 / 8;
  griddep_wait();
  griddep_launch();
  auto sum2 = [&](float2 s) {
    s.x = warp_sum(s.x);
    s.y = warp_sum(s.y);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = s;
    __syncthreads();
    s = (threadIdx.x & 31) < THREADS / 32 ? scratch[threadIdx.x & 31] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(s.x), warp_sum(s.y));
  };
  float xv[PACKS][8], v[PACKS][8], v2[FORM == kAddTwo ? PACKS : 1][8];
  float2 sq = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    if (p.src) {
      load8<T>(reinterpret_cast<const T *>(p.src) + row * p.lds + c * 8, xv[i]);
      if (p.src2) {
        float f[8];
        load8<T>(reinterpret_cast<const T *>(p.src2) + row * p.lds2 + c * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) xv[i][e] += f[e];
      }
    } else {
      load8<float>(p.x + row * p.ldx + c * 8, xv[i]);
    }
    if (FORM >= kAddMix) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] = 0.f;
      float self = 0.f;
      constexpr int kAhead = FORM == kAddMixFew ? 4 : 1;
      for (int k0 = 0; k0 < p.top; k0 += kAhead) {
        float s[kAhead], f[kAhead][8];
        long long src[kAhead];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
          const bool in = k0 + k < p.top;
          const long long a = row * p.top + (in ? k0 + k : 0);
          const int ex = p.idx[a];
          s[k] = p.weights[a];
          src[k] = p.rows ? p.rows[a] : a;
          if (in && ex >= p.experts) self += s[k];
          if (!in || ex < 0 || ex >= p.experts) src[k] = -1;
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k)
          if (src[k] >= 0) load8<T>(reinterpret_cast<const T *>(p.y) + src[k] * p.ldy + c * 8, f[k]);
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
          if (src[k] < 0) continue;
#pragma unroll
          for (int e = 0; e < 8; ++e) v[i][e] = fmaf(s[k], f[k][e], v[i][e]);
        }
      }
      if (self != 0.f) {
        float f[8];
        load8<T>(reinterpret_cast<const T *>(p.ident) + row * p.ldi + c * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = fmaf(self, f[e], v[i][e]);
      }
      if (p.shared) {
        const float s = p.gate[row];
        float f[8];
        load8<T>(reinterpret_cast<const T *>(p.shared) + row * p.ldsh + c * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = fmaf(s, f[e], v[i][e]);
      }
    } else if (p.y) {
      load8<T>(reinterpret_cast<const T *>(p.y) + row * p.ldy + c * 8, v[i]);
    }
    if (FORM == kAddTwo) {
      load8<T>(reinterpret_cast<const T *>(p.y2) + row * p.ldy2 + c * 8, v2[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        sq.x = fmaf(v[i][e], v[i][e], sq.x);
        sq.y = fmaf(v2[i][e], v2[i][e], sq.y);
      }
    }
  }
  if (FORM == kAddTwo) {
    sq = sum2(sq);
    const float r1 = rsqrtf(sq.x * p.inv_count + p.eps), r2 = rsqrtf(sq.y * p.inv_count + p.eps);
#pragma unroll
    for (int i = 0; i < PACKS; ++i) {
      const int c = threadIdx.x + i * THREADS;
      if (c >= packs) break;
      float a[8], b[8];
      load8<float>(p.w + c * 8, a);
      load8<float>(p.w2 + c * 8, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] = v[i][e] * r1 * a[e] + v2[i][e] * r2 * b[e];
    }
  }
  float sx = 0.f;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    if (FORM != kAddRow || p.y) {
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[i][e] = fmaf(p.scale, v[i][e], xv[i][e]);
    }
    if (p.src || p.y) store8<float>(p.x + row * p.ldx + c * 8, xv[i]);
#pragma unroll
    for (int e = 0; e < 8; ++e) sx = fmaf(xv[i][e], xv[i][e], sx);
  }
  if (!p.w_next) return;
  const float r = rsqrtf(sum2(make_float2(sx, 0.f)).x * p.inv_count + p.eps) * p.next_scale;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    float wv[8];
    load8<T>(reinterpret_cast<const T *>(p.w_next) + c * 8, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) wv[e] *= xv[i][e] * r;
    store8<T>(reinterpret_cast<T *>(p.h) + row * p.ldh + c * 8, wv);
    if (p.router) {
      // the router reads the row as the products do: rounded to the operand type
#pragma unroll
      for (int e = 0; e < 8; ++e) dyn[c * 8 + e] = to_f32<T>(from_f32<T>(wv[e]));
    }
  }
  if (!p.router) return;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float *z = dyn + p.n2;                           // the rule's numbers lie behind the choices' logits; the gate's is not among them
  for (int e = warp; e < p.choices + (p.r_gate ? 1 : 0); e += THREADS / 32) {
    const T *wr = reinterpret_cast<const T *>(p.router) + (long long)e * p.n2;
    float acc = 0.f;
#pragma unroll 4
    for (int c = lane; c < packs; c += 32) {
      float f[8];
      load8<T>(wr + c * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc = fmaf(f[j], dyn[c * 8 + j], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) {
      if (e < p.choices) z[e] = acc;
      else p.r_gate[row] = 1.f / (1.f + expf(-acc));
    }
  }
  __syncthreads();
  if (warp == 0) route_warp_rule<true>(z, p.choices, p.r_top, p.rule, p.r_idx + row * p.r_top, p.r_weights + row * p.r_top, nullptr, nullptr);
}

template <typename T, int FORM> int launch_add(const AddParams &p, int n1, cudaStream_t st) {
  const int packs = p.n2 / 8, threads = p.router ? 1024 : kNormThreads, per = (packs + threads - 1) / threads;
  const size_t smem = p.router ? (size_t)(p.n2 + rule_floats(p.choices, p.rule)) * sizeof(float) : 0;
  const dim3 g(n1), b(threads);
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "stream_add: cannot reserve %zu bytes of shared memory", smem);
    }
    launch_pdl(kern, g, b, smem, st, p);
    return check_launch("stream_add");
  };
  if (p.router) return per <= 1 ? go(stream_add_kernel<T, 1, FORM, 1024>) : go(stream_add_kernel<T, 2, FORM, 1024>);
  if (per <= 1) return go(stream_add_kernel<T, 1, FORM, kNormThreads>);
  if (per <= 2) return go(stream_add_kernel<T, 2, FORM, kNormThreads>);
  if (per <= 4) return go(stream_add_kernel<T, 4, FORM, kNormThreads>);
  return go(stream_add_kernel<T, 8, FORM, kNormThreads>);
}

template <typename T, int PACKS>
__global__ void __launch_bounds__(kNormThreads) stream_update_kernel(const StreamParams p) {
  constexpr int THREADS = kNormThreads;
  __shared__ float scratch[THREADS / 32];
  const long long row = blockIdx.x;
  const int packs = p.n2 / 8;
  griddep_wait();
  griddep_launch();
  float v[PACKS][8];
  float r = 0.f;
  if (p.y) {
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < PACKS; ++i) {
      const int c = threadIdx.x + i * THREADS;
      if (c >= packs) break;
      load8<T>(reinterpret_cast<const T *>(p.y) + row * p.ldy + c * 8, v[i]);
      if (p.gate) {
        float g[8];
        load8<T>(reinterpret_cast<const T *>(p.gate) + row * p.ldg + c * 8, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = v[i][e] / (1.f + __expf(-g[e]));
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) sq = fmaf(v[i][e], v[i][e], sq);
    }
    r = rsqrtf(block_sum<THREADS>(sq, scratch) * p.inv_count + p.eps);
  }
  float sx = 0.f;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    float xv[8];
    if (p.src) {
      load8<T>(reinterpret_cast<const T *>(p.src) + row * p.lds + c * 8, xv);
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[e] *= p.src_scale;
    } else {
      load8<float>(p.x + row * p.ldx + c * 8, xv);
    }
    if (p.y) {
      float wv[8];
      load8<float>(p.w_out + c * 8, wv);
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[e] = fmaf(v[i][e] * r, wv[e], xv[e]);
    }
    store8<float>(p.x + row * p.ldx + c * 8, xv);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      sx = fmaf(xv[e], xv[e], sx);
      v[i][e] = xv[e];
    }
  }
  if (!p.w_next) return;
  r = rsqrtf(block_sum<THREADS>(sx, scratch) * p.inv_count + p.eps);
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= packs) break;
    float wv[8];
    load8<T>(reinterpret_cast<const T *>(p.w_next) + c * 8, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) wv[e] *= v[i][e] * r;
    store8<T>(reinterpret_cast<T *>(p.h) + row * p.ldh + c * 8, wv);
  }
}

template <typename T> int launch_stream(const StreamParams &p, int n1, cudaStream_t st) {
  const int packs = p.n2 / 8, per = (packs + kNormThreads - 1) / kNormThreads;
  const dim3 g(n1), b(kNormThreads);
  if (per <= 1) launch_pdl(stream_update_kernel<T, 1>, g, b, 0, st, p);
  else if (per <= 2) launch_pdl(stream_update_kernel<T, 2>, g, b, 0, st, p);
  else if (per <= 4) launch_pdl(stream_update_kernel<T, 4>, g, b, 0, st, p);
  else launch_pdl(stream_update_kernel<T, 8>, g, b, 0, st, p);
  return check_launch("stream_update");
}

template <typename TI, typename TO>
int launch_rms(const RmsParams &p, int n1, cudaStream_t st) {
  const int packs = p.n2 / 8, per = (packs + kNormThreads - 1) / kNormThreads;
  const dim3 g(n1), b(kNormThreads);
  const dim3 gw((n1 + kNormThreads / 32 - 1) / (kNormThreads / 32));
  if (packs <= 32) launch_pdl(rms_norm_kernel<TI, TO, 1, 32>, gw, b, 0, st, p);
  else if (packs <= 64) launch_pdl(rms_norm_kernel<TI, TO, 2, 32>, gw, b, 0, st, p);
  else if (packs <= 128) launch_pdl(rms_norm_kernel<TI, TO, 4, 32>, gw, b, 0, st, p);
  else if (per <= 1) launch_pdl(rms_norm_kernel<TI, TO, 1, kNormThreads>, g, b, 0, st, p);
  else if (per <= 2) launch_pdl(rms_norm_kernel<TI, TO, 2, kNormThreads>, g, b, 0, st, p);
  else if (per <= 4) launch_pdl(rms_norm_kernel<TI, TO, 4, kNormThreads>, g, b, 0, st, p);
  else launch_pdl(rms_norm_kernel<TI, TO, 8, kNormThreads>, g, b, 0, st, p);
  return check_launch("rms_norm");
}

template <typename T, bool COMBINE>
int launch_residual(const ResidualParams &p, int n1, cudaStream_t st) {
  const int packs = p.n2 / 8, threads = p.router ? 1024 : kNormThreads, per = (packs + threads - 1) / threads;
  const size_t smem = p.router ? (size_t)(p.n2 + p.experts) * sizeof(float) : 0;
  const dim3 g(n1), b(threads);
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      return fail(EB_ECUDA, "rms_residual: cannot reserve %zu bytes of shared memory", smem);
    }
    launch_pdl(kern, g, b, smem, st, p);
    return check_launch("rms_residual");
  };
  if (p.router) return per <= 1 ? go(rms_residual_kernel<T, 1, COMBINE, 1024>) : go(rms_residual_kernel<T, 2, COMBINE, 1024>);
  if (per <= 1) return go(rms_residual_kernel<T, 1, COMBINE, kNormThreads>);
  if (per <= 2) return go(rms_residual_kernel<T, 2, COMBINE, kNormThreads>);
  if (per <= 4) return go(rms_residual_kernel<T, 4, COMBINE, kNormThreads>);
  return go(rms_residual_kernel<T, 8, COMBINE, kNormThreads>);
}

constexpr int kMaxNormWidth = 8 * 8 * kNormThreads;

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_rms_norm(const void *x, long long ldx, int in_dtype, const void *w, float w_offset, float eps, void *y, long long ldy,
                           int out_dtype, int n1, int n2, int count, void *ring, long long ring_batch_stride, long long ring_ld,
                           int ring_rows, int rows_per_batch, const int32_t *pos_device, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(in_dtype) && dtype_ok(out_dtype), "rms_norm: bad dtype %d / %d", in_dtype, out_dtype);
  EB_REQUIRE(in_dtype == EB_F32 || in_dtype == out_dtype, "rms_norm: the input is fp32 or of the output type");
  EB_REQUIRE(x && w && (y || ring), "rms_norm: null pointer");
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && n2 <= kMaxNormWidth, "rms_norm: width %d must be a multiple of 8, at most %d", n2, kMaxNormWidth);
  EB_REQUIRE(count > 0 && count <= n2, "rms_norm: the mean is over 1..n2 elements");
  EB_REQUIRE(ldx >= n2 && ldx % 8 == 0 && (!y || (ldy >= n2 && ldy % 8 == 0)), "rms_norm: row strides must be multiples of 8 and >= n2");
  EB_REQUIRE(aligned16(x) && aligned16(w) && aligned16(y) && aligned16(ring), "rms_norm: pointers must be 16-byte aligned");
  if (ring) {
    EB_REQUIRE(ring_rows > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0, "rms_norm: the ring needs its rows and rows_per_batch");
    EB_REQUIRE(ring_ld >= n2 && ring_ld % 8 == 0 && ring_batch_stride % 8 == 0, "rms_norm: ring strides must be multiples of 8");
  }
  RmsParams p{};
  p.x = x; p.ldx = ldx; p.w = w; p.w_offset = w_offset; p.eps = eps; p.inv_count = 1.f / (float)count;
  p.y = y; p.ldy = ldy; p.n1 = n1; p.n2 = n2;
  p.ring = ring; p.ring_bs = ring_batch_stride; p.ring_ld = ring_ld; p.ring_rows = ring_rows; p.rows_per_batch = rows_per_batch;
  p.pos_dev = pos_device;
  cudaStream_t st = as_stream(stream);
  if (in_dtype == EB_F32) {
    if (out_dtype == EB_F32) return launch_rms<float, float>(p, n1, st);
    if (out_dtype == EB_F16) return launch_rms<float, __half>(p, n1, st);
    return launch_rms<float, __nv_bfloat16>(p, n1, st);
  }
  if (out_dtype == EB_F16) return launch_rms<__half, __half>(p, n1, st);
  return launch_rms<__nv_bfloat16, __nv_bfloat16>(p, n1, st);
}

extern "C" int eb_rms_residual(const void *y, long long ldy, int dtype, const int32_t *idx, const int32_t *rows, const float *weights,
                               int top, const void *w, float w_offset, float eps, float *x, long long ldx, void *xt, long long ldt,
                               int n1, int n2, int count, const void *router, int experts, int router_top, int32_t *router_idx,
                               float *router_weights, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "rms_residual: bad dtype %d", dtype);
  EB_REQUIRE(y && w && x, "rms_residual: null pointer");
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && n2 <= kMaxNormWidth, "rms_residual: width %d must be a multiple of 8, at most %d", n2, kMaxNormWidth);
  EB_REQUIRE(count > 0 && count <= n2, "rms_residual: the mean is over 1..n2 elements");
  EB_REQUIRE(ldy >= n2 && ldy % 8 == 0 && ldx >= n2 && ldx % 8 == 0 && (!xt || (ldt >= n2 && ldt % 8 == 0)),
             "rms_residual: row strides must be multiples of 8 and >= n2");
  EB_REQUIRE(aligned16(y) && aligned16(w) && aligned16(x) && aligned16(xt) && aligned16(router), "rms_residual: pointers must be 16-byte aligned");
  EB_REQUIRE(!idx || (weights && top > 0), "rms_residual: a combination needs weights and top");
  if (router) {
    EB_REQUIRE(router_idx && router_weights, "rms_residual: the router needs its outputs");
    EB_REQUIRE(experts > 0 && experts <= kMaxExperts && router_top > 0 && router_top <= experts,
               "rms_residual: bad router (%d experts, top %d)", experts, router_top);
  }
  ResidualParams p{};
  p.y = y; p.ldy = ldy; p.idx = idx; p.rows = rows; p.weights = weights; p.top = top;
  p.w = w; p.w_offset = w_offset; p.eps = eps; p.inv_count = 1.f / (float)count;
  p.x = x; p.ldx = ldx; p.xt = xt; p.ldt = ldt; p.n2 = n2;
  p.router = router; p.experts = experts; p.r_top = router_top; p.r_idx = router_idx; p.r_weights = router_weights;
  cudaStream_t st = as_stream(stream);
#define EB_RES(T) (idx ? launch_residual<T, true>(p, n1, st) : launch_residual<T, false>(p, n1, st))
  if (dtype == EB_F32) return EB_RES(float);
  if (dtype == EB_F16) return EB_RES(__half);
  return EB_RES(__nv_bfloat16);
#undef EB_RES
}

extern "C" int eb_stream_update(const void *src, long long lds, float src_scale, const void *y, long long ldy, const void *gate, long long ldg,
                                const float *w_out, float *x, long long ldx, const void *w_next, void *h, long long ldh, float eps, int n1, int n2, int count, int dtype, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "stream_update: bad dtype %d", dtype);
  EB_REQUIRE(x && (src || y || w_next), "stream_update: null pointer");
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && n2 <= kMaxNormWidth, "stream_update: width %d must be a multiple of 8, at most %d", n2, kMaxNormWidth);
  EB_REQUIRE(count > 0 && count <= n2, "stream_update: the mean is over 1..n2 elements");
  EB_REQUIRE(ldx >= n2 && ldx % 8 == 0 && (!src || (lds >= n2 && lds % 8 == 0)) && (!y || (ldy >= n2 && ldy % 8 == 0)) &&
                 (!gate || (ldg >= n2 && ldg % 8 == 0)) && (!w_next || (ldh >= n2 && ldh % 8 == 0)),
             "stream_update: row strides must be multiples of 8 and >= n2");
  EB_REQUIRE(!y || w_out, "stream_update: the added row needs its weight");
  EB_REQUIRE(!gate || y, "stream_update: a gate without a row");
  EB_REQUIRE(!w_next || h, "stream_update: no place for the normalised row");
  EB_REQUIRE(aligned16(src) && aligned16(y) && aligned16(gate) && aligned16(w_out) && aligned16(x) && aligned16(w_next) && aligned16(h),
             "stream_update: pointers must be 16-byte aligned");
  StreamParams p{};
  p.src = src; p.lds = lds; p.src_scale = src_scale; p.y = y; p.ldy = ldy; p.gate = gate; p.ldg = ldg; p.w_out = w_out;
  p.x = x; p.ldx = ldx; p.w_next = w_next; p.h = h; p.ldh = ldh;
  p.eps = eps; p.inv_count = 1.f / (float)count; p.n2 = n2;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_stream<float>(p, n1, st);
  if (dtype == EB_F16) return launch_stream<__half>(p, n1, st);
  return launch_stream<__nv_bfloat16>(p, n1, st);
}

extern "C" int eb_stream_add(const void *src, long long lds, const void *src2, long long lds2, const void *y, long long ldy, const float *w,
                             const void *y2, long long ldy2, const float *w2, const int32_t *idx, const int32_t *rows, const float *weights, int top,
                             int experts, const void *ident, long long ldi, const void *shared, long long ldsh, const float *gate, float scale,
                             float *x, long long ldx, const void *w_next, float next_scale, void *h, long long ldh, float eps, int n1, int n2,
                             int count, const void *router, int choices, int r_experts, int r_top, const float *r_correction, int r_groups,
                             int r_keep, int32_t *r_idx, float *r_weights, float *r_gate, int dtype, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "stream_add: bad dtype %d", dtype);
  EB_REQUIRE(x && (src || y || w_next), "stream_add: null pointer");
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && n2 <= kMaxNormWidth, "stream_add: width %d must be a multiple of 8, at most %d", n2, kMaxNormWidth);
  EB_REQUIRE(count > 0 && count <= n2, "stream_add: the mean is over 1..n2 elements");
  const void *rows_p[] = {src, src2, y, y2, ident, shared, h};
  const long long rows_ld[] = {lds, lds2, ldy, ldy2, ldi, ldsh, ldh};
  for (int i = 0; i < 7; ++i)
    EB_REQUIRE(!rows_p[i] || (rows_ld[i] >= n2 && rows_ld[i] % 8 == 0 && aligned16(rows_p[i])), "stream_add: row strides must be multiples of 8 and >= n2, rows 16-byte aligned");
  EB_REQUIRE(ldx >= n2 && ldx % 8 == 0 && aligned16(x) && aligned16(w) && aligned16(w2) && aligned16(w_next) && aligned16(router),
             "stream_add: row strides must be multiples of 8 and >= n2, pointers 16-byte aligned");
  EB_REQUIRE(!src2 || src, "stream_add: a second start row without a first");
  EB_REQUIRE(!y2 || (y && w && w2 && !idx), "stream_add: two rows need their weights");
  EB_REQUIRE(y2 || !w, "stream_add: a weight without a second row");
  EB_REQUIRE(!idx || (y && weights && ident && top > 0 && experts >= 0), "stream_add: a mixture needs expert rows, weights, top and the input rows");
  EB_REQUIRE(!shared || (idx && gate), "stream_add: a shared expert goes with a mixture and its gate");
  EB_REQUIRE(!w_next || h, "stream_add: no place for the normalised row");
  AddParams p{};
  if (router) {
    EB_REQUIRE(w_next && r_idx && r_weights, "stream_add: the router reads h and needs its outputs");
    if (int rc = make_rule("stream_add", choices, r_experts, r_top, r_correction, r_groups, r_keep, &p.rule)) return rc;
  }
  p.src = src; p.lds = lds; p.src2 = src2; p.lds2 = lds2; p.y = y; p.ldy = ldy; p.y2 = y2; p.ldy2 = ldy2; p.w = w; p.w2 = w2;
  p.idx = idx; p.rows = rows; p.weights = weights; p.gate = gate; p.top = top; p.experts = experts; p.ident = ident; p.ldi = ldi;
  p.shared = shared; p.ldsh = ldsh; p.scale = scale; p.x = x; p.ldx = ldx; p.w_next = w_next; p.next_scale = next_scale; p.h = h; p.ldh = ldh;
  p.eps = eps; p.inv_count = 1.f / (float)count; p.n2 = n2;
  p.router = router; p.choices = choices; p.r_top = r_top; p.r_idx = r_idx; p.r_weights = r_weights; p.r_gate = r_gate;
  cudaStream_t st = as_stream(stream);
#define EB_ADD(T) (idx ? (n1 < 4 * sm_count() ? launch_add<T, kAddMixFew>(p, n1, st) : launch_add<T, kAddMix>(p, n1, st)) : y2 ? launch_add<T, kAddTwo>(p, n1, st) : launch_add<T, kAddRow>(p, n1, st))
  if (dtype == EB_F32) return EB_ADD(float);
  if (dtype == EB_F16) return EB_ADD(__half);
  return EB_ADD(__nv_bfloat16);
#undef EB_ADD
}
