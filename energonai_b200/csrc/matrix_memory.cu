// Matrix memory: a recurrent layer whose state per head is a matrix S [dk][dv], a normaliser n [dk] and
// a running maximum m of the log gates (all fp32, see eb_memory_scan in the header for the equations).
//
//   memory_scan     a whole prompt, token by token: the path of 32-bit models and of head sizes that the
//                   chunked tensor-core kernel (matrix_memory_tc.cu) does not have.  A CTA owns 32
//                   columns of S of one (sequence, head); S stays in shared memory.
//   memory_step     one token per sequence, a pass over the state (HBM-bound: S is read and written
//                   once).  The columns of a head are split over a cluster of 1 to 8 CTAs, which also
//                   forms the head's norm through distributed shared memory, so that the output
//                   gate and the projection's operand come out of the same launch.
//   head_norm_gate  that tail alone, for the rows of a prompt.
#include "common.cuh"
#include "memory_gates.cuh"
#include "state_pass.cuh"

namespace eb {
namespace {

template <typename T> __device__ __forceinline__ T store_cast(float v) { return from_f32<T>(v); }
template <> __device__ __forceinline__ __half store_cast<__half>(float v) { return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }

// ---- prompt, token by token ------------------------------------------------------------------------
constexpr int kScanCols = 32, kScanThreads = 256, kScanWarps = kScanThreads / 32;

struct ScanParams {
  const void *q, *k, *v;
  long long ldp;
  const float *gates;
  long long ldg;
  const float *bias_i, *bias_f;
  float cap, scale;
  const int *first;
  void *o;
  long long ldo;
  float *S, *n, *m;
  int seq, heads, dk, dv;
};

template <typename T>
__global__ void __launch_bounds__(kScanThreads) memory_scan_kernel(const ScanParams p) {
  extern __shared__ float sm[];
  float *S = sm, *n = S + p.dk * kScanCols, *qs = n + p.dk, *ks = qs + p.dk;
  __shared__ float red[kScanWarps][kScanCols + 1], nred[kScanWarps];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, b = blockIdx.z;
  const int col = blockIdx.x * kScanCols + lane;
  const bool has = col < p.dv;
  for (int i = threadIdx.x; i < p.dk * kScanCols; i += kScanThreads) S[i] = 0.f;
  for (int i = threadIdx.x; i < p.dk; i += kScanThreads) n[i] = 0.f;
  const float bi = p.bias_i[h], bf = p.bias_f[h];
  float m = 0.f;
  const int t0 = p.first ? p.first[b] : 0;
  const long long row0 = (long long)b * p.seq;
  T *o = reinterpret_cast<T *>(p.o) + h * p.dv + col;
  if (warp == 0 && has)
    for (int t = 0; t < min(t0, p.seq); ++t) o[(row0 + t) * p.ldo] = from_f32<T>(0.f);
  for (int t = t0; t < p.seq; ++t) {
    const long long row = row0 + t;
    const T *q = reinterpret_cast<const T *>(p.q) + row * p.ldp + h * p.dk, *k = reinterpret_cast<const T *>(p.k) + row * p.ldp + h * p.dk;
    const float v = has ? to_f32<T>(reinterpret_cast<const T *>(p.v)[row * p.ldp + h * p.dv + col]) : 0.f;
    const float li = log_input_gate(p.gates[row * p.ldg + h], bi, p.cap), lf = log_forget_gate(p.gates[row * p.ldg + p.heads + h], bf, p.cap);
    const float mn = fmaxf(lf + m, li), a = expf(lf + m - mn), w = expf(li - mn);
    m = mn;
    for (int d = threadIdx.x; d < p.dk; d += kScanThreads) {
      qs[d] = to_f32<T>(q[d]) * p.scale;
      ks[d] = to_f32<T>(k[d]);
    }
    __syncthreads();
    float acc = 0.f, nq = 0.f;
    for (int d = warp; d < p.dk; d += kScanWarps) {
      const float s = fmaf(a, S[d * kScanCols + lane], w * ks[d] * v);
      S[d * kScanCols + lane] = s;
      acc = fmaf(s, qs[d], acc);
    }
    for (int d = threadIdx.x; d < p.dk; d += kScanThreads) {
      const float x = fmaf(a, n[d], w * ks[d]);
      n[d] = x;
      nq = fmaf(x, qs[d], nq);
    }
    red[warp][lane] = acc;
    nq = warp_sum(nq);
    if (lane == 0) nred[warp] = nq;
    __syncthreads();
    if (warp == 0) {
      float num = 0.f, den = 0.f;
#pragma unroll
      for (int i = 0; i < kScanWarps; ++i) { num += red[i][lane]; den += nred[i]; }
      if (has) o[row * p.ldo] = store_cast<T>(num / (fmaxf(fabsf(den), expf(-m)) + kMemoryDenomEps));
    }
    __syncthreads();
  }
  const long long bh = (long long)b * p.heads + h;
  if (has)
    for (int d = warp; d < p.dk; d += kScanWarps) p.S[(bh * p.dk + d) * p.dv + col] = S[d * kScanCols + lane];
  if (blockIdx.x == 0) {
    for (int d = threadIdx.x; d < p.dk; d += kScanThreads) p.n[bh * p.dk + d] = n[d];
    if (threadIdx.x == 0) p.m[bh] = m;
  }
}

template <typename T> int launch_scan(const ScanParams &p, int B, cudaStream_t st) {
  const size_t smem = (size_t)p.dk * (kScanCols + 3) * sizeof(float);
  auto kern = memory_scan_kernel<T>;
  if (smem > 200 * 1024) return fail(EB_EUNSUPPORTED, "memory_scan: head size %d is too large", p.dk);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return fail(EB_ECUDA, "memory_scan: cannot reserve %zu bytes of shared memory", smem);
  }
  launch_pdl(kern, dim3((p.dv + kScanCols - 1) / kScanCols, p.heads, B), dim3(kScanThreads), smem, st, p);
  return check_launch("memory_scan");
}

// ---- one token per sequence ------------------------------------------------------------------------
struct StepParams {
  const void *q, *k, *v, *g;
  long long ldp;
  const float *gates;
  long long ldg;
  const float *bias_i, *bias_f;
  float cap, scale;
  const void *norm;
  float inv_count, eps;
  void *out;
  long long ldo;
  float *S, *n, *m;
  int heads, dk, dv, cols;     // cols: columns per CTA, a multiple of 4
};

template <typename T>
__global__ void __launch_bounds__(kStepThreads, 4) memory_step_kernel(const StepParams p) {
  extern __shared__ float sm[];
  float *qs = sm, *ks = qs + p.dk, *ns = ks + p.dk, *vs = ns + p.dk, *red = vs + p.cols;      // red: [row groups][cols]
  __shared__ float scratch[kStepThreads / 32];
  __shared__ __align__(8) ClusterSum head_sum;
  const int peers = gridDim.x;
  cluster_sum_begin(head_sum, peers);
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int c0 = blockIdx.x * p.cols, width = min(p.cols, p.dv - c0);           // (width may be <= 0 for a CTA behind the last column)
  const long long bh = (long long)b * p.heads + h;
  const T *q = reinterpret_cast<const T *>(p.q) + b * p.ldp + h * p.dk, *k = reinterpret_cast<const T *>(p.k) + b * p.ldp + h * p.dk,
          *v = reinterpret_cast<const T *>(p.v) + b * p.ldp + h * p.dv + c0, *g = reinterpret_cast<const T *>(p.g) + b * p.ldp + h * p.dv + c0;
  StatePass pass(p.S + bh * p.dk * p.dv + c0, p.dk, p.dv, p.cols, width);
  pass.begin();
  const float m0 = p.m[bh];
  const float li = log_input_gate(p.gates[b * p.ldg + h], p.bias_i[h], p.cap), lf = log_forget_gate(p.gates[b * p.ldg + p.heads + h], p.bias_f[h], p.cap);
  const float m1 = fmaxf(lf + m0, li), a = expf(lf + m0 - m1), w = expf(li - m1);
  float nq = 0.f;
  for (int d = tid; d < p.dk; d += kStepThreads) {
    const float qv = to_f32<T>(q[d]) * p.scale, kv = w * to_f32<T>(k[d]), nv = fmaf(a, p.n[bh * p.dk + d], kv);
    qs[d] = qv;
    ks[d] = kv;
    ns[d] = nv;
    nq = fmaf(nv, qv, nq);
  }
  for (int c = tid; c < width; c += kStepThreads) vs[c] = to_f32<T>(v[c]);
  nq = block_sum<kStepThreads>(nq, scratch);                                   // (also makes qs, ks, vs visible)
  const float den = fmaxf(fabsf(nq), expf(-m1)) + kMemoryDenomEps;

  pass.run([a](int) { return a; }, ks, qs, vs, red);
  __syncthreads();
  float sq = 0.f;
  for (int c = tid; c < width; c += kStepThreads) {
    float x = 0.f;
    for (int r = 0; r < pass.R; ++r) x += red[r * p.cols + c];
    x /= den;
    red[c] = x;                                     // (row group 0: only this thread has read column c of it)
    sq = fmaf(x, x, sq);
  }
  sq = block_sum<kStepThreads>(sq, scratch);
  sq = cluster_sum(head_sum, peers, sq);
  const float rs = rsqrtf(sq * p.inv_count + p.eps);
  T *out = reinterpret_cast<T *>(p.out) + b * p.ldo + h * p.dv + c0;
  const T *norm = reinterpret_cast<const T *>(p.norm) + h * p.dv + c0;
  for (int c = tid; c < width; c += kStepThreads) out[c] = from_f32<T>(red[c] * rs * to_f32<T>(norm[c]) * sigmoid(to_f32<T>(g[c])));
  // every CTA of the head has read n and m: its sum, which depends on them, is here
  if (blockIdx.x == 0) {
    for (int d = tid; d < p.dk; d += kStepThreads) p.n[bh * p.dk + d] = ns[d];
    if (tid == 0) p.m[bh] = m1;
  }
}

template <typename T> int launch_step(StepParams p, int B, cudaStream_t st) {
  const int split = state_split((long long)B * p.heads, p.dv);
  p.cols = ((p.dv + split - 1) / split + 3) / 4 * 4;
  if (p.cols > 4 * kStepThreads) return fail(EB_EUNSUPPORTED, "memory_step: value head size %d is too large", p.dv);
  const int R = kStepThreads / (p.cols / 4);
  const size_t smem = (size_t)(3 * p.dk + p.cols + R * p.cols) * sizeof(float);
  if (smem > 48 * 1024) return fail(EB_EUNSUPPORTED, "memory_step: head sizes %d / %d are too large", p.dk, p.dv);
  return launch_state_step("memory_step", memory_step_kernel<T>, p, dim3(split, p.heads, B), split, smem, st);
}

// ---- the tail of a prompt's rows ---------------------------------------------------------------------
struct HeadNormParams {
  const void *o, *g, *norm;
  long long ldo, ldg, ld_out;
  void *out;
  float inv_count, eps;
  int rows, heads, dv, silu;   // silu: the gate is g * sigmoid(g)
};

// A warp per (row, head), heads in packs of 8 elements.
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const HeadNormParams p) {
  griddep_wait();
  griddep_launch();
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (unit >= (long long)p.rows * p.heads) return;
  const long long row = unit / p.heads;
  const int h = (int)(unit - row * p.heads);
  constexpr int N = Vec16<T>::N, kKeep = 4;         // the first kKeep vectors per lane stay in registers
  const T *o = reinterpret_cast<const T *>(p.o) + row * p.ldo + h * p.dv, *g = reinterpret_cast<const T *>(p.g) + row * p.ldg + h * p.dv,
          *norm = reinterpret_cast<const T *>(p.norm) + h * p.dv;
  T *out = reinterpret_cast<T *>(p.out) + row * p.ld_out + h * p.dv;
  const int vecs = p.dv / N;
  Vec16<T> keep[kKeep];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = lane + 32 * i;
    if (c >= vecs) break;
    float f[N];
    keep[i].load(o + c * N);
    keep[i].unpack(f);
#pragma unroll
    for (int e = 0; e < N; ++e) sq = fmaf(f[e], f[e], sq);
  }
  for (int c = lane + 32 * kKeep; c < vecs; c += 32) {
    Vec16<T> a;
    float f[N];
    a.load(o + c * N);
    a.unpack(f);
#pragma unroll
    for (int e = 0; e < N; ++e) sq = fmaf(f[e], f[e], sq);
  }
  const float rs = rsqrtf(warp_sum(sq) * p.inv_count + p.eps);
  auto tail = [&](const Vec16<T> &a, int c) {
    Vec16<T> gv, wv, y;
    float f[N], gf[N], wf[N];
    a.unpack(f);
    gv.load(g + c * N);
    gv.unpack(gf);
    wv.load(norm + c * N);
    wv.unpack(wf);
#pragma unroll
    for (int e = 0; e < N; ++e) f[e] = f[e] * rs * wf[e] * __fdividef(p.silu ? gf[e] : 1.f, 1.f + __expf(-gf[e]));
    y.pack(f);
    y.store(out + c * N);
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = lane + 32 * i;
    if (c >= vecs) break;
    tail(keep[i], c);
  }
  for (int c = lane + 32 * kKeep; c < vecs; c += 32) {
    Vec16<T> a;
    a.load(o + c * N);
    tail(a, c);
  }
}

int check_memory(const char *name, const void *q, const void *k, const void *v, const float *gates, const float *bi, const float *bf, const float *S,
                 const float *n, const float *m, long long ldp, long long ldg, int batch, int heads, int dk, int dv, float cap, int dtype) {
  if (!dtype_ok(dtype)) return fail(EB_EINVAL, "%s: bad dtype %d", name, dtype);
  if (!q || !k || !v || !gates || !bi || !bf || !S || !n || !m) return fail(EB_EINVAL, "%s: null pointer", name);
  if (batch < 0 || batch > 65535 || heads <= 0 || heads > 65535 || dk <= 0 || dv <= 0) return fail(EB_EINVAL, "%s: bad sizes", name);
  if (dv % 8 != 0 || dk % 8 != 0) return fail(EB_EINVAL, "%s: head sizes must be multiples of 8 (%d, %d)", name, dk, dv);
  if (ldp % 8 != 0 || ldg < 2 * heads) return fail(EB_EINVAL, "%s: row strides must be multiples of 8 and hold a row", name);
  if (!(cap > 0.f)) return fail(EB_EINVAL, "%s: the gates' cap must be positive", name);
  if (!aligned16(S) || !aligned16(q) || !aligned16(k) || !aligned16(v)) return fail(EB_EINVAL, "%s: pointers must be 16-byte aligned", name);
  return EB_OK;
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_memory_scan(const void *q, const void *k, const void *v, long long ldp, const float *gates, long long ldg, const float *bias_i,
                              const float *bias_f, float cap, float scale, const int32_t *first, void *o, long long ldo, float *S, float *n,
                              float *m, int batch, int seq, int heads, int dk, int dv, int dtype, void *stream) {
  if (batch == 0 || seq == 0) return EB_OK;
  if (int rc = check_memory("memory_scan", q, k, v, gates, bias_i, bias_f, S, n, m, ldp, ldg, batch, heads, dk, dv, cap, dtype)) return rc;
  EB_REQUIRE(seq > 0 && o && ldo >= (long long)heads * dv, "memory_scan: bad output");
  ScanParams p{};
  p.q = q; p.k = k; p.v = v; p.ldp = ldp; p.gates = gates; p.ldg = ldg; p.bias_i = bias_i; p.bias_f = bias_f; p.cap = cap; p.scale = scale;
  p.first = first; p.o = o; p.ldo = ldo; p.S = S; p.n = n; p.m = m; p.seq = seq; p.heads = heads; p.dk = dk; p.dv = dv;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_scan<float>(p, batch, st);
  if (dtype == EB_F16) return launch_scan<__half>(p, batch, st);
  return launch_scan<__nv_bfloat16>(p, batch, st);
}

extern "C" int eb_memory_step(const void *q, const void *k, const void *v, const void *g, long long ldp, const float *gates, long long ldg,
                              const float *bias_i, const float *bias_f, float cap, float scale, const void *norm, int dv_count, float eps,
                              void *out, long long ldo, float *S, float *n, float *m, int batch, int heads, int dk, int dv, int dtype,
                              void *stream) {
  if (batch == 0) return EB_OK;
  if (int rc = check_memory("memory_step", q, k, v, gates, bias_i, bias_f, S, n, m, ldp, ldg, batch, heads, dk, dv, cap, dtype)) return rc;
  EB_REQUIRE(g && norm && out && ldo >= (long long)heads * dv, "memory_step: bad output");
  EB_REQUIRE(dv_count > 0 && dv_count <= dv, "memory_step: the mean is over 1..dv elements");
  StepParams p{};
  p.q = q; p.k = k; p.v = v; p.g = g; p.ldp = ldp; p.gates = gates; p.ldg = ldg; p.bias_i = bias_i; p.bias_f = bias_f; p.cap = cap; p.scale = scale;
  p.norm = norm; p.inv_count = 1.f / (float)dv_count; p.eps = eps; p.out = out; p.ldo = ldo; p.S = S; p.n = n; p.m = m;
  p.heads = heads; p.dk = dk; p.dv = dv;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_step<float>(p, batch, st);
  if (dtype == EB_F16) return launch_step<__half>(p, batch, st);
  return launch_step<__nv_bfloat16>(p, batch, st);
}

extern "C" int eb_head_norm_gate_act(const void *o, long long ldo, const void *g, long long ldg, const void *norm, float eps, void *out,
                                     long long ld_out, int rows, int heads, int dv, int dv_count, int silu, int dtype, void *stream) {
  if (rows == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "head_norm_gate: bad dtype %d", dtype);
  EB_REQUIRE(o && g && norm && out, "head_norm_gate: null pointer");
  EB_REQUIRE(rows > 0 && heads > 0 && dv > 0 && dv % 8 == 0 && dv_count > 0 && dv_count <= dv, "head_norm_gate: bad sizes");
  EB_REQUIRE(ldo % 8 == 0 && ldg % 8 == 0 && ld_out % 8 == 0 && ldo >= (long long)heads * dv && ldg >= (long long)heads * dv && ld_out >= (long long)heads * dv,
             "head_norm_gate: row strides must be multiples of 8 and hold a row");
  EB_REQUIRE(aligned16(o) && aligned16(g) && aligned16(norm) && aligned16(out), "head_norm_gate: pointers must be 16-byte aligned");
  EB_REQUIRE(((long long)rows * heads + 7) / 8 < (1ll << 31), "head_norm_gate: too many rows");
  HeadNormParams p{};
  p.o = o; p.g = g; p.norm = norm; p.ldo = ldo; p.ldg = ldg; p.ld_out = ld_out; p.out = out;
  p.inv_count = 1.f / (float)dv_count; p.eps = eps; p.rows = rows; p.heads = heads; p.dv = dv; p.silu = silu;
  const dim3 grid((unsigned)(((long long)rows * heads + 7) / 8)), block(256);
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) launch_pdl(head_norm_gate_kernel<float>, grid, block, 0, st, p);
  else if (dtype == EB_F16) launch_pdl(head_norm_gate_kernel<__half>, grid, block, 0, st, p);
  else launch_pdl(head_norm_gate_kernel<__nv_bfloat16>, grid, block, 0, st, p);
  return check_launch("head_norm_gate");
}

extern "C" int eb_head_norm_gate(const void *o, long long ldo, const void *g, long long ldg, const void *norm, float eps, void *out,
                                 long long ld_out, int rows, int heads, int dv, int dv_count, int dtype, void *stream) {
  return eb_head_norm_gate_act(o, ldo, g, ldg, norm, eps, out, ld_out, rows, heads, dv, dv_count, 0, dtype, stream);
}
