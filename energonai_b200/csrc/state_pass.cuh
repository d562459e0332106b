// What the generation-step kernels of recurrent layers share (matrix_memory.cu, decay_memory.cu): one pass
// over a CTA's columns of a head's fp32 state S [dk][dv], HBM-bound (read and written once),
//
//   S[d] = decay(d) S[d] + k[d] v,    y = sum_d q[d] S[d],
//
// and the sum that the CTAs of a head form together.
#pragma once

#include "common.cuh"

namespace eb {
namespace {

constexpr int kStepThreads = 256, kStepBatch = 8;

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// Thread = 4 columns of every R-th row; kStepBatch rows in flight per thread, the first of them requested
// (begin) before anything else is worked out.
struct StatePass {
  float4 s[kStepBatch];
  float *S;                    // this thread's column of row 0
  int dk, dv, cols, cg4, rg, R;
  bool active;
  // cols: columns of the CTA (a multiple of 4, at most 4 * kStepThreads), of which `width` exist
  __device__ __forceinline__ StatePass(float *state, int dk_, int dv_, int cols_, int width) : dk(dk_), dv(dv_), cols(cols_) {
    const int groups = cols / 4;
    R = kStepThreads / groups;
    cg4 = threadIdx.x % groups;
    rg = threadIdx.x / groups;
    active = rg < R && cg4 * 4 < width;
    S = state + cg4 * 4;
  }
  __device__ __forceinline__ void fetch(int d0) {
#pragma unroll
    for (int i = 0; i < kStepBatch; ++i)
      if (d0 + i * R < dk) s[i] = __ldcs(reinterpret_cast<const float4 *>(S + (long long)(d0 + i * R) * dv));
  }
  __device__ __forceinline__ void begin() {
    if (active) fetch(rg);
  }
  // ks, qs [dk], vs [cols] in shared memory; the row groups' sums go to red [R][cols]
  template <class Decay> __device__ __forceinline__ void run(Decay decay, const float *ks, const float *qs, const float *vs, float *red) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active) {
      const float4 vv = *reinterpret_cast<const float4 *>(vs + cg4 * 4);
      for (int d0 = rg; d0 < dk; d0 += R * kStepBatch) {
        if (d0 != rg) fetch(d0);
#pragma unroll
        for (int i = 0; i < kStepBatch; ++i) {
          const int d = d0 + i * R;
          if (d < dk) {
            const float a = decay(d), kd = ks[d], qd = qs[d];
            s[i].x = fmaf(a, s[i].x, kd * vv.x); s[i].y = fmaf(a, s[i].y, kd * vv.y);
            s[i].z = fmaf(a, s[i].z, kd * vv.z); s[i].w = fmaf(a, s[i].w, kd * vv.w);
            __stcs(reinterpret_cast<float4 *>(S + (long long)d * dv), s[i]);
            acc.x = fmaf(s[i].x, qd, acc.x); acc.y = fmaf(s[i].y, qd, acc.y);
            acc.z = fmaf(s[i].z, qd, acc.z); acc.w = fmaf(s[i].w, qd, acc.w);
          }
        }
      }
    }
    if (rg < R) *reinterpret_cast<float4 *>(red + rg * cols + cg4 * 4) = acc;
  }
};

// The CTAs of a head show each other a number: every one sends its own to all with an asynchronous store
// that completes on the receiver's mbarrier.  (A cluster barrier would do, but its release waits for
// the stores of the whole state.)
struct ClusterSum {
  float part[8];
  uint64_t arrived;
};
__device__ __forceinline__ void cluster_sum_begin(ClusterSum &c, int peers) {
  if (peers <= 1) return;
  if (threadIdx.x == 0) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_addr(&c.arrived)) : "memory");
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_addr(&c.arrived)), "r"(peers * 4) : "memory");
  }
  __syncwarp();
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
}
// Once per launch; every thread of the CTA calls it with the CTA's number.
__device__ __forceinline__ float cluster_sum(ClusterSum &c, int peers, float v) {
  if (peers <= 1) return v;
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");         // every CTA's mbarrier is set up
  if (threadIdx.x < peers) {
    uint32_t dst, bar;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_addr(&c.part[blockIdx.x])), "r"(threadIdx.x));
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(bar) : "r"(smem_addr(&c.arrived)), "r"(threadIdx.x));
    asm volatile("st.async.shared::cluster.mbarrier::complete_tx::bytes.b32 [%0], %1, [%2];" ::"r"(dst), "r"(__float_as_uint(v)), "r"(bar) : "memory");
  }
  // (the numbers of all CTAs arrive without further waits of theirs; the limit only keeps a defect from hanging)
  for (int it = 0; it < (1 << 20); ++it) {
    uint32_t ok;
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], 0;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(ok) : "r"(smem_addr(&c.arrived)) : "memory");
    if (ok) break;
  }
  v = 0.f;
  for (int r = 0; r < peers; ++r) v += c.part[r];
  return v;
}

// Columns of a head over as many CTAs (1, 2, 4, 8) as it takes to have two per SM, at least 32 columns
// each; more where a CTA would hold more than 1024.
inline int state_split(long long heads, int dv) {
  int split = 1;
  while (split < 8 && (heads * split < 2 * sm_count() || dv > 1024 * split) && (dv + 2 * split - 1) / (2 * split) >= 32) split *= 2;
  return split;
}

// Launch with the CTAs of a head (gridDim.x) as a cluster.
template <typename P> int launch_state_step(const char *name, void (*kern)(P), const P &p, dim3 grid, int cluster, size_t smem, cudaStream_t st) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(kStepThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  cudaLaunchKernelEx(&cfg, kern, p);
  return check_launch(name);
}

}  // namespace
}  // namespace eb
