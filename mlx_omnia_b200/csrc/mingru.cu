// A gated recurrence over independent channels whose gates read only the current token:
//
//   z_t = sigmoid(zh_t + bz)          u_t = uh_t + bu                  (zh, uh, gh: projected columns)
//   cand_t = u_t + 1/2 where u_t >= 0, sigmoid(u_t) where u_t < 0
//   S_t = (1 - z_t) S_(t-1) + z_t cand_t
//   out_t = S_t * silu(gh_t)
//
// Everything but the projected columns and the output is float32. A portion's tokens are cut into
// segments: a warp folds its segment (32 lanes of one or two channels) to (product of 1 - z, value from
// zero), a cluster of blocks exchanges its blocks' folds through distributed shared memory, and every
// warp then walks its segment again from its start. Cutting is the same recurrence regrouped.
// A step of single tokens is one multiply and one fused multiply-add a channel, in a kernel of its own.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int MAX_WARPS = 16, MAX_CLUSTER = 8;

__device__ __forceinline__ float sigmoid_f(float v) {
  const float e = expf(-fabsf(v)), big = __fdividef(1.f, 1.f + e);
  return v >= 0.f ? big : e * big;
}

// 1 - z and z * cand of a token's channel, both sigmoids from one exponential of -|z| (no difference near one).
__device__ __forceinline__ void gates_of(float z, float u, float& keep, float& take) {
  const float e = expf(-fabsf(z)), big = __fdividef(1.f, 1.f + e), small = e * big;
  keep = z >= 0.f ? small : big;
  take = (z >= 0.f ? big : small) * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
}

template <typename T>
__global__ void mingru_step_kernel(const T* __restrict__ proj, int stride, int z_col, int u_col, int g_col,
                                   const float* __restrict__ z_bias, const float* __restrict__ u_bias, int C,
                                   float* __restrict__ S_state, const int* __restrict__ cu_seqlens,
                                   const int* __restrict__ state_slots, T* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int t = cu_seqlens[seq];
  if (c >= C || cu_seqlens[seq + 1] <= t) return;
  const T* row = proj + (size_t)t * stride;
  float* S = S_state + (size_t)state_slots[seq] * C + c;
  float keep, take;
  gates_of(to_f32(row[z_col + c]) + (z_bias ? z_bias[c] : 0.f), to_f32(row[u_col + c]) + (u_bias ? u_bias[c] : 0.f), keep, take);
  const float s = fmaf(keep, *S, take);
  *S = s;
  const float g = to_f32(row[g_col + c]);
  out[(size_t)t * C + c] = from_f32<T>(s * g * sigmoid_f(g));
}

// V neighbouring channels a lane; BATCH tokens' columns are asked for before the first is used.
template <typename T, int V>
struct alignas(sizeof(T) * V) Lanes {
  T v[V];
};
constexpr int BATCH = 8;

// grid (cluster, ceil(C / 32 V), requests), clusters along x; block 32 x warps.
template <typename T, int V>
__global__ void __launch_bounds__(32 * MAX_WARPS, 2)
mingru_scan_kernel(const T* __restrict__ proj, int stride, int z_col, int u_col, int g_col,
                   const float* __restrict__ z_bias, const float* __restrict__ u_bias, int C, float* __restrict__ S_state,
                   const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, T* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  typedef Lanes<T, V> L;
  __shared__ float fold_a[MAX_WARPS][32 * V], fold_b[MAX_WARPS][32 * V];
  __shared__ float block_a[32 * V], block_b[32 * V];
  __shared__ float start[MAX_WARPS][32 * V];  // what every warp's segment starts from
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = (int)blockIdx.x, ranks = (int)gridDim.x;  // one cluster spans the grid's x
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int at = lane * V, c = blockIdx.y * 32 * V + at, seq = blockIdx.z;
  const int begin = cu_seqlens[seq], n = max(0, cu_seqlens[seq + 1] - begin);
  const bool live = c < C;  // C is a multiple of V
  const int per = (n + ranks * warps - 1) / (ranks * warps);
  const int seg = rank * warps + warp;
  const int t0 = begin + min(n, seg * per), t1 = live ? begin + min(n, (seg + 1) * per) : t0;
  float zb[V], ub[V], A[V], B[V];
  float* state = S_state + (size_t)state_slots[seq] * C;
#pragma unroll
  for (int e = 0; e < V; ++e) {
    zb[e] = live && z_bias ? z_bias[c + e] : 0.f, ub[e] = live && u_bias ? u_bias[c + e] : 0.f;
    A[e] = 1.f, B[e] = 0.f;
  }
  // Thread i < 32 V looks after channel i's folds. Every block reads the carried state before any block's last
  // warp writes it (behind the barriers).
  const int mine = blockIdx.y * 32 * V + (int)threadIdx.x;
  const bool folds = threadIdx.x < 32 * V;
  float carried = folds && mine < C && n > 0 ? state[mine] : 0.f;
  for (int t = t0; t < t1; t += BATCH) {
    L z[BATCH], u[BATCH];
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const T* row = proj + (size_t)min(t + i, t1 - 1) * stride + c;
      z[i] = *reinterpret_cast<const L*>(row + z_col), u[i] = *reinterpret_cast<const L*>(row + u_col);
    }
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      if (t + i >= t1) break;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float keep, take;
        gates_of(to_f32(z[i].v[e]) + zb[e], to_f32(u[i].v[e]) + ub[e], keep, take);
        B[e] = fmaf(keep, B[e], take);
        A[e] *= keep;
      }
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) fold_a[warp][at + e] = A[e], fold_b[warp][at + e] = B[e];
  __syncthreads();
  if (ranks > 1) {
    if (folds) {
      float a = 1.f, b = 0.f;
#pragma unroll 4
      for (int w = 0; w < warps; ++w) {
        const float fa = fold_a[w][threadIdx.x];
        b = fmaf(fa, b, fold_b[w][threadIdx.x]), a *= fa;
      }
      block_a[threadIdx.x] = a, block_b[threadIdx.x] = b;
    }
    cluster.sync();
    if (folds) {
      float ra[MAX_CLUSTER], rb[MAX_CLUSTER];  // the blocks before this one, all asked for at once
#pragma unroll
      for (int r = 0; r < MAX_CLUSTER; ++r)
        if (r < rank)
          ra[r] = *cluster.map_shared_rank(&block_a[threadIdx.x], r), rb[r] = *cluster.map_shared_rank(&block_b[threadIdx.x], r);
#pragma unroll
      for (int r = 0; r < MAX_CLUSTER; ++r)
        if (r < rank) carried = fmaf(ra[r], carried, rb[r]);
    }
  }
  if (folds) {
#pragma unroll 4
    for (int w = 0; w < warps; ++w) {
      start[w][threadIdx.x] = carried;
      carried = fmaf(fold_a[w][threadIdx.x], carried, fold_b[w][threadIdx.x]);
    }
  }
  __syncthreads();
  float S[V];
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = start[warp][at + e];
  for (int t = t0; t < t1; t += BATCH) {
    L z[BATCH], u[BATCH], g[BATCH];
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const T* row = proj + (size_t)min(t + i, t1 - 1) * stride + c;
      z[i] = *reinterpret_cast<const L*>(row + z_col), u[i] = *reinterpret_cast<const L*>(row + u_col);
      g[i] = *reinterpret_cast<const L*>(row + g_col);
    }
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      if (t + i >= t1) break;
      L o;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float keep, take;
        gates_of(to_f32(z[i].v[e]) + zb[e], to_f32(u[i].v[e]) + ub[e], keep, take);
        S[e] = fmaf(keep, S[e], take);
        const float gate = to_f32(g[i].v[e]);
        o.v[e] = from_f32<T>(S[e] * gate * sigmoid_f(gate));
      }
      *reinterpret_cast<L*>(out + (size_t)(t + i) * C + c) = o;
    }
  }
  if (t0 < t1 && t1 == begin + n)
#pragma unroll
    for (int e = 0; e < V; ++e) state[c + e] = S[e];
  if (ranks > 1) cluster.sync();  // nobody leaves while another block may still read its folds
}

}  // namespace

// S_state float32 [slots, C], moved on; out [tokens, C]. single: every request brings one token (or none).
// Otherwise warps (1 .. 16) x cluster (1, 2, 4, 8) segments a request.
extern "C" int omnia_mingru(const void* proj, int stride, int z_col, int u_col, int g_col, const float* z_bias,
                            const float* u_bias, int C, float* S_state, const int* cu_seqlens, const int* state_slots,
                            int num_seqs, int single, int warps, int cluster, void* out, int dtype, cudaStream_t stream) {
  if (num_seqs == 0) return 0;
  if (C < 1 || warps < 1 || warps > MAX_WARPS || cluster < 1 || cluster > MAX_CLUSTER || (cluster & (cluster - 1)))
    return (int)cudaErrorInvalidValue;
  if (single) {
    const int threads = C >= 128 ? 128 : 32;
    OMNIA_DISPATCH_DTYPE(dtype, (launch_pdl(mingru_step_kernel<T>, dim3((C + threads - 1) / threads, num_seqs), dim3(threads), 0,
                                            stream, (const T*)proj, stride, z_col, u_col, g_col, z_bias, u_bias, C, S_state,
                                            cu_seqlens, state_slots, (T*)out)));
    return OMNIA_LAUNCH_RESULT();
  }
  // Two channels a lane where they come in aligned pairs (a block then needs 64 threads to look after
  // the folds of 64 channels).
  const bool pairs = warps >= 2 && C % 2 == 0 && stride % 2 == 0 && z_col % 2 == 0 && u_col % 2 == 0 && g_col % 2 == 0 &&
                     (((uintptr_t)proj | (uintptr_t)out) & 7) == 0;
  const int lanes = pairs ? 64 : 32;
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(cluster, (C + lanes - 1) / lanes, num_seqs);
  config.blockDim = dim3(32 * warps);
  config.stream = stream;
  cudaLaunchAttribute attributes[2];
  attributes[0].id = cudaLaunchAttributeClusterDimension;
  attributes[0].val.clusterDim.x = cluster, attributes[0].val.clusterDim.y = 1, attributes[0].val.clusterDim.z = 1;
  attributes[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attributes[1].val.programmaticStreamSerializationAllowed = 1;
  config.attrs = attributes;
  config.numAttrs = 2;
  OMNIA_DISPATCH_DTYPE(dtype, {
    cudaLaunchKernelEx(&config, pairs ? mingru_scan_kernel<T, 2> : mingru_scan_kernel<T, 1>, (const T*)proj, stride, z_col, u_col,
                       g_col, z_bias, u_bias, C, S_state, cu_seqlens, state_slots, (T*)out);
  });
  return OMNIA_LAUNCH_RESULT();
}
