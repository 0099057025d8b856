// A gated recurrence over independent channels whose gates read only the current token:
//
//   z_t = sigmoid(zh_t + bz)          u_t = uh_t + bu                  (zh, uh, gh: projected columns)
//   cand_t = u_t + 1/2 where u_t >= 0, sigmoid(u_t) where u_t < 0
//   S_t = (1 - z_t) S_(t-1) + z_t cand_t
//   out_t = S_t * silu(gh_t)
//
// Everything but the projected columns and the output is float32. A portion's tokens are cut into
// segments: a warp folds its segment (32 channels, lane = channel) to (product of 1 - z, value from
// zero), a cluster of blocks exchanges its blocks' folds through distributed shared memory, and every
// warp then walks its segment again from its start. Cutting is the same recurrence regrouped.
// A step of single tokens is one multiply and one fused multiply-add a channel, in a kernel of its own.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int MAX_WARPS = 16, MAX_CLUSTER = 8;

__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }

// 1 - z and z * cand of a token's channel. 1 - sigmoid(z) is sigmoid(-z): no difference near one.
__device__ __forceinline__ void gates_of(float z, float u, float& keep, float& take) {
  keep = sigmoid_f(-z);
  take = sigmoid_f(z) * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
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

// grid (cluster, ceil(C / 32), requests), clusters along x; block 32 x warps.
template <typename T>
__global__ void __launch_bounds__(32 * MAX_WARPS)
mingru_scan_kernel(const T* __restrict__ proj, int stride, int z_col, int u_col, int g_col,
                   const float* __restrict__ z_bias, const float* __restrict__ u_bias, int C, float* __restrict__ S_state,
                   const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, T* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float fold_a[MAX_WARPS][32], fold_b[MAX_WARPS][32];
  __shared__ float block_a[32], block_b[32];
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = (int)blockIdx.x, ranks = (int)gridDim.x;  // one cluster spans the grid's x
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int c = blockIdx.y * 32 + lane, seq = blockIdx.z;
  const int begin = cu_seqlens[seq], n = max(0, cu_seqlens[seq + 1] - begin);
  const bool live = c < C;
  const int per = (n + ranks * warps - 1) / (ranks * warps);
  const int seg = rank * warps + warp;
  const int t0 = begin + min(n, seg * per), t1 = begin + min(n, (seg + 1) * per);
  const float zb = live && z_bias ? z_bias[c] : 0.f, ub = live && u_bias ? u_bias[c] : 0.f;
  float* state = S_state + (size_t)state_slots[seq] * C + c;
  float A = 1.f, B = 0.f;
  if (live) {
#pragma unroll 8
    for (int t = t0; t < t1; ++t) {
      const T* row = proj + (size_t)t * stride;
      float keep, take;
      gates_of(to_f32(row[z_col + c]) + zb, to_f32(row[u_col + c]) + ub, keep, take);
      B = fmaf(keep, B, take);
      A *= keep;
    }
  }
  fold_a[warp][lane] = A, fold_b[warp][lane] = B;
  // Every block reads the carried state before any block's last warp writes it (behind the barrier).
  float S = live && n > 0 ? *state : 0.f;
  __syncthreads();
  if (warp == 0) {
    float a = 1.f, b = 0.f;
    for (int w = 0; w < warps; ++w) b = fmaf(fold_a[w][lane], b, fold_b[w][lane]), a *= fold_a[w][lane];
    block_a[lane] = a, block_b[lane] = b;
  }
  cluster.sync();
  for (int r = 0; r < rank; ++r)
    S = fmaf(*cluster.map_shared_rank(&block_a[lane], r), S, *cluster.map_shared_rank(&block_b[lane], r));
  for (int w = 0; w < warp; ++w) S = fmaf(fold_a[w][lane], S, fold_b[w][lane]);
  if (live) {
#pragma unroll 8
    for (int t = t0; t < t1; ++t) {
      const T* row = proj + (size_t)t * stride;
      float keep, take;
      gates_of(to_f32(row[z_col + c]) + zb, to_f32(row[u_col + c]) + ub, keep, take);
      S = fmaf(keep, S, take);
      const float g = to_f32(row[g_col + c]);
      out[(size_t)t * C + c] = from_f32<T>(S * g * sigmoid_f(g));
    }
    if (t0 < t1 && t1 == begin + n) *state = S;
  }
  cluster.sync();  // nobody leaves while another block may still read its folds
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
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(cluster, (C + 31) / 32, num_seqs);
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
    cudaLaunchKernelEx(&config, mingru_scan_kernel<T>, (const T*)proj, stride, z_col, u_col, g_col, z_bias, u_bias, C, S_state,
                       cu_seqlens, state_slots, (T*)out);
  });
  return OMNIA_LAUNCH_RESULT();
}
