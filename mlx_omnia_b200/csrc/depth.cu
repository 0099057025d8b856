// Layer norm, and the end of a parallel block: the residual takes both branches at once, the depth
// average mixes it with what earlier layers left, and the next reader's norm is applied, in one
// pass over a row.
//
//   layernorm    h = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b       float32 in, T out
//   depth_step   r   = x + a + m                 (a, m: the branches; m may be absent, or be the weighted
//                                                 sum of rows of routed experts, taken here in float32)
//                x'  = sum_(j < count) c_j X_j + c_count r     (X_0 = the embedding output, X_j = result
//                                                 of layer j - 1; without coefficients x' = r)
//                h   = norm(x')                  (layer norm, or RMS norm where there is no bias; may be absent)
//                r is kept as X_count for the layers after.
//
// A block owns a row; the row waits in shared memory as float32 between the passes. The mean and the
// mean of the squared deviations are taken one after the other (no difference of large sums).
#include "common.cuh"

namespace {

constexpr int DEPTH_THREADS = 256;

// Statistics of the row in `row` (every thread has written its own entries, i = threadIdx.x * V ...), then
// the normed row to `h`. `bias` null: RMS norm.
template <typename T>
__device__ __forceinline__ void norm_row(const float* row, const float* __restrict__ w, const float* __restrict__ b,
                                         int layer, float eps, T* __restrict__ h, int hidden, float sum, float* scratch) {
  float mean = 0.f;
  if (layer) mean = block_sum(sum, scratch) / (float)hidden;
  else __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float d = row[i] - mean;
    ss += d * d;
  }
  const float r = rsqrtf(block_sum(ss, scratch) / (float)hidden + eps);
  constexpr int VEC = 8;
  if (hidden % VEC == 0 && ((uintptr_t)h & 15) == 0 && ((uintptr_t)w & 15) == 0 && ((uintptr_t)b & 15) == 0) {
    for (int i = threadIdx.x * VEC; i < hidden; i += blockDim.x * VEC) {
      alignas(16) T o[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e += 4) {
        const float4 x = *reinterpret_cast<const float4*>(row + i + e);
        const float4 wv = w ? __ldg(reinterpret_cast<const float4*>(w + i + e)) : make_float4(1.f, 1.f, 1.f, 1.f);
        const float4 bv = b ? __ldg(reinterpret_cast<const float4*>(b + i + e)) : make_float4(0.f, 0.f, 0.f, 0.f);
        o[e] = from_f32<T>((x.x - mean) * r * wv.x + bv.x);
        o[e + 1] = from_f32<T>((x.y - mean) * r * wv.y + bv.y);
        o[e + 2] = from_f32<T>((x.z - mean) * r * wv.z + bv.z);
        o[e + 3] = from_f32<T>((x.w - mean) * r * wv.w + bv.w);
      }
#pragma unroll
      for (int q = 0; q < (int)(VEC * sizeof(T) / 16); ++q)
        reinterpret_cast<uint4*>(h + i)[q] = reinterpret_cast<const uint4*>(o)[q];
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
      h[i] = from_f32<T>((row[i] - mean) * r * (w ? w[i] : 1.f) + (b ? b[i] : 0.f));
  }
}

template <typename T>
__global__ void __launch_bounds__(DEPTH_THREADS)
layernorm_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, float eps,
                 T* __restrict__ h, int hidden) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float row_s[];
  __shared__ float scratch[33];
  const float* xr = x + (size_t)blockIdx.x * hidden;
  float sum = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = xr[i];
    row_s[i] = v;
    sum += v;
  }
  norm_row(row_s, w, b, 1, eps, h + (size_t)blockIdx.x * hidden, hidden, sum, scratch);
}

struct DepthArgs {
  const float* x;          // [rows, hidden] the residual the block was handed
  const void* a;           // [rows, hidden] T
  const void* m;           // [rows, hidden] T, or null
  const void* expert_rows; // [sorted pairs, hidden] T, or null: m = sum_k weight[t, k] * expert_rows[place[t, k]]
  const int* place;        // [rows, top]
  const float* weight;     // [rows, top]
  int top;
  const float* first;      // X_0 [rows, hidden]
  float* results;          // X_1 .. side by side, [layers, rows, hidden]; X_count is written when `keep`
  int count, keep;
  const float* coef;       // [count + 1], or null: no average
  float* x_out;            // [rows, hidden]
  const float* norm_w;
  const float* norm_b;
  int norm;                // 0 none, 1 layer norm, 2 RMS norm
  float eps;
  void* h;                 // [rows, hidden] T
  int rows, hidden;
};

template <typename T, int V>
struct alignas(sizeof(T) * V) Pack {
  T v[V];
};

template <typename T, int V>
__global__ void __launch_bounds__(DEPTH_THREADS) depth_step_kernel(const DepthArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float row_s[];
  __shared__ float scratch[33];
  const int t = blockIdx.x, hidden = p.hidden;
  const size_t base = (size_t)t * hidden, slab = (size_t)p.rows * hidden;
  typedef Pack<float, V> F;
  typedef Pack<T, V> E;
  const float own = p.coef ? __ldg(p.coef + p.count) : 1.f;
  float sum = 0.f;
  for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
    F r = *reinterpret_cast<const F*>(p.x + base + i);
    const E a = *reinterpret_cast<const E*>((const T*)p.a + base + i);
    float branch[V];
#pragma unroll
    for (int e = 0; e < V; ++e) branch[e] = to_f32(a.v[e]);
    if (p.expert_rows) {
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = 0.f;
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        const int at = p.place[(size_t)t * p.top + k];
        const float w = p.weight[(size_t)t * p.top + k];
        const E y = *reinterpret_cast<const E*>((const T*)p.expert_rows + (size_t)at * hidden + i);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w, to_f32(y.v[e]), acc[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) branch[e] += acc[e];
    } else if (p.m) {
      const E m = *reinterpret_cast<const E*>((const T*)p.m + base + i);
#pragma unroll
      for (int e = 0; e < V; ++e) branch[e] += to_f32(m.v[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) r.v[e] += branch[e];
    F out = r;
    if (p.coef) {
      if (p.keep) *reinterpret_cast<F*>(p.results + (size_t)(p.count - 1) * slab + base + i) = r;
      const float c0 = __ldg(p.coef);
      const F x0 = *reinterpret_cast<const F*>(p.first + base + i);
#pragma unroll
      for (int e = 0; e < V; ++e) out.v[e] = c0 * x0.v[e];
#pragma unroll 8
      for (int j = 1; j < p.count; ++j) {
        const float c = __ldg(p.coef + j);
        const F xj = *reinterpret_cast<const F*>(p.results + (size_t)(j - 1) * slab + base + i);
#pragma unroll
        for (int e = 0; e < V; ++e) out.v[e] = fmaf(c, xj.v[e], out.v[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) out.v[e] = fmaf(own, r.v[e], out.v[e]);
    }
    *reinterpret_cast<F*>(p.x_out + base + i) = out;
    if (p.norm) {
      *reinterpret_cast<F*>(row_s + i) = out;
#pragma unroll
      for (int e = 0; e < V; ++e) sum += out.v[e];
    }
  }
  if (p.norm)
    norm_row(row_s, p.norm_w, p.norm_b, p.norm == 1, p.eps, (T*)p.h + base, hidden, sum, scratch);
}

template <typename K>
int allow_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 200 * 1024) return (int)cudaErrorInvalidValue;
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <typename T, int V>
int launch_depth(const DepthArgs& p, cudaStream_t stream) {
  const size_t smem = p.norm ? (size_t)p.hidden * sizeof(float) : 0;
  const int code = allow_smem(depth_step_kernel<T, V>, smem);
  if (code != 0) return code;
  launch_pdl(depth_step_kernel<T, V>, dim3(p.rows), dim3(DEPTH_THREADS), smem, stream, p);
  return OMNIA_LAUNCH_RESULT();
}

}  // namespace

extern "C" int omnia_layernorm(const float* x, const float* w, const float* b, float eps, void* h, int rows, int hidden,
                               int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  const size_t smem = (size_t)hidden * sizeof(float);
  OMNIA_DISPATCH_DTYPE(dtype, {
    const int code = allow_smem(layernorm_kernel<T>, smem);
    if (code != 0) return code;
    launch_pdl(layernorm_kernel<T>, dim3(rows), dim3(DEPTH_THREADS), smem, stream, x, w, b, eps, (T*)h, hidden);
  });
  return OMNIA_LAUNCH_RESULT();
}

// See the head of the file. `place` entries must be rows of `expert_rows`.
extern "C" int omnia_depth_step(const float* x, const void* a, const void* m, const void* expert_rows, const int* place,
                                const float* weight, int top, const float* first, float* results, int count, int keep,
                                const float* coef, float* x_out, const float* norm_w, const float* norm_b, int norm,
                                float eps, void* h, int rows, int hidden, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (hidden < 1 || norm < 0 || norm > 2 || (coef && (count < 1 || first == nullptr)) || (expert_rows && top < 1))
    return (int)cudaErrorInvalidValue;
  DepthArgs p;
  p.x = x, p.a = a, p.m = m, p.expert_rows = expert_rows, p.place = place, p.weight = weight, p.top = top;
  p.first = first, p.results = results, p.count = count, p.keep = keep, p.coef = coef, p.x_out = x_out;
  p.norm_w = norm_w, p.norm_b = norm_b, p.norm = norm, p.eps = eps, p.h = h, p.rows = rows, p.hidden = hidden;
  const uintptr_t all = (uintptr_t)x | (uintptr_t)a | (uintptr_t)m | (uintptr_t)expert_rows | (uintptr_t)first |
                        (uintptr_t)results | (uintptr_t)x_out;
  const bool wide = hidden % 4 == 0 && (all & 15) == 0;
  OMNIA_DISPATCH_DTYPE(dtype, { return wide ? launch_depth<T, 4>(p, stream) : launch_depth<T, 1>(p, stream); });
  return (int)cudaErrorInvalidValue;
}
