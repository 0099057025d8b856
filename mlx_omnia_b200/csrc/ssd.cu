// A state-space mixer of the Mamba-2 form around its recurrence. The projected row of a token holds, from
// `col0`, [z: inner | x: inner | B: G * N | C: G * N | dt: H] with inner = H * dv; per head h, its B and C those of
// group h / (H / G):
//
//   x, B, C = silu(causal convolution per channel + bias)   (the C channels x | B | C together, K taps, the
//             last one the current token's; a request's last K - 1 inputs carried in a state slot)
//   dt = softplus(dt + dt_bias[h]),  a = exp(-exp(A_log[h]) dt)
//   S_t = a S_(t-1) + dt B_t x_t^T   [N, dv],   y_t = S_t^T C_t + D_h x_t
//   out = RMSnorm(y * silu(z)) * w, the norm taken over `norm_groups` equal runs of the heads side by side
//
// Three kernels, everything in float32 up to what they hand on:
//
//   inputs   a thread walks a channel (or a head's dt) over a run of tokens with the taps' window in registers,
//            so every projected value is read once. Out: float32 rows [C | B | x | (a, dt) a head] for the token-by-
//            token recurrence (state_recurrence.cu), or for the chunked one (ssd_chunk.cu) float16 rows
//            [x | B | C] beside float32 pairs (log a, dt).
//   step     a step in which every request brings one token: convolution, step sizes and recurrence in one
//            kernel, a block per (request, head, run of columns).
//   out      per token: y (the skip in it) times silu(z), norm and weight, rounded once; and, after the last token,
//            per request: the convolution's carried inputs moved on.
//
// The projected rows may be float32 where the rest of the model is bfloat16.
#include "common.cuh"

#include <cuda_fp16.h>

// float16 holds the convolution's outputs for the chunked recurrence; what is beyond its range is held at its end.
template <>
__device__ __forceinline__ __half from_f32<__half>(float v) {
  return __float2half_rn(v > 65504.f ? 65504.f : v < -65504.f ? -65504.f : v);
}

namespace {

constexpr int MAX_TAPS = 16;
constexpr int RUN = 16;  // tokens a thread of the input step walks

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }

// The request that token t belongs to.
__device__ __forceinline__ int request_of(const int* __restrict__ cu, int num_seqs, int t) {
  int lo = 0, hi = num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid + 1] > t) hi = mid;
    else lo = mid + 1;
  }
  return lo;
}

struct Sizes {
  int H, dv, G, N;
  __host__ __device__ int inner() const { return H * dv; }
  __host__ __device__ int channels() const { return H * dv + 2 * G * N; }
};

// VC neighbouring elements as float32, or as O.
template <int VC>
__device__ __forceinline__ void load_vec(const float* p, float* v) {
  if constexpr (VC == 2) {
    const float2 q = *reinterpret_cast<const float2*>(p);
    v[0] = q.x, v[1] = q.y;
  } else {
    v[0] = p[0];
  }
}
template <int VC>
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float* v) {
  if constexpr (VC == 2) {
    const __nv_bfloat162 q = *reinterpret_cast<const __nv_bfloat162*>(p);
    v[0] = __low2float(q), v[1] = __high2float(q);
  } else {
    v[0] = to_f32(p[0]);
  }
}
template <int VC>
__device__ __forceinline__ void store_vec(float* p, const float* v) {
  if constexpr (VC == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else p[0] = v[0];
}
template <int VC>
__device__ __forceinline__ void store_vec(__half* p, const float* v) {
  if constexpr (VC == 2) *reinterpret_cast<__half2*>(p) = __halves2half2(from_f32<__half>(v[0]), from_f32<__half>(v[1]));
  else p[0] = from_f32<__half>(v[0]);
}

// grid (ceil((channels / VC + H) / 128), ceil(tokens / RUN)), 128 threads. KT: taps held in registers (>= taps); VC:
// channels a thread walks (2 where every width and place is even). Places of x, B and C in an output row are at_x,
// at_b, at_c; the pairs' rows are pair_stride floats apart.
template <typename T, typename O, int KT, int VC>
__global__ void __launch_bounds__(128)
ssd_inputs_kernel(const T* __restrict__ proj, int stride, int col0, Sizes s, const float* __restrict__ taps,
                  const float* __restrict__ conv_bias, int K, const float* __restrict__ conv_state,
                  const float* __restrict__ dt_bias, const float* __restrict__ A_log, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ state_slots, int num_seqs, int tokens, O* __restrict__ rows, int row_stride,
                  int at_x, int at_b, int at_c, float* __restrict__ pairs, int pair_stride, int log_decay) {
  pdl_wait();
  pdl_launch_dependents();
  const int C = s.channels(), inner = s.inner(), gn = s.G * s.N;
  const int unit = blockIdx.x * blockDim.x + threadIdx.x;
  if (unit >= C / VC + s.H) return;
  const int t0 = blockIdx.y * RUN, t1 = min(tokens, t0 + RUN);
  if (unit >= C / VC) {
    const int h = unit - C / VC;
    const float bias = dt_bias[h], rate = expf(A_log[h]);
#pragma unroll 8
    for (int t = t0; t < t1; ++t) {
      const float dt = softplus(to_f32(proj[(size_t)t * stride + col0 + inner + C + h]) + bias);
      float2* pair = reinterpret_cast<float2*>(pairs + (size_t)t * pair_stride) + h;
      *pair = make_float2(log_decay ? -rate * dt : expf(-rate * dt), dt);
    }
    return;
  }
  const int c = unit * VC;
  // taps [C, K]: w[KT - 1] the current token's, zeros ahead of the first.
  float w[KT][VC], u[KT][VC], bias[VC];
#pragma unroll
  for (int e = 0; e < VC; ++e) {
    bias[e] = conv_bias[c + e];
#pragma unroll
    for (int j = 0; j < KT; ++j) {
      const int tap = j - (KT - K);
      w[j][e] = tap >= 0 ? taps[(size_t)(c + e) * K + tap] : 0.f;
      u[j][e] = 0.f;
    }
  }
  const T* column = proj + col0 + inner + c;
  O* out = rows + (c < inner ? at_x + c : c < inner + gn ? at_b + (c - inner) : at_c + (c - inner - gn));
  int seq = request_of(cu_seqlens, num_seqs, t0);
  int begin = cu_seqlens[seq], end = cu_seqlens[seq + 1];
  // The K - 1 inputs ahead of token t of the request: in the batch, or carried in its slot.
  auto window = [&](int t) {
    const float* held = conv_state + (size_t)state_slots[seq] * max(K - 1, 1) * C + c;
#pragma unroll
    for (int j = 0; j < KT - 1; ++j) {
      const int back = KT - 1 - j;  // how many tokens before t
      if (back > K - 1) {
#pragma unroll
        for (int e = 0; e < VC; ++e) u[j + 1][e] = 0.f;
        continue;
      }
      const int at = t - back;
      if (at >= begin) load_vec<VC>(column + (size_t)at * stride, u[j + 1]);
      else load_vec<VC>(held + (size_t)(K - 1 + at - begin) * C, u[j + 1]);
    }
  };
  // One token: u[1 .. KT - 1] are the inputs before it, oldest first.
  auto token = [&](int t, const float* now) {
    float y[VC];
#pragma unroll
    for (int e = 0; e < VC; ++e) {
      y[e] = bias[e];
#pragma unroll
      for (int j = 0; j < KT - 1; ++j) u[j][e] = u[j + 1][e], y[e] = fmaf(w[j][e], u[j][e], y[e]);
      u[KT - 1][e] = now[e];
      y[e] = silu(fmaf(w[KT - 1][e], now[e], y[e]));
    }
    store_vec<VC>(out + (size_t)t * row_stride, y);
  };
  if (t1 - t0 == RUN && t1 <= end) {
    // The whole run in one request: all its inputs asked for at once.
    float now[RUN][VC];
#pragma unroll
    for (int i = 0; i < RUN; ++i) load_vec<VC>(column + (size_t)(t0 + i) * stride, now[i]);
    window(t0);
#pragma unroll
    for (int i = 0; i < RUN; ++i) token(t0 + i, now[i]);
    return;
  }
  window(t0);
  for (int t = t0; t < t1; ++t) {
    if (t >= end) {
      do {
        ++seq;
        begin = end, end = cu_seqlens[seq + 1];
      } while (t >= end && seq + 1 < num_seqs);
      window(t);
    }
    float now[VC];
    load_vec<VC>(column + (size_t)t * stride, now);
    token(t, now);
  }
}

// A block per (head x run of columns, request), 256 threads: the token's B and C (its group's) and x columns from the
// convolution, then S moved on in place, four columns and every `teams`-th row a thread, the teams' sums added in
// their order. y float32 [tokens, inner].
template <typename T, int VEC>
__global__ void __launch_bounds__(256, 4)
ssd_step_kernel(const T* __restrict__ proj, int stride, int col0, Sizes s, int cols, const float* __restrict__ taps,
                const float* __restrict__ conv_bias, int K, const float* __restrict__ conv_state,
                const float* __restrict__ dt_bias, const float* __restrict__ A_log, const float* __restrict__ D,
                float* __restrict__ S_state, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                float* __restrict__ y) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float step_s[];
  const int parts = (s.dv + cols - 1) / cols;
  const int head = blockIdx.x / parts, j0 = (blockIdx.x % parts) * cols, mine = min(cols, s.dv - j0), seq = blockIdx.y;
  const int t = cu_seqlens[seq];
  if (cu_seqlens[seq + 1] <= t) return;
  const int C = s.channels(), inner = s.inner(), gn = s.G * s.N, N = s.N, group = head / (s.H / s.G);
  float* b_s = step_s;                          // [N]
  float* c_s = b_s + N;                         // [N]
  float* x_s = c_s + N;                         // [cols]
  float* part = x_s + ((cols + 3) & ~3);        // [teams][mine]
  const T* row = proj + (size_t)t * stride + col0;
  const int slot = state_slots[seq];
  float* S = S_state + ((size_t)slot * s.H + head) * N * s.dv + j0;
  const int runs = mine / VEC, teams = max(1, (int)blockDim.x / max(runs, 1));
  // The first rows of S are asked for ahead of everything else: they come from memory, the rest is arithmetic.
  constexpr int AHEAD = 8;
  float ahead[AHEAD][VEC];
  if ((int)threadIdx.x < teams * runs) {
    const float* at = S + (size_t)(threadIdx.x / runs) * s.dv + (threadIdx.x % runs) * VEC;
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if ((int)threadIdx.x / runs + i * teams < N) {
        if constexpr (VEC == 4) {
          const float4 v = *reinterpret_cast<const float4*>(at + (size_t)i * teams * s.dv);
          ahead[i][0] = v.x, ahead[i][1] = v.y, ahead[i][2] = v.z, ahead[i][3] = v.w;
        } else {
          ahead[i][0] = at[(size_t)i * teams * s.dv];
        }
      }
  }
  const float* held = conv_state + (size_t)slot * max(K - 1, 1) * C;
  for (int i = threadIdx.x; i < 2 * N + mine; i += blockDim.x) {
    const int c = i < N ? inner + group * N + i : i < 2 * N ? inner + gn + group * N + (i - N) : head * s.dv + j0 + (i - 2 * N);
    float v = conv_bias[c];
    for (int j = 0; j < K - 1; ++j) v = fmaf(taps[(size_t)c * K + j], held[(size_t)j * C + c], v);
    v = fmaf(taps[(size_t)c * K + K - 1], to_f32(row[inner + c]), v);
    (i < 2 * N ? b_s[i] : x_s[i - 2 * N]) = silu(v);
  }
  const float dt = softplus(to_f32(row[inner + C + head]) + dt_bias[head]);
  const float a = expf(-expf(A_log[head]) * dt);
  __syncthreads();
  for (int item = threadIdx.x; item < teams * runs; item += blockDim.x) {
    const int m = item / runs, j = (item % runs) * VEC;
    float sum[VEC], v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum[e] = 0.f, v[e] = dt * x_s[j + e];
    auto move_on = [&](int r, float* st) {
      const float b = b_s[r], c = c_s[r];
      float* at = S + (size_t)r * s.dv + j;
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[e] = fmaf(b, v[e], a * st[e]), sum[e] = fmaf(st[e], c, sum[e]);
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(at) = make_float4(st[0], st[1], st[2], st[3]);
      else at[0] = st[0];
    };
    int r = m;
    if (item == (int)threadIdx.x) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i, r += teams)
        if (r < N) move_on(r, ahead[i]);
    }
#pragma unroll 8
    for (; r < N; r += teams) {
      const float* at = S + (size_t)r * s.dv + j;
      float st[VEC];
      if constexpr (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(at);
        st[0] = q.x, st[1] = q.y, st[2] = q.z, st[3] = q.w;
      } else {
        st[0] = at[0];
      }
      move_on(r, st);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) part[m * mine + j + e] = sum[e];
  }
  __syncthreads();
  for (int j = threadIdx.x; j < mine; j += blockDim.x) {
    float o = 0.f;
    for (int m = 0; m < teams; ++m) o += part[m * mine + j];
    y[(size_t)t * inner + head * s.dv + j0 + j] = fmaf(D[head], x_s[j], o);
  }
}

constexpr int OUT_ITEMS = 4;  // runs of four channels a thread of the output step keeps in registers

// Four neighbouring elements of the gate's columns as float32.
__device__ __forceinline__ void load_four(const float* p, float* v) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
}
__device__ __forceinline__ void load_four(const __nv_bfloat16* p, float* v) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&q.x), b = *reinterpret_cast<const __nv_bfloat162*>(&q.y);
  v[0] = __low2float(a), v[1] = __high2float(a), v[2] = __low2float(b), v[3] = __high2float(b);
}
__device__ __forceinline__ void store_four(float* p, const float* v) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_four(__nv_bfloat16* p, const float* v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// Blocks 0 .. tokens - 1: a token each; the others: blockDim channels of a request's carried inputs each.
// WHOLE: one norm group, its channels in fours and in the threads' registers.
template <typename T, typename O, bool WHOLE>
__global__ void __launch_bounds__(1024)
ssd_out_kernel(const float* __restrict__ y, const T* __restrict__ proj, int stride, int col0, Sizes s, int norm_groups,
               float eps, const float* __restrict__ norm_w, int K, float* __restrict__ conv_state,
               const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, int tokens, O* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) float out_s[];
  __shared__ float red[33];
  const int inner = s.inner(), C = s.channels();
  if ((int)blockIdx.x >= tokens) {
    const int blocks = (C + blockDim.x - 1) / blockDim.x, item = blockIdx.x - tokens;
    const int seq = item / blocks, c = (item % blocks) * blockDim.x + threadIdx.x;
    const int begin = cu_seqlens[seq], n = cu_seqlens[seq + 1] - begin;
    if (n <= 0 || K < 2 || c >= C) return;
    float* held = conv_state + (size_t)state_slots[seq] * (K - 1) * C + c;
    // Place j of the new window is n tokens further on than place j of the old one.
    float v[MAX_TAPS - 1];
#pragma unroll
    for (int j = 0; j < MAX_TAPS - 1; ++j)
      if (j < K - 1)
        v[j] = j + n < K - 1 ? held[(size_t)(j + n) * C] : to_f32(proj[(size_t)(begin + j + n - (K - 1)) * stride + col0 + inner + c]);
#pragma unroll
    for (int j = 0; j < MAX_TAPS - 1; ++j)
      if (j < K - 1) held[(size_t)j * C] = v[j];
    return;
  }
  const size_t t = blockIdx.x;
  const float* yt = y + t * inner;
  const T* z = proj + t * stride + col0;
  const int run = inner / norm_groups;
  if constexpr (WHOLE) {
    float v[OUT_ITEMS][4], ss = 0.f;
#pragma unroll
    for (int i = 0; i < OUT_ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < inner) {
        float gate[4];
        load_four(yt + c, v[i]);
        load_four(z + c, gate);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i][e] *= silu(gate[e]), ss += v[i][e] * v[i][e];
      }
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)inner + eps);
#pragma unroll
    for (int i = 0; i < OUT_ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < inner) {
        float w[4];
        load_four(norm_w + c, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i][e] *= r * w[e];
        store_four(out + t * inner + c, v[i]);
      }
    }
    return;
  }
  if (norm_groups == 1) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < inner; c += blockDim.x) {
      const float v = yt[c] * silu(to_f32(z[c]));
      out_s[c] = v;
      ss += v * v;
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)run + eps);
    for (int c = threadIdx.x; c < inner; c += blockDim.x) out[t * inner + c] = from_f32<O>(out_s[c] * r * norm_w[c]);
    return;
  }
  // A warp takes a group at a time.
  const int lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  for (int g = threadIdx.x >> 5; g < norm_groups; g += warps) {
    const int c0 = g * run;
    float ss = 0.f;
#pragma unroll 4
    for (int i = lane; i < run; i += 32) {
      const float v = yt[c0 + i] * silu(to_f32(z[c0 + i]));
      out_s[c0 + i] = v;
      ss += v * v;
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)run + eps);
    __syncwarp();
#pragma unroll 4
    for (int i = lane; i < run; i += 32) out[t * inner + c0 + i] = from_f32<O>(out_s[c0 + i] * r * norm_w[c0 + i]);
  }
}

template <typename T, typename O>
int launch_inputs(const void* proj, int stride, int col0, const Sizes& s, const float* taps, const float* conv_bias, int K,
                  const float* conv_state, const float* dt_bias, const float* A_log, const int* cu_seqlens,
                  const int* state_slots, int num_seqs, int tokens, void* rows, int row_stride, int at_x, int at_b, int at_c,
                  float* pairs, int pair_stride, int log_decay, cudaStream_t stream) {
  // Two channels a thread where every width, place and stride is even and every base on two elements.
  const bool even = ((s.inner() | (s.G * s.N) | stride | col0 | row_stride | at_x | at_b | at_c) & 1) == 0 &&
                    ((uintptr_t)proj % (2 * sizeof(T))) == 0 && ((uintptr_t)rows % (2 * sizeof(O))) == 0 &&
                    ((uintptr_t)conv_state & 7) == 0;
  const dim3 grid((s.channels() / (even ? 2 : 1) + s.H + 127) / 128, (tokens + RUN - 1) / RUN);
#define OMNIA_SSD_INPUTS_AS(KT, VC)                                                                                       \
  launch_pdl(ssd_inputs_kernel<T, O, KT, VC>, grid, dim3(128), 0, stream, (const T*)proj, stride, col0, s, taps, conv_bias, K, \
             conv_state, dt_bias, A_log, cu_seqlens, state_slots, num_seqs, tokens, (O*)rows, row_stride, at_x, at_b, at_c,  \
             pairs, pair_stride, log_decay)
#define OMNIA_SSD_INPUTS(KT)                 \
  do {                                       \
    if (even) OMNIA_SSD_INPUTS_AS(KT, 2);    \
    else OMNIA_SSD_INPUTS_AS(KT, 1);         \
  } while (0)
  if (K <= 4) OMNIA_SSD_INPUTS(4);
  else if (K <= 8) OMNIA_SSD_INPUTS(8);
  else OMNIA_SSD_INPUTS(MAX_TAPS);
#undef OMNIA_SSD_INPUTS
#undef OMNIA_SSD_INPUTS_AS
  return OMNIA_LAUNCH_RESULT();
}

bool sizes_ok(const Sizes& s, int K) {
  return s.H >= 1 && s.dv >= 1 && s.G >= 1 && s.N >= 1 && s.H % s.G == 0 && K >= 1 && K <= MAX_TAPS;
}

}  // namespace

// wide_rows != 0: float32 rows and (a, dt) pairs; else float16 rows and (log a, dt) pairs. Places and strides in elements of what they index; pairs must start on 8 bytes in every row.
extern "C" int omnia_ssd_inputs(const void* proj, int stride, int col0, int H, int dv, int G, int N, const float* taps,
                                const float* conv_bias, int K, const float* conv_state, const float* dt_bias,
                                const float* A_log, const int* cu_seqlens, const int* state_slots, int num_seqs, int tokens,
                                void* rows, int row_stride, int at_x, int at_b, int at_c, float* pairs, int pair_stride,
                                int wide_rows, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  const Sizes s{H, dv, G, N};
  if (!sizes_ok(s, K) || num_seqs < 1 || pair_stride % 2 || ((uintptr_t)pairs & 7)) return (int)cudaErrorInvalidValue;
  OMNIA_DISPATCH_DTYPE(dtype, {
    if (wide_rows)
      return launch_inputs<T, float>(proj, stride, col0, s, taps, conv_bias, K, conv_state, dt_bias, A_log, cu_seqlens,
                                     state_slots, num_seqs, tokens, rows, row_stride, at_x, at_b, at_c, pairs, pair_stride, 0, stream);
    return launch_inputs<T, __half>(proj, stride, col0, s, taps, conv_bias, K, conv_state, dt_bias, A_log, cu_seqlens, state_slots,
                               num_seqs, tokens, rows, row_stride, at_x, at_b, at_c, pairs, pair_stride, 1, stream);
  });
  return (int)cudaErrorInvalidValue;
}

// cols: value columns a block takes (a multiple of 4 where dv is one).
extern "C" int omnia_ssd_step(const void* proj, int stride, int col0, int H, int dv, int G, int N, int cols, const float* taps,
                              const float* conv_bias, int K, const float* conv_state, const float* dt_bias,
                              const float* A_log, const float* D, float* S_state, const int* cu_seqlens,
                              const int* state_slots, int num_seqs, float* y, int dtype, cudaStream_t stream) {
  if (num_seqs == 0) return 0;
  const Sizes s{H, dv, G, N};
  if (!sizes_ok(s, K) || cols < 1 || cols > dv) return (int)cudaErrorInvalidValue;
  const bool fours = dv % 4 == 0 && cols % 4 == 0 && ((uintptr_t)S_state & 15) == 0;
  // The teams' partial sums: a float for each thread's column, or more columns than threads.
  const size_t floats = 2 * (size_t)N + ((cols + 3) & ~3) + (cols > 1024 ? cols : 1024);
  const size_t smem = floats * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const dim3 grid(H * ((dv + cols - 1) / cols), num_seqs);
#define OMNIA_SSD_STEP(VEC)                                                                                               \
  do {                                                                                                                    \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(ssd_step_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize,       \
                                                 (int)smem) != cudaSuccess)                                               \
      return (int)cudaGetLastError();                                                                                     \
    launch_pdl(ssd_step_kernel<T, VEC>, grid, dim3(256), smem, stream, (const T*)proj, stride, col0, s, cols, taps, conv_bias, \
               K, conv_state, dt_bias, A_log, D, S_state, cu_seqlens, state_slots, y);                                     \
  } while (0)
  OMNIA_DISPATCH_DTYPE(dtype, {
    if (fours) OMNIA_SSD_STEP(4);
    else OMNIA_SSD_STEP(1);
  });
#undef OMNIA_SSD_STEP
  return OMNIA_LAUNCH_RESULT();
}

extern "C" int omnia_ssd_out(const float* y, const void* proj, int stride, int col0, int H, int dv, int G, int N,
                             int norm_groups, float eps, const float* norm_w, int K, float* conv_state,
                             const int* cu_seqlens, const int* state_slots, int num_seqs, int tokens, void* out, int dtype,
                             int out_dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  const Sizes s{H, dv, G, N};
  if (!sizes_ok(s, K) || norm_groups < 1 || s.inner() % norm_groups) return (int)cudaErrorInvalidValue;
  // One norm group in fours: from registers, as many threads as hold it. Anything else: through shared memory.
  const int quads = s.inner() / 4, whole_threads = ((quads + OUT_ITEMS - 1) / OUT_ITEMS + 31) / 32 * 32;
  const bool whole = norm_groups == 1 && s.inner() % 4 == 0 && whole_threads <= 1024 && stride % 4 == 0 && col0 % 4 == 0 &&
                     (((uintptr_t)y | (uintptr_t)proj | (uintptr_t)norm_w | (uintptr_t)out) & 15) == 0;
  const size_t smem = whole ? 0 : (size_t)s.inner() * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const int threads = whole ? (whole_threads < 128 ? 128 : whole_threads) : 256;
  const dim3 grid(tokens + (K > 1 ? num_seqs * ((s.channels() + threads - 1) / threads) : 0));
#define OMNIA_SSD_OUT(WHOLE)                                                                                                 \
  do {                                                                                                                       \
    if (smem > 47 * 1024 && cudaFuncSetAttribute(ssd_out_kernel<T, O, WHOLE>, cudaFuncAttributeMaxDynamicSharedMemorySize,         \
                                                 (int)smem) != cudaSuccess)                                                  \
      return (int)cudaGetLastError();                                                                                        \
    launch_pdl(ssd_out_kernel<T, O, WHOLE>, grid, dim3(threads), smem, stream, y, (const T*)proj, stride, col0, s, norm_groups,    \
               eps, norm_w, K, conv_state, cu_seqlens, state_slots, tokens, (O*)out);                                         \
  } while (0)
  // The output in the projected rows' type, or bfloat16 from float32 rows.
  if (dtype == OMNIA_F32 && out_dtype == OMNIA_BF16) {
    using T = float;
    using O = __nv_bfloat16;
    if (whole) OMNIA_SSD_OUT(true);
    else OMNIA_SSD_OUT(false);
  } else if (dtype == out_dtype) {
    OMNIA_DISPATCH_DTYPE(dtype, {
      using O = T;
      if (whole) OMNIA_SSD_OUT(true);
      else OMNIA_SSD_OUT(false);
    });
  } else {
    return (int)cudaErrorInvalidValue;
  }
#undef OMNIA_SSD_OUT
  return OMNIA_LAUNCH_RESULT();
}
