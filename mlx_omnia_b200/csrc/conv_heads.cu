// What a token's projected row becomes before an attention whose projections pass a short causal
// convolution over time and whose heads may have several softmax maps. Per channel of q, k
// and v a bias, then y_t = sum_j taps[K - 1 - j] in_(t - j) over the request's inputs (zeros ahead of its
// start; inputs before this step come from the request's state slot), then on q and k the rotation of
// the first `rot` dims of every map of every head. A head has `maps` maps of `dk` dims each. A head of
// the cache is `d` wide: a key row is the head's maps side by side, a value row the head's values, both
// filled up with zeros; and a query row (head, map) is zero but for its own map's dims. A query row's
// product with a key row is then its own map's score, every map of a head shares one key row and one
// value row, and the attention kernels see ordinary grouped-query attention: heads * maps query heads
// of d over kv_heads key/value heads.
//
// Float32 from the projected row on; rounded once where a row is stored.
#include "common.cuh"

#define CONV_MAX_TAPS 16

namespace {

template <typename T>
struct Pair {
  T a, b;
};

struct ConvArgs {
  const void* proj;        // [tokens, stride] T; channels from col0 on: q, then k, then v
  int stride, col0;
  const float* bias;       // [channels] or null
  const float* taps;       // [K][channels], the last row the current token's
  int K, channels;
  float* state;            // [slots][K - 1][channels], oldest first: a request's last inputs
  const int* cu_seqlens;
  const int* state_slots;
  int num_seqs;
  int heads, kv_heads, maps, dk, dv, d;  // kv_heads 0: queries only
  const float* inv_freq;   // [rot / 2] or null
  int rot, half_pairs;
  float amount;            // multiplies cosine and sine
  const int* positions;
  const long long* slot_mapping;
  void* q_out;             // [tokens, heads * maps, d]
  void* k_pages;           // key row: k_pages + page * page_stride + (head * page_size + offset) * d
  void* v_pages;
  long long page_stride;
  int page_size;
  long long num_slots;
  int tokens, advance;     // advance: every request brings one token and its state is moved on here
  int* err;
};

// The convolution's value of channel c for token t of a request that began at `begin` in this step.
template <typename T>
__device__ __forceinline__ float conv_at(const ConvArgs& p, const float* state, int t, int begin, int c) {
  const T* col = (const T*)p.proj + p.col0 + c;
  const float bias = p.bias ? p.bias[c] : 0.f;
  float acc = 0.f;
  for (int j = 0; j < p.K; ++j) {
    const int src = t - j;
    const float x = src >= begin ? to_f32(col[(size_t)src * p.stride]) + bias
                                 : state[(size_t)(p.K - 1 - (begin - src)) * p.channels + c];
    acc = fmaf(p.taps[(size_t)(p.K - 1 - j) * p.channels + c], x, acc);
  }
  return acc;
}

// Two neighbouring channels at once. With `advance` their inputs in the state are moved on by the token.
template <typename T>
__device__ __forceinline__ float2 conv_pair_at(const ConvArgs& p, float* state, int t, int begin, int c) {
  const T* col = (const T*)p.proj + p.col0 + c;
  const float2 bias = p.bias ? *reinterpret_cast<const float2*>(p.bias + c) : make_float2(0.f, 0.f);
  float2 acc = make_float2(0.f, 0.f), now = make_float2(0.f, 0.f);
#pragma unroll 4
  for (int j = 0; j < p.K; ++j) {
    const int src = t - j;
    float2 x;
    if (src >= begin) {
      const Pair<T> raw = *reinterpret_cast<const Pair<T>*>(col + (size_t)src * p.stride);
      x = make_float2(to_f32(raw.a) + bias.x, to_f32(raw.b) + bias.y);
    } else {
      x = *reinterpret_cast<const float2*>(state + (size_t)(p.K - 1 - (begin - src)) * p.channels + c);
    }
    if (j == 0) now = x;
    const float2 w = __ldg(reinterpret_cast<const float2*>(p.taps + (size_t)(p.K - 1 - j) * p.channels + c));
    acc.x = fmaf(w.x, x.x, acc.x), acc.y = fmaf(w.y, x.y, acc.y);
  }
  if (p.advance && p.K > 1) {
    for (int i = 0; i + 1 < p.K - 1; ++i)
      *reinterpret_cast<float2*>(state + (size_t)i * p.channels + c) =
          *reinterpret_cast<const float2*>(state + (size_t)(i + 1) * p.channels + c);
    *reinterpret_cast<float2*>(state + (size_t)(p.K - 2) * p.channels + c) = now;
  }
  return acc;
}

// grid (tokens, parts of a row's outputs). PAIRS: a thread makes two neighbouring elements (all widths
// even, pairs of neighbours turn together); otherwise one, and works its partner's value out as well.
template <typename T, bool PAIRS>
__global__ void __launch_bounds__(256) conv_heads_prepare_kernel(const ConvArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float cos_s[128], sin_s[128];
  const int t = blockIdx.x;
  int lo = 0, hi = p.num_seqs;  // the token's request: the last whose tokens begin at or before t
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_seqlens[mid] <= t) lo = mid;
    else hi = mid;
  }
  const int begin = p.cu_seqlens[lo];
  float* state = p.state + (size_t)p.state_slots[lo] * (p.K - 1) * p.channels;
  const int half = p.inv_freq ? p.rot / 2 : 0;
  const float pos = (float)p.positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * p.inv_freq[i], &s, &c);
    cos_s[i] = c * p.amount, sin_s[i] = s * p.amount;
  }
  __syncthreads();
  long long slot = -1;
  if (p.kv_heads > 0) {
    slot = p.slot_mapping[t];
    if (slot >= p.num_slots) {
      if (threadIdx.x == 0) atomicOr(p.err, OMNIA_ERR_SLOT);
      slot = -1;
    }
  }
  const long long page = slot >= 0 ? slot / p.page_size : 0, off = slot >= 0 ? slot % p.page_size : 0;
  const int q_outs = p.heads * p.maps * p.d, k_outs = p.kv_heads * p.d, outs = q_outs + 2 * k_outs;
  const int k_chan = p.heads * p.maps * p.dk, v_chan = k_chan + p.kv_heads * p.maps * p.dk;
  constexpr int N = PAIRS ? 2 : 1;
  for (int o = (blockIdx.y * blockDim.x + threadIdx.x) * N; o < outs; o += gridDim.y * blockDim.x * N) {
    // Which channel (if any) the element holds, its dim within a map, and where it goes.
    int c = -1, dim = -1;
    T* dst;
    if (o < q_outs) {
      const int row = o / p.d, e = o - row * p.d, i = e - (row % p.maps) * p.dk;
      if (i >= 0 && i < p.dk) c = row * p.dk + i, dim = i;
      dst = (T*)p.q_out + (size_t)t * q_outs + o;
    } else {
      const bool value = o >= q_outs + k_outs;
      const int x = o - q_outs - (value ? k_outs : 0), head = x / p.d, e = x - head * p.d;
      if (value) {
        if (e < p.dv) c = v_chan + head * p.dv + e;
      } else if (e < p.maps * p.dk) {
        c = k_chan + head * p.maps * p.dk + e, dim = e % p.dk;
      }
      dst = (T*)(value ? p.v_pages : p.k_pages) + page * p.page_stride + ((long long)head * p.page_size + off) * p.d + e;
    }
    const bool store = o < q_outs || slot >= 0;
    if (PAIRS) {
      float2 y = make_float2(0.f, 0.f);
      if (c >= 0) {
        y = conv_pair_at<T>(p, state, t, begin, c);
        if (dim >= 0 && dim < 2 * half) {
          const float co = cos_s[dim >> 1], si = sin_s[dim >> 1];
          y = make_float2(y.x * co - y.y * si, y.y * co + y.x * si);
        }
      }
      if (store) *reinterpret_cast<Pair<T>*>(dst) = Pair<T>{from_f32<T>(y.x), from_f32<T>(y.y)};
    } else {
      float y = 0.f;
      if (c >= 0) {
        y = conv_at<T>(p, state, t, begin, c);
        if (dim >= 0 && dim < 2 * half) {
          const bool second = p.half_pairs ? dim >= half : (dim & 1);
          const int i = p.half_pairs ? dim % half : dim >> 1;
          const int away = p.half_pairs ? half : 1;
          const float other = conv_at<T>(p, state, t, begin, second ? c - away : c + away);
          y = second ? y * cos_s[i] + other * sin_s[i] : y * cos_s[i] - other * sin_s[i];
        }
      }
      if (store) *dst = from_f32<T>(y);
    }
  }
}

// Many tokens: a thread owns eight neighbouring elements of the outputs and walks a run of tokens with the
// last K - 1 inputs in registers, so an input is read once; what the elements are and where they go is worked
// out once a run. grid (runs of RUN tokens, ceil(outputs / 8 / threads)); every width in eights.
constexpr int RUN = 16, AHEAD = 4;  // AHEAD tokens' inputs are asked for together
template <typename T>
struct alignas(16) Octet {
  T v[8];
};

template <typename T, int K>
__global__ void __launch_bounds__(256) conv_heads_runs_kernel(const ConvArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ float2 turn_s[];  // [RUN][half] (cos, sin)
  __shared__ long long slot_s[RUN];
  const int t0 = blockIdx.x * RUN, t1 = min(p.tokens, t0 + RUN);
  const int half = p.inv_freq ? p.rot / 2 : 0;
  for (int i = threadIdx.x; i < (t1 - t0) * half; i += blockDim.x) {
    float s, c;
    sincosf((float)p.positions[t0 + i / half] * p.inv_freq[i % half], &s, &c);
    turn_s[i] = make_float2(c * p.amount, s * p.amount);
  }
  if (threadIdx.x < t1 - t0) {
    long long slot = p.kv_heads > 0 ? p.slot_mapping[t0 + threadIdx.x] : -1;
    if (slot >= p.num_slots) {
      if (blockIdx.y == 0) atomicOr(p.err, OMNIA_ERR_SLOT);
      slot = -1;
    }
    slot_s[threadIdx.x] = slot;
  }
  __syncthreads();
  const int q_outs = p.heads * p.maps * p.d, k_outs = p.kv_heads * p.d, outs = q_outs + 2 * k_outs;
  const int k_chan = p.heads * p.maps * p.dk, v_chan = k_chan + p.kv_heads * p.maps * p.dk;
  const int o = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (o >= outs) return;
  int c = -1, dim = -1, head = 0, e = 0;
  const bool query = o < q_outs, value = o >= q_outs + k_outs;
  if (query) {
    const int row = o / p.d, i = o - row * p.d - (row % p.maps) * p.dk;
    if (i >= 0 && i < p.dk) c = row * p.dk + i, dim = i;
  } else {
    const int x = o - q_outs - (value ? k_outs : 0);
    head = x / p.d, e = x - head * p.d;
    if (value) {
      if (e < p.dv) c = v_chan + head * p.dv + e;
    } else if (e < p.maps * p.dk) {
      c = k_chan + head * p.maps * p.dk + e, dim = e % p.dk;
    }
  }
  T* pages = (T*)(value ? p.v_pages : p.k_pages);
  auto store = [&](int t, const Octet<T>& y) {
    T* dst;
    if (query) {
      dst = (T*)p.q_out + (size_t)t * q_outs + o;
    } else {
      const long long slot = slot_s[t - t0];
      if (slot < 0) return;
      dst = pages + (slot / p.page_size) * p.page_stride + ((long long)head * p.page_size + slot % p.page_size) * p.d + e;
    }
    *reinterpret_cast<Octet<T>*>(dst) = y;
  };
  if (c < 0) {
    Octet<T> zero;
#pragma unroll
    for (int i = 0; i < 8; ++i) zero.v[i] = from_f32<T>(0.f);
    for (int t = t0; t < t1; ++t) store(t, zero);
    return;
  }
  float w[K][8], bias[8], before[K > 1 ? K - 1 : 1][8];  // before[j]: the input j + 1 tokens back
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    bias[i] = p.bias ? p.bias[c + i] : 0.f;
#pragma unroll
    for (int j = 0; j < K; ++j) w[j][i] = p.taps[(size_t)(K - 1 - j) * p.channels + c + i];
  }
  const T* col = (const T*)p.proj + p.col0 + c;
  int lo = 0, hi = p.num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.cu_seqlens[mid] <= t0) lo = mid;
    else hi = mid;
  }
  int end = t0;  // the first token of the run finds its request's inputs like the first of any request
  Octet<T> raw[AHEAD];
  for (int t = t0; t < t1; ++t) {
    if ((t - t0) % AHEAD == 0) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        raw[i] = *reinterpret_cast<const Octet<T>*>(col + (size_t)min(t + i, t1 - 1) * p.stride);
    }
    if (t >= end) {
      while (p.cu_seqlens[lo + 1] <= t) ++lo;
      end = p.cu_seqlens[lo + 1];
      const int begin = p.cu_seqlens[lo];
      const float* state = p.state + (size_t)p.state_slots[lo] * (K - 1) * p.channels + c;
#pragma unroll
      for (int j = 0; j < K - 1; ++j) {
        const int src = t - 1 - j;
#pragma unroll
        for (int i = 0; i < 8; ++i)
          before[j][i] = src >= begin ? to_f32(col[(size_t)src * p.stride + i]) + bias[i]
                                      : state[(size_t)(K - 1 - (begin - src)) * p.channels + i];
      }
    }
    float y[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float x = to_f32(raw[0].v[i]) + bias[i];
      y[i] = w[0][i] * x;
#pragma unroll
      for (int j = 1; j < K; ++j) y[i] = fmaf(w[j][i], before[j - 1][i], y[i]);
#pragma unroll
      for (int j = K - 2; j > 0; --j) before[j][i] = before[j - 1][i];
      if (K > 1) before[0][i] = x;
    }
    Octet<T> out;
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      if (dim >= 0 && dim + i < 2 * half) {
        const float2 turn = turn_s[(t - t0) * half + ((dim + i) >> 1)];
        const float u = y[i] * turn.x - y[i + 1] * turn.y;
        y[i + 1] = y[i + 1] * turn.x + y[i] * turn.y;
        y[i] = u;
      }
      out.v[i] = from_f32<T>(y[i]), out.v[i + 1] = from_f32<T>(y[i + 1]);
    }
    store(t, out);
#pragma unroll
    for (int i = 0; i + 1 < AHEAD; ++i) raw[i] = raw[i + 1];
  }
}

// A request's last K - 1 inputs, oldest first, after this step. grid (ceil(channels / 128), requests)
template <typename T>
__global__ void conv_heads_advance_kernel(const ConvArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
  const int begin = p.cu_seqlens[seq], n = p.cu_seqlens[seq + 1] - begin;
  if (c >= p.channels || n <= 0) return;
  float* state = p.state + (size_t)p.state_slots[seq] * (p.K - 1) * p.channels + c;
  const float bias = p.bias ? p.bias[c] : 0.f;
  float keep[CONV_MAX_TAPS];
#pragma unroll
  for (int i = 0; i < CONV_MAX_TAPS; ++i) {
    if (i >= p.K - 1) break;
    const int at = n - (p.K - 1) + i;  // among this step's tokens; negative: still of the old state
    keep[i] = at >= 0 ? to_f32(((const T*)p.proj)[(size_t)(begin + at) * p.stride + p.col0 + c]) + bias
                      : state[(size_t)(i + n) * p.channels];
  }
#pragma unroll
  for (int i = 0; i < CONV_MAX_TAPS; ++i) {
    if (i >= p.K - 1) break;
    state[(size_t)i * p.channels] = keep[i];
  }
}

}  // namespace

extern "C" int omnia_conv_heads_prepare(const void* proj, int stride, int col0, const float* bias, const float* taps, int K,
                                        int channels, float* state, const int* cu_seqlens, const int* state_slots,
                                        int num_seqs, int heads, int kv_heads, int maps, int dk, int dv, int d,
                                        const float* inv_freq, int rot, int half_pairs, float amount, const int* positions,
                                        const long long* slot_mapping, void* q_out, void* k_pages, void* v_pages,
                                        long long page_stride, int page_size, long long num_slots, int tokens, int single,
                                        int dtype, int* err, cudaStream_t stream) {
  if (tokens == 0) return 0;
  if (K < 1 || K > CONV_MAX_TAPS || maps < 1 || maps * dk > d || dv > d || rot > dk || rot > 256 || (rot & 1) || num_seqs < 1 ||
      heads < 1 || channels != heads * maps * dk + kv_heads * (maps * dk + dv))
    return (int)cudaErrorInvalidValue;
  ConvArgs p;
  p.proj = proj, p.stride = stride, p.col0 = col0, p.bias = bias, p.taps = taps, p.K = K, p.channels = channels;
  p.state = state, p.cu_seqlens = cu_seqlens, p.state_slots = state_slots, p.num_seqs = num_seqs;
  p.heads = heads, p.kv_heads = kv_heads, p.maps = maps, p.dk = dk, p.dv = dv, p.d = d;
  p.inv_freq = inv_freq, p.rot = rot, p.half_pairs = half_pairs, p.amount = amount, p.positions = positions;
  p.slot_mapping = slot_mapping, p.q_out = q_out, p.k_pages = k_pages, p.v_pages = v_pages, p.page_stride = page_stride;
  p.page_size = page_size, p.num_slots = num_slots, p.tokens = tokens, p.err = err;
  const size_t pair_bytes = dtype == OMNIA_BF16 ? 4 : 8;
  const bool pairs = !half_pairs && dk % 2 == 0 && dv % 2 == 0 && d % 2 == 0 && stride % 2 == 0 && col0 % 2 == 0 &&
                     page_stride % 2 == 0 &&
                     (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & (pair_bytes - 1)) == 0 &&
                     (((uintptr_t)bias | (uintptr_t)taps | (uintptr_t)state) & 7) == 0;
  p.advance = single && pairs;
  const int outs = (heads * maps + 2 * kv_heads) * d, per = 256 * (pairs ? 2 : 1);
  int parts = (outs + per - 1) / per;
  const int enough = (4 * omnia_sm_count() + tokens - 1) / tokens;  // many tokens: fewer, longer blocks
  if (parts > enough) parts = enough;
  const dim3 grid(tokens, parts);
  const bool runs = pairs && !single && tokens >= 2 * RUN && K <= 4 && dk % 8 == 0 && dv % 8 == 0 && d % 8 == 0 && stride % 8 == 0 &&
                    col0 % 8 == 0 && page_stride % 8 == 0 &&
                    (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15) == 0;
  const size_t turns = inv_freq ? (size_t)RUN * (rot / 2) * sizeof(float2) : 0;
  const dim3 run_grid((tokens + RUN - 1) / RUN, (outs / 8 + 255) / 256);
  OMNIA_DISPATCH_DTYPE(dtype, {
    if (runs && K == 1) launch_pdl(conv_heads_runs_kernel<T, 1>, run_grid, dim3(256), turns, stream, p);
    else if (runs && K == 2) launch_pdl(conv_heads_runs_kernel<T, 2>, run_grid, dim3(256), turns, stream, p);
    else if (runs && K == 3) launch_pdl(conv_heads_runs_kernel<T, 3>, run_grid, dim3(256), turns, stream, p);
    else if (runs && K == 4) launch_pdl(conv_heads_runs_kernel<T, 4>, run_grid, dim3(256), turns, stream, p);
    else if (pairs) launch_pdl(conv_heads_prepare_kernel<T, true>, grid, dim3(256), 0, stream, p);
    else launch_pdl(conv_heads_prepare_kernel<T, false>, grid, dim3(256), 0, stream, p);
  });
  if (!p.advance && K > 1) {
    const int code = OMNIA_LAUNCH_RESULT();
    if (code != 0) return code;
    OMNIA_DISPATCH_DTYPE(dtype, (launch_pdl(conv_heads_advance_kernel<T>, dim3((channels + 127) / 128, num_seqs), dim3(128), 0,
                                            stream, p)));
  }
  return OMNIA_LAUNCH_RESULT();
}
