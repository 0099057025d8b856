// Paged causal attention for any batch shape, head sizes (<= 512; keys and values may differ in
// width), page size and element type: the kernel of the 32-bit path, and of sizes the tiled kernels
// refuse. A window may keep the request's first `keep_first` positions visible for good, and the
// softmax's denominator may hold one more term exp(sink[head]) that has no key and no value.
// With `chunk` > 0 a query sees the keys of its own run of `chunk` positions only (runs counted from
// position 0 of the request); with `maps` 2 two neighbouring query heads are the two maps of one head of
// differential attention, and their difference is written (see MapDifference); with `softcap` > 0 a scaled score s becomes softcap * tanh(s / softcap).
//
// One warp per (token, query head). Keys are visited in chunks of 32 starting at the
// lowest visible position; in a chunk every lane scores one key (a full dot product in
// float32), the chunk's softmax statistics are merged online, and for the values every
// lane owns the output dims lane, lane+32, ... The order of all additions depends only on
// the token's own position and window, never on how the batch was cut.
#include "common.cuh"

// MOST: a multiple of 32 that neither width exceeds (a lane holds MOST / 32 of the output's dims).
template <typename T, int MOST>
__global__ void paged_attention_generic_kernel(
    const T* __restrict__ q,                // [tokens, nq, d]
    const T* __restrict__ k_pages,          // key row: k_pages + page * page_stride + (kvh * page_size + off) * d
    const T* __restrict__ v_pages,          // value row: v_pages + page * page_stride + (kvh * page_size + off) * dv
    long long page_stride,
    const int* __restrict__ block_table,    // [num_seqs, max_pages]
    const int* __restrict__ cu_seqlens,     // [num_seqs + 1]
    const int* __restrict__ positions,      // [tokens]
    const T* __restrict__ gate, int gate_stride,  // gate[t * gate_stride + h * d + i], or null
    T* __restrict__ out,                    // [tokens, nq * dv]
    const float* __restrict__ sink,         // [nq] or null
    int num_seqs, int max_pages, int num_pages, int nq, int nkv, int d, int dv, int page_size,
    int window, int keep_first, float scale, int chunk, float softcap, int maps, const MapDifference difference,
    int* err) {
  constexpr int ACC = MOST / 32;
  __shared__ float qs[4][MOST];
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * 4 + warp;
  if (head >= nq) return;
  // The request this token belongs to: the last s with cu_seqlens[s] <= t.
  int lo_s = 0, hi_s = num_seqs - 1;
  while (lo_s < hi_s) {
    const int mid = (lo_s + hi_s + 1) >> 1;
    if (cu_seqlens[mid] <= t) lo_s = mid; else hi_s = mid - 1;
  }
  const int seq = lo_s;
  const int pos = positions[t];
  const int kvh = head / (nq / nkv);
  int first = window > 0 ? max(0, pos - window + 1) : 0;
  if (chunk > 0) first = max(first, pos - pos % chunk);

  const T* qrow = q + ((size_t)t * nq + head) * d;
  for (int i = lane; i < d; i += 32) qs[warp][i] = to_f32(qrow[i]) * scale;
  __syncwarp();

  float m = -INFINITY, l = 0.f;
  float acc[ACC];
#pragma unroll
  for (int k = 0; k < ACC; ++k) acc[k] = 0.f;
  const int* table = block_table + (size_t)seq * max_pages;

  // Two runs of keys: the kept first positions below the window, then the window itself.
  const int kept = min(keep_first, first);
  for (int run = 0; run < 2; ++run) {
  const int run_lo = run == 0 ? 0 : first, run_hi = run == 0 ? kept - 1 : pos;
  for (int base = run_lo; base <= run_hi; base += 32) {
    const int j = base + lane;
    float s = -INFINITY;
    long long vrow = -1;
    if (j <= run_hi) {
      const int page = table[j / page_size];
      if (page < 0 || page >= num_pages) {
        atomicOr(err, OMNIA_ERR_PAGE);
      } else {
        const long long in_page = (long long)kvh * page_size + j % page_size;
        vrow = (long long)page * page_stride + in_page * dv;
        const T* kp = k_pages + (long long)page * page_stride + in_page * d;
        float dot = 0.f;
        for (int i = 0; i < d; ++i) dot += qs[warp][i] * to_f32(kp[i]);
        s = softcap > 0.f ? softcap * tanhf(dot / softcap) : dot;
      }
    }
    const float m_new = fmaxf(m, warp_max(s));
    if (m_new == -INFINITY) continue;
    const float alpha = expf(m - m_new);
    const float p = s == -INFINITY ? 0.f : expf(s - m_new);
    l = l * alpha + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int k = 0; k < ACC; ++k) acc[k] *= alpha;
    const int count = min(32, run_hi - base + 1);
    for (int jj = 0; jj < count; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const long long vr = __shfl_sync(0xffffffffu, vrow, jj);
      if (vr < 0) continue;
      const T* vp = v_pages + vr;
#pragma unroll
      for (int k = 0; k < ACC; ++k) {
        const int i = lane + 32 * k;
        if (i < dv) acc[k] += pj * to_f32(vp[i]);
      }
    }
  }
  }
  if (sink != nullptr) {  // one more term of the denominator, with no value: the sum only
    const float z = sink[head];
    const float m_new = fmaxf(m, z);
    const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * alpha + expf(z - m_new);
#pragma unroll
    for (int k = 0; k < ACC; ++k) acc[k] *= alpha;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  if (maps == 2) {
    // The odd warp of a pair hands its map over (nq is even, so the pair is there or gone together).
    if (warp & 1)
#pragma unroll
      for (int k = 0; k < ACC; ++k) qs[warp][lane + 32 * k] = acc[k] * inv;
    __syncthreads();
    if (warp & 1) return;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < ACC; ++k) {
      acc[k] = lane + 32 * k < difference.dv ? acc[k] * inv - difference.lambda * qs[warp + 1][lane + 32 * k] : 0.f;
      ss += acc[k] * acc[k];
    }
    const float f = rsqrtf(warp_sum(ss) / (float)difference.dv + difference.eps) * difference.factor;
    T* drow = out + ((size_t)t * (nq / 2) + head / 2) * difference.dv;
#pragma unroll
    for (int k = 0; k < ACC; ++k)
      if (lane + 32 * k < difference.dv) drow[lane + 32 * k] = from_f32<T>(acc[k] * f);
    return;
  }
  T* orow = out + ((size_t)t * nq + head) * dv;
#pragma unroll
  for (int k = 0; k < ACC; ++k) {
    const int i = lane + 32 * k;
    if (i >= dv) continue;
    float v = acc[k] * inv;
    if (gate != nullptr) {
      const float g = to_f32(gate[(size_t)t * gate_stride + (size_t)head * dv + i]);
      v *= 1.f / (1.f + expf(-g));
    }
    orow[i] = from_f32<T>(v);
  }
}

extern "C" int omnia_paged_attention_generic(
    const void* q, const void* k_pages, const void* v_pages, long long page_stride, const int* block_table,
    const int* cu_seqlens, const int* positions, const void* gate, int gate_stride, void* out, const float* sink,
    int tokens, int num_seqs, int max_pages, int num_pages, int nq, int nkv, int d, int dv, int page_size, int window,
    int keep_first, float scale, int chunk, float softcap, int maps, float lambda, float diff_eps, float diff_factor, int out_dv,
    int dtype, int* err, cudaStream_t stream) {
  if (tokens == 0) return 0;
  if (maps < 1 || maps > 2 || (maps == 2 && (nq % 2 || gate != nullptr || out_dv < 1 || out_dv > dv)))
    return (int)cudaErrorInvalidValue;
  const MapDifference difference{lambda, diff_eps, diff_factor, out_dv};
  if (d > 512 || dv > 512 || nkv <= 0 || nq % nkv != 0 || keep_first < 0 || (keep_first > 0 && window <= 0) ||
      chunk < 0 || softcap < 0.f || (chunk > 0 && keep_first > 0))
    return (int)cudaErrorInvalidValue;
  dim3 grid(tokens, (nq + 3) / 4);
  OMNIA_DISPATCH_DTYPE(dtype, {
    if (d <= 256 && dv <= 256)
      paged_attention_generic_kernel<T, 256><<<grid, 128, 0, stream>>>(
          (const T*)q, (const T*)k_pages, (const T*)v_pages, page_stride, block_table, cu_seqlens, positions, (const T*)gate,
          gate_stride, (T*)out, sink, num_seqs, max_pages, num_pages, nq, nkv, d, dv, page_size, window, keep_first, scale,
          chunk, softcap, maps, difference, err);
    else
      paged_attention_generic_kernel<T, 512><<<grid, 128, 0, stream>>>(
          (const T*)q, (const T*)k_pages, (const T*)v_pages, page_stride, block_table, cu_seqlens, positions, (const T*)gate,
          gate_stride, (T*)out, sink, num_seqs, max_pages, num_pages, nq, nkv, d, dv, page_size, window, keep_first, scale,
          chunk, softcap, maps, difference, err);
  });
  return OMNIA_LAUNCH_RESULT();
}
