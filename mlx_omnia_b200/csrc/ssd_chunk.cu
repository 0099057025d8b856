// The state-space recurrence of ssd.cu over a portion's tokens, a chunk of SSD_L tokens at a time on the tensor
// cores. With l_t the running sum of log a within a chunk, S the state ahead of it:
//
//   y_t = e^(l_t) S^T C_t + sum_(s <= t) e^(l_t - l_s) dt_s (C_t . B_s) x_s + D x_t
//   S  <- e^(l_last) S + sum_s e^(l_last - l_s) dt_s B_s x_s^T
//
// Four products a chunk: C B^T, its weighted lower triangle times x, C S, and B^T times the weighted x. B, C and x
// are float16 (three bits more than bfloat16 would keep of what the convolution makes in float32; their size needs
// no wider exponent); everything else that enters a product (the weighted triangle, the weighted x, the state) is
// split into the sum of two float16 numbers, 22 bits of mantissa, the state and the triangle after a scaling by a
// power of two that keeps their largest entries in range. Sums, decays and the carried state are float32. All exponents are of differences
// that are at most zero.
//
// A block owns SSD_COLS value columns of one head of one request and walks its chunks in order; a column of S needs
// no other column. Warp w has 16 of the chunk's tokens for the first three products (the tokens dealt so that the two
// warps of a scheduler have equal shares of the triangle) and 16 of the state's rows for the last, whose float32
// values never leave its registers; the other warps read them as pairs of float16 from shared memory. The next
// chunk's B, C, x and step sizes come in by asynchronous copies meanwhile.
//
// Compiled per state size and columns: -DSSD_N=<N> (a multiple of 16), -DSSD_COLS=<16 or 32>.
#include "common.cuh"

#include <cuda_fp16.h>

#ifndef SSD_N
#define SSD_N 128
#endif
#ifndef SSD_COLS
#define SSD_COLS 32
#endif

namespace {

typedef __half f16;

constexpr int N = SSD_N, COLS = SSD_COLS;
static_assert(N % 16 == 0 && (COLS == 16 || COLS == 32), "sizes the tensor cores' tiles fit");
constexpr int NROW = N + 8, XROW = COLS + 8;  // rows of shared memory in elements: an odd number of 16-byte pieces

constexpr size_t smem_bytes(int L) {
  return sizeof(f16) * (2 * (size_t)L * (2 * NROW + XROW) + 2 * N * XROW + 2 * L * XROW) + 2 * sizeof(float2) * L +
         3 * sizeof(float) * L + sizeof(float) * 8;
}
constexpr int L = N <= 128 && smem_bytes(128) <= 227 * 1024 ? 128 : 64;
static_assert(smem_bytes(L) <= 227 * 1024, "a chunk fits shared memory");
constexpr int WARPS = L / 16, THREADS = 32 * WARPS;
// The state's tiles of 16 rows x 8 columns: MPW row tiles a warp, or several warps to a row tile.
constexpr int MT = N / 16, MPW = (MT + WARPS - 1) / WARPS;
constexpr int share(int warps_a_tile) {
  return warps_a_tile >= 4 && COLS >= 32 ? 4 : warps_a_tile >= 2 ? 2 : 1;
}
constexpr int CW = share(WARPS / MT);  // warps that share a row tile's columns
constexpr int NT = COLS / 8, NTW = NT / CW;

__device__ __forceinline__ uint32_t shared_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy16(const void* smem, const void* gmem, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(shared_address(smem)), "l"(gmem), "r"(valid ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void copy8(const void* smem, const void* gmem, bool valid) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;\n" ::"r"(shared_address(smem)), "l"(gmem), "r"(valid ? 8 : 0)
               : "memory");
}
__device__ __forceinline__ void ldmatrix(uint32_t* r, const f16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(shared_address(p)));
}
__device__ __forceinline__ void ldmatrix_t(uint32_t* r, const f16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(shared_address(p)));
}
__device__ __forceinline__ void mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (u, v) as two pairs of float16 whose sum has 22 bits of mantissa (numbers beyond float16's range are held at its end).
__device__ __forceinline__ void split(float u, float v, uint32_t& hi, uint32_t& lo) {
  u = u > 65504.f ? 65504.f : u < -65504.f ? -65504.f : u;
  v = v > 65504.f ? 65504.f : v < -65504.f ? -65504.f : v;
  const __half2 h = __floats2half2_rn(u, v);
  const __half2 l = __floats2half2_rn(u - __low2float(h), v - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float power_of_two(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}

// rows: bfloat16 [tokens, row_stride], x, B and C at their places; pairs: (log a, dt) [tokens, H]; y: float32 [tokens, H * dv].
__global__ void __launch_bounds__(THREADS, 1)
ssd_chunk_kernel(const f16* __restrict__ rows, int row_stride, int at_x, int at_b, int at_c, const float2* __restrict__ pairs,
                 int H, int G, int dv, const float* __restrict__ D, float* __restrict__ S_state,
                 const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, float* __restrict__ y) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  f16* stage0 = reinterpret_cast<f16*>(chunk_smem);  // two stages of [L][NROW] B, [L][NROW] C, [L][XROW] x
  constexpr int STAGE = L * (2 * NROW + XROW);
  f16* Sh = stage0 + 2 * STAGE;  // [N][XROW] the state's upper halves, then the lower ones
  f16* Sl = Sh + N * XROW;
  f16* Wh = Sl + N * XROW;    // [L][XROW] the weighted x
  f16* Wl = Wh + L * XROW;
  float2* ps = reinterpret_cast<float2*>(Wl + L * XROW);  // [2][L] (log a, dt)
  float* cum = reinterpret_cast<float*>(ps + 2 * L);  // running sum of log2 a
  float* dts = cum + L;
  float* wgt = dts + L;                              // what a token's x is weighted with on its way into the state
  float* peaks = wgt + L;                            // each warp's largest entry of the state

  const int parts = dv / COLS, head = blockIdx.x / parts, col0 = (blockIdx.x % parts) * COLS, seq = blockIdx.y;
  const int begin = cu_seqlens[seq], end = cu_seqlens[seq + 1];
  if (end <= begin) return;
  const int group = head / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const float skip = D[head];
  const f16* b_rows = rows + at_b + group * N;
  const f16* c_rows = rows + at_c + group * N;
  const f16* x_rows = rows + at_x + head * dv + col0;

  auto fetch = [&](int t0, int n, int b) {
    f16* Bd = stage0 + b * STAGE;
    f16* Cd = Bd + L * NROW;
    f16* Xd = Cd + L * NROW;
    const int fill = min(L, (n + 31) & ~31);  // rows past the portion's end are zeros, up to a whole block of keys
    for (int i = tid; i < fill * (N / 8); i += THREADS) {
      const int r = i / (N / 8), c = (i % (N / 8)) * 8;
      const size_t from = (size_t)(t0 + (r < n ? r : 0)) * row_stride + c;
      copy16(Bd + r * NROW + c, b_rows + from, r < n);
      copy16(Cd + r * NROW + c, c_rows + from, r < n);
    }
    for (int i = tid; i < fill * (COLS / 8); i += THREADS) {
      const int r = i / (COLS / 8), c = (i % (COLS / 8)) * 8;
      copy16(Xd + r * XROW + c, x_rows + (size_t)(t0 + (r < n ? r : 0)) * row_stride + c, r < n);
    }
    for (int r = tid; r < L; r += THREADS) copy8(ps + b * L + r, pairs + (size_t)(t0 + (r < n ? r : 0)) * H + head, r < n);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };

  // This warp's part of the state: row tiles m0, m0 + 1, ..., columns from c0.
  const int m0 = (warp / CW) * MPW, c0 = (warp % CW) * NTW * 8;
  float S[MPW][NTW][4];
  float* mine = S_state + ((size_t)state_slots[seq] * H + head) * N * dv + col0 + c0 + 2 * t4;
#pragma unroll
  for (int m = 0; m < MPW; ++m)
#pragma unroll
    for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
      for (int side = 0; side < 2; ++side) {
        float2 v = make_float2(0.f, 0.f);
        if (m0 + m < MT) v = *reinterpret_cast<const float2*>(mine + (size_t)((m0 + m) * 16 + g + 8 * side) * dv + nt * 8);
        S[m][nt][2 * side] = v.x, S[m][nt][2 * side + 1] = v.y;
      }

  auto note_peak = [&]() {
    float peak = 0.f;
#pragma unroll
    for (int m = 0; m < MPW; ++m)
#pragma unroll
      for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) peak = fmaxf(peak, fabsf(S[m][nt][e]));
    peak = warp_max(peak);
    if (lane == 0) peaks[warp] = peak;
  };
  note_peak();
  const int tile = WARPS == 8 && warp >= 4 ? 11 - warp : warp, row0 = tile * 16;
  const int chunks = (end - begin + L - 1) / L;
  fetch(begin, min(L, end - begin), 0);
  for (int c = 0; c < chunks; ++c) {
    const int t0 = begin + c * L, n = min(L, end - t0), b = c & 1;
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();  // the chunk has arrived, and everybody is done with the last one
    if (c + 1 < chunks) fetch(t0 + L, min(L, end - t0 - L), b ^ 1);
    const f16 *Bc = stage0 + b * STAGE, *Cc = Bc + L * NROW, *Xc = Cc + L * NROW;
    // A state beyond 2^15 goes down by a power of two on its way into the product, whose result goes up by it.
    float peak = peaks[0];
#pragma unroll
    for (int i = 1; i < WARPS; ++i) peak = fmaxf(peak, peaks[i]);
    const int shift = max((int)(__float_as_uint(peak) >> 23) - 127 - 14, 0);
    const float down = __uint_as_float((uint32_t)(127 - shift) << 23), up = __uint_as_float((uint32_t)(127 + shift) << 23);
#pragma unroll
    for (int m = 0; m < MPW; ++m)
      if (m0 + m < MT)
#pragma unroll
        for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
          for (int side = 0; side < 2; ++side) {
            const int place = ((m0 + m) * 16 + g + 8 * side) * XROW + c0 + nt * 8 + 2 * t4;
            uint32_t hi, lo;
            split(S[m][nt][2 * side] * down, S[m][nt][2 * side + 1] * down, hi, lo);
            *reinterpret_cast<uint32_t*>(Sh + place) = hi;
            *reinterpret_cast<uint32_t*>(Sl + place) = lo;
          }
    if (warp == 0) {
      // The running sums: L / 32 neighbouring tokens a lane.
      constexpr int PER = L / 32;
      float sum[PER], dt[PER], total = 0.f;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const float2 pair = ps[b * L + lane * PER + i];  // zeros past the portion's end
        total += pair.x * 1.4426950408889634f;
        sum[i] = total, dt[i] = pair.y;
      }
      float before = total;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += v;
      }
      const float all = __shfl_sync(0xffffffffu, before, 31);
      before -= total;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int t = lane * PER + i;
        cum[t] = before + sum[i];
        dts[t] = dt[i];
        wgt[t] = power_of_two(fminf(all - (before + sum[i]), 0.f)) * dt[i];
      }
    }
    __syncthreads();
    const int key_rows = (n + 15) & ~15;
#pragma unroll 8
    for (int i = tid; i < key_rows * (COLS / 2); i += THREADS) {
      const int r = i / (COLS / 2), place = r * XROW + (i % (COLS / 2)) * 2;
      const float w = wgt[r];
      const __half2 v = *reinterpret_cast<const __half2*>(Xc + place);
      uint32_t hi, lo;
      split(w * __low2float(v), w * __high2float(v), hi, lo);
      *reinterpret_cast<uint32_t*>(Wh + place) = hi;
      *reinterpret_cast<uint32_t*>(Wl + place) = lo;
    }
    if (row0 < n) {
      uint32_t cf[N / 16][4];
#pragma unroll
      for (int ks = 0; ks < N / 16; ++ks) ldmatrix(cf[ks], Cc + (row0 + (mat & 1) * 8 + r8) * NROW + ks * 16 + (mat >> 1) * 8);
      float acc[NT][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < N / 16; ++ks)
#pragma unroll
        for (int pair = 0; pair < NT / 2; ++pair) {
          const int place = (ks * 16 + (mat & 1) * 8 + r8) * XROW + pair * 16 + (mat >> 1) * 8;
          uint32_t hi[4], lo[4];
          ldmatrix_t(hi, Sh + place);
          ldmatrix_t(lo, Sl + place);
          mma(acc[2 * pair], cf[ks], hi[0], hi[1]);
          mma(acc[2 * pair + 1], cf[ks], hi[2], hi[3]);
          mma(acc[2 * pair], cf[ks], lo[0], lo[1]);
          mma(acc[2 * pair + 1], cf[ks], lo[2], lo[3]);
        }
      const float cum_a = cum[row0 + g], cum_b = cum[row0 + g + 8];
      const float ea = power_of_two(cum_a) * up, eb = power_of_two(cum_b) * up;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) acc[nt][0] *= ea, acc[nt][1] *= ea, acc[nt][2] *= eb, acc[nt][3] *= eb;
      // The keys in blocks of 32, up to this warp's last token.
      const int blocks = (min(row0 + 16, n) + 31) / 32;
#pragma unroll 1
      for (int kb = 0; kb < blocks; ++kb) {
        float p[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) p[j][0] = p[j][1] = p[j][2] = p[j][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < N / 16; ++ks)
#pragma unroll
          for (int j2 = 0; j2 < 2; ++j2) {
            uint32_t bm[4];
            ldmatrix(bm, Bc + (kb * 32 + j2 * 16 + (mat >> 1) * 8 + r8) * NROW + ks * 16 + (mat & 1) * 8);
            mma(p[2 * j2], cf[ks], bm[0], bm[1]);
            mma(p[2 * j2 + 1], cf[ks], bm[2], bm[3]);
          }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int key = kb * 32 + j * 8 + 2 * t4 + e;
            const float ck = cum[key], dk = dts[key];
            p[j][e] *= key <= row0 + g ? power_of_two(cum_a - ck) * dk : 0.f;
            p[j][2 + e] *= key <= row0 + g + 8 ? power_of_two(cum_b - ck) * dk : 0.f;
          }
        // Weights beyond 2^15 (a whole warp's matter, and a rare one): they and the sums so far go down by a power of
        // two, and the sums come up again.
        float most = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) most = fmaxf(most, fabsf(p[j][e]));
        const bool wide = __any_sync(0xffffffffu, most > 32768.f);
        float raise = 1.f;
        if (wide) {
          const int places = max((int)(__float_as_uint(warp_max(most)) >> 23) - 127 - 14, 0);
          const float lower = __uint_as_float((uint32_t)(127 - places) << 23);
          raise = __uint_as_float((uint32_t)(127 + places) << 23);
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) p[j][e] *= lower;
#pragma unroll
          for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] *= lower;
        }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
          uint32_t hi[4], lo[4];
          split(p[2 * kk][0], p[2 * kk][1], hi[0], lo[0]);
          split(p[2 * kk][2], p[2 * kk][3], hi[1], lo[1]);
          split(p[2 * kk + 1][0], p[2 * kk + 1][1], hi[2], lo[2]);
          split(p[2 * kk + 1][2], p[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
          for (int pair = 0; pair < NT / 2; ++pair) {
            uint32_t xv[4];
            ldmatrix_t(xv, Xc + (kb * 32 + kk * 16 + (mat & 1) * 8 + r8) * XROW + pair * 16 + (mat >> 1) * 8);
            mma(acc[2 * pair], hi, xv[0], xv[1]);
            mma(acc[2 * pair + 1], hi, xv[2], xv[3]);
            mma(acc[2 * pair], lo, xv[0], xv[1]);
            mma(acc[2 * pair + 1], lo, xv[2], xv[3]);
          }
        }
        if (wide)
#pragma unroll
          for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] *= raise;
      }
#pragma unroll
      for (int side = 0; side < 2; ++side) {
        const int r = row0 + g + 8 * side;
        if (r >= n) continue;
        float* out = y + (size_t)(t0 + r) * H * dv + head * dv + col0 + 2 * t4;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const __half2 v = *reinterpret_cast<const __half2*>(Xc + r * XROW + nt * 8 + 2 * t4);
          *reinterpret_cast<float2*>(out + nt * 8) = make_float2(fmaf(skip, __low2float(v), acc[nt][2 * side]),
                                                                 fmaf(skip, __high2float(v), acc[nt][2 * side + 1]));
        }
      }
    }
    __syncthreads();  // the weighted x is complete, and the state as an operand has been read
    const float kept = power_of_two(cum[L - 1]);
#pragma unroll
    for (int m = 0; m < MPW; ++m) {
      if (m0 + m >= MT) continue;
#pragma unroll
      for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][nt][e] *= kept;
#pragma unroll 2
      for (int ks = 0; ks < key_rows / 16; ++ks) {
        uint32_t bt[4];
        ldmatrix_t(bt, Bc + (ks * 16 + (mat >> 1) * 8 + r8) * NROW + (m0 + m) * 16 + (mat & 1) * 8);
        if constexpr (NTW == 1) {
          // One tile of eight columns: its upper and lower halves in one load.
          uint32_t w[4];
          const f16* part = (mat >> 1) ? Wl : Wh;
          ldmatrix_t(w, part + (ks * 16 + (mat & 1) * 8 + r8) * XROW + c0);
          mma(S[m][0], bt, w[0], w[1]);
          mma(S[m][0], bt, w[2], w[3]);
        } else {
#pragma unroll
          for (int pair = 0; pair < NTW / 2; ++pair) {
            const int place = (ks * 16 + (mat & 1) * 8 + r8) * XROW + c0 + pair * 16 + (mat >> 1) * 8;
            uint32_t hi[4], lo[4];
            ldmatrix_t(hi, Wh + place);
            ldmatrix_t(lo, Wl + place);
            mma(S[m][2 * pair], bt, hi[0], hi[1]);
            mma(S[m][2 * pair + 1], bt, hi[2], hi[3]);
            mma(S[m][2 * pair], bt, lo[0], lo[1]);
            mma(S[m][2 * pair + 1], bt, lo[2], lo[3]);
          }
        }
      }
    }
    note_peak();
  }
#pragma unroll
  for (int m = 0; m < MPW; ++m)
    if (m0 + m < MT)
#pragma unroll
      for (int nt = 0; nt < NTW; ++nt)
#pragma unroll
        for (int side = 0; side < 2; ++side)
          *reinterpret_cast<float2*>(mine + (size_t)((m0 + m) * 16 + g + 8 * side) * dv + nt * 8) =
              make_float2(S[m][nt][2 * side], S[m][nt][2 * side + 1]);
}

}  // namespace

extern "C" int omnia_ssd_chunk_tokens(void) { return L; }

// Every place and stride of `rows` a multiple of 8 elements and the base on 16 bytes; dv a multiple of SSD_COLS.
extern "C" int omnia_ssd_chunk(const void* rows, int row_stride, int at_x, int at_b, int at_c, const float* pairs, int H, int G,
                               int dv, const float* D, float* S_state, const int* cu_seqlens, const int* state_slots,
                               int num_seqs, float* y, cudaStream_t stream) {
  if (num_seqs == 0) return 0;
  if (H < 1 || G < 1 || H % G || dv < COLS || dv % COLS || row_stride % 8 || at_x % 8 || at_b % 8 || at_c % 8 ||
      (((uintptr_t)rows | (uintptr_t)S_state | (uintptr_t)y) & 15) || ((uintptr_t)pairs & 7))
    return (int)cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e =
        cudaFuncSetAttribute(ssd_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes(L));
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  launch_pdl(ssd_chunk_kernel, dim3(H * (dv / COLS), num_seqs), dim3(THREADS), smem_bytes(L), stream, (const f16*)rows,
             row_stride, at_x, at_b, at_c, (const float2*)pairs, H, G, dv, D, S_state, cu_seqlens, state_slots, y);
  return OMNIA_LAUNCH_RESULT();
}
