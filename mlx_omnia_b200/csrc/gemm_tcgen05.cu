// out[m, n] = sum_k a[m, k] * w[n, k] in bfloat16 on the 5th-generation tensor cores:
// TMA (cp.async.bulk.tensor) stages 128-byte-swizzled tiles of both operands in shared
// memory, one elected thread issues tcgen05.mma with the accumulator in tensor memory,
// and four warps read the accumulator back with tcgen05.ld for the epilogue.
//
// Blocks are persistent (one per SM) and take 128 x BLOCK_N tiles of the output round-robin
// (BLOCK_N = 256, or 128 for narrow problems), each over all of k in steps of 64, through a
// ring of STAGES shared-memory stages and two accumulators in tensor memory, so the epilogue
// of one tile runs while the next tile is being multiplied:
//   warp 0   producer: waits for a free stage, arms its "full" barrier with the byte count
//            and issues the two TMA loads (rows beyond m or n and columns beyond k are
//            zero-filled by the TMA unit);
//   warp 1   allocates tensor memory, then its elected lane waits for a drained accumulator and
//            for each full stage issues four MMAs (k = 16 each); tcgen05.commit frees the
//            stage when they have read it, and after the last step signals "accumulator full";
//   warps 2-5  wait for that signal, read their 32 accumulator rows 32 columns at a time,
//            apply the epilogue, store, and signal "accumulator empty".
// Epilogues: 0 store bfloat16; 1 SwiGLU: the B tile holds 128 gate rows and the matching
// 128 up rows of w, the block stores silu(gate) * up (BLOCK_N 256 only); 2 soft cap to float32.
//
// Grouped form (routed experts): the rows of `a` are sorted by expert, w holds every expert's matrix one
// after the other, and a list made on the device says which runs of at most 128 rows belong to which
// expert: a row tile is then (expert, first row, rows) from that list instead of a multiple of 128, its
// weight rows start at expert * rows-per-expert, and the epilogue stores only the tile's own rows (the
// TMA box of `a` reaches into the next expert's rows, whose products are dropped). How many row tiles
// there are is read from device memory, so the host never learns where the tokens went.
//
// Every wait on a barrier is bounded: when the bound is hit the block raises OMNIA_ERR_TIMEOUT
// in the error word, every role leaves its loop, the block waits (bounded again) for the TMA
// loads it still has in flight, frees its tensor memory and returns.
#include <cuda.h>

#include "common.cuh"

#define OMNIA_ERR_TIMEOUT 8

namespace {

typedef __nv_bfloat16 bf16;

constexpr int BLOCK_M = 128;
constexpr int BLOCK_K = 64;   // 128 bytes of bfloat16: one swizzle row
constexpr int UMMA_K = 16;
constexpr int THREADS = 192;  // producer warp, MMA warp, four epilogue warps
constexpr uint32_t WAIT_LIMIT = 1u << 20;

enum { EPI_STORE = 0, EPI_SWIGLU = 1, EPI_SOFTCAP = 2 };

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ bool mbar_try(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\n\t"  // sleeps up to the hint (ns)
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(bar), "r"(parity), "r"(2000u)
      : "memory");
  return ok != 0;
}
// Bounded wait; false when the block is giving up (its own limit, or another role's).
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag) {
  if (omnia_mbar_test(bar, parity)) return true;
  for (uint32_t i = 0; i < WAIT_LIMIT; ++i) {
    if (mbar_try(bar, parity)) return true;
    if ((i & 63) == 63 && *abort_flag) return false;
  }
  *abort_flag = 1;
  return false;
}

__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y)
      : "memory");
}

// Shared-memory matrix descriptor of a K-major tile with 128-byte swizzle: rows of 128 bytes,
// eight-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t umma_desc(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr >> 4) & 0x3FFF);  // start address
  d |= (uint64_t)1 << 16;                       // leading byte offset (unused with swizzle)
  d |= (uint64_t)(1024 >> 4) << 32;             // stride byte offset between 8-row groups
  d |= (uint64_t)1 << 46;                       // descriptor version of sm_100
  d |= (uint64_t)2 << 61;                       // SWIZZLE_128B
  return d;
}

// kind::f16 instruction descriptor: float32 accumulator, bfloat16 A and B, both K-major.
__host__ __device__ constexpr uint32_t umma_idesc(int m, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

__device__ __forceinline__ void umma(uint32_t tmem_d, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void umma_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tmem_load32(uint32_t addr, uint32_t* v) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
        "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
        "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
        "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
      : "r"(addr));
}

template <int BLOCK_N, int STAGES, int EPI>
__global__ void __launch_bounds__(THREADS, 1)
gemm_tcgen05_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
                    void* __restrict__ out, int m, int n, int k, int pair_offset, float multiplier,
                    float cap, int m_tiles, int n_tiles, const int* __restrict__ group_tiles,
                    const int* __restrict__ group_count, int group_rows, int* err) {
  constexpr uint32_t A_BYTES = BLOCK_M * BLOCK_K * sizeof(bf16);
  constexpr uint32_t B_BYTES = BLOCK_N * BLOCK_K * sizeof(bf16);
  constexpr uint32_t STAGE_BYTES = A_BYTES + B_BYTES;
  constexpr int TILE_COLS = EPI == EPI_SWIGLU ? BLOCK_N / 2 : BLOCK_N;
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* tiles = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t* bars = reinterpret_cast<uint64_t*>(tiles + STAGES * STAGE_BYTES);
  // bars: [0, S) stage full, [S, 2S) stage empty, [2S, 2S+2) accumulator full, [2S+2, 2S+4) accumulator empty
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int k_blocks = (k + BLOCK_K - 1) / BLOCK_K;
  const uint32_t full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
  const uint32_t acc_full0 = smem_u32(bars + 2 * STAGES), acc_empty0 = smem_u32(bars + 2 * STAGES + 2);

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(acc_full0 + 8 * b, 1);
      mbar_init(acc_empty0 + 8 * b, 4);  // one arrival per epilogue warp
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_holder)),
                 "r"((uint32_t)(2 * BLOCK_N)));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = *tmem_holder;
  // Everything so far needed nothing from the kernel before this one and ran while it finished
  // (the launch is a programmatic dependent launch); from here on its results are read.
  pdl_wait();
  pdl_launch_dependents();
  // Grouped: the list's length is what the kernel before this one wrote; m_tiles is then its capacity.
  if (group_tiles != nullptr) m_tiles = min(*group_count, m_tiles);
  const int total_tiles = m_tiles * n_tiles;
  // Row tile `mt`: its first row, how many of its 128 rows are its own, and where its weight rows begin.
  auto row_tile = [&](int mt, int& m0, int& rows, int& w0) {
    if (group_tiles != nullptr) {
      w0 = group_tiles[3 * mt] * group_rows, m0 = group_tiles[3 * mt + 1], rows = group_tiles[3 * mt + 2];
    } else {
      w0 = 0, m0 = mt * BLOCK_M, rows = BLOCK_M;
    }
  };

  // Tiles are dealt round-robin; consecutive tiles share the same columns of the output (the
  // same rows of w), so blocks running side by side read the same weight tile out of L2.
  if (warp == 0) {
    // ---- producer ----------------------------------------------------------------------
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total_tiles && ok; tile += gridDim.x) {
        int m0, tile_rows, w0;
        row_tile(tile % m_tiles, m0, tile_rows, w0);
        const int n0 = (tile / m_tiles) * TILE_COLS;
        for (int kb = 0; kb < k_blocks; ++kb, ++it) {
          const int s = it % STAGES;
          ok = mbar_wait(empty0 + 8 * s, ((it / STAGES) & 1) ^ 1, abort_flag);
          if (!ok) break;
          const uint32_t a_dst = smem_u32(tiles + s * STAGE_BYTES), b_dst = a_dst + A_BYTES;
          mbar_expect_tx(full0 + 8 * s, STAGE_BYTES);
          tma_load_2d(a_dst, &map_a, full0 + 8 * s, kb * BLOCK_K, m0);
          if (EPI == EPI_SWIGLU) {
            tma_load_2d(b_dst, &map_b, full0 + 8 * s, kb * BLOCK_K, w0 + n0);
            tma_load_2d(b_dst + B_BYTES / 2, &map_b, full0 + 8 * s, kb * BLOCK_K, w0 + pair_offset + n0);
          } else {
            tma_load_2d(b_dst, &map_b, full0 + 8 * s, kb * BLOCK_K, w0 + n0);
          }
        }
      }
      if (*abort_flag) {
        // Giving up: let the loads already issued land before the block's memory goes away.
        for (uint32_t back = 0; back < (uint32_t)STAGES && back < it; ++back) {
          const uint32_t j = it - 1 - back;
          for (uint32_t i = 0; i < WAIT_LIMIT && !mbar_try(full0 + 8 * (j % STAGES), (j / STAGES) & 1); ++i) {
          }
        }
      }
    }
  } else if (warp == 1) {
    // ---- MMA issuer ----------------------------------------------------------------------
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc(BLOCK_M, BLOCK_N);
      uint32_t it = 0, local = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total_tiles && ok; tile += gridDim.x, ++local) {
        const uint32_t buf = local & 1;
        ok = mbar_wait(acc_empty0 + 8 * buf, ((local >> 1) & 1) ^ 1, abort_flag);  // the epilogue has drained it
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t acc = tmem_base + buf * BLOCK_N;
        for (int kb = 0; kb < k_blocks; ++kb, ++it) {
          const int s = it % STAGES;
          ok = mbar_wait(full0 + 8 * s, (it / STAGES) & 1, abort_flag);
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint32_t a_addr = smem_u32(tiles + s * STAGE_BYTES), b_addr = a_addr + A_BYTES;
#pragma unroll
          for (int kk = 0; kk < BLOCK_K / UMMA_K; ++kk) {
            const uint64_t a_desc = umma_desc(a_addr + kk * UMMA_K * sizeof(bf16));
            const uint64_t b_desc = umma_desc(b_addr + kk * UMMA_K * sizeof(bf16));
            umma(acc, a_desc, b_desc, idesc, (kb | kk) != 0);
          }
          umma_commit(empty0 + 8 * s);  // the stage is free once these MMAs have read it
        }
        if (ok) umma_commit(acc_full0 + 8 * buf);
      }
    }
  } else {
    // ---- epilogue (warps 2..5 own accumulator rows 32 * (warp % 4) .. + 31) -------------------
    const int quarter = warp & 3;
    uint32_t local = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < total_tiles && ok; tile += gridDim.x, ++local) {
      int m0, tile_rows, w0;
      row_tile(tile % m_tiles, m0, tile_rows, w0);
      const int n0 = (tile / m_tiles) * TILE_COLS;
      const int row = quarter * 32 + lane < tile_rows ? m0 + quarter * 32 + lane : m;  // m: not one of the tile's own
      const uint32_t buf = local & 1;
      ok = mbar_wait(acc_full0 + 8 * buf, (local >> 1) & 1, abort_flag);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t lane_base = tmem_base + buf * BLOCK_N + ((uint32_t)(quarter * 32) << 16);
      if (EPI == EPI_SWIGLU) {
        bf16* dst = reinterpret_cast<bf16*>(out) + (size_t)row * pair_offset + n0;
#pragma unroll 1
        for (int c = 0; c < BLOCK_N / 2; c += 32) {
          uint32_t gate[32], up[32];
          tmem_load32(lane_base + c, gate);
          tmem_load32(lane_base + BLOCK_N / 2 + c, up);
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
          if (row < m) {
#pragma unroll
            for (int j = 0; j < 32; j += 2) {
              float v[2];
#pragma unroll
              for (int e = 0; e < 2; ++e) {
                // Both halves are rounded to bfloat16 first, as a separate product would round them.
                const float g = __bfloat162float(__float2bfloat16_rn(__uint_as_float(gate[j + e])));
                const float u = __bfloat162float(__float2bfloat16_rn(__uint_as_float(up[j + e])));
                // cap > 0: the clamped unit (gate below cap, up within +-cap and moved by one, slope `multiplier`).
                const float gc = cap > 0.f ? fminf(g, cap) : g;
                const float uc = cap > 0.f ? fminf(fmaxf(u, -cap), cap) + 1.f : u;
                // cap -1: the gate through a relu; cap -2: through the tanh form of GELU, g sigmoid(2 a).
                const float z = cap < OMNIA_UNIT_RELU ? 1.5957691216057308f * (g + 0.044715f * g * g * g) : multiplier * gc;
                v[e] = cap == OMNIA_UNIT_RELU ? fmaxf(g, 0.f) * u : __fdividef(gc, 1.f + __expf(-z)) * uc;
              }
              const int col = n0 + c + j;
              if (col + 1 < pair_offset && (pair_offset & 1) == 0) {
                *reinterpret_cast<__nv_bfloat162*>(dst + c + j) = __floats2bfloat162_rn(v[0], v[1]);
              } else {
                if (col < pair_offset) dst[c + j] = __float2bfloat16_rn(v[0]);
                if (col + 1 < pair_offset) dst[c + j + 1] = __float2bfloat16_rn(v[1]);
              }
            }
          }
        }
      } else {
#pragma unroll 1
        for (int c = 0; c < BLOCK_N; c += 32) {
          uint32_t acc[32];
          tmem_load32(lane_base + c, acc);
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
          if (row >= m) continue;
          if (EPI == EPI_SOFTCAP) {
            float* dst = reinterpret_cast<float*>(out) + (size_t)row * n + n0 + c;
#pragma unroll
            for (int j = 0; j < 32; ++j) {
              if (n0 + c + j >= n) break;
              const float z = __bfloat162float(__float2bfloat16_rn(__uint_as_float(acc[j]))) * multiplier;
              dst[j] = cap > 0.f ? cap * tanhf(z / cap) : z;
            }
          } else {
            bf16* dst = reinterpret_cast<bf16*>(out) + (size_t)row * n + n0 + c;
            // cap 5: the exact GELU of the product, as bfloat16 would hold it (a separate kernel would read it so).
            if (cap == 5.f) {
#pragma unroll
              for (int j = 0; j < 32; ++j)
                acc[j] = __float_as_uint(gelu_erf(__bfloat162float(__float2bfloat16_rn(__uint_as_float(acc[j])))));
            }
            if (n0 + c + 32 <= n && (n & 7) == 0) {
#pragma unroll
              for (int j = 0; j < 32; j += 8) {
                uint4 packed;
                __nv_bfloat162 p0 = __floats2bfloat162_rn(__uint_as_float(acc[j]), __uint_as_float(acc[j + 1]));
                __nv_bfloat162 p1 = __floats2bfloat162_rn(__uint_as_float(acc[j + 2]), __uint_as_float(acc[j + 3]));
                __nv_bfloat162 p2 = __floats2bfloat162_rn(__uint_as_float(acc[j + 4]), __uint_as_float(acc[j + 5]));
                __nv_bfloat162 p3 = __floats2bfloat162_rn(__uint_as_float(acc[j + 6]), __uint_as_float(acc[j + 7]));
                packed.x = *reinterpret_cast<uint32_t*>(&p0);
                packed.y = *reinterpret_cast<uint32_t*>(&p1);
                packed.z = *reinterpret_cast<uint32_t*>(&p2);
                packed.w = *reinterpret_cast<uint32_t*>(&p3);
                *reinterpret_cast<uint4*>(dst + j) = packed;
              }
            } else {
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (n0 + c + j < n) dst[j] = __float2bfloat16_rn(__uint_as_float(acc[j]));
            }
          }
        }
      }
      // This warp has read its rows of the accumulator: hand the buffer back to the MMA warp.
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty0 + 8 * buf);
    }
  }

  // ---- teardown: everyone meets, the allocating warp frees the tensor memory ---------------
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((uint32_t)(2 * BLOCK_N)));
  }
  if (threadIdx.x == 0 && *abort_flag) atomicOr(err, OMNIA_ERR_TIMEOUT);
}

// ---- host side ---------------------------------------------------------------------------

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encode_tiled() {
  static EncodeTiled fn = nullptr;
  if (fn == nullptr) {
    void* symbol = nullptr;
    cudaDriverEntryPointQueryResult result;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &symbol, cudaEnableDefault, &result) == cudaSuccess &&
        result == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiled>(symbol);
  }
  return fn;
}

// A [rows, k] bfloat16 row-major matrix as a 2-D tensor map with boxes of 64 x box_rows, 128-byte swizzle.
bool make_map(CUtensorMap* map, const void* base, int rows, int k, int box_rows) {
  EncodeTiled encode = encode_tiled();
  if (encode == nullptr) return false;
  const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows};
  const cuuint64_t strides[1] = {(cuuint64_t)k * sizeof(bf16)};
  const cuuint32_t box[2] = {(cuuint32_t)BLOCK_K, (cuuint32_t)box_rows};
  const cuuint32_t elem[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem,
                CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BLOCK_N, int STAGES, int EPI>
int launch(const void* a, const void* w, void* out, int m, int n, int k, int pair_offset, float multiplier,
           float cap, int* err, cudaStream_t stream) {
  CUtensorMap map_a, map_b;
  const int b_box = EPI == EPI_SWIGLU ? BLOCK_N / 2 : BLOCK_N;
  if (!make_map(&map_a, a, m, k, BLOCK_M) || !make_map(&map_b, w, n, k, b_box)) return (int)cudaErrorInvalidValue;
  constexpr size_t smem = (size_t)STAGES * (BLOCK_M + BLOCK_N) * BLOCK_K * sizeof(bf16) + 1024 + 256;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(gemm_tcgen05_kernel<BLOCK_N, STAGES, EPI>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int cols = EPI == EPI_SWIGLU ? pair_offset : n;
  const int tile_cols = EPI == EPI_SWIGLU ? BLOCK_N / 2 : BLOCK_N;
  const int n_tiles = (cols + tile_cols - 1) / tile_cols, m_tiles = (m + BLOCK_M - 1) / BLOCK_M;
  const int sm_count = omnia_sm_count();
  const long long total = (long long)n_tiles * m_tiles;
  const int grid = (int)(total < sm_count ? total : sm_count);  // one persistent block per SM
  launch_pdl(gemm_tcgen05_kernel<BLOCK_N, STAGES, EPI>, grid, THREADS, smem, stream,
             map_a, map_b, out, m, n, k, pair_offset, multiplier, cap, m_tiles, n_tiles, (const int*)nullptr,
             (const int*)nullptr, 0, err);
  return OMNIA_LAUNCH_RESULT();
}

// The grouped form: a [m, k] sorted by expert, w [experts * n, k], tiles [max_tiles, 3] and tile_count on the device.
template <int BLOCK_N, int STAGES, int EPI>
int launch_grouped(const void* a, const void* w, void* out, int m, int n, int k, int experts, int pair_offset,
                   const int* tiles, const int* tile_count, int max_tiles, float multiplier, float cap, int* err,
                   cudaStream_t stream) {
  CUtensorMap map_a, map_b;
  const int b_box = EPI == EPI_SWIGLU ? BLOCK_N / 2 : BLOCK_N;
  if (!make_map(&map_a, a, m, k, BLOCK_M) || !make_map(&map_b, w, experts * n, k, b_box)) return (int)cudaErrorInvalidValue;
  constexpr size_t smem = (size_t)STAGES * (BLOCK_M + BLOCK_N) * BLOCK_K * sizeof(bf16) + 1024 + 256;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(gemm_tcgen05_kernel<BLOCK_N, STAGES, EPI>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int cols = EPI == EPI_SWIGLU ? pair_offset : n;
  const int tile_cols = EPI == EPI_SWIGLU ? BLOCK_N / 2 : BLOCK_N;
  const int n_tiles = (cols + tile_cols - 1) / tile_cols;
  const int sm_count = omnia_sm_count();
  const long long total = (long long)n_tiles * max_tiles;
  const int grid = (int)(total < sm_count ? total : sm_count);
  launch_pdl(gemm_tcgen05_kernel<BLOCK_N, STAGES, EPI>, grid, THREADS, smem, stream,
             map_a, map_b, out, m, n, k, pair_offset, multiplier, cap, max_tiles, n_tiles, tiles, tile_count, n, err);
  return OMNIA_LAUNCH_RESULT();
}

}  // namespace

// epilogue: 0 store bfloat16 [m, n] (cap 5: the exact GELU of the product); 1 SwiGLU, w = [gate rows | up rows] with n = 2 * inner,
// out bfloat16 [m, inner] (cap > 0: the clamped unit, the sigmoid's slope in `multiplier`); 2 soft cap, out float32 [m, n]. a and w must be 16-byte aligned and
// k a multiple of 8 (rows of both matrices start on 16 bytes).
extern "C" int omnia_gemm_tcgen05(const void* a, const void* w, void* out, int m, int n, int k, int epilogue,
                                  float multiplier, float cap, int* err, cudaStream_t stream) {
  if (m == 0 || n == 0) return 0;
  if (k <= 0 || k % 8 != 0 || ((uintptr_t)a & 15) || ((uintptr_t)w & 15)) return (int)cudaErrorInvalidValue;
  if (epilogue == EPI_SWIGLU) {
    if (n % 2) return (int)cudaErrorInvalidValue;
    return launch<256, 4, EPI_SWIGLU>(a, w, out, m, n, k, n / 2, cap > 0.f ? multiplier : 1.f, cap, err, stream);
  }
  if (epilogue == EPI_SOFTCAP) return launch<256, 4, EPI_SOFTCAP>(a, w, out, m, n, k, 0, multiplier, cap, err, stream);
  if (epilogue != EPI_STORE || (cap != 0.f && cap != 5.f)) return (int)cudaErrorInvalidValue;
  // 256-wide tiles do twice the work per byte staged; 128-wide tiles win only when they fill
  // SMs that the wide tiling would leave idle. Cost in units of one wide tile per round of all SMs.
  const long long m_tiles = (m + 127) / 128, sms = omnia_sm_count();
  const long long wide_rounds = (((n + 255) / 256) * m_tiles + sms - 1) / sms;
  const long long narrow_rounds = (((n + 127) / 128) * m_tiles + sms - 1) / sms;
  if (wide_rounds * 100 <= narrow_rounds * 65) return launch<256, 4, EPI_STORE>(a, w, out, m, n, k, 0, 1.f, cap, err, stream);
  return launch<128, 6, EPI_STORE>(a, w, out, m, n, k, 0, 1.f, cap, err, stream);
}

// The grouped product of routed experts: a [m, k] rows sorted by expert; w [experts, n, k]; tiles
// [max_tiles, 3] = (expert, first row, rows <= 128) and tile_count [1] in device memory. epilogue 0:
// out [m, n] = a w_e^T (cap 5: its exact GELU); 1: n = 2 * inner (gate rows, then up rows), out [m, inner] = silu(gate) * up, or with
// cap > 0 the clamped unit (the sigmoid's slope in `multiplier`), with cap -1 relu(gate) * up, -2 tanh-GELU(gate) * up.
extern "C" int omnia_gemm_tcgen05_grouped(const void* a, const void* w, void* out, int m, int n, int k, int experts,
                                          int epilogue, const int* tiles, const int* tile_count, int max_tiles,
                                          float multiplier, float cap, int* err, cudaStream_t stream) {
  if (m == 0 || n == 0 || max_tiles == 0) return 0;
  if (k <= 0 || k % 8 != 0 || ((uintptr_t)a & 15) || ((uintptr_t)w & 15) || experts < 1) return (int)cudaErrorInvalidValue;
  if (epilogue == EPI_SWIGLU) {
    if (n % 2) return (int)cudaErrorInvalidValue;
    return launch_grouped<256, 4, EPI_SWIGLU>(a, w, out, m, n, k, experts, n / 2, tiles, tile_count, max_tiles,
                                              cap > 0.f ? multiplier : 1.f, cap, err, stream);
  }
  if (epilogue != EPI_STORE || (cap != 0.f && cap != 5.f)) return (int)cudaErrorInvalidValue;
  return launch_grouped<256, 4, EPI_STORE>(a, w, out, m, n, k, experts, 0, tiles, tile_count, max_tiles, 1.f, cap, err, stream);
}

