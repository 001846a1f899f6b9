// GEMM for a few tokens: y[M, N] = alpha * x[M, K] W[N, K]^T with bf16 weights, M up to 128 per tile.
//
// A decode step is bound by reading the weights once, so W is the 128-row A operand of tcgen05.mma (the
// tokens are the narrow N side) and the reduction is split over the CTAs of a cluster until enough bytes
// are in flight. Each CTA streams its k-blocks of W and x through a TMA ring into one TMEM accumulator,
// stages the fp32 result in shared memory, and after a cluster barrier every CTA sums a share of the
// tokens over the peers' shared memory and stores it: no atomics, no accumulator to clear, the same
// result every time. With `f_off` > 0 a tile takes 64 rows of each half of a gate / up matrix and stores
// the gated activation. One launch can hold several products side by side (one per attention head) or a
// list of row segments that meet a matrix each (routed experts).
//
// gemm_segments: the row-segment form for prompts. Persistent over (segment tile, weight tile), 128 tokens
// x 256 weight rows, two accumulators in TMEM so that storing a tile overlaps the next one's products.
#include "api.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "host_util.h"
#include "tc.cuh"

namespace mb {
namespace {

constexpr int GD_THREADS = 128;
constexpr int GD_BM = 128;       // weight rows per tile
constexpr int GD_BK = 64;
constexpr int GD_MAX_STAGES = 8;
constexpr int GD_A_BYTES = GD_BM * GD_BK * 2;

__device__ __forceinline__ uint32_t gd_ctarank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ void gd_cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t gd_mapa(uint32_t addr, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
__device__ __forceinline__ float gd_ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

// Value of one output element before it is stored.
__device__ __forceinline__ float gd_tail(const GemmTail& tail, float y, int token, int n, int batch) {
  if (tail.gate != nullptr)
    return y * sigmoid_f(__bfloat162float(static_cast<const __nv_bfloat16*>(tail.gate)[token * tail.ld_gate + batch * tail.gate_batch + n]));
  if (tail.cap > 0.f) return soft_cap_f(y, tail.cap);
  if (tail.mul == nullptr) return y;
  const int id = min(max(tail.mul_ids[token], 0), tail.vocab - 1);
  return gelu_tanh_f(y) * __bfloat162float(static_cast<const __nv_bfloat16*>(tail.mul)[id * tail.ld_mul + n]);
}

// grid (tiles of W, K splits = cluster size, token tiles x products or entries of the tile list)
template <typename OUT>
__global__ void __launch_bounds__(GD_THREADS)
gemm_decode_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, OUT* __restrict__ out,
                   long long ldo, int M, int N, int K, int mt, int stages, float alpha, const __grid_constant__ GemmTail tail,
                   int m_tiles, long long out_batch, TileList list, int* status) {
  const int f_off = tail.f_off;
  int matrix, m0, x_batch;
  if (list.tiles) {
    if ((int)blockIdx.z >= *list.count) return;      // the same for every CTA of a cluster
    const int* tile = list.tiles + 3 * blockIdx.z;
    matrix = tile[0];
    m0 = tile[1];
    M = m0 + tile[2];
    x_batch = 0;
  } else {
    matrix = x_batch = blockIdx.z / m_tiles;
    m0 = (blockIdx.z % m_tiles) * mt;
    out += matrix * out_batch;
  }
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[GD_MAX_STAGES], empty[GD_MAX_STAGES], done;
  __shared__ uint32_t tmem_ptr;
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int splits = gridDim.y;
  const int kblocks = (K + GD_BK - 1) / GD_BK;
  const int kb0 = (int)((long long)kblocks * blockIdx.y / splits), kb1 = (int)((long long)kblocks * (blockIdx.y + 1) / splits);
  const int n0 = blockIdx.x * (f_off ? GD_BM / 2 : GD_BM);
  const int stage_bytes = GD_A_BYTES + mt * GD_BK * 2;
  const uint32_t tmem_cols = mt <= 32 ? 32 : (mt <= 64 ? 64 : 128);
  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&done, 1);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_x);
  }
  if (warp == 1) {
    tmem_alloc(&tmem_ptr, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_ptr;
  if (warp == 0) {
    if (lane == 0) {
      int st = 0;
      uint32_t ph = 0;
      for (int kb = kb0; kb < kb1; ++kb) {
        if (!mbar_wait(&empty[st], ph ^ 1, abort_flag, status, 90)) break;
        uint8_t* a = smem + st * stage_bytes;
        mbar_arrive_expect_tx(&full[st], (uint32_t)stage_bytes);
        tma_load_3d(a, &tm_w, &full[st], kb * GD_BK, n0, matrix);
        if (f_off) tma_load_3d(a + GD_A_BYTES / 2, &tm_w, &full[st], kb * GD_BK, f_off + n0, matrix);
        tma_load_3d(a + GD_A_BYTES, &tm_x, &full[st], kb * GD_BK, x_batch, m0);
        if (++st == stages) { st = 0; ph ^= 1; }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16(GD_BM, mt, false, false);
      int st = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int kb = kb0; kb < kb1; ++kb) {
        if (!mbar_wait(&full[st], ph, abort_flag, status, 91)) { ok = false; break; }
        tc_fence_after();
        const uint32_t a = smem_u32(smem + st * stage_bytes), b = a + GD_A_BYTES;
#pragma unroll
        for (int k = 0; k < GD_BK / 16; ++k)
          umma_f16(tmem, umma_desc_sw128(a + k * 32, 0, 1024), umma_desc_sw128(b + k * 32, 0, 1024), idesc,
                   (kb > kb0 || k > 0) ? 1u : 0u);
        umma_commit(&empty[st]);
        if (++st == stages) { st = 0; ph ^= 1; }
      }
      if (ok) umma_commit(&done);
    }
    __syncwarp();
  }
  bool ok = mbar_wait(&done, 0, abort_flag, status, 92);
  ok = __all_sync(0xffffffffu, ok);
  // every load has been consumed: the ring now holds the staged result, [token][128 rows] fp32
  float* acc = reinterpret_cast<float*>(smem);
  if (ok) {
    tc_fence_after();
    const uint32_t t_row = tmem + ((uint32_t)(warp * 32) << 16);
    for (int c = 0; c < mt; c += 16) {
      uint32_t v[16];
      tmem_ld16(t_row + c, v);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 16; ++j) acc[(c + j) * GD_BM + threadIdx.x] = __uint_as_float(v[j]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {               // copies in flight land in this CTA's memory: give them time
    const long long t0 = clock64();
    while (clock64() - t0 < 10000000LL) {}
    __syncthreads();
  }
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem, tmem_cols);
  gd_cluster_sync();
  const int rank = (int)gd_ctarank();
  const uint32_t acc_addr = smem_u32(acc);
  const int tokens = min(mt, M - m0);
  uint32_t peer[8];
#pragma unroll
  for (int p = 0; p < 8; ++p) peer[p] = gd_mapa(acc_addr, p < splits ? p : 0);
  if (f_off == 0) {
    const int n = n0 + threadIdx.x;
    for (int t = rank; t < tokens; t += splits) {
      float y = 0.f;
#pragma unroll
      for (int p = 0; p < 8; ++p)
        if (p < splits) y += gd_ld_cluster(peer[p] + (t * GD_BM + threadIdx.x) * 4);
      if (n < N) stf(out + (long long)(m0 + t) * ldo + n, gd_tail(tail, y * alpha, m0 + t, n, x_batch));
    }
  } else {
    const int i = threadIdx.x & 63, n = n0 + i;
    for (int t = rank * 2 + (threadIdx.x >> 6); t < tokens; t += 2 * splits) {
      float g = 0.f, u = 0.f;
#pragma unroll
      for (int p = 0; p < 8; ++p)
        if (p < splits) {
          g += gd_ld_cluster(peer[p] + (t * GD_BM + i) * 4);
          u += gd_ld_cluster(peer[p] + (t * GD_BM + 64 + i) * 4);
        }
      if (n < N) stf(out + (long long)(m0 + t) * ldo + n, gate_act(tail.act, g * alpha, u * alpha));
    }
  }
  gd_cluster_sync();               // nobody leaves while a peer still reads its shared memory
}

template <typename OUT>
void launch_gd(const CUtensorMap& tw, const CUtensorMap& tx, OUT* out, long long ldo, int M, int N, int K, int mt, int stages,
               int smem, dim3 grid, float alpha, const GemmTail& tail, int m_tiles, long long out_batch, const TileList& list,
               int* status, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(gemm_decode_kernel<OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    configured = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(GD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = grid.y;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  MB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, gemm_decode_kernel<OUT>, tw, tx, out, ldo, M, N, K, mt, stages, alpha, tail, m_tiles,
                                   out_batch, list, status));
}

// Weights [matrices][rows][K] as a 3-D map, one box = box_rows rows x 64 columns of one matrix.
CUtensorMap weight_map(const void* W, long long ldw, long long w_batch, int matrices, int rows, int K, int box_rows) {
  uint64_t d[3] = {(uint64_t)K, (uint64_t)rows, (uint64_t)matrices};
  uint64_t st[2] = {(uint64_t)ldw * 2, (uint64_t)(matrices > 1 ? w_batch : ldw * (long long)rows) * 2};
  uint32_t b[3] = {GD_BK, (uint32_t)box_rows, 1};
  return make_tensor_map(W, TmaDType::BF16, 3, d, st, b, true);
}

// ---------------------------------------------------------------------------------------------
constexpr int GS_THREADS = 192;     // TMA producer, MMA issuer, four epilogue warps
constexpr int GS_BM = 128;          // tokens per tile (the A operand)
constexpr int GS_BN = 256;          // weight rows per tile
constexpr int GS_STAGES = 4;
constexpr int GS_A = GS_BM * GD_BK * 2, GS_B = GS_BN * GD_BK * 2, GS_STAGE = GS_A + GS_B;
constexpr int GS_BAR = GS_STAGES * GS_STAGE;
constexpr int GS_SMEM = GS_BAR + (2 * GS_STAGES + 4) * 8 + 16 + 1024;

__global__ void __launch_bounds__(GS_THREADS, 1)
gemm_segments_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x,
                     __nv_bfloat16* __restrict__ out, long long ldo, int N, int K, int tiles_n,
                     const __grid_constant__ GemmTail tail, TileList list, int* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + GS_BAR);
  uint64_t* empty = full + GS_STAGES;
  uint64_t* tfull = empty + GS_STAGES;
  uint64_t* tempty = tfull + 2;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(tempty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kblocks = (K + GD_BK - 1) / GD_BK;
  const int total = min(*list.count, list.max_tiles) * tiles_n;
  const bool gated = tail.f_off > 0;
  const int per_tile = gated ? GS_BN / 2 : GS_BN;       // output columns of a tile

  if (threadIdx.x == 0) {
    for (int s = 0; s < GS_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&tfull[i], 1);
      mbar_init(&tempty[i], 4);
    }
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_x);
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_ptr;

  if (warp == 0) {
    if (lane == 0) {
      int st = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int w = blockIdx.x; w < total && ok; w += gridDim.x) {
        const int* tile = list.tiles + 3 * (w / tiles_n);
        const int n0 = (w % tiles_n) * per_tile;
        const int second = gated ? tail.f_off + n0 : n0 + 128;
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&empty[st], ph ^ 1, abort_flag, status, 95)) { ok = false; break; }
          uint8_t* a = smem + st * GS_STAGE;
          mbar_arrive_expect_tx(&full[st], GS_STAGE);
          tma_load_2d(a, &tm_x, &full[st], kb * GD_BK, tile[1]);
          tma_load_3d(a + GS_A, &tm_w, &full[st], kb * GD_BK, n0, tile[0]);
          tma_load_3d(a + GS_A + GS_B / 2, &tm_w, &full[st], kb * GD_BK, second, tile[0]);
          if (++st == GS_STAGES) { st = 0; ph ^= 1; }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t IDESC = umma_idesc_bf16(GS_BM, GS_BN, false, false);
      int st = 0, acc = 0;
      uint32_t ph = 0, acc_ph = 0;
      bool ok = true;
      for (int w = blockIdx.x; w < total && ok; w += gridDim.x) {
        if (!mbar_wait(&tempty[acc], acc_ph ^ 1, abort_flag, status, 96)) break;
        tc_fence_after();
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&full[st], ph, abort_flag, status, 97)) { ok = false; break; }
          tc_fence_after();
          const uint32_t a = smem_u32(smem + st * GS_STAGE), b = a + GS_A;
#pragma unroll
          for (int k = 0; k < GD_BK / 16; ++k)
            umma_f16(tmem + acc * GS_BN, umma_desc_sw128(a + k * 32, 0, 1024), umma_desc_sw128(b + k * 32, 0, 1024), IDESC,
                     (kb > 0 || k > 0) ? 1u : 0u);
          umma_commit(&empty[st]);
          if (++st == GS_STAGES) { st = 0; ph ^= 1; }
        }
        if (!ok) break;
        umma_commit(&tfull[acc]);
        acc ^= 1;
        if (acc == 0) acc_ph ^= 1;
      }
    }
  } else {
    const int quarter = warp & 3;                        // TMEM lanes this warp may read
    const int r = quarter * 32 + lane;
    int acc = 0;
    uint32_t acc_ph = 0;
    for (int w = blockIdx.x; w < total; w += gridDim.x) {
      const int* tile = list.tiles + 3 * (w / tiles_n);
      const int n0 = (w % tiles_n) * per_tile;
      const bool live = r < tile[2];
      __nv_bfloat16* dst = out + (long long)(tile[1] + r) * ldo + n0;
      bool ok = mbar_wait(&tfull[acc], acc_ph, abort_flag, status, 98);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t t_row = tmem + acc * GS_BN + ((uint32_t)(quarter * 32) << 16);
      const int cols = min(per_tile, N - n0);
#pragma unroll 1
      for (int c = 0; c < cols; c += 16) {
        uint32_t g[16], u[16];
        tmem_ld16(t_row + c, g);
        if (gated) tmem_ld16(t_row + GS_BN / 2 + c, u);
        tmem_ld_wait();
        float y[16];
#pragma unroll
        for (int j = 0; j < 16; ++j)
          y[j] = gated ? gate_act(tail.act, __uint_as_float(g[j]), __uint_as_float(u[j])) : __uint_as_float(g[j]);
        if (live) {
#pragma unroll
          for (int h = 0; h < 2; ++h)
            if (c + 8 * h < cols) {                      // N is a multiple of 8
              uint4 v;
              v.x = pack_bf16x2(y[8 * h + 0], y[8 * h + 1]);
              v.y = pack_bf16x2(y[8 * h + 2], y[8 * h + 3]);
              v.z = pack_bf16x2(y[8 * h + 4], y[8 * h + 5]);
              v.w = pack_bf16x2(y[8 * h + 6], y[8 * h + 7]);
              *reinterpret_cast<uint4*>(dst + c + 8 * h) = v;
            }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tempty[acc]);
      acc ^= 1;
      if (acc == 0) acc_ph ^= 1;
    }
  }
  __syncthreads();
  if (*abort_flag) {               // copies in flight land in this CTA's memory: give them time
    const long long t0 = clock64();
    while (clock64() - t0 < 10000000LL) {}
    __syncthreads();
  }
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

}  // namespace

void gemm_decode(const void* x, long long ldx, const void* W, long long ldw, void* out, bool out_f32, long long ldo, int M,
                 int N, int K, float alpha, const GemmTail& tail, const GemmGroup& group, int* status, cudaStream_t stream) {
  const int f_off = tail.f_off, batch = group.list ? 1 : (group.batch > 0 ? group.batch : 1);
  const bool many = batch > 1 || group.list;
  MB_REQUIRE(M > 0 && N > 0 && K > 0, "gemm_decode: empty problem");
  MB_REQUIRE(ldx % 8 == 0 && ldw % 8 == 0 && (!many || (group.x_batch % 8 == 0 && group.w_batch % 8 == 0)),
             "gemm_decode: strides must be multiples of 8 elements");
  MB_REQUIRE(f_off == 0 || f_off >= N, "gemm_decode: the up half starts after the gate half");
  MB_REQUIRE((tail.mul != nullptr) + (f_off > 0) + (tail.cap > 0.f) + (tail.gate != nullptr) <= 1, "gemm_decode: one tail at a time");
  int mt = (M + 15) / 16 * 16;
  if (mt > 128) mt = 128;
  if (group.list) mt = group.mt;
  MB_REQUIRE(mt % 16 == 0 && mt >= 16 && mt <= 128, "gemm_decode: tile rows");
  const int m_tiles = group.list ? 1 : (M + mt - 1) / mt;
  const int z = group.list ? group.list->max_tiles : m_tiles * batch;
  const int rows_per_tile = f_off ? GD_BM / 2 : GD_BM;
  const int tiles = (N + rows_per_tile - 1) / rows_per_tile;
  const int kblocks = (K + GD_BK - 1) / GD_BK;
  int splits = 1;
  while (splits < 8 && splits * 2 <= kblocks / 2 && (long long)tiles * z * splits * 2 <= 3 * sm_count()) splits *= 2;
  const int stage = GD_A_BYTES + mt * GD_BK * 2;
  int stages = (100 * 1024) / stage;
  if (stages > GD_MAX_STAGES) stages = GD_MAX_STAGES;
  const int smem = stages * stage + 1024;          // >= mt * 512 bytes of staged result for every mt
  const int matrices = group.list ? group.batch : batch;
  const CUtensorMap tw = weight_map(W, ldw, group.w_batch, matrices, f_off ? f_off + N : N, K, rows_per_tile);
  uint64_t xd[3] = {(uint64_t)K, (uint64_t)batch, (uint64_t)M}, xs[2] = {(uint64_t)(batch > 1 ? group.x_batch : ldx) * 2, (uint64_t)ldx * 2};
  uint32_t xb[3] = {GD_BK, 1, (uint32_t)mt};
  const CUtensorMap tx = make_tensor_map(x, TmaDType::BF16, 3, xd, xs, xb, true);
  const TileList list = group.list ? *group.list : TileList{nullptr, nullptr, 0};
  const dim3 grid(tiles, splits, z);
  if (out_f32)
    launch_gd<float>(tw, tx, (float*)out, ldo, M, N, K, mt, stages, smem, grid, alpha, tail, m_tiles, group.out_batch, list,
                     status, stream);
  else
    launch_gd<__nv_bfloat16>(tw, tx, (__nv_bfloat16*)out, ldo, M, N, K, mt, stages, smem, grid, alpha, tail, m_tiles,
                             group.out_batch, list, status, stream);
  count_launch();
  check_launch();
}

void gemm_segments(const void* x, long long ldx, const void* W, long long ldw, long long w_batch, int matrices, void* out,
                   long long ldo, int total_rows, int N, int K, const GemmTail& tail, const TileList& list, int* status,
                   cudaStream_t stream) {
  MB_REQUIRE(total_rows > 0 && N > 0 && K > 0 && list.tiles && list.count, "gemm_segments: empty problem");
  MB_REQUIRE(ldx % 8 == 0 && ldw % 8 == 0 && w_batch % 8 == 0 && ldo % 8 == 0 && N % 8 == 0 &&
                 (reinterpret_cast<uintptr_t>(out) & 15) == 0, "gemm_segments: alignment");
  MB_REQUIRE(tail.f_off == 0 || tail.f_off >= N, "gemm_segments: the up half starts after the gate half");
  MB_REQUIRE(tail.mul == nullptr && tail.gate == nullptr && tail.cap <= 0.f, "gemm_segments: gated tail only");
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(gemm_segments_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, GS_SMEM));
    configured = true;
  }
  const int per_tile = tail.f_off ? GS_BN / 2 : GS_BN, tiles_n = (N + per_tile - 1) / per_tile;
  const CUtensorMap tw = weight_map(W, ldw, w_batch, matrices, tail.f_off ? tail.f_off + N : N, K, 128);
  uint64_t xd[2] = {(uint64_t)K, (uint64_t)total_rows}, xs[1] = {(uint64_t)ldx * 2};
  uint32_t xb[2] = {GD_BK, GS_BM};
  const CUtensorMap tx = make_tensor_map(x, TmaDType::BF16, 2, xd, xs, xb, true);
  const long long work = (long long)list.max_tiles * tiles_n;
  const int grid = (int)(work < sm_count() ? work : sm_count());
  gemm_segments_kernel<<<grid, GS_THREADS, GS_SMEM, stream>>>(tw, tx, (__nv_bfloat16*)out, ldo, N, K, tiles_n, tail, list, status);
  count_launch();
  check_launch();
}

}  // namespace mb
