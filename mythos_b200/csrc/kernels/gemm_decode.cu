// GEMM for a few tokens: y[M, N] = alpha * x[M, K] W[N, K]^T with bf16 weights, M up to 128 per tile.
//
// A decode step is bound by reading the weights once, so W is the 128-row A operand of tcgen05.mma (the
// tokens are the narrow N side) and the reduction is split over the CTAs of a cluster until enough bytes
// are in flight. Each CTA streams its k-blocks of W and x through a TMA ring into one TMEM accumulator,
// stages the fp32 result in shared memory, and after a cluster barrier every CTA sums a share of the
// tokens over the peers' shared memory and stores it: no atomics, no accumulator to clear, the same
// result every time. With `f_off` > 0 a tile takes 64 rows of each half of a gate / up matrix and stores
// silu(gate) * up.
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

// grid (tiles of W, K splits = cluster size, token tiles)
template <typename OUT>
__global__ void __launch_bounds__(GD_THREADS)
gemm_decode_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, OUT* __restrict__ out,
                   long long ldo, int M, int N, int K, int mt, int stages, int f_off, float alpha, int* status) {
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
  const int m0 = blockIdx.z * mt;
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
        tma_load_2d(a, &tm_w, &full[st], kb * GD_BK, n0);
        if (f_off) tma_load_2d(a + GD_A_BYTES / 2, &tm_w, &full[st], kb * GD_BK, f_off + n0);
        tma_load_2d(a + GD_A_BYTES, &tm_x, &full[st], kb * GD_BK, m0);
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
      if (n < N) stf(out + (long long)(m0 + t) * ldo + n, y * alpha);
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
      if (n < N) stf(out + (long long)(m0 + t) * ldo + n, silu_f(g * alpha) * (u * alpha));
    }
  }
  gd_cluster_sync();               // nobody leaves while a peer still reads its shared memory
}

template <typename OUT>
void launch_gd(const CUtensorMap& tw, const CUtensorMap& tx, OUT* out, long long ldo, int M, int N, int K, int mt, int stages,
               int smem, int tiles, int splits, int m_tiles, int f_off, float alpha, int* status, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(gemm_decode_kernel<OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    configured = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, splits, m_tiles);
  cfg.blockDim = dim3(GD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = splits;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  MB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, gemm_decode_kernel<OUT>, tw, tx, out, ldo, M, N, K, mt, stages, f_off, alpha, status));
}

}  // namespace

void gemm_decode(const void* x, long long ldx, const void* W, long long ldw, void* out, bool out_f32, long long ldo, int M,
                 int N, int K, int f_off, float alpha, int* status, cudaStream_t stream) {
  MB_REQUIRE(M > 0 && N > 0 && K > 0, "gemm_decode: empty problem");
  MB_REQUIRE(ldx % 8 == 0 && ldw % 8 == 0, "gemm_decode: row strides must be multiples of 8 elements");
  MB_REQUIRE(f_off == 0 || f_off >= N, "gemm_decode: the up half starts after the gate half");
  int mt = (M + 15) / 16 * 16;
  if (mt > 128) mt = 128;
  const int m_tiles = (M + mt - 1) / mt;
  const int rows_per_tile = f_off ? GD_BM / 2 : GD_BM;
  const int tiles = (N + rows_per_tile - 1) / rows_per_tile;
  const int kblocks = (K + GD_BK - 1) / GD_BK;
  int splits = 1;
  while (splits < 8 && splits * 2 <= kblocks / 2 && tiles * m_tiles * splits * 2 <= 3 * sm_count()) splits *= 2;
  const int stage = GD_A_BYTES + mt * GD_BK * 2;
  int stages = (100 * 1024) / stage;
  if (stages > GD_MAX_STAGES) stages = GD_MAX_STAGES;
  const int smem = stages * stage + 1024;          // >= mt * 512 bytes of staged result for every mt
  const long long w_rows = f_off ? (long long)f_off + N : N;
  uint64_t wd[2] = {(uint64_t)K, (uint64_t)w_rows}, ws[1] = {(uint64_t)ldw * 2};
  uint32_t wb[2] = {GD_BK, (uint32_t)rows_per_tile};
  uint64_t xd[2] = {(uint64_t)K, (uint64_t)M}, xs[1] = {(uint64_t)ldx * 2};
  uint32_t xb[2] = {GD_BK, (uint32_t)mt};
  const CUtensorMap tw = make_tensor_map(W, TmaDType::BF16, 2, wd, ws, wb, true);
  const CUtensorMap tx = make_tensor_map(x, TmaDType::BF16, 2, xd, xs, xb, true);
  if (out_f32)
    launch_gd<float>(tw, tx, (float*)out, ldo, M, N, K, mt, stages, smem, tiles, splits, m_tiles, f_off, alpha, status, stream);
  else
    launch_gd<__nv_bfloat16>(tw, tx, (__nv_bfloat16*)out, ldo, M, N, K, mt, stages, smem, tiles, splits, m_tiles, f_off, alpha,
                             status, stream);
  count_launch();
  check_launch();
}

}  // namespace mb
