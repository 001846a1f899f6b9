// Routing of tokens to experts for serving (hybrid_api.h).
//
//   expert_select  one warp per token: scores of all router logits (softmax or sigmoid), choice scores (score +
//                  correction), the best groups of neighbouring experts, the best experts in them, a place inside each
//                  chosen expert's row segment. The last CTA to finish turns the counts into segments and a
//                  tile list for the grouped GEMMs and clears the counts for the next launch.
//   expert_gather  token rows into their segments.
//
// All arithmetic is fp32. Which place a token gets inside a segment depends on the order in which warps
// arrive; its result does not, because rows of a GEMM do not mix.
#include "common.cuh"
#include "host_util.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"

namespace mb {
namespace {

constexpr int ER_WARPS = 8;
constexpr int ER_MAX_EXPERTS = 1024;

// Largest value and, among equals, lowest index over the warp.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}

__global__ void __launch_bounds__(ER_WARPS * 32)
expert_select_kernel(const float* __restrict__ logits, long long ldz, const float* __restrict__ correction, RouterSpec s,
                     RouterBuffers b, int tile_rows, int rows) {
  extern __shared__ float sm[];
  __shared__ int s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = s.experts, size = E / s.groups;
  float* score = sm + warp * (2 * E + s.groups);
  float* choice = score + E;
  float* best = choice + E;          // per group: its largest choice score, then 1 (kept) or 0
  const int t = blockIdx.x * ER_WARPS + warp;
  if (t < rows) {
    const float* z = logits + (long long)t * ldz;
    if (s.sigmoid) {
      for (int e = lane; e < E; e += 32) {
        const float p = sigmoid_f(z[e]);
        score[e] = p;
        choice[e] = p + (correction ? correction[e] : 0.f);
      }
    } else {
      float mx = -INFINITY;
      for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
      mx = warp_max(mx);
      float sum = 0.f;
      for (int e = lane; e < E; e += 32) {
        const float p = expf(z[e] - mx);
        score[e] = p;
        sum += p;
      }
      sum = warp_sum(sum);
      for (int e = lane; e < E; e += 32) {
        const float p = score[e] / sum;
        score[e] = p;
        choice[e] = p + (correction ? correction[e] : 0.f);
      }
    }
    __syncwarp();
    if (s.keep < s.groups) {
      for (int g = lane; g < s.groups; g += 32) {
        float m = choice[g * size], m2 = -INFINITY;     // the two largest
        for (int i = 1; i < size; ++i) {
          const float c = choice[g * size + i];
          m2 = fmaxf(m2, fminf(m, c));
          m = fmaxf(m, c);
        }
        best[g] = s.group_best == 2 && size > 1 ? m + m2 : m;
      }
      __syncwarp();
      for (int j = 0; j < s.groups - s.keep; ++j) {      // strike out the worst groups
        float v = -INFINITY;
        int at = -1;
        for (int g = lane; g < s.groups; g += 32)
          if (best[g] != INFINITY && (at < 0 || -best[g] >= v)) {
            v = -best[g];
            at = g;
          }
        // among equals the highest index goes: the lowest one is the one that is kept
        int key = at < 0 ? 0x7fffffff : -at;
        if (at < 0) v = -INFINITY;
        warp_argmax(v, key);
        const int g = -key;
        if (g >= 0 && g < s.groups) {
          for (int i = lane; i < size; i += 32) choice[g * size + i] = -INFINITY;
          if (lane == 0) best[g] = INFINITY;
        }
        __syncwarp();
      }
    }
    float mine = 0.f, total = 0.f;                      // lane j keeps the score of choice j
    for (int j = 0; j < s.top; ++j) {
      float v = -INFINITY;
      int at = 0x7fffffff;
      for (int e = lane; e < E; e += 32)
        if (choice[e] > v) {
          v = choice[e];
          at = e;
        }
      warp_argmax(v, at);
      at = min(at, E - 1);
      const float p = score[at];
      total += p;
      if (lane == j) mine = p;
      if (lane == 0) {
        choice[at] = -INFINITY;
        const long long o = (long long)t * s.top + j;
        b.idx[o] = at;
        b.slot[o] = atomicAdd(&b.counts[at], 1);
      }
      __syncwarp();
    }
    if (lane < s.top) b.weight[(long long)t * s.top + lane] = s.normalise ? mine / (total + 1e-20f) * s.scale : mine;
  }
  // ---- the last CTA plans the segments
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(&b.counts[E], 1) == (int)gridDim.x - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  int* cnt = reinterpret_cast<int*>(sm);
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    cnt[e] = atomicExch(&b.counts[e], 0);
    if (e == 0) b.counts[E] = 0;
  }
  __syncthreads();
  if (warp != 0) return;
  const int per = (E + 31) / 32, lo = min(E, lane * per), hi = min(E, lo + per);
  int n = 0, tiles = 0;
  for (int e = lo; e < hi; ++e) {
    n += cnt[e];
    tiles += (cnt[e] + tile_rows - 1) / tile_rows;
  }
  int row = n, tile = tiles;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int a = __shfl_up_sync(0xffffffffu, row, o), c = __shfl_up_sync(0xffffffffu, tile, o);
    if (lane >= o) {
      row += a;
      tile += c;
    }
  }
  if (lane == 31) *b.tile_count = min(tile, b.max_tiles);
  row -= n;
  tile -= tiles;
  for (int e = lo; e < hi; ++e) {
    b.offset[e] = row;
    for (int r = 0; r < cnt[e]; r += tile_rows, ++tile)
      if (tile < b.max_tiles) {
        b.tiles[3 * tile] = e;
        b.tiles[3 * tile + 1] = row + r;
        b.tiles[3 * tile + 2] = min(tile_rows, cnt[e] - r);
      }
    row += cnt[e];
  }
}

// One warp per (token, choice).
__global__ void __launch_bounds__(256)
expert_gather_kernel(const uint8_t* __restrict__ h, long long ldh, RouterSpec s, RouterBuffers b, uint8_t* __restrict__ out,
                     int* __restrict__ row, long long row_bytes, long long pairs) {
  const int lane = threadIdx.x & 31;
  for (long long p = (long long)blockIdx.x * 8 + (threadIdx.x >> 5); p < pairs; p += (long long)gridDim.x * 8) {
    const int to = b.offset[b.idx[p]] + b.slot[p];
    if (lane == 0) row[p] = to;
    const uint4* src = reinterpret_cast<const uint4*>(h + (p / s.top) * ldh);
    uint4* dst = reinterpret_cast<uint4*>(out + (long long)to * row_bytes);
    for (long long i = lane; i < row_bytes / 16; i += 32) dst[i] = src[i];
  }
}

}  // namespace

void expert_select(const float* logits, long long ldz, const float* correction, const RouterSpec& s, const RouterBuffers& b,
                   int tile_rows, int rows, cudaStream_t stream) {
  MB_REQUIRE(s.experts > 0 && s.experts <= ER_MAX_EXPERTS, "expert_select: at most 1024 experts");
  MB_REQUIRE(s.groups > 0 && s.experts % s.groups == 0 && s.keep > 0 && s.keep <= s.groups &&
                 s.top > 0 && s.top <= 32 && s.top <= s.experts / s.groups * s.keep && (s.group_best == 1 || s.group_best == 2),
             "expert_select: groups / top");
  MB_REQUIRE(tile_rows > 0, "expert_select: tile rows");
  if (rows == 0) return;
  const int smem = ER_WARPS * (2 * s.experts + s.groups) * 4;
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(expert_select_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    configured = true;
  }
  expert_select_kernel<<<(rows + ER_WARPS - 1) / ER_WARPS, ER_WARPS * 32, smem, stream>>>(logits, ldz, correction, s, b,
                                                                                         tile_rows, rows);
  count_launch();
  check_launch();
}

void expert_gather(const void* h, long long ldh_bytes, const RouterSpec& s, const RouterBuffers& b, void* out, int* row,
                   long long row_bytes, int rows, cudaStream_t stream) {
  MB_REQUIRE(row_bytes % 16 == 0 && ldh_bytes % 16 == 0, "expert_gather: rows of whole 16-byte units");
  if (rows == 0) return;
  const long long pairs = (long long)rows * s.top, want = (pairs + 7) / 8, cap = (long long)sm_count() * 8;
  expert_gather_kernel<<<(int)(want < cap ? want : cap), 256, 0, stream>>>((const uint8_t*)h, ldh_bytes, s, b, (uint8_t*)out, row,
                                                                           row_bytes, pairs);
  count_launch();
  check_launch();
}

}  // namespace mb
