// Attention of absorbed latent queries over the paged latent cache on the tcgen05 tensor cores: every query head of a token
// reads the same cache rows, so the heads are the N columns of both products and the cache streams once per group of heads.
//   MMA 1  S^T[128 keys, G]     = C_tile[128 keys, wide + rot] . Q[G heads, wide + rot]^T          (both K-major)
//   MMA 2  O^T[128 dims, 2 G] (m) += C_tile[:, 128 dims of block m]^T . [P_hi; P_lo][2 G, 128 keys]^T   (C MN-major)
// The value of a key is its latent, so one tile in shared memory serves both.  Softmax weights stay 32-bit: they enter MMA 2
// as two 16-bit terms, whose sums lie in separate columns and are added at the end (the product is bound by reading the
// tile, so twice the columns cost nothing).
//
// A cluster of C CTAs shares one (token, group of heads, part); each CTA takes a contiguous range of keys, keeps its
// accumulator in tensor memory, and after one cluster barrier the CTAs merge their heads through distributed shared memory.
// Ranges are dealt in granules of 32 keys over all SMs.  A tile (up to 147 KB) has one buffer, but MMA 1 starts on each box
// of 64 entries as it arrives, and the boxes of a block of entries are refilled as soon as MMA 2 has read that block.
#include <cuda.h>
#include <cuda_runtime.h>
#include <math.h>
#include <type_traits>
#include "latent_internal.h"
#include "launch_util.cuh"
#include "ortb200_kernels.h"
#include "ptx_sm100.cuh"
#include "tensor_map.h"

namespace ortb200 {

namespace {

constexpr int kTile = 128;
constexpr int kBox = 128 * 128;           // [128 keys][64 entries] of 16-bit data
constexpr int kThreads = 160;             // 4 softmax warps + 1 TMA / MMA warp
constexpr int kMaxBoxes = 9;              // e.g. a latent of 512 and a rotated part of 64
constexpr int kMaxWideBoxes = 8;
constexpr int kGranule = 32;              // keys: unit of the ranges and of what is fetched and multiplied
constexpr float kNegBig = -1.0e30f;
constexpr float kRaise = 8.f;             // the reference maximum is raised only past 2^8
constexpr int kMaxCluster = 4;
constexpr int kMaxBlocks = kMaxWideBoxes / 2;

enum { BAR_Q = 0, BAR_S, BAR_P, BAR_FULL0, BAR_O0 = BAR_FULL0 + kMaxBoxes, BAR_COUNT = BAR_O0 + kMaxBlocks };

struct LatentTcParams {
  const int* cu_seqlens;
  const int* past_seqlens;
  const int* block_table;
  float* o;
  float* ml;
  int* status;
  int B, N, rank, wide, wide_boxes, boxes, parts, cluster;
  int block_size, max_blocks, num_blocks, piece_rows;
  float scale_log2;
};

__device__ __forceinline__ float redux_max(float v) {
  float r;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t map_to_cta(uint32_t local_smem_addr, uint32_t cta) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local_smem_addr), "r"(cta));
  return r;
}
__device__ __forceinline__ float ld_dsmem(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_dsmem4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr));
  return v;
}
__device__ __forceinline__ void tmem_st_x16(uint32_t taddr, const float* v) {
  uint32_t w[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) w[i] = __float_as_uint(v[i]);
  tmem_st_x16_u32(taddr, w);
}

template <int G>
struct Layout {
  static constexpr int kHeadBox = G * 128;               // [G heads][64 entries]
  static constexpr int kPBox = 2 * G * 128;              // [G leading terms, G remainders][64 keys]
  static constexpr int kPBytes = 2 * kPBox;
  // maxima, sums, (max, sum) per head, merge factors, barriers
  static constexpr int kSmall = 2 * 4 * G * 4 + 2 * G * 4 + G * kMaxCluster * 4 + 256;
  static constexpr int kTmemCols = G == 32 ? 512 : 256;   // S^T (G of the first 2 G columns), then up to four blocks of O^T (2 G each)
  // Shared memory is asked for so that the allocations of the CTAs on an SM always fit together: a CTA that waits for
  // tensor memory while its cluster waits for it must not depend on other clusters.
  static constexpr int kMinSmem = (G == 32 ? 120 : 100) * 1024;
  static int bytes(int boxes) { return boxes * (kBox + kHeadBox) + kPBytes + kSmall + 1024; }
};

template <typename T, int G>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_qr, const __grid_constant__ CUtensorMap tm_c,
                        const __grid_constant__ CUtensorMap tm_cr, const LatentTcParams p) {
  using L = Layout<G>;
  constexpr bool kBf16 = std::is_same<T, __nv_bfloat16>::value;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sm_q = smem + p.boxes * kBox;
  uint8_t* sm_p = sm_q + p.boxes * L::kHeadBox;
  float* sm_max = reinterpret_cast<float*>(sm_p + L::kPBytes);   // [4][G]
  float* sm_sum = sm_max + 4 * G;                                // [4][G]
  float* sm_ml = sm_sum + 4 * G;                                 // [G][2]
  float* sm_coef = sm_ml + 2 * G;                                // [heads merged here][kMaxCluster]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sm_coef + G * kMaxCluster);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + BAR_COUNT);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int part = blockIdx.x / p.cluster, rank = blockIdx.x % p.cluster;
  const int head0 = blockIdx.y * G, t = blockIdx.z;
  const int n_heads = min(G, p.N - head0);

  if (tid == 0) {
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_qr);
    tma_prefetch_desc(&tm_c);
    tma_prefetch_desc(&tm_cr);
    for (int i = 0; i < BAR_COUNT; ++i) mbar_init(&bars[i], i == BAR_P ? 128 : 1);
    fence_mbar_init();
  }
  if (warp == 4) {
    tmem_alloc(tmem_slot, L::kTmemCols);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 2 * G;

  pdl_wait_prior_grids();
  const int b = sequence_of(p.cu_seqlens, p.B, t);
  int len = p.past_seqlens[b] + (t - p.cu_seqlens[b]) + 1;
  if (len > p.max_blocks * p.block_size || len < 0) {
    if (tid == 0 && p.status) atomicExch(p.status, kStatusBadLength);
    len = len < 0 ? 0 : p.max_blocks * p.block_size;
  }
  const int ctas = p.parts * p.cluster, granules = (len + kGranule - 1) / kGranule;
  const int range = (granules + ctas - 1) / ctas * kGranule;
  const int k_begin = static_cast<int>(blockIdx.x) * range, k_end = min(len, k_begin + range);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + kTile - 1) / kTile : 0;
  const int o_blocks = (p.wide_boxes + 1) / 2;

  if (warp == 4) {
    // ---------------------------------------------------------- TMA producer + MMA issuer (lane i fetches piece i of a tile)
    const uint32_t idesc_s = umma_idesc_f16(kBf16, kTile, G);
    const uint32_t idesc_o = umma_idesc_f16(kBf16, 128, 2 * G) | (1u << 15);   // A (the tile read along its entries) is MN-major
    const uint32_t c_addr = smem_u32(smem), q_addr = smem_u32(sm_q), p_addr = smem_u32(sm_p);
    const int granule_pieces = kGranule / p.piece_rows;
    bool ok = true;
    if (n_tiles > 0 && lane == 0) {
      mbar_expect_tx(&bars[BAR_Q], static_cast<uint32_t>(p.boxes) * L::kHeadBox);
      for (int bx = 0; bx < p.boxes; ++bx) {
        if (bx < p.wide_boxes) tma_load_2d(sm_q + bx * L::kHeadBox, &tm_q, &bars[BAR_Q], bx * 64, t * p.N + head0);
        else tma_load_2d(sm_q + bx * L::kHeadBox, &tm_qr, &bars[BAR_Q], (bx - p.wide_boxes) * 64, t * p.N + head0);
      }
    }
    for (int i = 0; i < n_tiles && ok; ++i) {
      const int key0 = k_begin + i * kTile;
      const int live = (min(kTile, k_end - key0) + kGranule - 1) / kGranule;   // granules
      const int pieces = live * granule_pieces;   // at most 16: lanes take a piece of one of two boxes each
      const int sub = lane / pieces, piece = lane - sub * pieces, key = key0 + piece * p.piece_rows;
      // blocks outside the sequence or the pool are clamped: masked keys only have to be finite
      const int bi = min(key / p.block_size, p.max_blocks - 1);
      const int blk = min(max(p.block_table[static_cast<long long>(b) * p.max_blocks + bi], 0), p.num_blocks - 1);
      const int row = blk * p.block_size + key % p.block_size;
      for (int bx0 = 0; bx0 < p.boxes && ok; bx0 += 2) {
        if (i > 0 && bx0 / 2 < o_blocks && !mbar_wait(&bars[BAR_O0 + bx0 / 2], (i - 1) & 1)) { ok = false; break; }
        const int n = min(2, p.boxes - bx0);
        if (lane < n) mbar_expect_tx(&bars[BAR_FULL0 + bx0 + lane], static_cast<uint32_t>(live) * (kGranule * 128));
        __syncwarp();
        if (sub < n) {
          const int bx = bx0 + sub;
          uint8_t* dst = smem + bx * kBox + piece * p.piece_rows * 128;
          if (bx < p.wide_boxes) tma_load_2d(dst, &tm_c, &bars[BAR_FULL0 + bx], bx * 64, row);
          else tma_load_2d(dst, &tm_cr, &bars[BAR_FULL0 + bx], (bx - p.wide_boxes) * 64, row);
        }
        __syncwarp();
      }
      if (!ok) break;
      if (i == 0 && !mbar_wait(&bars[BAR_Q], 0)) { ok = false; break; }
      for (int bx = 0; bx < p.boxes && ok; ++bx) {
        if (!mbar_wait(&bars[BAR_FULL0 + bx], i & 1)) { ok = false; break; }
        if (lane == 0) {
          tcgen05_fence_after();
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_f16(tmem_s, umma_desc_sw128(c_addr + bx * kBox + kk * 32), umma_desc_sw128(q_addr + bx * L::kHeadBox + kk * 32), idesc_s,
                     bx > 0 || kk > 0 ? 1u : 0u);
        }
        __syncwarp();
      }
      if (!ok) break;
      if (lane == 0) {
        umma_commit(&bars[BAR_S]);
      }
      __syncwarp();
      if (!mbar_wait(&bars[BAR_P], i & 1)) { ok = false; break; }
      if (lane == 0) {
        tcgen05_fence_after();
        for (int m = 0; m < o_blocks; ++m) {
          for (int kk = 0; kk < live * (kGranule / 16); ++kk)
            umma_f16(tmem_o + m * 2 * G, umma_desc_mn_sw128(c_addr + 2 * m * kBox + kk * 2048, kBox, 1024),
                     umma_desc_sw128(p_addr + (kk / 4) * L::kPBox + (kk % 4) * 32), idesc_o, i > 0 || kk > 0 ? 1u : 0u);
          umma_commit(&bars[BAR_O0 + m]);
        }
      }
      __syncwarp();
    }
    if (!ok && lane == 0 && p.status) atomicExch(p.status, kStatusTimeoutMma);
  }

  if (warp < 4) {
    // ---------------------------------------------------------- softmax: thread = key of the tile, then entry of the latent
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    float m_ref[G], l_part[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {
      m_ref[g] = kNegBig;
      l_part[g] = 0.f;
    }
    // A wait that gives up clears `ok`; the loop still runs to its end (without further waits) so that every thread keeps
    // meeting the others at the named barriers and publishes P for the MMA warp.
    bool ok = true;
    for (int i = 0; i < n_tiles; ++i) {
      if (ok && !mbar_wait(&bars[BAR_S], i & 1)) ok = false;
      tcgen05_fence_after();
      float sv[G];
#pragma unroll
      for (int c = 0; c < G; c += 16) tmem_ld_x16(tmem_s + lane_addr + c, sv + c);
      tmem_ld_wait();
      const bool valid = k_begin + i * kTile + tid < k_end;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        sv[g] = valid ? sv[g] * p.scale_log2 : kNegBig;
        const float wm = redux_max(sv[g]);
        if (lane == 0) sm_max[warp * G + g] = wm;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      float corr[G];
      bool raise = false;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float mt = fmaxf(fmaxf(sm_max[g], sm_max[G + g]), fmaxf(sm_max[2 * G + g], sm_max[3 * G + g]));
        corr[g] = 1.f;
        if (mt > m_ref[g] + kRaise) {
          corr[g] = m_ref[g] <= kNegBig ? 0.f : exp2f(m_ref[g] - mt);
          m_ref[g] = mt;
          raise = true;
        }
      }
      if (raise) {   // uniform over the CTA: every thread saw the same maxima
#pragma unroll
        for (int g = 0; g < G; ++g) l_part[g] *= corr[g];
        if (i > 0) {
          if (ok && !mbar_wait(&bars[BAR_O0 + o_blocks - 1], (i - 1) & 1)) ok = false;
          tcgen05_fence_after();
          for (int m = 0; m < o_blocks; ++m) {
#pragma unroll
            for (int c = 0; c < 2 * G; c += 16) {
              float ov[16];
              tmem_ld_x16(tmem_o + m * 2 * G + lane_addr + c, ov);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 16; ++j) ov[j] *= corr[(c + j) % G];
              tmem_st_x16(tmem_o + m * 2 * G + lane_addr + c, ov);
            }
          }
          tmem_st_wait();
        }
      }
      // weights of this key for every head, as leading term + remainder in the swizzled K-major layout MMA 2 reads
      uint8_t* pb = sm_p + (tid >> 6) * L::kPBox;
      const int col = tid & 63;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float pr = valid ? exp2f(sv[g] - m_ref[g]) : 0.f;
        const T hi = from_float<T>(pr);
        l_part[g] += pr;
        uint8_t* dst = pb + g * 128 + (((col >> 3) ^ (g & 7)) << 4) + (col & 7) * 2;
        *reinterpret_cast<T*>(dst) = hi;
        *reinterpret_cast<T*>(dst + L::kHeadBox) = from_float<T>(pr - to_float<T>(hi));
      }
      fence_proxy_async();
      tcgen05_fence_before();
      mbar_arrive(&bars[BAR_P]);
      asm volatile("bar.sync 1, 128;" ::: "memory");   // sm_max is free again
    }
    // sums over the warp's keys: halving exchanges leave lane j with head j % G
    float acc[G];
#pragma unroll
    for (int g = 0; g < G; ++g) acc[g] = l_part[g];
#pragma unroll
    for (int o = G / 2; o >= 1; o >>= 1) {
#pragma unroll
      for (int g = 0; g < o; ++g) {
        const float send = lane & o ? acc[g] : acc[g + o], keep = lane & o ? acc[g + o] : acc[g];
        acc[g] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    if (G == 16) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 16);
    if (lane < G) sm_sum[warp * G + lane] = acc[0];
    if (tid == 0) {
#pragma unroll
      for (int g = 0; g < G; ++g) sm_ml[2 * g] = m_ref[g];
    }
    if (n_tiles > 0 && ok && !mbar_wait(&bars[BAR_O0 + o_blocks - 1], (n_tiles - 1) & 1)) ok = false;
    tcgen05_fence_after();
    if (!ok && p.status) atomicExch(p.status, kStatusTimeoutEpilogue);
    // O^T -> [G][wide_boxes * 64] fp32 in the tile's place
    const int pitch = p.wide_boxes * 64;
    if (n_tiles > 0) {
      float* stage = reinterpret_cast<float*>(smem);
      for (int m = 0; m < o_blocks; ++m) {
        float ov[2 * G];
#pragma unroll
        for (int c = 0; c < 2 * G; c += 16) tmem_ld_x16(tmem_o + m * 2 * G + lane_addr + c, ov + c);
        tmem_ld_wait();
        if (m * 128 + tid < pitch) {
#pragma unroll
          for (int g = 0; g < G; ++g) stage[g * pitch + m * 128 + tid] = ov[g] + ov[G + g];
        }
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (tid < G) sm_ml[2 * tid + 1] = sm_sum[tid] + sm_sum[G + tid] + sm_sum[2 * G + tid] + sm_sum[3 * G + tid];
  }
  tcgen05_fence_before();
  if (p.cluster > 1) cluster_sync_all();
  else __syncthreads();
  pdl_launch_dependents();
  // ------------------------------------------------------------ merge: CTA r of C takes heads r, r + C, ...
  const int mine = n_heads > rank ? (n_heads - rank + p.cluster - 1) / p.cluster : 0;
  const int pitch = p.wide_boxes * 64, vecs = p.wide / 4;   // wide is a multiple of eight
  const uint32_t stage_addr = smem_u32(smem), ml_addr = smem_u32(sm_ml);
  const long long at0 = static_cast<long long>(t) * p.N + head0;
  if (tid < mine) {
    const int g = rank + tid * p.cluster;
    float mc[kMaxCluster], lc[kMaxCluster], mm = kNegBig, sum = 0.f;
#pragma unroll
    for (int c = 0; c < kMaxCluster; ++c) {
      mc[c] = c < p.cluster ? ld_dsmem(map_to_cta(ml_addr + g * 8, c)) : kNegBig;
      lc[c] = c < p.cluster ? ld_dsmem(map_to_cta(ml_addr + g * 8 + 4, c)) : 0.f;
    }
#pragma unroll
    for (int c = 0; c < kMaxCluster; ++c) mm = fmaxf(mm, mc[c]);
#pragma unroll
    for (int c = 0; c < kMaxCluster; ++c) {
      const float w = mc[c] <= kNegBig ? 0.f : exp2f(mc[c] - mm);
      sum = fmaf(w, lc[c], sum);
      sm_coef[tid * kMaxCluster + c] = w;
    }
    p.ml[((at0 + g) * p.parts + part) * 2] = mm;
    p.ml[((at0 + g) * p.parts + part) * 2 + 1] = sum;
  }
  // a thread has four vectors of all CTAs in flight; what a CTA without keys has not staged is not used
  constexpr int kBatch = 4;
  for (int j0 = tid; j0 < mine * vecs || j0 == tid; j0 += kBatch * kThreads) {
    float4 v[kBatch][kMaxCluster];
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      const int j = j0 + i * kThreads, k = j / vecs, d = (j - k * vecs) * 4, g = rank + k * p.cluster;
#pragma unroll
      for (int c = 0; c < kMaxCluster; ++c)
        if (j < mine * vecs && c < p.cluster) v[i][c] = ld_dsmem4(map_to_cta(stage_addr + (g * pitch + d) * 4, c));
    }
    if (j0 == tid) __syncthreads();   // every thread comes by once: the factors are complete
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      const int j = j0 + i * kThreads, k = j / vecs, d = (j - k * vecs) * 4, g = rank + k * p.cluster;
      if (j >= mine * vecs) continue;
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int c = 0; c < kMaxCluster; ++c) {
        const float w = c < p.cluster ? sm_coef[k * kMaxCluster + c] : 0.f;
        if (w == 0.f) continue;
        o.x = fmaf(w, v[i][c].x, o.x); o.y = fmaf(w, v[i][c].y, o.y); o.z = fmaf(w, v[i][c].z, o.z); o.w = fmaf(w, v[i][c].w, o.w);
      }
      *reinterpret_cast<float4*>(p.o + ((at0 + g) * p.parts + part) * p.wide + d) = o;
    }
  }
  if (p.cluster > 1) cluster_sync_all();   // staged accumulators stay until the others have read them
  else __syncthreads();
  if (warp == 4) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_s, L::kTmemCols);
  }
}

int cluster_for(int max_blocks, int block_size) {
  const long long tiles = (static_cast<long long>(max_blocks) * block_size + kTile - 1) / kTile;
  return tiles >= 4 ? 4 : (tiles >= 2 ? 2 : 1);   // larger clusters leave too many SMs without a place for a whole one
}

template <typename T, int G>
int launch_tc(const ortb200_latent_decode_args& a, cudaStream_t stream) {
  using L = Layout<G>;
  const CUtensorMapDataType dt = std::is_same<T, __nv_bfloat16>::value ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
  LatentTcParams p{};
  p.cu_seqlens = a.cu_seqlens; p.past_seqlens = a.past_seqlens; p.block_table = a.block_table;
  p.o = a.o; p.ml = a.ml; p.status = a.status;
  p.B = a.B; p.N = a.N; p.rank = a.rank; p.wide = a.wide; p.parts = a.parts;
  p.wide_boxes = (a.wide + 63) / 64;
  p.boxes = p.wide_boxes + (a.width - a.wide + 63) / 64;
  p.cluster = cluster_for(a.max_blocks, a.block_size);
  p.block_size = a.block_size; p.max_blocks = a.max_blocks; p.num_blocks = a.num_blocks;
  p.piece_rows = a.block_size < kGranule ? a.block_size : kGranule;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  const int rot = a.width - a.wide;
  const int64_t rows = static_cast<int64_t>(a.num_blocks) * a.block_size, heads = static_cast<int64_t>(a.T) * a.N, pitch = static_cast<int64_t>(a.width) * 2;
  const char *q = static_cast<const char*>(a.q_abs), *c = static_cast<const char*>(a.cache);
  CUtensorMap tq, tqr, tc, tcr;
  if (make_tensor_map_2d(&tq, q, dt, 2, a.wide, heads, pitch, 64, G) != 0 || make_tensor_map_2d(&tc, c, dt, 2, a.wide, rows, pitch, 64, p.piece_rows) != 0)
    return -6;
  tqr = tq;
  tcr = tc;
  if (rot > 0 && (make_tensor_map_2d(&tqr, q + static_cast<int64_t>(a.wide) * 2, dt, 2, rot, heads, pitch, 64, G) != 0 ||
                  make_tensor_map_2d(&tcr, c + static_cast<int64_t>(a.wide) * 2, dt, 2, rot, rows, pitch, 64, p.piece_rows) != 0))
    return -6;
  const int need = L::bytes(p.boxes), smem = need > L::kMinSmem ? need : L::kMinSmem;
  auto kern = latent_decode_tc_kernel<T, G>;
  static int attr_smem = 0;
  if (smem > attr_smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
    attr_smem = smem;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.cluster * p.parts, (a.N + G - 1) / G, a.T);
  cfg.blockDim = dim3(kThreads, 1, 1);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attrs[2];
  int n = 0;
  attrs[n].id = cudaLaunchAttributeClusterDimension;
  attrs[n].val.clusterDim.x = p.cluster;
  attrs[n].val.clusterDim.y = 1;
  attrs[n++].val.clusterDim.z = 1;
  if (a.use_pdl) {
    attrs[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attrs[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  cfg.attrs = attrs;
  cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, kern, tq, tqr, tc, tcr, p) == cudaSuccess ? 0 : -11;
}

bool sizes_fit(int N, int wide, int width, int block_size, int dtype) {
  if (dtype != ORTB200_F16 && dtype != ORTB200_BF16) return false;
  if (N <= 0 || wide <= 0 || wide % 8 || width % 8 || width < wide) return false;
  if (block_size < 8 || (block_size & (block_size - 1)) != 0) return false;
  const int wide_boxes = (wide + 63) / 64, boxes = wide_boxes + (width - wide + 63) / 64;
  // an odd number of latent boxes is completed by the first box behind them
  return wide_boxes <= kMaxWideBoxes && boxes <= kMaxBoxes && (wide_boxes % 2 == 0 || boxes > wide_boxes);
}

// Sixteen heads per CTA as long as the groups of a token run side by side, else 32: the cache is then read half as often.
int heads_per_cta(int T, int N, int max_blocks, int block_size) {
  return N > 16 && static_cast<long long>(T) * ((N + 15) / 16) * cluster_for(max_blocks, block_size) > 148 ? 32 : 16;
}

}  // namespace

int launch_latent_decode_tc(const ortb200_latent_decode_args* a, cudaStream_t stream) {
  if (!sizes_fit(a->N, a->wide, a->width, a->block_size, a->dtype) || a->T > 65535) return -2;
  const bool wide_group = heads_per_cta(a->T, a->N, a->max_blocks, a->block_size) == 32;
  if (a->dtype == ORTB200_BF16) return wide_group ? launch_tc<__nv_bfloat16, 32>(*a, stream) : launch_tc<__nv_bfloat16, 16>(*a, stream);
  return wide_group ? launch_tc<__half, 32>(*a, stream) : launch_tc<__half, 16>(*a, stream);
}

}  // namespace ortb200

using namespace ortb200;

extern "C" int ortb200_latent_decode_plan(int T, int N, int wide, int width, int block_size, int max_blocks, int dtype, int* parts) {
  if (parts) *parts = 1;
  if (T <= 0 || T > 65535 || max_blocks <= 0 || !sizes_fit(N, wide, width, block_size, dtype)) return 0;
  // one resident CTA per SM; a part should have at least half a tile per CTA when the cache is full
  const int cluster = cluster_for(max_blocks, block_size);
  const int G = heads_per_cta(T, N, max_blocks, block_size);
  const long long ctas = static_cast<long long>(T) * ((N + G - 1) / G) * cluster;
  long long n = 148 / ctas;
  const long long tiles = (static_cast<long long>(max_blocks) * block_size + kTile - 1) / kTile;
  if (n > 2 * tiles / cluster) n = 2 * tiles / cluster;
  if (n > 16) n = 16;
  if (parts && n > 1) *parts = static_cast<int>(n);
  return 1;
}
