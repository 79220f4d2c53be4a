// Attention of absorbed latent queries over the paged latent cache on the tcgen05 tensor cores: every query head of a token
// reads the same cache rows, so the heads are the N columns of both products and the cache streams once per group of heads.
//   MMA 1  S^T[128 keys, G]     = C_tile[128 keys, wide + rot] . Q[G heads, wide + rot]^T          (both K-major)
//   MMA 2  O^T[128 dims, G] (m) += C_tile[:, 128 dims of block m]^T . (P_hi + P_lo)[G heads, 128 keys]^T   (C MN-major)
// The value of a key is its latent, so one tile in shared memory serves both.  Softmax weights stay 32-bit: they enter MMA 2
// as the sum of two 16-bit terms.
//
// A cluster of C CTAs shares one (token, group of heads, part); each CTA takes a contiguous range of 128-key tiles, keeps its
// accumulator in tensor memory, and after one cluster barrier the CTAs merge their heads through distributed shared memory.
// A tile (up to 147 KB) has one buffer; ranges are short because the tiles are dealt to all SMs.
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
constexpr int kTmemCols = 256;            // S^T (G), then up to four blocks of O^T (G each)
constexpr float kNegBig = -1.0e30f;
constexpr float kRaise = 8.f;             // the reference maximum is raised only past 2^8
// At most two CTAs per SM, so that their tensor-memory allocations always fit: a CTA that waits for an allocation while its
// cluster waits for it must not depend on other clusters.
constexpr int kMinSmem = 100 * 1024;

enum { BAR_Q = 0, BAR_FULL, BAR_S, BAR_P, BAR_O, BAR_COUNT };

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
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
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
  static constexpr int kPBytes = 4 * kHeadBox;           // two key boxes of leading terms, two of remainders
  static constexpr int kSmall = 2 * 4 * G * 4 + 2 * G * 4 + 128;   // maxima, sums, (max, sum) per head, barriers
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
  uint64_t* bars = reinterpret_cast<uint64_t*>(sm_ml + 2 * G);
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
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + G;

  pdl_wait_prior_grids();
  const int b = sequence_of(p.cu_seqlens, p.B, t);
  int len = p.past_seqlens[b] + (t - p.cu_seqlens[b]) + 1;
  if (len > p.max_blocks * p.block_size || len < 0) {
    if (tid == 0 && p.status) atomicExch(p.status, kStatusBadLength);
    len = len < 0 ? 0 : p.max_blocks * p.block_size;
  }
  const int all_tiles = (len + kTile - 1) / kTile;
  const int per_cta = (all_tiles + p.parts * p.cluster - 1) / (p.parts * p.cluster);
  const int tile0 = static_cast<int>(blockIdx.x) * per_cta;
  const int n_tiles = max(0, min(all_tiles - tile0, per_cta));
  const int o_blocks = (p.wide_boxes + 1) / 2;

  if (warp == 4) {
    // ---------------------------------------------------------- TMA producer + MMA issuer (lane i fetches piece i of a tile)
    const uint32_t idesc_s = umma_idesc_f16(kBf16, kTile, G);
    const uint32_t idesc_o = umma_idesc_f16(kBf16, 128, G) | (1u << 15);   // A (the tile read along its entries) is MN-major
    const uint32_t c_addr = smem_u32(smem), q_addr = smem_u32(sm_q), p_addr = smem_u32(sm_p);
    const int pieces = kTile / p.piece_rows;
    bool ok = true;
    if (n_tiles > 0 && lane == 0) {
      mbar_expect_tx(&bars[BAR_Q], static_cast<uint32_t>(p.boxes) * L::kHeadBox);
      for (int bx = 0; bx < p.boxes; ++bx) {
        if (bx < p.wide_boxes) tma_load_2d(sm_q + bx * L::kHeadBox, &tm_q, &bars[BAR_Q], bx * 64, t * p.N + head0);
        else tma_load_2d(sm_q + bx * L::kHeadBox, &tm_qr, &bars[BAR_Q], (bx - p.wide_boxes) * 64, t * p.N + head0);
      }
    }
    for (int i = 0; i < n_tiles && ok; ++i) {
      if (i > 0 && !mbar_wait(&bars[BAR_O], (i - 1) & 1)) { ok = false; break; }   // the tile before has been read
      if (lane == 0) mbar_expect_tx(&bars[BAR_FULL], static_cast<uint32_t>(p.boxes) * kBox);
      __syncwarp();
      if (lane < pieces) {
        // blocks outside the sequence or the pool are clamped: masked keys only have to be finite
        const int key = (tile0 + i) * kTile + lane * p.piece_rows;
        const int bi = min(key / p.block_size, p.max_blocks - 1);
        const int blk = min(max(p.block_table[static_cast<long long>(b) * p.max_blocks + bi], 0), p.num_blocks - 1);
        const int row = blk * p.block_size + key % p.block_size;
        uint8_t* dst = smem + lane * p.piece_rows * 128;
        for (int bx = 0; bx < p.boxes; ++bx) {
          if (bx < p.wide_boxes) tma_load_2d(dst + bx * kBox, &tm_c, &bars[BAR_FULL], bx * 64, row);
          else tma_load_2d(dst + bx * kBox, &tm_cr, &bars[BAR_FULL], (bx - p.wide_boxes) * 64, row);
        }
      }
      __syncwarp();
      if (i == 0 && !mbar_wait(&bars[BAR_Q], 0)) { ok = false; break; }
      if (!mbar_wait(&bars[BAR_FULL], i & 1)) { ok = false; break; }
      if (lane == 0) {
        tcgen05_fence_after();
        for (int bx = 0; bx < p.boxes; ++bx) {
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_f16(tmem_s, umma_desc_sw128(c_addr + bx * kBox + kk * 32), umma_desc_sw128(q_addr + bx * L::kHeadBox + kk * 32), idesc_s,
                     bx > 0 || kk > 0 ? 1u : 0u);
        }
        umma_commit(&bars[BAR_S]);
      }
      __syncwarp();
      if (!mbar_wait(&bars[BAR_P], i & 1)) { ok = false; break; }
      if (lane == 0) {
        tcgen05_fence_after();
        for (int m = 0; m < o_blocks; ++m) {
#pragma unroll
          for (int kk = 0; kk < kTile / 16; ++kk) {
            const uint64_t cdesc = umma_desc_mn_sw128(c_addr + 2 * m * kBox + kk * 2048, kBox, 1024);
            const uint32_t po = p_addr + (kk / 4) * L::kHeadBox + (kk % 4) * 32;
            umma_f16(tmem_o + m * G, cdesc, umma_desc_sw128(po), idesc_o, i > 0 || kk > 0 ? 1u : 0u);
            umma_f16(tmem_o + m * G, cdesc, umma_desc_sw128(po + 2 * L::kHeadBox), idesc_o, 1u);
          }
        }
        umma_commit(&bars[BAR_O]);
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
      const bool valid = (tile0 + i) * kTile + tid < len;
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
          if (ok && !mbar_wait(&bars[BAR_O], (i - 1) & 1)) ok = false;
          tcgen05_fence_after();
          for (int m = 0; m < o_blocks; ++m) {
#pragma unroll
            for (int c = 0; c < G; c += 16) {
              float ov[16];
              tmem_ld_x16(tmem_o + m * G + lane_addr + c, ov);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 16; ++j) ov[j] *= corr[c + j];
              tmem_st_x16(tmem_o + m * G + lane_addr + c, ov);
            }
          }
          tmem_st_wait();
        }
      }
      // weights of this key for every head, as leading term + remainder in the swizzled K-major layout MMA 2 reads
      uint8_t* pb = sm_p + (tid >> 6) * L::kHeadBox;
      const int col = tid & 63;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float pr = valid ? exp2f(sv[g] - m_ref[g]) : 0.f;
        const T hi = from_float<T>(pr);
        l_part[g] += pr;
        uint8_t* dst = pb + g * 128 + (((col >> 3) ^ (g & 7)) << 4) + (col & 7) * 2;
        *reinterpret_cast<T*>(dst) = hi;
        *reinterpret_cast<T*>(dst + 2 * L::kHeadBox) = from_float<T>(pr - to_float<T>(hi));
      }
      fence_proxy_async();
      tcgen05_fence_before();
      mbar_arrive(&bars[BAR_P]);
      asm volatile("bar.sync 1, 128;" ::: "memory");   // sm_max is free again
    }
    if (n_tiles > 0 && ok && !mbar_wait(&bars[BAR_O], (n_tiles - 1) & 1)) ok = false;
    tcgen05_fence_after();
    if (!ok && p.status) atomicExch(p.status, kStatusTimeoutEpilogue);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float s = warp_sum(l_part[g]);
      if (lane == 0) sm_sum[warp * G + g] = s;
      if (tid == 0) sm_ml[2 * g] = m_ref[g];
    }
    // O^T -> [G][wide_boxes * 64] fp32 in the tile's place
    const int pitch = p.wide_boxes * 64;
    if (n_tiles > 0) {
      float* stage = reinterpret_cast<float*>(smem);
      for (int m = 0; m < o_blocks; ++m) {
#pragma unroll
        for (int c = 0; c < G; c += 16) {
          float ov[16];
          tmem_ld_x16(tmem_o + m * G + lane_addr + c, ov);
          tmem_ld_wait();
          if (m * 128 + tid < pitch) {
#pragma unroll
            for (int j = 0; j < 16; ++j) stage[(c + j) * pitch + m * 128 + tid] = ov[j];
          }
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
  // ------------------------------------------------------------ merge: the CTAs of a cluster take every C-th head each
  if (warp < 4) {
    const int pitch = p.wide_boxes * 64;
    const uint32_t stage = smem_u32(smem), ml = smem_u32(sm_ml);
    for (int g = rank; g < n_heads; g += p.cluster) {
      float mc[8], w[8];
      float mm = kNegBig, sum = 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        mc[c] = c < p.cluster ? ld_dsmem(map_to_cta(ml + g * 8, c)) : kNegBig;
        mm = fmaxf(mm, mc[c]);
      }
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        w[c] = mc[c] <= kNegBig ? 0.f : exp2f(mc[c] - mm);
        if (c < p.cluster) sum = fmaf(w[c], ld_dsmem(map_to_cta(ml + g * 8 + 4, c)), sum);
      }
      const long long at = (static_cast<long long>(t) * p.N + head0 + g) * p.parts + part;
      for (int d = tid * 4; d < p.wide; d += 512) {   // wide is a multiple of eight
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          if (w[c] == 0.f) continue;                  // no keys: nothing was staged
          const float4 v = ld_dsmem4(map_to_cta(stage + (g * pitch + d) * 4, c));
          o.x = fmaf(w[c], v.x, o.x); o.y = fmaf(w[c], v.y, o.y); o.z = fmaf(w[c], v.z, o.z); o.w = fmaf(w[c], v.w, o.w);
        }
        *reinterpret_cast<float4*>(p.o + at * p.wide + d) = o;
      }
      if (tid == 0) {
        p.ml[at * 2] = mm;
        p.ml[at * 2 + 1] = sum;
      }
    }
  }
  if (p.cluster > 1) cluster_sync_all();   // staged accumulators stay until the others have read them
  else __syncthreads();
  if (warp == 4) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_s, kTmemCols);
  }
}

int cluster_for(int max_blocks, int block_size) {
  const long long tiles = (static_cast<long long>(max_blocks) * block_size + kTile - 1) / kTile;
  return tiles >= 8 ? 8 : (tiles >= 4 ? 4 : (tiles >= 2 ? 2 : 1));
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
  p.piece_rows = a.block_size < kTile ? a.block_size : kTile;
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
  const int need = L::bytes(p.boxes), smem = need > kMinSmem ? need : kMinSmem;
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

int heads_per_cta(int N) { return N > 16 ? 32 : 16; }

}  // namespace

int launch_latent_decode_tc(const ortb200_latent_decode_args* a, cudaStream_t stream) {
  if (!sizes_fit(a->N, a->wide, a->width, a->block_size, a->dtype) || a->T > 65535) return -2;
  const bool wide_group = heads_per_cta(a->N) == 32;
  if (a->dtype == ORTB200_BF16) return wide_group ? launch_tc<__nv_bfloat16, 32>(*a, stream) : launch_tc<__nv_bfloat16, 16>(*a, stream);
  return wide_group ? launch_tc<__half, 32>(*a, stream) : launch_tc<__half, 16>(*a, stream);
}

}  // namespace ortb200

using namespace ortb200;

extern "C" int ortb200_latent_decode_plan(int T, int N, int wide, int width, int block_size, int max_blocks, int dtype, int* parts) {
  if (parts) *parts = 1;
  if (T <= 0 || T > 65535 || max_blocks <= 0 || !sizes_fit(N, wide, width, block_size, dtype)) return 0;
  // one resident CTA per SM; a part should have at least a tile per CTA when the cache is full
  const int cluster = cluster_for(max_blocks, block_size);
  const int G = heads_per_cta(N);
  const long long ctas = static_cast<long long>(T) * ((N + G - 1) / G) * cluster;
  long long n = 148 / ctas;
  const long long tiles = (static_cast<long long>(max_blocks) * block_size + kTile - 1) / kTile;
  if (n > tiles / cluster) n = tiles / cluster;
  if (n > 16) n = 16;
  if (parts && n > 1) *parts = static_cast<int>(n);
  return 1;
}
