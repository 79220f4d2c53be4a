// Flash attention of packed prompts whose softmax weights stay 32-bit up to the product with V: P enters MMA 2 as the sum of
// two 16-bit terms.  Causal, optionally within a window or a chunk of the sequence.
//
//   MMA 1  S[128 q, 64 keys]   = Q . K^T                      (shared memory, both K-major)
//   softmax threads (one per query row) read their row of S from tensor memory into registers and write P back over it:
//   leading terms in columns [0, 32) of the buffer, remainders in [32, 64), as packed pairs
//   MMA 2  O[128 q, dv]       += (P_hi + P_lo) . V            (A from tensor memory, V MN-major)
// P needs no shared memory and S / P take two buffers of 64 columns, so two CTAs share an SM (96 KB and 256 columns each) and
// one's tensor-core work hides behind the other's softmax.
//
// Two forms.  Paged: keys and values of a head lie in cache blocks named by the block table.  Latent: queries and keys are an
// unrotated part per head and a rotated part (of the keys one that all heads share), keys and values were expanded from
// their latents and lie packed, sequence behind sequence; tensor maps zero-fill heads narrower than a box of 64.
#include <cuda.h>
#include <cuda_runtime.h>
#include <math.h>
#include "attn_internal.h"
#include "ortb200_kernels.h"
#include "ptx_sm100.cuh"
#include "tensor_map.h"

namespace ortb200 {

namespace {

constexpr int kQT = 128;      // query rows per CTA
constexpr int kKT = 64;       // keys per tile
constexpr int kThreads = 192; // TMA warp, MMA warp, four softmax warps
constexpr int kTmemCols = 256;

struct SplitParams {
  AttnParams a;
  // latent form
  int plain_boxes;       // leading boxes of a query / key tile that hold the unrotated part
  int dv;                // value head size (columns of a head that are stored)
  const void* gate;      // optional [T, gate_ld]: sigmoid factor per token and head
  long long gate_ld;
};

// KB / VB: 64-element boxes of a query / key tile and of a value tile; STAGES: key and value tiles in flight
template <int KB, int VB, int STAGES>
struct Smem {
  static constexpr int kQBox = 128 * 128, kBox = kKT * 128;
  static constexpr int kStageBytes = (KB + VB) * kBox;
  static constexpr int kOffKV = KB * kQBox;
  static constexpr int kOffBar = kOffKV + STAGES * kStageBytes;
  static constexpr int kTotal = kOffBar + 256 + 1024;
};

enum { BAR_Q = 0, BAR_K_FULL, BAR_K_EMPTY = BAR_K_FULL + 2, BAR_V_FULL = BAR_K_EMPTY + 2, BAR_V_EMPTY = BAR_V_FULL + 2, BAR_S = BAR_V_EMPTY + 2,
       BAR_P = BAR_S + 2, BAR_O = BAR_P + 2, BAR_END, BAR_COUNT };

template <int KB, int VB, int STAGES, bool LATENT>
__global__ void __launch_bounds__(kThreads, 2)
attn_split_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                  const __grid_constant__ CUtensorMap tm_qr, const __grid_constant__ CUtensorMap tm_kr, const SplitParams sp) {
  using L = Smem<KB, VB, STAGES>;
  constexpr int HD = VB * 64;   // columns of O
  const AttnParams& p = sp.a;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kOffBar);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + BAR_COUNT);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // query tiles of all sequences are numbered from the last sequence's last tile (most keys) on; the grid is an upper bound
  pdl_wait_prior_grids();
  int b, q0 = 0, q_row0 = 0, S = 0, k_row0 = 0, tile = blockIdx.x;
  for (b = p.B - 1; b >= 0; --b) {
    q_row0 = p.cu_seqlens[b];
    S = p.cu_seqlens[b + 1] - q_row0;
    const int tiles = (S + kQT - 1) / kQT;
    if (tile < tiles) {
      q0 = (tiles - 1 - tile) * kQT;
      break;
    }
    tile -= tiles;
  }
  if (b < 0) return;
  if (LATENT) {
    for (int i = 0; i < b; ++i) k_row0 += p.past_seqlens[i];
    k_row0 += q_row0;
  }
  const int head = blockIdx.y, kvh = LATENT ? head : head / (p.N / p.Nk);

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
    if (LATENT) {
      tma_prefetch_desc(&tm_qr);
      tma_prefetch_desc(&tm_kr);
    }
    for (int i = 0; i < BAR_COUNT; ++i) mbar_init(&bars[i], i == BAR_P || i == BAR_P + 1 ? 128 : 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_s = *tmem_slot;          // S / P: two buffers of 64 columns
  const uint32_t tmem_o = tmem_s + 2 * kKT;    // O, accumulated over all key tiles

  const int past = p.past_seqlens[b], total = past + S;
  const int kv_end = min(total, past + q0 + kQT);
  int kv_begin = 0;
  if (p.window > 0) kv_begin = max(0, past + q0 - p.window + 1) / kKT * kKT;
  if (p.chunk > 0) kv_begin = max(kv_begin, (past + q0) / p.chunk * p.chunk / kKT * kKT);
  const int n_tiles = (kv_end - kv_begin + kKT - 1) / kKT;

  if (warp == 0) {
    if (lane == 0 && n_tiles > 0) {
      mbar_expect_tx(&bars[BAR_Q], KB * L::kQBox);
      for (int bx = 0; bx < KB; ++bx) {
        if (LATENT && bx >= sp.plain_boxes) tma_load_4d(smem + bx * L::kQBox, &tm_qr, &bars[BAR_Q], (bx - sp.plain_boxes) * 64, q_row0 + q0, head, 0);
        else tma_load_4d(smem + bx * L::kQBox, &tm_q, &bars[BAR_Q], bx * 64, q_row0 + q0, head, 0);
      }
      bool ok = true;
      for (int t = 0; t < n_tiles && ok; ++t) {
        const int s = t % STAGES, parity = (t / STAGES - 1) & 1, key0 = kv_begin + t * kKT;
        // coordinates behind the entry: (row, head, 0), or (position in block, head, block)
        int c1 = k_row0 + key0, c3 = 0;
        if (!LATENT) {
          const int bi = min(key0 / p.block_size, p.max_blocks - 1);
          c1 = key0 % p.block_size;
          c3 = min(max(p.block_table[static_cast<long long>(b) * p.max_blocks + bi], 0), p.num_blocks - 1);
        }
        uint8_t* st = smem + L::kOffKV + s * L::kStageBytes;
        if (t >= STAGES && !mbar_wait(&bars[BAR_K_EMPTY + s], parity)) { ok = false; break; }
        mbar_expect_tx(&bars[BAR_K_FULL + s], KB * L::kBox);
        for (int bx = 0; bx < KB; ++bx) {
          if (LATENT && bx >= sp.plain_boxes)   // one rotated part for all heads
            tma_load_4d(st + bx * L::kBox, &tm_kr, &bars[BAR_K_FULL + s], (bx - sp.plain_boxes) * 64, c1, 0, 0);
          else
            tma_load_4d(st + bx * L::kBox, &tm_k, &bars[BAR_K_FULL + s], bx * 64, c1, kvh, c3);
        }
        if (t >= STAGES && !mbar_wait(&bars[BAR_V_EMPTY + s], parity)) { ok = false; break; }
        mbar_expect_tx(&bars[BAR_V_FULL + s], VB * L::kBox);
        for (int bx = 0; bx < VB; ++bx) tma_load_4d(st + (KB + bx) * L::kBox, &tm_v, &bars[BAR_V_FULL + s], bx * 64, c1, kvh, c3);
      }
      if (!ok && p.status) atomicExch(p.status, kStatusTimeoutProducer);
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      const uint32_t idesc_s = umma_idesc_f16(p.bf16 != 0, kQT, kKT);
      const uint32_t idesc_o = umma_idesc_f16_bmn(p.bf16 != 0, kQT, HD);
      const uint32_t q_addr = smem_u32(smem);
      auto issue_s = [&](int t) {
        const uint32_t k_addr = smem_u32(smem + L::kOffKV + (t % STAGES) * L::kStageBytes);
#pragma unroll
        for (int kk = 0; kk < KB * 4; ++kk)
          umma_f16(tmem_s + (t & 1) * kKT, umma_desc_sw128(q_addr + (kk / 4) * L::kQBox + (kk % 4) * 32),
                   umma_desc_sw128(k_addr + (kk / 4) * L::kBox + (kk % 4) * 32), idesc_s, kk > 0 ? 1u : 0u);
        umma_commit(&bars[BAR_S + (t & 1)]);
        umma_commit(&bars[BAR_K_EMPTY + t % STAGES]);
      };
      bool ok = mbar_wait(&bars[BAR_Q], 0) && mbar_wait(&bars[BAR_K_FULL], 0);
      if (ok) {
        tcgen05_fence_after();
        issue_s(0);
      }
      for (int t = 0; t < n_tiles && ok; ++t) {
        const int s = t % STAGES;
        if (t + 1 < n_tiles) {
          // S of the next tile goes over P of tile t - 1, whose product has to be finished
          if (t > 0 && !mbar_wait(&bars[BAR_O], (t - 1) & 1)) { ok = false; break; }
          if (!mbar_wait(&bars[BAR_K_FULL + (t + 1) % STAGES], ((t + 1) / STAGES) & 1)) { ok = false; break; }
          tcgen05_fence_after();
          issue_s(t + 1);
        }
        if (!mbar_wait(&bars[BAR_V_FULL + s], (t / STAGES) & 1) || !mbar_wait(&bars[BAR_P + (t & 1)], (t >> 1) & 1)) { ok = false; break; }
        tcgen05_fence_after();
        const uint32_t v_addr = smem_u32(smem + L::kOffKV + s * L::kStageBytes + KB * L::kBox);
        const uint32_t tmem_p = tmem_s + (t & 1) * kKT;
#pragma unroll
        for (int kk = 0; kk < kKT / 16; ++kk) {
          const uint64_t vdesc = umma_desc_mn_sw128(v_addr + kk * 2048, L::kBox, 1024);
          umma_f16_ts(tmem_o, tmem_p + kk * 8, vdesc, idesc_o, t > 0 || kk > 0 ? 1u : 0u);
          umma_f16_ts(tmem_o, tmem_p + kKT / 2 + kk * 8, vdesc, idesc_o, 1u);
        }
        umma_commit(&bars[BAR_O]);
        umma_commit(&bars[BAR_V_EMPTY + s]);
        if (t == n_tiles - 1) umma_commit(&bars[BAR_END]);
      }
      if (!ok && p.status) atomicExch(p.status, kStatusTimeoutMma);
    }
  } else {
    const int qw = warp & 3, s_idx = q0 + qw * 32 + lane, pos = past + s_idx;
    const uint32_t lane_addr = static_cast<uint32_t>(qw * 32) << 16;
    // The reference maximum of a row is raised only when a tile exceeds it by 2^8 (weights stay below 256), so the
    // accumulator in tensor memory is rescaled a few times per row instead of once per tile.
    constexpr float kRaise = 8.f;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int t = 0; t < n_tiles; ++t) {
      // S of this tile was issued after the product of tile t - 2 had finished: BAR_O is at most one phase back below
      if (ok && !mbar_wait(&bars[BAR_S + (t & 1)], (t >> 1) & 1)) ok = false;
      tcgen05_fence_after();
      const int key0 = kv_begin + t * kKT;
      const uint32_t s_addr = tmem_s + (t & 1) * kKT + lane_addr;
      float sv[kKT];
      tmem_ld_x32(s_addr, sv);
      tmem_ld_x32(s_addr + 32, sv + 32);
      tmem_ld_wait();
      // interior tiles (every key visible to every row of this query tile) skip the per-element mask
      if (key0 + kKT - 1 > past + q0 || p.window > 0 || (p.chunk > 0 && key0 < (past + q0 + kQT - 1) / p.chunk * p.chunk)) {
        const int hi = min(total, pos + 1) - key0;
        int lo = p.window > 0 ? pos - p.window + 1 - key0 : -kKT;
        if (p.chunk > 0) lo = max(lo, pos / p.chunk * p.chunk - key0);
#pragma unroll
        for (int j = 0; j < kKT; ++j) sv[j] = (j < hi && j >= lo) ? sv[j] : -INFINITY;
      }
      float m_raw = -INFINITY;
#pragma unroll
      for (int j = 0; j < kKT; j += 2) m_raw = fmax3(m_raw, sv[j], sv[j + 1]);
      const float m_tile = m_raw * p.scale_log2;     // scale > 0: -inf stays -inf
      const bool raise = m_tile > m + kRaise;        // also the first finite maximum of a row (m = -inf)
      if (__any_sync(0xffffffffu, raise)) {
        // tensor-memory accesses are warp-wide: every lane takes part, rows that keep their maximum scale by 1
        const float corr = raise ? (m == -INFINITY ? 0.f : exp2f(m - m_tile)) : 1.f;
        if (t > 0) {
          if (ok && !mbar_wait(&bars[BAR_O], (t - 1) & 1)) ok = false;
          tcgen05_fence_after();
#pragma unroll 1
          for (int c = 0; c < HD; c += 32) {
            float v[32];
            tmem_ld_x32(tmem_o + lane_addr + c, v);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] *= corr;
            tmem_st_x32(tmem_o + lane_addr + c, v);
          }
        }
        l *= corr;
        if (raise) m = m_tile;
      }
      const float neg_m = m == -INFINITY ? 0.f : -m;   // a row without a visible key so far: weights 0
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int c = 0; c < kKT; c += 32) {
        uint32_t hi[16], rest[16];
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
          const float p0 = ex2_approx(fmaf(sv[c + j], p.scale_log2, neg_m));
          const float p1 = ex2_approx(fmaf(sv[c + j + 1], p.scale_log2, neg_m));
          sum0 += p0;
          sum1 += p1;
          if (p.bf16) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
            const __nv_bfloat162 e = __floats2bfloat162_rn(p0 - __bfloat162float(h.x), p1 - __bfloat162float(h.y));
            hi[j / 2] = *reinterpret_cast<const uint32_t*>(&h);
            rest[j / 2] = *reinterpret_cast<const uint32_t*>(&e);
          } else {
            const __half2 h = __floats2half2_rn(p0, p1);
            const __half2 e = __floats2half2_rn(p0 - __half2float(h.x), p1 - __half2float(h.y));
            hi[j / 2] = *reinterpret_cast<const uint32_t*>(&h);
            rest[j / 2] = *reinterpret_cast<const uint32_t*>(&e);
          }
        }
        tmem_st_x16_u32(s_addr + c / 2, hi);
        tmem_st_x16_u32(s_addr + kKT / 2 + c / 2, rest);
      }
      l += sum0 + sum1;
      tmem_st_wait();
      tcgen05_fence_before();
      mbar_arrive(&bars[BAR_P + (t & 1)]);
    }
    // (BAR_O may still be two phases back here, where its parity would already read as done)
    if (n_tiles > 0 && ok && !mbar_wait(&bars[BAR_END], 0)) ok = false;
    tcgen05_fence_after();
    if (!ok && p.status) atomicExch(p.status, kStatusTimeoutEpilogue);
    pdl_launch_dependents();
    float denom = l, rescale = 1.f;
    if (p.head_sink) {
      const float sink = (p.bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.head_sink)[head])
                                 : __half2float(static_cast<const __half*>(p.head_sink)[head])) * 1.4426950408889634f;
      const float mm = fmaxf(m, sink);
      rescale = m == -INFINITY ? 0.f : exp2f(m - mm);
      denom = l * rescale + exp2f(sink - mm);
    }
    float inv = denom > 0.f && n_tiles > 0 ? rescale / denom : 0.f;
    if (LATENT && sp.gate != nullptr && s_idx < S) {
      const long long gi = (q_row0 + s_idx) * sp.gate_ld + head;
      const float g = p.bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(sp.gate)[gi]) : __half2float(static_cast<const __half*>(sp.gate)[gi]);
      inv *= 1.f / (1.f + __expf(-g));
    }
    uint8_t* orow = static_cast<uint8_t*>(p.out) + 2 * ((q_row0 + s_idx) * p.o_strides[1] + head * p.o_strides[2]);
#pragma unroll 1
    for (int c0 = 0; c0 < HD; c0 += 32) {
      float v[32];
      tmem_ld_x32(tmem_o + lane_addr + c0, v);
      tmem_ld_wait();
      if (ok && n_tiles > 0 && s_idx < S) {
#pragma unroll
        for (int c = 0; c < 32; c += 8) {
          if (c0 + c >= sp.dv) break;
          uint32_t w[4];
#pragma unroll
          for (int j = 0; j < 8; j += 2) {
            if (p.bf16) {
              const __nv_bfloat162 h = __floats2bfloat162_rn(v[c + j] * inv, v[c + j + 1] * inv);
              w[j / 2] = *reinterpret_cast<const uint32_t*>(&h);
            } else {
              const __half2 h = __floats2half2_rn(v[c + j] * inv, v[c + j + 1] * inv);
              w[j / 2] = *reinterpret_cast<const uint32_t*>(&h);
            }
          }
          *reinterpret_cast<uint4*>(orow + (c0 + c) * 2) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
  }

  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_s, kTmemCols);
  }
}

template <int KB, int VB, int STAGES, bool LATENT>
int launch_split(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tqr, const CUtensorMap& tkr,
                 const SplitParams& p, int T, cudaStream_t stream) {
  using L = Smem<KB, VB, STAGES>;
  auto kern = attn_split_kernel<KB, VB, STAGES, LATENT>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal) != cudaSuccess) return -10;
    attr_set = true;
  }
  // every sequence has at most one partly filled query tile
  const dim3 grid(T / kQT + (p.a.B < T ? p.a.B : T), p.a.N, 1);
  kern<<<grid, kThreads, L::kTotal, stream>>>(tq, tk, tv, tqr, tkr, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

int launch_latent(const ortb200_latent_prefill_args* a, cudaStream_t stream) {
  const CUtensorMapDataType dt = a->dtype == ORTB200_BF16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
  CUtensorMap tq, tk, tv, tqr, tkr;
  // [rows, heads, size] operands with `ld` elements between rows and `step` between heads
  auto map = [&](CUtensorMap* m, const void* base, int64_t size, int64_t rows, int64_t heads, int64_t ld, int64_t step, int box_rows) {
    const int64_t dims[4] = {size, rows, heads, 1};
    const int64_t strides[3] = {ld * 2, step * 2, rows * ld * 2};
    return make_tensor_map_4d(m, base, dt, 2, dims, strides, 64, box_rows) == 0;
  };
  const char* kv = static_cast<const char*>(a->kv);
  if (!map(&tq, a->q, a->dk, a->T, a->N, a->q_ld, a->dk + a->dr, kQT) ||
      !map(&tqr, a->q_rot, a->dr, a->T, a->N, static_cast<int64_t>(a->N) * a->dr, a->dr, kQT) ||
      !map(&tk, kv, a->dk, a->key_rows, a->N, a->kv_ld, a->dk, kKT) ||
      !map(&tv, kv + static_cast<int64_t>(a->N) * a->dk * 2, a->dv, a->key_rows, a->N, a->kv_ld, a->dv, kKT) ||
      !map(&tkr, a->k_rot, a->dr, a->key_rows, 1, a->k_rot_ld, a->k_rot_ld, kKT))
    return -6;
  SplitParams p{};
  p.a.head_sink = a->head_sink;
  p.a.out = a->out;
  p.a.B = a->B; p.a.N = a->N; p.a.Nk = a->N;
  p.a.o_strides[1] = a->out_ld; p.a.o_strides[2] = a->dv;
  p.a.scale_log2 = a->scale * 1.4426950408889634f;
  p.a.bf16 = a->dtype == ORTB200_BF16 ? 1 : 0;
  p.a.status = a->status;
  p.a.cu_seqlens = a->cu_seqlens; p.a.past_seqlens = a->past_seqlens;
  p.plain_boxes = (a->dk + 63) / 64;
  p.dv = a->dv; p.gate = a->gate; p.gate_ld = a->gate_ld;
  const int kb = p.plain_boxes + (a->dr + 63) / 64, vb = (a->dv + 63) / 64;
  if (kb == 2 && vb == 1) return launch_split<2, 1, 2, true>(tq, tk, tv, tqr, tkr, p, a->T, stream);
  if (kb == 2 && vb == 2) return launch_split<2, 2, 2, true>(tq, tk, tv, tqr, tkr, p, a->T, stream);
  if (kb == 3 && vb == 1) return launch_split<3, 1, 1, true>(tq, tk, tv, tqr, tkr, p, a->T, stream);
  if (kb == 3 && vb == 2) return launch_split<3, 2, 1, true>(tq, tk, tv, tqr, tkr, p, a->T, stream);
  return -2;
}

}  // namespace

int launch_attn_split(const ortb200_attn_prefill_args* a, cudaStream_t stream) {
  if (a->softcap > 0.f || !a->causal || a->block_size % kKT != 0) return -2;
  const int HD = a->H;
  const CUtensorMapDataType dt = a->dtype == ORTB200_BF16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16;
  CUtensorMap tq, tk, tv;
  const int64_t q_dims[4] = {HD, a->T, a->N, 1};
  const int64_t q_strides[3] = {a->q_strides[1] * 2, a->q_strides[2] * 2, a->T * a->q_strides[1] * 2};
  const int64_t row = static_cast<int64_t>(a->Nk) * HD * 2;
  const int64_t dims[4] = {HD, a->block_size, a->Nk, a->num_blocks};
  const int64_t strides[3] = {row, HD * 2, row * a->block_size};
  if (make_tensor_map_4d(&tq, a->q, dt, 2, q_dims, q_strides, 64, kQT) != 0 || make_tensor_map_4d(&tk, a->k, dt, 2, dims, strides, 64, kKT) != 0 ||
      make_tensor_map_4d(&tv, a->v, dt, 2, dims, strides, 64, kKT) != 0)
    return -6;
  SplitParams p{};
  p.a.head_sink = a->head_sink;
  p.a.out = a->out;
  p.a.B = a->B; p.a.N = a->N; p.a.Nk = a->Nk;
  for (int i = 0; i < 3; ++i) p.a.o_strides[i] = a->o_strides[i];
  p.a.window = a->window; p.a.chunk = a->chunk;
  p.a.scale_log2 = (a->scale != 0.f ? a->scale : 1.0f / sqrtf(static_cast<float>(HD))) * 1.4426950408889634f;
  p.a.bf16 = a->dtype == ORTB200_BF16 ? 1 : 0;
  p.a.status = a->status;
  p.a.block_table = a->block_table; p.a.cu_seqlens = a->cu_seqlens; p.a.past_seqlens = a->past_seqlens;
  p.a.block_size = a->block_size; p.a.max_blocks = a->max_blocks; p.a.num_blocks = a->num_blocks;
  p.plain_boxes = HD / 64;
  p.dv = HD;
  return HD == 128 ? launch_split<2, 2, 2, false>(tq, tk, tv, tq, tk, p, a->T, stream) : launch_split<1, 1, 2, false>(tq, tk, tv, tq, tk, p, a->T, stream);
}

}  // namespace ortb200

using namespace ortb200;

extern "C" int ortb200_latent_prefill_supported(int dk, int dr, int dv, int dtype) {
  if (dtype != ORTB200_BF16 && dtype != ORTB200_F16) return 0;
  if (dk <= 0 || dr <= 0 || dv <= 0 || dk % 8 || dr % 8 || dv % 8 || dv > 128) return 0;
  return (dk + 63) / 64 + (dr + 63) / 64 <= 3 ? 1 : 0;
}

extern "C" int ortb200_latent_prefill(const ortb200_latent_prefill_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->q || !a->q_rot || !a->kv || !a->k_rot || !a->out || !a->cu_seqlens || !a->past_seqlens) return -1;
  if (a->B <= 0 || a->T <= 0 || a->N <= 0 || a->N > 65535 || a->key_rows <= 0 || !(a->scale > 0.f)) return -1;
  if (!ortb200_latent_prefill_supported(a->dk, a->dr, a->dv, a->dtype)) return -2;
  if (a->q_ld < static_cast<int64_t>(a->N) * (a->dk + a->dr) || a->kv_ld < static_cast<int64_t>(a->N) * (a->dk + a->dv) || a->k_rot_ld < a->dr ||
      a->out_ld < static_cast<int64_t>(a->N) * a->dv || (a->gate && a->gate_ld < a->N))
    return -2;
  if (a->q_ld % 8 || a->kv_ld % 8 || a->k_rot_ld % 8 || a->out_ld % 8) return -3;
  if ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->q_rot) | reinterpret_cast<uintptr_t>(a->kv) |
       reinterpret_cast<uintptr_t>(a->k_rot) | reinterpret_cast<uintptr_t>(a->out)) & 15)
    return -3;
  return launch_latent(a, stream);
}
