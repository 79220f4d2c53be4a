// Latent attention around its attention kernels (ortb200_kernels.h describes the two forms):
//   latent_prep     rotation of the queries, norm + rotation + append of the new cache entries
//   latent_absorb   the same, and the queries folded through the key map: q -> Uk^T q
//   latent_gather   cached entries of all sequences behind one another, as the input of the expanding GEMM
//   latent_attn     attention over the cache on CUDA cores, fp32, any sizes up to a latent of 1024: the path of fp32 models and
//                   of sizes outside the tensor-core kernel
//   latent_out      merge of the key ranges, sink, value map, output gate
#include <cuda_runtime.h>
#include <math.h>
#include "launch_util.cuh"
#include "latent_internal.h"
#include "ortb200_kernels.h"
#include "ptx_sm100.cuh"

namespace ortb200 {

namespace {

constexpr float kNeg = -1.0e30f;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kTok = 8;            // tokens that share one pass over the weights
constexpr int kMaxLatent = 1024;

template <typename T, int E>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[E]) {
  if constexpr (E == 1) {
    v[0] = to_float<T>(p[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < E; i += 4) {
      const float4 q = *reinterpret_cast<const float4*>(p + i);
      v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
    }
  } else {
    const uint4 q = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&q);
#pragma unroll
    for (int i = 0; i < E; ++i) v[i] = to_float<T>(e[i]);
  }
}

// E entries as they lie in memory: converted where they are used, so that a group of loads goes out together
template <typename T, int E>
struct Raw {
  static constexpr int kWords = E * sizeof(T) / 16;
  uint4 q[kWords > 0 ? kWords : 1];
  T one;
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (E == 1) {
      one = p[0];
    } else {
#pragma unroll
      for (int i = 0; i < kWords; ++i) q[i] = reinterpret_cast<const uint4*>(p)[i];
    }
  }
  __device__ __forceinline__ float at(int e) const {
    if constexpr (E == 1) return to_float<T>(one);
    else return to_float<T>(reinterpret_cast<const T*>(q)[e]);
  }
};

struct TokenPlace {
  int pos;          // position in its sequence, clamped into the rotary tables
  long long entry;  // cache entry, -1 when the block table does not hold the position
};
__device__ __forceinline__ TokenPlace place_of(const ortb200_latent_prep_args& a, int t) {
  // one token per sequence: everything that does not depend on the search is loaded at once
  const int guess = min(t, a.B - 1), c0 = a.cu_seqlens[guess], c1 = a.cu_seqlens[guess + 1], past = a.past_seqlens[guess];
  int b = guess, pos = past;
  if (c0 != t || c1 != t + 1) {
    b = sequence_of(a.cu_seqlens, a.B, t);
    pos = a.past_seqlens[b] + (t - a.cu_seqlens[b]);
  }
  const int bi = pos / a.block_size;
  const int blk = pos >= 0 && bi < a.max_blocks ? a.block_table[static_cast<long long>(b) * a.max_blocks + bi] : -1;
  const bool ok = blk >= 0 && blk < a.num_blocks && (a.rot_dim == 0 || pos < a.table_rows);
  return {ok ? pos : 0, ok ? static_cast<long long>(blk) * a.block_size + pos % a.block_size : -1};
}

// entry d of a rotated part x of dr entries
template <typename T>
__device__ __forceinline__ float rotated(const ortb200_latent_prep_args& a, const T* x, int d, int pos) {
  const float v = to_float<T>(x[d]);
  if (d >= a.rot_dim) return v;
  const long long i = static_cast<long long>(pos) * (a.rot_dim / 2) + d / 2;
  const float c = a.cos_table[i], s = a.sin_table[i], w = to_float<T>(x[d ^ 1]);
  return d & 1 ? fmaf(v, c, w * s) : fmaf(v, c, -(w * s));
}

// One warp: the cache entry of token t, and its optional copies.
template <typename T>
__device__ __forceinline__ void append_entry(const ortb200_latent_prep_args& a, int t, int lane) {
  const TokenPlace at = place_of(a, t);
  if (at.entry < 0 && lane == 0 && a.status) atomicExch(a.status, kStatusBadArgument);
  const T* c = static_cast<const T*>(a.packed) + static_cast<long long>(t) * a.ld + static_cast<long long>(a.N) * (a.dk + a.dr);
  T* dst = at.entry >= 0 ? static_cast<T*>(a.cache) + at.entry * a.width : nullptr;
  T* co = a.c_out ? static_cast<T*>(a.c_out) + static_cast<long long>(t) * a.rank : nullptr;
  T* ko = a.k_rot_out ? static_cast<T*>(a.k_rot_out) + static_cast<long long>(t) * (a.width - a.wide) : nullptr;
  float ss = 0.f;
  if (sizeof(T) == 2 && a.rank % 8 == 0 && a.wide == a.rank && (reinterpret_cast<uintptr_t>(c) & 15) == 0) {   // whole vectors, held in registers
    constexpr int kVecs = kMaxLatent / 256;
    float x[kVecs][8];
#pragma unroll
    for (int k = 0; k < kVecs; ++k) {
      const int d = (k * 32 + lane) * 8;
#pragma unroll
      for (int e = 0; e < 8; ++e) x[k][e] = 0.f;
      if (d < a.rank) load_vec<T, 8>(c + d, x[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(x[k][e], x[k][e], ss);
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / a.rank + a.eps);
#pragma unroll
    for (int k = 0; k < kVecs; ++k) {
      const int d = (k * 32 + lane) * 8;
      if (d >= a.rank) continue;
      __align__(16) T y[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = from_float<T>(x[k][e] * r * a.norm[d + e]);
      if (dst) *reinterpret_cast<uint4*>(dst + d) = *reinterpret_cast<const uint4*>(y);
      if (co) *reinterpret_cast<uint4*>(co + d) = *reinterpret_cast<const uint4*>(y);
    }
  } else {
    for (int d = lane; d < a.rank; d += 32) {
      const float x = to_float<T>(c[d]);
      ss = fmaf(x, x, ss);
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / a.rank + a.eps);
    for (int d = lane; d < a.wide; d += 32) {
      const T y = from_float<T>(d < a.rank ? to_float<T>(c[d]) * r * a.norm[d] : 0.f);
      if (dst) dst[d] = y;
      if (co && d < a.rank) co[d] = y;
    }
  }
  const T* kr = c + a.rank;
  for (int d = lane; d < a.width - a.wide; d += 32) {
    const T y = from_float<T>(d < a.dr ? rotated<T>(a, kr, d, at.pos) : 0.f);
    if (dst) dst[a.wide + d] = y;
    if (ko) ko[d] = y;
  }
}

// One block per token: warp 0 appends the entry, all warps rotate query heads.
template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const ortb200_latent_prep_args a) {
  pdl_wait_prior_grids();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) append_entry<T>(a, t, lane);
  const int pos = place_of(a, t).pos;
  const T* __restrict__ q = static_cast<const T*>(a.packed) + static_cast<long long>(t) * a.ld + a.dk;
  T* __restrict__ dst = static_cast<T*>(a.q_rot) + static_cast<long long>(t) * a.N * a.dr;
  const int n = a.N * a.dr;
  if (((a.dr | a.dk | a.ld) & 1) == 0) {   // whole pairs in one access
    struct __align__(2 * sizeof(T)) Pair {
      T u, v;
    };
    const int half = a.dr / 2;
    const float* __restrict__ cs = a.cos_table + static_cast<long long>(pos) * (a.rot_dim / 2);
    const float* __restrict__ sn = a.sin_table + static_cast<long long>(pos) * (a.rot_dim / 2);
    constexpr int kBatch = 4;
    for (int i0 = threadIdx.x; i0 < n / 2; i0 += kBatch * 128) {
      Pair x[kBatch];
      float c[kBatch], s[kBatch];
#pragma unroll
      for (int k = 0; k < kBatch; ++k) {
        const int i = min(i0 + k * 128, n / 2 - 1), h = i / half, j = i - h * half;
        x[k] = *reinterpret_cast<const Pair*>(q + static_cast<long long>(h) * (a.dk + a.dr) + 2 * j);
        c[k] = 2 * j < a.rot_dim ? cs[j] : 1.f;
        s[k] = 2 * j < a.rot_dim ? sn[j] : 0.f;
      }
#pragma unroll
      for (int k = 0; k < kBatch; ++k) {
        const int i = i0 + k * 128;
        if (i >= n / 2) break;
        const float u = to_float<T>(x[k].u), v = to_float<T>(x[k].v);
        x[k].u = from_float<T>(fmaf(u, c[k], -(v * s[k])));
        x[k].v = from_float<T>(fmaf(v, c[k], u * s[k]));
        *reinterpret_cast<Pair*>(dst + 2 * i) = x[k];
      }
    }
  } else {
    for (int i = threadIdx.x; i < n; i += 128) {
      const int h = i / a.dr, d = i - h * a.dr;
      dst[i] = from_float<T>(rotated<T>(a, q + static_cast<long long>(h) * (a.dk + a.dr), d, pos));
    }
  }
  pdl_launch_dependents();
}

// The x axis holds blocks (h, slice of 16 E latent entries), whose threads are (E entries, one of 16 shares of the head's dk
// rows); then blocks that rotate the queries' parts of eight heads each; then one that appends the new entries.  The y axis
// holds groups of kTok tokens.
constexpr int kRows = 8;           // rows of the key map that a thread has in flight

template <typename T, typename QT, int E>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const ortb200_latent_prep_args a, const int slices) {
  extern __shared__ __align__(16) float q_s[];           // [dk][kTok], then [8 warps][kTok][16 E]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.y * kTok, nt = min(kTok, a.T - t0);
  const int maps = a.N * slices, bx = blockIdx.x;
  if (bx >= maps) {
    pdl_wait_prior_grids();
    if (bx == static_cast<int>(gridDim.x) - 1) {
      if (warp < nt) append_entry<T>(a, t0 + warp, lane);
    } else {
      const int h = (bx - maps) * 8 + warp;
      const int mine = lane < nt ? place_of(a, t0 + lane).pos : 0;
      if (h < a.N) {
        const T* q = static_cast<const T*>(a.packed) + static_cast<long long>(h) * (a.dk + a.dr) + a.dk;
        QT* out = static_cast<QT*>(a.q_abs) + (static_cast<long long>(t0) * a.N + h) * a.width;
        int pos[kTok];
#pragma unroll
        for (int tk = 0; tk < kTok; ++tk) pos[tk] = __shfl_sync(0xffffffffu, mine, tk);
        for (int d = lane; d < a.width - a.wide; d += 32) {
          float v[kTok];   // all tokens are read before the first is stored
#pragma unroll
          for (int tk = 0; tk < kTok; ++tk) v[tk] = tk < nt && d < a.dr ? rotated<T>(a, q + static_cast<long long>(t0 + tk) * a.ld, d, pos[tk]) : 0.f;
#pragma unroll
          for (int tk = 0; tk < kTok; ++tk)
            if (tk < nt) out[static_cast<long long>(tk) * a.N * a.width + a.wide + d] = from_float<QT>(v[tk]);
        }
        for (int d = a.rank + lane; d < a.wide; d += 32)
          for (int tk = 0; tk < nt; ++tk) out[static_cast<long long>(tk) * a.N * a.width + d] = from_float<QT>(0.f);
      }
    }
    pdl_launch_dependents();
    return;
  }
  const int h = bx / slices, slice = bx % slices;
  const int cg = threadIdx.x & 15, share = threadIdx.x >> 4;
  const int c = (slice * 16 + cg) * E;
  const bool in = c < a.rank;   // E divides rank
  const T* w = static_cast<const T*>(a.up) + static_cast<long long>(h) * a.dk * a.rank + (in ? c : 0);
  Raw<T, E> wv[kRows];          // the first rows are constants: fetched before the kernel in front has finished
#pragma unroll
  for (int k = 0; k < kRows; ++k) wv[k].load(w + static_cast<long long>(min(share + 16 * k, a.dk - 1)) * a.rank);
  pdl_wait_prior_grids();
  const T* q = static_cast<const T*>(a.packed) + static_cast<long long>(t0) * a.ld + static_cast<long long>(h) * (a.dk + a.dr);
#pragma unroll
  for (int tk = 0; tk < kTok; ++tk)
    for (int d = threadIdx.x; d < a.dk; d += 256) q_s[d * kTok + tk] = tk < nt ? to_float<T>(q[static_cast<long long>(tk) * a.ld + d]) : 0.f;
  __syncthreads();
  float acc[kTok][E];
#pragma unroll
  for (int tk = 0; tk < kTok; ++tk)
#pragma unroll
    for (int e = 0; e < E; ++e) acc[tk][e] = 0.f;
  for (int d0 = share; d0 < a.dk; d0 += 16 * kRows) {
#pragma unroll
    for (int k = 0; k < kRows; ++k) {
      const int d = d0 + 16 * k;
      if (d >= a.dk) break;
      const float4 qa = *reinterpret_cast<const float4*>(q_s + d * kTok), qb = *reinterpret_cast<const float4*>(q_s + d * kTok + 4);
      const float qv[kTok] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
      for (int tk = 0; tk < kTok; ++tk)
#pragma unroll
        for (int e = 0; e < E; ++e) acc[tk][e] = fmaf(qv[tk], wv[k].at(e), acc[tk][e]);
    }
    if (d0 + 16 * kRows < a.dk) {
#pragma unroll
      for (int k = 0; k < kRows; ++k) wv[k].load(w + static_cast<long long>(min(d0 + 16 * (kRows + k), a.dk - 1)) * a.rank);
    }
  }
  float* red = q_s + a.dk * kTok;
#pragma unroll
  for (int tk = 0; tk < kTok; ++tk)
#pragma unroll
    for (int e = 0; e < E; ++e) {
      acc[tk][e] += __shfl_xor_sync(0xffffffffu, acc[tk][e], 16);
      if (lane < 16) red[(warp * kTok + tk) * 16 * E + cg * E + e] = acc[tk][e];
    }
  __syncthreads();
  QT* out = static_cast<QT*>(a.q_abs) + (static_cast<long long>(t0) * a.N + h) * a.width;
  for (int i = threadIdx.x; i < nt * 16 * E; i += 256) {
    const int tk = i / (16 * E), j = i % (16 * E), col = slice * 16 * E + j;
    if (col >= a.rank) continue;
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) v += red[(k * kTok + tk) * 16 * E + j];
    out[static_cast<long long>(tk) * a.N * a.width + col] = from_float<QT>(v);
  }
  pdl_launch_dependents();
}

// One warp per entry.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, const int* cu, const int* past, const int* table,
                                                            T* __restrict__ c_out, T* __restrict__ k_out, int rows, int B, int rank, int wide, int width,
                                                            int block_size, int max_blocks, int num_blocks, int* status) {
  pdl_wait_prior_grids();
  const int lane = threadIdx.x & 31;
  for (int row = blockIdx.x * 8 + (threadIdx.x >> 5); row < rows; row += gridDim.x * 8) {
    int b = 0, pos = row;
    for (; b < B - 1; ++b) {
      const int n = past[b] + cu[b + 1] - cu[b];
      if (pos < n) break;
      pos -= n;
    }
    const int bi = pos / block_size;
    int blk = bi < max_blocks ? table[static_cast<long long>(b) * max_blocks + bi] : -1;
    if (blk < 0 || blk >= num_blocks) {
      if (status && lane == 0) atomicExch(status, kStatusBadArgument);
      blk = 0;
    }
    const T* src = cache + (static_cast<long long>(blk) * block_size + pos % block_size) * width;
    T* c = c_out + static_cast<long long>(row) * rank;
    T* k = k_out + static_cast<long long>(row) * (width - wide);
    if (sizeof(T) == 2 && rank % 8 == 0) {   // width and wide are multiples of 8 then
      for (int d = lane * 8; d < rank; d += 256) *reinterpret_cast<uint4*>(c + d) = *reinterpret_cast<const uint4*>(src + d);
      for (int d = lane * 8; d < width - wide; d += 256) *reinterpret_cast<uint4*>(k + d) = *reinterpret_cast<const uint4*>(src + wide + d);
    } else {
      for (int d = lane; d < rank; d += 32) c[d] = src[d];
      for (int d = lane; d < width - wide; d += 32) k[d] = src[wide + d];
    }
  }
  pdl_launch_dependents();
}

// One block per (token, head): four warps take 32 keys at a time (one key per lane for the scores), keep an online softmax
// each and are merged at the end.  NI = ceil(rank / 32) rounded up: accumulator entries per lane.
template <typename T, int NI>
__global__ void __launch_bounds__(128) latent_attn_kernel(const ortb200_latent_decode_args a) {
  extern __shared__ __align__(16) float smem[];          // q [width], then [4][rank]
  __shared__ float m_s[4], l_s[4];
  float* q = smem;
  float* acc_s = smem + a.width;
  const int t = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait_prior_grids();
  const int b = sequence_of(a.cu_seqlens, a.B, t);
  const int end = min(a.past_seqlens[b] + (t - a.cu_seqlens[b]) + 1, a.max_blocks * a.block_size);
  const int* table = a.block_table + static_cast<long long>(b) * a.max_blocks;
  const float* qp = static_cast<const float*>(a.q_abs) + (static_cast<long long>(t) * a.N + h) * a.width;
  for (int d = tid; d < a.width; d += 128) q[d] = qp[d];
  __syncthreads();
  float m = kNeg, l = 0.f, acc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) acc[i] = 0.f;
  const float scale = a.scale * kLog2e;
  for (int k0 = warp * 32; k0 < end; k0 += 128) {
    const int key = k0 + lane;
    const bool in = key < end;
    long long row = 0;
    float s = kNeg;
    if (in) {
      int blk = table[key / a.block_size];
      blk = blk < 0 ? 0 : (blk >= a.num_blocks ? a.num_blocks - 1 : blk);
      row = (static_cast<long long>(blk) * a.block_size + key % a.block_size) * a.width;
      const T* kp = static_cast<const T*>(a.cache) + row;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
      for (int d = 0; d < a.width; d += 4) {   // width is a multiple of four
        float kv[4];
        if constexpr (sizeof(T) == 4) {
          load_vec<T, 4>(kp + d, kv);
        } else {
          const uint2 w = *reinterpret_cast<const uint2*>(kp + d);
          const T* e = reinterpret_cast<const T*>(&w);
#pragma unroll
          for (int i = 0; i < 4; ++i) kv[i] = to_float<T>(e[i]);
        }
        d0 = fmaf(q[d], kv[0], d0);
        d1 = fmaf(q[d + 1], kv[1], d1);
        d2 = fmaf(q[d + 2], kv[2], d2);
        d3 = fmaf(q[d + 3], kv[3], d3);
      }
      s = ((d0 + d1) + (d2 + d3)) * scale;
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float corr = m <= kNeg ? 0.f : exp2f(m - m_new);
    const float p = in ? exp2f(s - m_new) : 0.f;
    l = l * corr + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < NI; ++i) acc[i] *= corr;
    const int n = min(32, end - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const T* cp = static_cast<const T*>(a.cache) + __shfl_sync(0xffffffffu, row, j);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = i * 32 + lane;
        if (d < a.rank) acc[i] = fmaf(pj, to_float<T>(cp[d]), acc[i]);
      }
    }
  }
  if (lane == 0) {
    m_s[warp] = m;
    l_s[warp] = l;
  }
#pragma unroll
  for (int i = 0; i < NI; ++i)
    if (i * 32 + lane < a.rank) acc_s[warp * a.rank + i * 32 + lane] = acc[i];
  __syncthreads();
  pdl_launch_dependents();
  float mm = kNeg, den = 0.f, c[4];
#pragma unroll
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, m_s[w]);
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    c[w] = m_s[w] <= kNeg ? 0.f : exp2f(m_s[w] - mm);
    den += l_s[w] * c[w];
  }
  const long long at = static_cast<long long>(t) * a.N + h;   // one part
  for (int d = tid; d < a.rank; d += 128) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) o = fmaf(acc_s[w * a.rank + d], c[w], o);
    a.o[at * a.wide + d] = o;
  }
  if (tid == 0) {
    a.ml[at * 2] = mm;
    a.ml[at * 2 + 1] = den;
  }
}

constexpr int kOutRows = 32;   // value entries per block: four per warp

// Blocks (h, kOutRows value entries, kTok tokens).  Every lane keeps four rows x kTok tokens of partial sums over its share
// of the latent; a halving exchange then leaves one finished sum per lane.
template <typename T, int E>
__global__ void __launch_bounds__(256) latent_out_kernel(const ortb200_latent_out_args a, const int slices) {
  extern __shared__ __align__(16) float o_s[];            // [kTok][rank]
  __shared__ float coef[kTok][32];
  const int h = blockIdx.x / slices, j0 = (blockIdx.x % slices) * kOutRows;
  const int t0 = blockIdx.y * kTok, nt = min(kTok, a.T - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j = j0 + warp * 4;
  const T* w = static_cast<const T*>(a.up_v) + (static_cast<long long>(h) * a.dv + min(j, a.dv - 1)) * a.rank;
  // the lane's first two shares of its four rows are constants: fetched before the kernel in front has finished
  constexpr int kAhead = 2;
  Raw<T, E> wv[kAhead][4];
  auto fetch = [&](int c, Raw<T, E> (&v)[4]) {
#pragma unroll
    for (int r = 0; r < 4; ++r) v[r].load(w + static_cast<long long>(j + r < a.dv ? r : 0) * a.rank + (c < a.rank ? c : 0));
  };
#pragma unroll
  for (int k = 0; k < kAhead; ++k) fetch((k * 32 + lane) * E, wv[k]);
  pdl_wait_prior_grids();
  if (warp < nt) {   // factor of every part of token t0 + warp (parts <= 32)
    const float* ml = a.ml + (static_cast<long long>(t0 + warp) * a.N + h) * a.parts * 2;
    const float m = lane < a.parts ? ml[lane * 2] : kNeg, l = lane < a.parts ? ml[lane * 2 + 1] : 0.f;
    const float sink = a.sink ? a.sink[h] * kLog2e : kNeg;
    const float mm = fmaxf(warp_max(m), sink);
    const float w = m <= kNeg ? 0.f : exp2f(m - mm);
    const float den = warp_sum(l * w) + (a.sink ? exp2f(sink - mm) : 0.f);
    coef[warp][lane] = den > 0.f ? w / den : 0.f;
  }
  __syncthreads();
  if constexpr (E == 8) {   // rank and wide are multiples of four then
    const int vecs = a.rank / 4;
#pragma unroll 4
    for (int i = threadIdx.x; i < kTok * vecs; i += 256) {
      const int tk = i / vecs, c = (i - tk * vecs) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (tk < nt) {
        const float* o = a.o + (static_cast<long long>(t0 + tk) * a.N + h) * a.parts * a.wide + c;
        for (int p0 = 0; p0 < a.parts; p0 += 4) {   // factors of absent parts are 0
          float4 x[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) x[k] = *reinterpret_cast<const float4*>(o + static_cast<long long>(min(p0 + k, a.parts - 1)) * a.wide);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float f = coef[tk][p0 + k];
            v.x = fmaf(f, x[k].x, v.x); v.y = fmaf(f, x[k].y, v.y); v.z = fmaf(f, x[k].z, v.z); v.w = fmaf(f, x[k].w, v.w);
          }
        }
      }
      *reinterpret_cast<float4*>(o_s + tk * a.rank + c) = v;
    }
  } else {
    for (int i = threadIdx.x; i < kTok * a.rank; i += 256) {
      const int tk = i / a.rank, c = i - tk * a.rank;
      float v = 0.f;
      if (tk < nt) {
        const float* o = a.o + (static_cast<long long>(t0 + tk) * a.N + h) * a.parts * a.wide + c;
        for (int p = 0; p < a.parts; ++p) v = fmaf(coef[tk][p], o[static_cast<long long>(p) * a.wide], v);
      }
      o_s[i] = v;
    }
  }
  __syncthreads();
  float acc[4 * kTok];
#pragma unroll
  for (int i = 0; i < 4 * kTok; ++i) acc[i] = 0.f;
  if (j < a.dv) {
    for (int c0 = 0; c0 < a.rank; c0 += kAhead * 32 * E) {
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        const int c = c0 + (k * 32 + lane) * E;
        if (c < a.rank) {
#pragma unroll
          for (int tk = 0; tk < kTok; ++tk) {
            float ov[E];
            load_vec<float, E>(o_s + tk * a.rank + c, ov);
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
              for (int e = 0; e < E; ++e) acc[r * kTok + tk] = fmaf(wv[k][r].at(e), ov[e], acc[r * kTok + tk]);
          }
        }
        if (c0 + kAhead * 32 * E < a.rank) fetch(c + kAhead * 32 * E, wv[k]);
      }
    }
    // after the step of distance o, a lane holds the sums whose index has bit o equal to the lane's
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
#pragma unroll
      for (int i = 0; i < o; ++i) {
        const float send = lane & o ? acc[i] : acc[i + o], keep = lane & o ? acc[i + o] : acc[i];
        acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    const int r = lane / kTok, tk = lane % kTok;
    if (tk < nt && j + r < a.dv) {
      float v = acc[0];
      if (a.gate) v *= sigmoid_f(to_float<T>(static_cast<const T*>(a.gate)[(t0 + tk) * a.gate_ld + h]));
      static_cast<T*>(a.out)[(t0 + tk) * a.out_ld + static_cast<long long>(h) * a.dv + j + r] = from_float<T>(v);
    }
  }
  pdl_launch_dependents();
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename K>
int opt_in_smem(K kern, int bytes) {
  return bytes <= 48 * 1024 || cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) == cudaSuccess ? 0 : -10;
}

template <typename T, typename QT, int E>
int launch_absorb(const ortb200_latent_prep_args& a, cudaStream_t stream) {
  const int slices = (a.rank + 16 * E - 1) / (16 * E);
  const int smem = (a.dk * kTok + 8 * kTok * 16 * E) * 4;
  auto kern = latent_absorb_kernel<T, QT, E>;
  if (int rc = opt_in_smem(kern, smem)) return rc;
  return launch_kernel(kern, dim3(a.N * slices + (a.N + 7) / 8 + 1, (a.T + kTok - 1) / kTok), 256, smem, stream, a.use_pdl != 0, a, slices);
}
template <typename T>
int dispatch_absorb(const ortb200_latent_prep_args& a, cudaStream_t stream) {
  const bool vec = a.rank % 8 == 0 && aligned16(a.up);
  if (a.q_abs_f32 || sizeof(T) == 4) return vec ? launch_absorb<T, float, 8>(a, stream) : launch_absorb<T, float, 1>(a, stream);
  return vec ? launch_absorb<T, T, 8>(a, stream) : launch_absorb<T, T, 1>(a, stream);
}

template <typename T, int NI>
int launch_attn(const ortb200_latent_decode_args& a, cudaStream_t stream) {
  return launch_kernel(latent_attn_kernel<T, NI>, dim3(a.T, a.N), 128, (a.width + 4 * a.rank) * 4, stream, a.use_pdl != 0, a);
}
template <typename T>
int dispatch_attn(const ortb200_latent_decode_args& a, cudaStream_t stream) {
  if (a.rank <= 128) return launch_attn<T, 4>(a, stream);
  if (a.rank <= 256) return launch_attn<T, 8>(a, stream);
  if (a.rank <= 512) return launch_attn<T, 16>(a, stream);
  return launch_attn<T, 32>(a, stream);
}

template <typename T>
int dispatch_out(const ortb200_latent_out_args& a, cudaStream_t stream) {
  const int slices = (a.dv + kOutRows - 1) / kOutRows, smem = kTok * a.rank * 4;
  const dim3 grid(a.N * slices, (a.T + kTok - 1) / kTok);
  if (a.rank % 8 == 0 && aligned16(a.up_v)) return launch_kernel(latent_out_kernel<T, 8>, grid, 256, smem, stream, a.use_pdl != 0, a, slices);
  return launch_kernel(latent_out_kernel<T, 1>, grid, 256, smem, stream, a.use_pdl != 0, a, slices);
}

template <typename T>
int dispatch_gather(const void* cache, const int* cu, const int* past, const int* table, void* c, void* k, int rows, int B, int rank, int wide, int width,
                    int block_size, int max_blocks, int num_blocks, bool pdl, int* status, cudaStream_t stream) {
  const int blocks = (rows + 7) / 8 < 148 * 8 ? (rows + 7) / 8 : 148 * 8;
  return launch_kernel(latent_gather_kernel<T>, dim3(blocks), 256, 0, stream, pdl, static_cast<const T*>(cache), cu, past, table, static_cast<T*>(c),
                       static_cast<T*>(k), rows, B, rank, wide, width, block_size, max_blocks, num_blocks, status);
}

bool bad_prep(const ortb200_latent_prep_args* a) {
  if (!a || !a->packed || !a->cache || !a->norm || !a->cu_seqlens || !a->past_seqlens || !a->block_table) return true;
  if (a->T <= 0 || a->B <= 0 || a->N <= 0 || a->dk <= 0 || a->dr < 0 || a->rank <= 0 || a->rank > kMaxLatent) return true;
  if (a->wide < a->rank || a->width < a->wide + a->dr || a->ld < a->N * (a->dk + a->dr) + a->rank + a->dr) return true;
  if (a->rot_dim < 0 || a->rot_dim % 2 || a->rot_dim > a->dr || (a->rot_dim > 0 && (!a->cos_table || !a->sin_table || a->table_rows <= 0))) return true;
  return a->block_size <= 0 || a->max_blocks <= 0 || a->num_blocks <= 0;
}

}  // namespace

}  // namespace ortb200

using namespace ortb200;

extern "C" int ortb200_latent_prep(const ortb200_latent_prep_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (bad_prep(a) || (!a->q_rot && a->dr > 0)) return -1;
  switch (a->dtype) {
    case ORTB200_F16: return launch_kernel(latent_prep_kernel<__half>, dim3(a->T), 128, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_BF16: return launch_kernel(latent_prep_kernel<__nv_bfloat16>, dim3(a->T), 128, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_F32: return launch_kernel(latent_prep_kernel<float>, dim3(a->T), 128, 0, stream, a->use_pdl != 0, *a);
    default: return -4;
  }
}

extern "C" int ortb200_latent_absorb(const ortb200_latent_prep_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (bad_prep(a) || !a->up || !a->q_abs || a->dk > 4096 || (a->T + kTok - 1) / kTok > 65535) return -1;
  switch (a->dtype) {
    case ORTB200_F16: return dispatch_absorb<__half>(*a, stream);
    case ORTB200_BF16: return dispatch_absorb<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return dispatch_absorb<float>(*a, stream);
    default: return -4;
  }
}

extern "C" int ortb200_latent_gather(const void* cache, const int* cu, const int* past, const int* table, void* c, void* k, int rows, int B, int rank,
                                     int wide, int width, int block_size, int max_blocks, int num_blocks, int dtype, int use_pdl, int* status,
                                     ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!cache || !cu || !past || !table || !c || !k || rows <= 0 || B <= 0 || rank <= 0 || wide < rank || width < wide) return -1;
  if (block_size <= 0 || max_blocks <= 0 || num_blocks <= 0) return -1;
  if (dtype != ORTB200_F32 && (wide % 8 || width % 8 || !aligned16(cache) || !aligned16(c) || !aligned16(k))) return -3;
  const bool pdl = use_pdl != 0;
  switch (dtype) {
    case ORTB200_F16:
      return dispatch_gather<__half>(cache, cu, past, table, c, k, rows, B, rank, wide, width, block_size, max_blocks, num_blocks, pdl, status, stream);
    case ORTB200_BF16:
      return dispatch_gather<__nv_bfloat16>(cache, cu, past, table, c, k, rows, B, rank, wide, width, block_size, max_blocks, num_blocks, pdl, status,
                                            stream);
    case ORTB200_F32:
      return dispatch_gather<float>(cache, cu, past, table, c, k, rows, B, rank, wide, width, block_size, max_blocks, num_blocks, pdl, status, stream);
    default: return -4;
  }
}

extern "C" int ortb200_latent_decode(const ortb200_latent_decode_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->q_abs || !a->cache || !a->cu_seqlens || !a->past_seqlens || !a->block_table || !a->o || !a->ml) return -1;
  if (a->T <= 0 || a->B <= 0 || a->N <= 0 || a->N > 65535 || a->rank <= 0 || a->rank > kMaxLatent || a->wide < a->rank || a->width < a->wide) return -2;
  if (a->block_size <= 0 || a->max_blocks <= 0 || a->num_blocks <= 0 || a->parts <= 0 || a->parts > 32 || a->width % 4) return -2;
  if (!aligned16(a->q_abs) || !aligned16(a->cache) || !aligned16(a->o)) return -3;
  if (a->tensor_cores) return launch_latent_decode_tc(a, stream);
  if (a->parts != 1) return -2;
  switch (a->dtype) {
    case ORTB200_F16: return dispatch_attn<__half>(*a, stream);
    case ORTB200_BF16: return dispatch_attn<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return dispatch_attn<float>(*a, stream);
    default: return -4;
  }
}

extern "C" int ortb200_latent_out(const ortb200_latent_out_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->o || !a->ml || !a->up_v || !a->out) return -1;
  if (a->T <= 0 || a->N <= 0 || a->dv <= 0 || a->rank <= 0 || a->rank > kMaxLatent || a->wide < a->rank || a->parts <= 0 || a->parts > 32) return -2;
  if (a->out_ld < static_cast<int64_t>(a->N) * a->dv || (a->gate && a->gate_ld < a->N) || (a->T + kTok - 1) / kTok > 65535) return -2;
  switch (a->dtype) {
    case ORTB200_F16: return dispatch_out<__half>(*a, stream);
    case ORTB200_BF16: return dispatch_out<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return dispatch_out<float>(*a, stream);
    default: return -4;
  }
}
