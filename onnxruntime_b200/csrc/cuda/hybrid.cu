// Packed-token pieces of hybrid decoders that are not recurrences:
//   hyper_norm     residual copies ("hyper-connections"): write-back of one sublayer, read-out for the next and its RMS
//                  norm in one pass over the fp32 copies
//   softcap        cap * tanh(x / cap) on the logits
//   qk_norm_rope   per-head RMS norm, partial rotary embedding (fp32 tables), append to the paged cache
//   paged_attn     causal attention over the paged cache for any head sizes and types, fp32 on CUDA cores: the path for
//                  fp32 models and for head sizes outside the tensor-core kernels
//   head_gate      sigmoid output gate + removal of the head padding behind the tensor-core kernels
//   gated_unit     act(gate) * up of two inputs, written into columns of a wider tensor
#include <cuda_runtime.h>
#include <math.h>
#include "gemm_internal.h"
#include "launch_util.cuh"
#include "ortb200_kernels.h"
#include "ptx_sm100.cuh"

namespace ortb200 {

namespace {

constexpr int kMaxHead = 256;
constexpr float kNeg = -1.0e30f;

// ------------------------------------------------------------------------------------------------- hyper-connections
template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&v)[4]) {
  if constexpr (sizeof(T) == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  } else {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&q);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = to_float<T>(e[i]);
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&v)[4]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    __align__(8) T e[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) e[i] = from_float<T>(v[i]);
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(e);
  }
}

// One block per token.  E = elements per access (4 when the width allows it).  u stays in shared memory between the sum of
// squares and the scaled store.
template <typename T, int N, int E>
__global__ void __launch_bounds__(N <= 4 ? 1024 : 256) hyper_norm_kernel(const ortb200_hyper_norm_args a) {
  extern __shared__ __align__(16) float u[];
  __shared__ float red[32];
  float mix[N][N], w_out[N], w_in[N];
#pragma unroll
  for (int s = 0; s < N; ++s) {
    w_in[s] = a.w_in[s];
    w_out[s] = a.y ? a.w_out[s] : 0.f;
#pragma unroll
    for (int t = 0; t < N; ++t) mix[s][t] = a.y ? a.mix[s * N + t] : (s == t ? 1.f : 0.f);
  }
  pdl_wait_prior_grids();
  const int W = a.width;
  long long tok = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  if (tok < 0 || tok >= a.T) {
    if (a.status && threadIdx.x == 0) atomicExch(a.status, kStatusBadArgument);
    tok = 0;
  }
  const float* xs = a.x_shared ? nullptr : static_cast<const float*>(a.x) + tok * N * W;
  const T* x1 = a.x_shared ? static_cast<const T*>(a.x) + tok * W : nullptr;
  const T* y = a.y ? static_cast<const T*>(a.y) + tok * W : nullptr;
  float* xo = a.x_out ? a.x_out + tok * N * W : nullptr;
  float ss = 0.f;
  for (int c = threadIdx.x * E; c < W; c += blockDim.x * E) {
    float x[N][E], yv[E], uv[E];
    if constexpr (E == 4) {
#pragma unroll
      for (int s = 0; s < N; ++s) {
        if (xs) load4<float>(xs + static_cast<long long>(s) * W + c, x[s]);
        else load4<T>(x1 + c, x[s]);
      }
      if (y) load4<T>(y + c, yv);
    } else {
#pragma unroll
      for (int s = 0; s < N; ++s) x[s][0] = xs ? xs[static_cast<long long>(s) * W + c] : to_float<T>(x1[c]);
      if (y) yv[0] = to_float<T>(y[c]);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) uv[e] = 0.f;
#pragma unroll
    for (int t = 0; t < N; ++t) {
      float v[E];
#pragma unroll
      for (int e = 0; e < E; ++e) {
        if (y) {
          v[e] = w_out[t] * yv[e];
#pragma unroll
          for (int s = 0; s < N; ++s) v[e] = fmaf(mix[s][t], x[s][e], v[e]);
        } else {
          v[e] = x[t][e];
        }
        uv[e] = fmaf(w_in[t], v[e], uv[e]);
      }
      if (xo) {
        if constexpr (E == 4) store4<float>(xo + static_cast<long long>(t) * W + c, v);
        else xo[static_cast<long long>(t) * W + c] = v[0];
      }
    }
#pragma unroll
    for (int e = 0; e < E; ++e) {
      u[c + e] = uv[e];
      ss = fmaf(uv[e], uv[e], ss);
    }
  }
  pdl_launch_dependents();
  const float r = 1.f / sqrtf(block_sum_all(ss, red) / W + a.eps);
  T* out = static_cast<T*>(a.out) + static_cast<long long>(blockIdx.x) * W;
  for (int c = threadIdx.x * E; c < W; c += blockDim.x * E) {   // the same thread wrote u[c .. c + E)
    float v[E];
#pragma unroll
    for (int e = 0; e < E; ++e) v[e] = u[c + e] * r * a.gamma[c + e];
    if constexpr (E == 4) store4<T>(out + c, v);
    else out[c] = from_float<T>(v[0]);
  }
}

template <typename T, int N>
int launch_hyper(const ortb200_hyper_norm_args& a, cudaStream_t stream) {
  const int smem = a.width * 4;
  const bool vec = a.width % 4 == 0;
  auto kern = vec ? hyper_norm_kernel<T, N, 4> : hyper_norm_kernel<T, N, 1>;
  static int attr_smem[2] = {0, 0};
  if (smem > 48 * 1024 && smem > attr_smem[vec]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
    attr_smem[vec] = smem;
  }
  // few tokens: enough threads that a row is one round of loads per thread
  const int blocks = a.rows ? a.num_rows : a.T;
  int threads = 256;
  while (N <= 4 && blocks <= 296 && threads < 1024 && threads * (vec ? 4 : 1) < a.width) threads *= 2;
  return launch_kernel(kern, dim3(blocks), threads, smem, stream, a.use_pdl != 0, a);
}

template <typename T>
int dispatch_hyper(const ortb200_hyper_norm_args& a, cudaStream_t stream) {
  switch (a.streams) {
    case 1: return launch_hyper<T, 1>(a, stream);
    case 2: return launch_hyper<T, 2>(a, stream);
    case 3: return launch_hyper<T, 3>(a, stream);
    case 4: return launch_hyper<T, 4>(a, stream);
    case 5: return launch_hyper<T, 5>(a, stream);
    case 6: return launch_hyper<T, 6>(a, stream);
    case 7: return launch_hyper<T, 7>(a, stream);
    case 8: return launch_hyper<T, 8>(a, stream);
    default: return -2;
  }
}

// ------------------------------------------------------------------------------------------------------------ softcap
template <typename T>
__global__ void __launch_bounds__(256) softcap_kernel(const T* __restrict__ x, float* __restrict__ y, int64_t n, float cap) {
  pdl_wait_prior_grids();
  const int64_t stride = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += stride) y[i] = cap * tanhf(to_float<T>(x[i]) / cap);
}

// -------------------------------------------------------------------------------------------- norm + rotary + append
template <typename T>
__global__ void __launch_bounds__(256, 6) qk_norm_rope_kernel(const ortb200_qk_norm_rope_args a) {
  __shared__ float head[8][kMaxHead];
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait_prior_grids();
  const int b = sequence_of(a.cu_seqlens, a.B, t);
  const int pos = a.past_seqlens[b] + (t - a.cu_seqlens[b]);
  const int bi = pos / a.block_size;
  const int blk = pos >= 0 && bi < a.max_blocks ? a.block_table[static_cast<long long>(b) * a.max_blocks + bi] : -1;
  const bool ok = blk >= 0 && blk < a.num_blocks && pos < a.table_rows;
  if (!ok && threadIdx.x == 0 && a.status) atomicExch(a.status, kStatusBadArgument);
  const long long entry = ok ? static_cast<long long>(blk) * a.block_size + pos % a.block_size : 0;
  const int half = a.rot_dim / 2;
  const float* cs = a.cos_table + static_cast<long long>(ok ? pos : 0) * half;
  const float* sn = a.sin_table + static_cast<long long>(ok ? pos : 0) * half;
  const T* row = static_cast<const T*>(a.packed) + static_cast<long long>(t) * a.ld;
  const int units = a.N + (a.kv_shared ? 0 : 2 * a.Nk);
  const int first_unit = a.q_out ? 0 : a.N;
  for (int u = first_unit + blockIdx.y * 8 + warp; u < units; u += 8 * gridDim.y) {
    const bool is_q = u < a.N, is_v = u >= a.N + a.Nk;
    if (!is_q && !ok) continue;
    if (is_v) {
      const int h = u - a.N - a.Nk;
      const T* __restrict__ src = row + (a.N + a.Nk) * a.dk + h * a.dv;
      T* __restrict__ dst = static_cast<T*>(a.v_cache) + (entry * a.Nk + h) * a.dv_pad;
      if (a.first_values) {
        const T* __restrict__ first = static_cast<const T*>(a.first_values) + t * a.first_ld + h * a.dv;
        const float m = *a.v_mix;
#pragma unroll 4
        for (int d = lane; d < a.dv_pad; d += 32)
          dst[d] = from_float<T>(d < a.dv ? fmaf(m, to_float<T>(first[d]), (1.f - m) * to_float<T>(src[d])) : 0.f);
        continue;
      }
#pragma unroll 4
      for (int d = lane; d < a.dv_pad; d += 32) dst[d] = d < a.dv ? src[d] : from_float<T>(0.f);
      continue;
    }
    const T* __restrict__ src = row + u * a.dk;
    const float* w = is_q ? a.q_norm : a.k_norm;
    T* __restrict__ dst = is_q ? static_cast<T*>(a.q_out) + (static_cast<long long>(t) * a.N + u) * a.dk_pad
                               : static_cast<T*>(a.k_cache) + (entry * a.Nk + (u - a.N)) * a.dk_pad;
    if (!w && half == 0) {   // nothing to compute
#pragma unroll 4
      for (int d = lane; d < a.dk_pad; d += 32) dst[d] = d < a.dk ? src[d] : from_float<T>(0.f);
      continue;
    }
    float ss = 0.f;
    for (int d = lane; d < a.dk; d += 32) {
      const float x = to_float<T>(src[d]);
      head[warp][d] = x;
      ss = fmaf(x, x, ss);
    }
    const float r = w ? 1.f / sqrtf(warp_sum(ss) / a.dk + a.eps) : 1.f;
    __syncwarp();
    for (int d = lane; d < a.dk_pad; d += 32) {
      float y = 0.f;
      if (d < a.dk) {
        y = head[warp][d] * r * (w ? w[d] : 1.f);
        if (d < 2 * half) {
          const int pair = d < half ? d + half : d - half, i = d < half ? d : d - half;
          const float z = head[warp][pair] * r * (w ? w[pair] : 1.f);
          y = d < half ? y * cs[i] - z * sn[i] : y * cs[i] + z * sn[i];
        }
      }
      dst[d] = from_float<T>(y);
    }
    __syncwarp();
  }
  pdl_launch_dependents();
}

// --------------------------------------------------------------------------------------------------- paged attention
// One block per (token, query head): four warps take 32 keys at a time (one key per lane for the scores), keep an online
// softmax each and are merged at the end.
template <typename T>
__global__ void __launch_bounds__(128) paged_attn_kernel(const ortb200_paged_attn_args a) {
  __shared__ __align__(16) float q[kMaxHead];
  __shared__ float acc_s[4][kMaxHead], m_s[4], l_s[4];
  const int t = blockIdx.x, h = blockIdx.y;
  const int kvh = h / (a.N / a.Nk);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_wait_prior_grids();
  const int b = sequence_of(a.cu_seqlens, a.B, t);
  const int pos = a.past_seqlens[b] + (t - a.cu_seqlens[b]);
  const int* table = a.block_table + static_cast<long long>(b) * a.max_blocks;
  const T* qp = static_cast<const T*>(a.q) + (static_cast<long long>(t) * a.N + h) * a.dk_pad;
  for (int d = tid; d < a.dk_pad; d += 128) q[d] = to_float<T>(qp[d]);
  __syncthreads();
  int begin = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  if (a.chunk > 0) begin = max(begin, pos / a.chunk * a.chunk);
  const int end = min(pos + 1, a.max_blocks * a.block_size);
  float m = kNeg, l = 0.f, acc[kMaxHead / 32];
#pragma unroll
  for (int i = 0; i < kMaxHead / 32; ++i) acc[i] = 0.f;
  for (int k0 = begin + warp * 32; k0 < end; k0 += 128) {
    const int key = k0 + lane;
    const bool in = key < end;
    long long entry = 0;
    float s = kNeg;
    if (in) {
      int blk = table[key / a.block_size];
      blk = blk < 0 ? 0 : (blk >= a.num_blocks ? a.num_blocks - 1 : blk);
      entry = (static_cast<long long>(blk) * a.block_size + key % a.block_size) * a.Nk + kvh;
      const T* kp = static_cast<const T*>(a.k_cache) + entry * a.dk_pad;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
      for (int d = 0; d < a.dk_pad; d += 4) {   // cache rows are padded to multiples of four
        float kv[4];
        load4<T>(kp + d, kv);
        d0 = fmaf(q[d], kv[0], d0);
        d1 = fmaf(q[d + 1], kv[1], d1);
        d2 = fmaf(q[d + 2], kv[2], d2);
        d3 = fmaf(q[d + 3], kv[3], d3);
      }
      s = ((d0 + d1) + (d2 + d3)) * a.scale;
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float corr = m <= kNeg ? 0.f : expf(m - m_new);
    const float p = in ? expf(s - m_new) : 0.f;
    l = l * corr + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < kMaxHead / 32; ++i) acc[i] *= corr;
    const int n = min(32, end - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const long long ej = __shfl_sync(0xffffffffu, entry, j);
      const T* vp = static_cast<const T*>(a.v_cache) + ej * a.dv_pad;
#pragma unroll
      for (int i = 0; i < kMaxHead / 32; ++i) {
        const int d = i * 32 + lane;
        if (d < a.dv) acc[i] = fmaf(pj, to_float<T>(vp[d]), acc[i]);
      }
    }
  }
  if (lane == 0) {
    m_s[warp] = m;
    l_s[warp] = l;
  }
#pragma unroll
  for (int i = 0; i < kMaxHead / 32; ++i) acc_s[warp][i * 32 + lane] = acc[i];
  __syncthreads();
  pdl_launch_dependents();
  float mm = a.sink ? a.sink[h] : kNeg;
#pragma unroll
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, m_s[w]);
  float den = a.sink ? expf(a.sink[h] - mm) : 0.f, c[4];
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    c[w] = m_s[w] <= kNeg ? 0.f : expf(m_s[w] - mm);
    den += l_s[w] * c[w];
  }
  const float inv = den > 0.f ? 1.f / den : 0.f;
  const T* gate = a.gate ? static_cast<const T*>(a.gate) + t * a.gate_ld + h * a.dv : nullptr;
  T* out = static_cast<T*>(a.out) + t * (a.out_ld > 0 ? a.out_ld : static_cast<long long>(a.N) * a.dv) + h * a.dv;
  for (int d = tid; d < a.dv; d += 128) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) o = fmaf(acc_s[w][d], c[w], o);
    o *= inv;
    if (gate) o *= sigmoid_f(to_float<T>(gate[d]));
    out[d] = from_float<T>(o);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) head_gate_kernel(const T* __restrict__ x, const T* __restrict__ gate, T* __restrict__ out, int64_t n,
                                                        int heads, int dv, int x_pad, int64_t gate_ld, int64_t out_ld) {
  pdl_wait_prior_grids();
  const int64_t stride = static_cast<int64_t>(gridDim.x) * blockDim.x;
  const int row = heads * dv;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += stride) {
    const int64_t t = i / row;
    const int c = static_cast<int>(i % row), h = c / dv, j = c % dv;
    float v = to_float<T>(x[(t * heads + h) * x_pad + j]);
    if (gate) v *= sigmoid_f(to_float<T>(gate[t * gate_ld + c]));
    out[t * out_ld + c] = from_float<T>(v);
  }
  pdl_launch_dependents();
}

// the same for 16-bit types with dv, x_pad and gate_ld multiples of 8: one 16-byte access each
template <typename T>
__global__ void __launch_bounds__(256) head_gate_vec8_kernel(const T* __restrict__ x, const T* __restrict__ gate, T* __restrict__ out,
                                                             int64_t n8, int heads, int dv, int x_pad, int64_t gate_ld, int64_t out_ld) {
  pdl_wait_prior_grids();
  const int64_t stride = static_cast<int64_t>(gridDim.x) * blockDim.x;
  const int row8 = heads * dv / 8, dv8 = dv / 8;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n8; i += stride) {
    const int64_t t = i / row8;
    const int c = static_cast<int>(i % row8), h = c / dv8, j = c % dv8;
    const uint4 xv = *reinterpret_cast<const uint4*>(x + (t * heads + h) * x_pad + j * 8);
    uint4 gv = make_uint4(0, 0, 0, 0);
    if (gate) gv = *reinterpret_cast<const uint4*>(gate + t * gate_ld + static_cast<int64_t>(c) * 8);
    const T* xe = reinterpret_cast<const T*>(&xv);
    const T* ge = reinterpret_cast<const T*>(&gv);
    __align__(16) T o[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = from_float<T>(gate ? to_float<T>(xe[e]) * sigmoid_f(to_float<T>(ge[e])) : to_float<T>(xe[e]));
    *reinterpret_cast<uint4*>(out + t * out_ld + static_cast<int64_t>(c) * 8) = *reinterpret_cast<const uint4*>(o);
  }
  pdl_launch_dependents();
}

// 16-bit results: fast exponential and division; 32-bit: the accurate ones this file is compiled with
template <typename T>
__device__ __forceinline__ float gated_value(const GateFn& f, float gate, float up) {
  if constexpr (sizeof(T) == 2) {
    const float g = fminf(gate, f.limit);
    const float u = fminf(fmaxf(up, -f.limit), f.limit) + f.offset;
    return __fdividef(g, 1.f + __expf(g * (f.c1 + f.c3 * g * g))) * u;
  } else {
    const float g = fminf(gate, f.limit);
    const float u = fminf(fmaxf(up, -f.limit), f.limit) + f.offset;
    return g / (1.f + expf(g * (f.c1 + f.c3 * g * g))) * u;
  }
}

// E elements per access: 8 for 16-bit types on aligned rows, else 1
template <typename T, int E>
__global__ void __launch_bounds__(256) gated_unit_kernel(const T* __restrict__ gate, const T* __restrict__ up, T* __restrict__ out, int64_t rows,
                                                         int cols, int64_t ld_in, int64_t ld_out, const GateFn f) {
  pdl_wait_prior_grids();
  const int per_row = cols / E;
  const int64_t n = rows * per_row, stride = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += stride) {
    const int64_t r = i / per_row;
    const int c = static_cast<int>(i % per_row) * E;
    if constexpr (E == 8) {
      const uint4 gv = *reinterpret_cast<const uint4*>(gate + r * ld_in + c), uv = *reinterpret_cast<const uint4*>(up + r * ld_in + c);
      const T* ge = reinterpret_cast<const T*>(&gv);
      const T* ue = reinterpret_cast<const T*>(&uv);
      __align__(16) T o[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = from_float<T>(gated_value<T>(f, to_float<T>(ge[e]), to_float<T>(ue[e])));
      *reinterpret_cast<uint4*>(out + r * ld_out + c) = *reinterpret_cast<const uint4*>(o);
    } else {
      out[r * ld_out + c] = from_float<T>(gated_value<T>(f, to_float<T>(gate[r * ld_in + c]), to_float<T>(up[r * ld_in + c])));
    }
  }
  pdl_launch_dependents();
}

unsigned grid_1d(int64_t n) {
  const int64_t g = (n + 255) / 256;
  return static_cast<unsigned>(g < 148 * 16 ? (g > 0 ? g : 1) : 148 * 16);
}

template <typename T>
int run_head_gate(const void* x, const void* gate, void* out, int T_, int heads, int dv, int x_pad, int64_t gate_ld, int64_t out_ld, bool pdl,
                  cudaStream_t st) {
  const int64_t n = static_cast<int64_t>(T_) * heads * dv;
  const uintptr_t align = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out);
  const T *xp = static_cast<const T*>(x), *gp = static_cast<const T*>(gate);
  T* op = static_cast<T*>(out);
  if (sizeof(T) == 2 && dv % 8 == 0 && x_pad % 8 == 0 && gate_ld % 8 == 0 && out_ld % 8 == 0 && (align & 15) == 0)
    return launch_kernel(head_gate_vec8_kernel<T>, dim3(grid_1d(n / 8)), 256, 0, st, pdl, xp, gp, op, n / 8, heads, dv, x_pad, gate_ld, out_ld);
  return launch_kernel(head_gate_kernel<T>, dim3(grid_1d(n)), 256, 0, st, pdl, xp, gp, op, n, heads, dv, x_pad, gate_ld, out_ld);
}

template <typename T>
int run_gated_unit(const void* gate, const void* up, void* out, int64_t rows, int cols, int64_t ld_in, int64_t ld_out, const GateFn& f, bool pdl,
                   cudaStream_t st) {
  const uintptr_t align = reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(out);
  const T *g = static_cast<const T*>(gate), *u = static_cast<const T*>(up);
  T* o = static_cast<T*>(out);
  if constexpr (sizeof(T) == 2) {
    if (cols % 8 == 0 && ld_in % 8 == 0 && ld_out % 8 == 0 && (align & 15) == 0)
      return launch_kernel(gated_unit_kernel<T, 8>, dim3(grid_1d(rows * cols / 8)), 256, 0, st, pdl, g, u, o, rows, cols, ld_in, ld_out, f);
  }
  return launch_kernel(gated_unit_kernel<T, 1>, dim3(grid_1d(rows * cols)), 256, 0, st, pdl, g, u, o, rows, cols, ld_in, ld_out, f);
}

}  // namespace

}  // namespace ortb200

using namespace ortb200;

extern "C" int ortb200_gated_unit(const void* gate, const void* up, void* out, int64_t rows, int cols, int64_t ld_in, int64_t ld_out, int act,
                                  float limit, float alpha, float offset, int dtype, int use_pdl, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!gate || !up || !out || rows < 0 || cols <= 0 || ld_in < cols || ld_out < cols || !is_gated_act(act)) return -1;
  if (rows == 0) return 0;
  const GateFn f = make_gate_fn(act, limit, alpha, offset);
  switch (dtype) {
    case ORTB200_F16: return run_gated_unit<__half>(gate, up, out, rows, cols, ld_in, ld_out, f, use_pdl != 0, stream);
    case ORTB200_BF16: return run_gated_unit<__nv_bfloat16>(gate, up, out, rows, cols, ld_in, ld_out, f, use_pdl != 0, stream);
    case ORTB200_F32: return run_gated_unit<float>(gate, up, out, rows, cols, ld_in, ld_out, f, use_pdl != 0, stream);
    default: return -4;
  }
}

extern "C" int ortb200_hyper_norm(const ortb200_hyper_norm_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->x || !a->w_in || !a->gamma || !a->out) return -1;
  if (a->y && (!a->mix || !a->w_out)) return -1;
  if (a->rows && a->x_out) return -2;
  if (a->T < 0 || a->num_rows < 0 || a->width <= 0 || a->width > 48 * 1024) return -2;
  if ((a->rows ? a->num_rows : a->T) == 0) return 0;
  if (a->T == 0) return -2;
  if ((reinterpret_cast<uintptr_t>(a->x) | reinterpret_cast<uintptr_t>(a->y) | reinterpret_cast<uintptr_t>(a->x_out) |
       reinterpret_cast<uintptr_t>(a->out)) & 15)
    return -3;
  switch (a->dtype) {
    case ORTB200_F16: return dispatch_hyper<__half>(*a, stream);
    case ORTB200_BF16: return dispatch_hyper<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return dispatch_hyper<float>(*a, stream);
    default: return -4;
  }
}

extern "C" int ortb200_softcap(const void* x, float* y, int64_t n, float cap, int dtype, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!x || !y || n < 0 || !(cap > 0.f)) return -1;
  if (n == 0) return 0;
  switch (dtype) {
    case ORTB200_F16: return launch_kernel(softcap_kernel<__half>, dim3(grid_1d(n)), 256, 0, stream, false, static_cast<const __half*>(x), y, n, cap);
    case ORTB200_BF16:
      return launch_kernel(softcap_kernel<__nv_bfloat16>, dim3(grid_1d(n)), 256, 0, stream, false, static_cast<const __nv_bfloat16*>(x), y, n, cap);
    case ORTB200_F32: return launch_kernel(softcap_kernel<float>, dim3(grid_1d(n)), 256, 0, stream, false, static_cast<const float*>(x), y, n, cap);
    default: return -4;
  }
}

extern "C" int ortb200_qk_norm_rope(const ortb200_qk_norm_rope_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->packed || !a->cu_seqlens || !a->past_seqlens || !a->block_table) return -1;
  if (!a->q_out && (a->kv_shared || a->q_norm || a->rot_dim > 0)) return -1;
  if (!a->kv_shared && (!a->k_cache || !a->v_cache)) return -1;
  if (a->first_values && (!a->v_mix || a->first_ld < static_cast<int64_t>(a->Nk) * a->dv)) return -1;
  if (a->T <= 0 || a->B <= 0 || a->N <= 0 || a->Nk <= 0 || a->N % a->Nk != 0) return -2;
  if (a->dk <= 0 || a->dk > kMaxHead || a->dv <= 0 || a->dk_pad < a->dk || a->dv_pad < a->dv || a->dk_pad > kMaxHead) return -2;
  if (a->rot_dim < 0 || a->rot_dim > a->dk || a->rot_dim % 2 != 0 || (a->rot_dim > 0 && (!a->cos_table || !a->sin_table))) return -2;
  if (a->table_rows <= 0 || a->block_size <= 0 || a->max_blocks <= 0 || a->num_blocks <= 0) return -2;
  if (a->ld < a->N * a->dk + (a->kv_shared ? 0 : a->Nk * (a->dk + a->dv))) return -2;
  const int units = (a->q_out ? a->N : 0) + (a->kv_shared ? 0 : 2 * a->Nk);
  int gy = 1;   // few tokens: several blocks share the heads of one token
  while (gy * a->T < 148 && gy * 8 < units) gy *= 2;
  const dim3 grid(a->T, gy);
  switch (a->dtype) {
    case ORTB200_F16: return launch_kernel(qk_norm_rope_kernel<__half>, grid, 256, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_BF16: return launch_kernel(qk_norm_rope_kernel<__nv_bfloat16>, grid, 256, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_F32: return launch_kernel(qk_norm_rope_kernel<float>, grid, 256, 0, stream, a->use_pdl != 0, *a);
    default: return -4;
  }
}

extern "C" int ortb200_paged_attn(const ortb200_paged_attn_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->q || !a->k_cache || !a->v_cache || !a->out || !a->cu_seqlens || !a->past_seqlens || !a->block_table) return -1;
  if (a->T <= 0 || a->B <= 0 || a->N <= 0 || a->N > 65535 || a->Nk <= 0 || a->N % a->Nk != 0) return -2;
  if (a->dk_pad <= 0 || a->dk_pad > kMaxHead || a->dk_pad % 4 != 0 || a->dv <= 0 || a->dv > kMaxHead || a->dv_pad < a->dv) return -2;
  if (a->block_size <= 0 || a->max_blocks <= 0 || a->num_blocks <= 0) return -2;
  if ((reinterpret_cast<uintptr_t>(a->k_cache) | reinterpret_cast<uintptr_t>(a->v_cache)) & 15) return -3;
  const dim3 grid(a->T, a->N);
  switch (a->dtype) {
    case ORTB200_F16: return launch_kernel(paged_attn_kernel<__half>, grid, 128, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_BF16: return launch_kernel(paged_attn_kernel<__nv_bfloat16>, grid, 128, 0, stream, a->use_pdl != 0, *a);
    case ORTB200_F32: return launch_kernel(paged_attn_kernel<float>, grid, 128, 0, stream, a->use_pdl != 0, *a);
    default: return -4;
  }
}

extern "C" int ortb200_head_gate(const void* x, const void* gate, void* out, int T, int heads, int dv, int x_pad, int64_t gate_ld, int64_t out_ld,
                                 int dtype, int use_pdl, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!x || !out || T <= 0 || heads <= 0 || dv <= 0 || x_pad < dv || out_ld < static_cast<int64_t>(heads) * dv ||
      (gate && gate_ld < static_cast<int64_t>(heads) * dv))
    return -1;
  switch (dtype) {
    case ORTB200_F16: return run_head_gate<__half>(x, gate, out, T, heads, dv, x_pad, gate_ld, out_ld, use_pdl != 0, stream);
    case ORTB200_BF16: return run_head_gate<__nv_bfloat16>(x, gate, out, T, heads, dv, x_pad, gate_ld, out_ld, use_pdl != 0, stream);
    case ORTB200_F32: return run_head_gate<float>(x, gate, out, T, heads, dv, x_pad, gate_ld, out_ld, use_pdl != 0, stream);
    default: return -4;
  }
}
