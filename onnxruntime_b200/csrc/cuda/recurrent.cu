// Recurrent token mixers over packed sequences: the gated delta rule with a decay per key channel, and the
// exponentially gated matrix memory (mLSTM).  State and arithmetic are fp32 everywhere, and every token
// sees the exact state of the tokens before it, so a result does not depend on how a prompt is cut.
//
// Several tokens per sequence (prompts): three launches.
//   prep   short convolution + silu, unit norms, decays, gates -> fp32 rows, heads padded; a warp owns the channels of one
//          head and walks a run of tokens with the convolution window in registers
//   scan   one block per (16 * warps state columns, head, sequence).  State columns are independent of each other, so
//          the grid splits them; a warp holds a [dk, 16] slice of S in registers (8 row groups x 4 column groups of
//          lanes), streams the token rows through double-buffered shared memory with cp.async, and does the decay, the
//          two matrix-vector products and the rank-one update with packed fp32x2 instructions
//   post   norm over the value dimension, output gate, ring of convolution inputs
// One token per sequence (decode): one launch, one block per (head, sequence) that does all of it; the state is read
// once and written once, which is what bounds the step.
//
// The delta-rule scan takes four tokens at a time.  With P_t = g_1 ... g_t the decays since the block began,
//   S_t^T k_{t+1} etc. need only products with the state at the block's start:
//   a_t = S^T (P_t k_t) + sum_{j<t} (k_t . g_{j+1..t} k_j) u_j,   u_t = beta_t (v_t - a_t)
//   o_t = S^T (P_t q_t) + sum_{j<=t} (q_t . g_{j+1..t} k_j) u_j,  S' = P_4 S + sum_j (g_{j+1..4} k_j) u_j^T
// All factors are products of decays (no quotients), so nothing can overflow; the prep kernel forms them, and the scan
// does 13 multiply-adds per state element and block instead of 16, with one chain of reductions instead of four.
#include <cuda_runtime.h>
#include <math.h>
#include <type_traits>
#include "launch_util.cuh"
#include "ortb200_kernels.h"
#include "ptx_sm100.cuh"

namespace ortb200 {

namespace {

constexpr int kMaxHead = 256;     // key / value head sizes
constexpr int kChunk = 8;         // tokens per shared-memory stage of the scan
constexpr int kPrepRun = 16;      // tokens a prep warp walks
constexpr int kMaxTaps = 16;

int pad_dk(int dk) { return dk <= 64 ? 64 : (dk <= 128 ? 128 : 256); }
int pad4(int n) { return (n + 3) / 4 * 4; }

// fp32 scratch of a multi-token call.  mLSTM rows are indexed by packed token; the delta rule keeps blocks of kBlock tokens
// of one sequence: block i of sequence b is number cu_seqlens[b] / kBlock + b + i, which never collides.
constexpr int kBlock = 4;
constexpr int kVecs = 3 * kBlock + 1;     // P_t k_t, P_t q_t, g_{j+1..4} k_j, P_4
constexpr int kScal = 20;                 // beta_t (4), k_t . g k_j for j < t (6), q_t . g k_j for j <= t (10)
struct Scratch {
  float* vec;     // delta: [blocks, H, kVecs, dkp];  mLSTM: [T, H, 2, dkp] q row, then k row
  float* v;       // delta: [blocks, kBlock, H, dvp];  mLSTM: [T, H, dvp]
  float* scal;    // delta: [blocks, H, kScal];        mLSTM: [T, H, 4] log gates i, f
  float* o;       // [T, H, dvp]
  float* aux_out; // mLSTM: [B, H, dk + 1] n and m after the last token
};

struct ScratchSizes {
  int64_t vec, v, scal, o, aux;
  int64_t total() const { return vec + v + scal + o + aux; }
};
ScratchSizes delta_scratch(int64_t T, int64_t B, int64_t H, int64_t dkp, int64_t dvp) {
  const int64_t blocks = T / kBlock + B;
  return {blocks * H * kVecs * dkp, blocks * kBlock * H * dvp, blocks * H * kScal, T * H * dvp, 0};
}
ScratchSizes mlstm_scratch(int64_t T, int64_t B, int64_t H, int64_t dk, int64_t dkp, int64_t dvp) {
  return {T * H * 2 * dkp, T * H * dvp, T * H * 4, T * H * dvp, B * H * (dk + 1)};
}
Scratch split_scratch(float* w, const ScratchSizes& n) {
  Scratch s;
  s.vec = w;
  s.v = s.vec + n.vec;
  s.scal = s.v + n.v;
  s.o = s.scal + n.scal;
  s.aux_out = s.o + n.o;
  return s;
}

// ------------------------------------------------------------------------------------------------ delta rule pieces
// silu behind the short convolution and sigmoid of the output gate: results that 16-bit models round to 16 bits take the
// fast exponential and division
template <typename T>
__device__ __forceinline__ float act_sigmoid(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
  else return sigmoid_f(x);
}

// Convolution + silu of one channel for the token in packed row t (position pos, `before` rows of its sequence in this
// call); earlier inputs come from the packed rows, then from the ring, and are zero in front of the sequence.
template <typename T>
__device__ __forceinline__ float conv_silu(const ortb200_gated_delta_args& a, const T* ring, int channels, int ch, long long t, int pos,
                                           int before) {
  const T* x = static_cast<const T*>(a.qkvb) + t * a.ld + ch;
  const float* w = a.conv + static_cast<long long>(ch) * a.taps;
  float acc = 0.f;
  for (int j = a.taps - 1; j >= 1; --j) {
    float xv = 0.f;
    if (j <= before) xv = to_float<T>(x[-static_cast<long long>(j) * a.ld]);
    else if (pos - j >= 0) xv = to_float<T>(ring[static_cast<long long>((pos - j) % a.taps) * channels + ch]);
    acc = fmaf(w[a.taps - 1 - j], xv, acc);
  }
  acc = fmaf(w[a.taps - 1], to_float<T>(x[0]), acc);
  return acc * act_sigmoid<T>(acc);
}

__device__ __forceinline__ bool slot_ok(int slot, int num_slots, int* status) {
  if (slot >= 0 && slot < num_slots) return true;
  if (status && threadIdx.x == 0) atomicExch(status, kStatusBadArgument);
  return false;
}

// Inputs of one channel per lane and 32-column group, TAPS - 1 tokens back (newest last), for a warp that walks packed rows.
template <typename T, int TAPS, int NI>
struct ConvWindow {
  float w[NI][TAPS], x[NI][TAPS - 1 > 0 ? TAPS - 1 : 1];
  __device__ __forceinline__ void load_taps(const float* conv, int ch0, int n, int lane) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[i][j] = d < n ? conv[static_cast<long long>(ch0 + d) * TAPS + j] : 0.f;
    }
  }
  // `row` points at channel ch0 of the token's packed row
  __device__ __forceinline__ void refill(const T* row, long long ld, const T* ring, int channels, int ch0, int n, int lane, int pos, int before) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
#pragma unroll
      for (int j = 1; j < TAPS; ++j) {
        float v = 0.f;
        if (d < n) {
          if (j <= before) v = to_float<T>(row[d - j * ld]);
          else if (pos - j >= 0) v = to_float<T>(ring[static_cast<long long>((pos - j) % TAPS) * channels + ch0 + d]);
        }
        x[i][TAPS - 1 - j] = v;
      }
    }
  }
  __device__ __forceinline__ void step(const T* row, int n, int lane, float (&y)[NI]) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
      const float now = d < n ? to_float<T>(row[d]) : 0.f;
      float acc = now * w[i][TAPS - 1];
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) acc = fmaf(x[i][j], w[i][j], acc);
#pragma unroll
      for (int j = 0; j + 2 < TAPS; ++j) x[i][j] = x[i][j + 1];
      if (TAPS > 1) x[i][TAPS - 2 > 0 ? TAPS - 2 : 0] = now;
      y[i] = acc * act_sigmoid<T>(acc);
    }
  }
};
// any number of taps: every input is fetched again
template <typename T, int NI>
struct ConvWindow<T, 0, NI> {
  const ortb200_gated_delta_args* a;
  const T* ring;
  int channels, ch0, pos, before;
  long long t;
  __device__ __forceinline__ void step(int n, int lane, float (&y)[NI]) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
      y[i] = d < n ? conv_silu<T>(*a, ring, channels, ch0 + d, t, pos, before) : 0.f;
    }
  }
};

// Sums of 16 values over the warp: lane l ends with the sum of x[l & 15].
__device__ __forceinline__ float reduce16(const float (&x)[16], int lane) {
  float y[8], z[4], w[2];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const float send = (lane & 8) ? x[i] : x[8 + i], keep = (lane & 8) ? x[8 + i] : x[i];
    y[i] = keep + __shfl_xor_sync(0xffffffffu, send, 8);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float send = (lane & 4) ? y[i] : y[4 + i], keep = (lane & 4) ? y[4 + i] : y[i];
    z[i] = keep + __shfl_xor_sync(0xffffffffu, send, 4);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float send = (lane & 2) ? z[i] : z[2 + i], keep = (lane & 2) ? z[2 + i] : z[i];
    w[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
  }
  const float send = (lane & 1) ? w[0] : w[1], keep = (lane & 1) ? w[1] : w[0];
  const float r = keep + __shfl_xor_sync(0xffffffffu, send, 1);
  return r + __shfl_xor_sync(0xffffffffu, r, 16);
}

// A warp owns one head (q, k and decays, or values) and a run of kPrepRun tokens of one sequence.
template <typename T, int TAPS, int NI>
__global__ void __launch_bounds__(256, NI <= 4 ? 2 : 1) delta_prep_kernel(const ortb200_gated_delta_args a, const Scratch s, int dkp, int dvp) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = a.heads, G = a.kv_heads, dk = a.dk, dv = a.dv;
  const int channels = 2 * G * dk + H * dv;
  const int unit = blockIdx.y * 8 + warp;           // H key heads (one per value head: each has its own decays), H value heads
  pdl_wait_prior_grids();
  pdl_launch_dependents();
  if (unit >= 2 * H) return;
  int run = blockIdx.x, b = 0, first = 0, len = 0;  // runs of all sequences are numbered consecutively
  for (; b < a.B; ++b) {
    first = a.cu_seqlens[b];
    len = a.cu_seqlens[b + 1] - first;
    const int runs = (len + kPrepRun - 1) / kPrepRun;
    if (run < runs) break;
    run -= runs;
  }
  if (b == a.B) return;
  const int slot = a.slots[b], past = a.past_seqlens[b];
  const bool ok = slot >= 0 && slot < a.num_slots;
  if (!ok && a.status && lane == 0) atomicExch(a.status, kStatusBadArgument);
  const T* ring = static_cast<const T*>(a.conv_state) + static_cast<long long>(ok ? slot : 0) * a.taps * channels;
  const int i0 = run * kPrepRun, i1 = min(len, i0 + kPrepRun);
  const long long block0 = first / kBlock + b;
  const T* base = static_cast<const T*>(a.qkvb);
  if (unit < H) {
    const int h = unit, u = h / (H / G), cq = u * dk, ck = (G + u) * dk;
    ConvWindow<T, TAPS, NI> wq, wk;
    if constexpr (TAPS > 0) {
      wq.load_taps(a.conv, cq, dk, lane);
      wk.load_taps(a.conv, ck, dk, lane);
      const T* row = base + static_cast<long long>(first + i0) * a.ld;
      wq.refill(row + cq, a.ld, ring, channels, cq, dk, lane, past + i0, i0);
      wk.refill(row + ck, a.ld, ring, channels, ck, dk, lane, past + i0, i0);
    }
    const float root = 1.f / sqrtf(static_cast<float>(dk)), rate = expf(a.a_log[h]);
    for (int ib = i0; ib < i1; ib += kBlock) {
      float q[kBlock][NI], k[kBlock][NI], g[kBlock][NI], beta = 0.f;
#pragma unroll
      for (int j = 0; j < kBlock; ++j) {
        const int i = ib + j;
        if (i < i1) {
          const long long t = first + i;
          if constexpr (TAPS > 0) {
            const T* row = base + t * a.ld;
            wq.step(row + cq, dk, lane, q[j]);
            wk.step(row + ck, dk, lane, k[j]);
          } else {
            wq = {&a, ring, channels, cq, past + i, i, t};
            wk = {&a, ring, channels, ck, past + i, i, t};
            wq.step(dk, lane, q[j]);
            wk.step(dk, lane, k[j]);
          }
          float qq = 0.f, kk = 0.f;
#pragma unroll
          for (int n = 0; n < NI; ++n) {
            qq = fmaf(q[j][n], q[j][n], qq);
            kk = fmaf(k[j][n], k[j][n], kk);
          }
#pragma unroll
          for (int off = 16; off > 0; off >>= 1) {
            qq += __shfl_xor_sync(0xffffffffu, qq, off);
            kk += __shfl_xor_sync(0xffffffffu, kk, off);
          }
          const float qs = root / sqrtf(qq + a.unit_eps), ks = 1.f / sqrtf(kk + a.unit_eps);
          const T* low = static_cast<const T*>(a.low) + t * H * (dk + dv) + h * dk;
#pragma unroll
          for (int n = 0; n < NI; ++n) {
            const int d = n * 32 + lane;
            q[j][n] *= qs;
            k[j][n] *= ks;
            g[j][n] = d < dk ? expf(-rate * softplus_f(to_float<T>(low[d]) + a.dt_bias[h * dk + d])) : 1.f;
          }
          if (lane == j) beta = sigmoid_f(to_float<T>(base[t * a.ld + channels + h]));
        } else {   // behind the end: tokens that leave the state alone
#pragma unroll
          for (int n = 0; n < NI; ++n) {
            q[j][n] = k[j][n] = 0.f;
            g[j][n] = 1.f;
          }
        }
      }
      const long long blk = block0 + ib / kBlock;
      float* out = s.vec + (blk * H + h) * kVecs * dkp + lane;
      float dots[16];
#pragma unroll
      for (int n = 0; n < 16; ++n) dots[n] = 0.f;
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        float P = 1.f;
#pragma unroll
        for (int j = 0; j < kBlock; ++j) {
          P *= g[j][n];
          out[j * dkp + n * 32] = P * k[j][n];
          out[(kBlock + j) * dkp + n * 32] = P * q[j][n];
        }
        out[3 * kBlock * dkp + n * 32] = P;
        // k_t . g k_j ordered by t, then j < t; behind them q_t . g k_j ordered by t, then j <= t
#pragma unroll
        for (int j = 0; j < kBlock; ++j) {
          float x = k[j][n];
          dots[6 + j * (j + 1) / 2 + j] = fmaf(q[j][n], x, dots[6 + j * (j + 1) / 2 + j]);
#pragma unroll
          for (int t = j + 1; t < kBlock; ++t) {
            x *= g[t][n];
            dots[t * (t - 1) / 2 + j] = fmaf(k[t][n], x, dots[t * (t - 1) / 2 + j]);
            dots[6 + t * (t + 1) / 2 + j] = fmaf(q[t][n], x, dots[6 + t * (t + 1) / 2 + j]);
          }
          out[(2 * kBlock + j) * dkp + n * 32] = x;
        }
      }
      const float sum = reduce16(dots, lane);
      float* sc = s.scal + (blk * H + h) * kScal;
      if (lane < kBlock) sc[lane] = beta;
      if (lane < 16) sc[kBlock + lane] = sum;
    }
  } else {
    const int h = unit - H, cv = 2 * G * dk + h * dv;
    for (int c0 = 0; c0 < dvp; c0 += NI * 32) {
      const int n = dv - c0;
      ConvWindow<T, TAPS, NI> wv;
      if constexpr (TAPS > 0) {
        wv.load_taps(a.conv, cv + c0, n, lane);
        wv.refill(base + static_cast<long long>(first + i0) * a.ld + cv + c0, a.ld, ring, channels, cv + c0, n, lane, past + i0, i0);
      }
      const int padded = (i1 + kBlock - 1) / kBlock * kBlock;
      for (int i = i0; i < padded; ++i) {
        const long long t = first + i;
        float v[NI];
        if (i < i1) {
          if constexpr (TAPS > 0) {
            wv.step(base + t * a.ld + cv + c0, n, lane, v);
          } else {
            wv = {&a, ring, channels, cv + c0, past + i, i, t};
            wv.step(n, lane, v);
          }
        } else {
#pragma unroll
          for (int e = 0; e < NI; ++e) v[e] = 0.f;
        }
        float* out = s.v + ((block0 * kBlock + i) * H + h) * dvp + c0;
#pragma unroll
        for (int e = 0; e < NI; ++e)
          if (c0 + e * 32 + lane < dvp) out[e * 32 + lane] = v[e];
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) mlstm_prep_kernel(const ortb200_mlstm_args a, const Scratch s, int dkp, int dvp) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = a.heads, dk = a.dk, dv = a.dv;
  const int h = blockIdx.y * 8 + warp;
  pdl_wait_prior_grids();
  pdl_launch_dependents();
  const T* row = static_cast<const T*>(a.packed) + static_cast<long long>(t) * a.ld;
  const float qs = 1.f / sqrtf(static_cast<float>(dk));
  if (h < H) {
    float* qk = s.vec + (static_cast<long long>(t) * H + h) * 2 * dkp;
    for (int d = lane; d < dkp; d += 32) {
      const float q = d < dk ? to_float<T>(row[h * dk + d]) * qs : 0.f;
      const float k = d < dk ? to_float<T>(row[(H + h) * dk + d]) : 0.f;
      qk[d] = q;
      qk[dkp + d] = k;
    }
    const T* v = row + 2 * H * dk + h * dv;
    float* vr = s.v + (static_cast<long long>(t) * H + h) * dvp;
    for (int d = lane; d < dvp; d += 32) vr[d] = d < dv ? to_float<T>(v[d]) : 0.f;
    if (lane == 0) {
      const T* gates = row + 2 * H * (dk + dv);
      float* sc = s.scal + (static_cast<long long>(t) * H + h) * 4;
      sc[0] = a.gate_cap * tanhf((to_float<T>(gates[h]) + a.i_bias[h]) / a.gate_cap);
      sc[1] = logsigmoid_f(a.gate_cap * tanhf((to_float<T>(gates[H + h]) + a.f_bias[h]) / a.gate_cap));
    }
  }
}

// --------------------------------------------------------------------------------------------------------- the scans
struct ScanParams {
  Scratch s;
  float* state;            // [num_slots, H, dk, dv]
  float* aux;              // mLSTM: [num_slots, H, dk + 1]
  const int* cu_seqlens;
  const int* past_seqlens;
  const int* slots;
  int H, dk, dv, dvp, num_slots;
  float den_eps;
  int* status;
};

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// The warp's slice of the state in registers: lane (rg = lane & 7, cg = lane >> 3) holds rows j * 32 + rg * 4 + {0..3},
// j < NJ, of the columns col0 ... col0 + 3, as pairs of rows.
template <int NJ>
struct StateSlice {
  f32x2 S[NJ][4][2];
  __device__ __forceinline__ void load(const float* g, int rg, int col0, int dk, int dv, bool fresh) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int r = j * 32 + rg * 4 + hh * 2;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float lo = 0.f, hi = 0.f;
          if (!fresh && col0 + c < dv) {
            if (r < dk) lo = g[static_cast<long long>(r) * dv + col0 + c];
            if (r + 1 < dk) hi = g[static_cast<long long>(r + 1) * dv + col0 + c];
          }
          S[j][c][hh] = pack2(lo, hi);
        }
      }
    }
  }
  __device__ __forceinline__ void store(float* g, int rg, int col0, int dk, int dv) const {
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int r = j * 32 + rg * 4 + hh * 2;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          if (col0 + c >= dv) continue;
          float lo, hi;
          unpack2(S[j][c][hh], lo, hi);
          if (r < dk) g[static_cast<long long>(r) * dv + col0 + c] = lo;
          if (r + 1 < dk) g[static_cast<long long>(r + 1) * dv + col0 + c] = hi;
        }
      }
    }
  }
};
__device__ __forceinline__ float hsum(f32x2 v) {
  float lo, hi;
  unpack2(v, lo, hi);
  return lo + hi;
}

constexpr int kStageBlocks = 2;   // delta blocks per shared-memory stage

// R = state rows per lane; dkp = 8 R.
template <int R>
__global__ void __launch_bounds__(128, R <= 16 ? 4 : 2) delta_scan_kernel(const ScanParams p) {
  constexpr int DKP = 8 * R, NJ = R / 4;
  const int cs = (blockDim.x >> 5) * 16;           // columns per block
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane & 7, cg = lane >> 3;
  const int h = blockIdx.y, b = blockIdx.z;
  const int base_col = blockIdx.x * cs;
  const int wcol = warp * 16 + cg * 4;             // column within the block's slice
  const int col0 = base_col + wcol;
  extern __shared__ __align__(16) float sm[];
  const int block_floats = kVecs * DKP + kBlock * cs + kScal;
  const int stage_floats = kStageBlocks * block_floats;

  pdl_wait_prior_grids();
  const int t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len <= 0) return;
  const int slot = p.slots[b];
  if (!slot_ok(slot, p.num_slots, p.status)) return;
  const bool fresh = p.past_seqlens[b] == 0;
  const long long block0 = t0 / kBlock + b;
  const int blocks = (len + kBlock - 1) / kBlock;

  auto fetch = [&](int stage) {
    float* st = sm + (stage & 1) * stage_floats;
    const int n = min(kStageBlocks, blocks - stage * kStageBlocks);
    for (int i = 0; i < n; ++i) {
      const long long blk = block0 + stage * kStageBlocks + i;
      float* dst = st + i * block_floats;
      const float* vec = p.s.vec + (blk * p.H + h) * kVecs * DKP;
      for (int c = threadIdx.x; c < kVecs * DKP / 4; c += blockDim.x) cp_async16(dst + c * 4, vec + c * 4);
      dst += kVecs * DKP;
      const int vq = cs / 4;
      for (int c = threadIdx.x; c < kBlock * vq; c += blockDim.x) {
        const int tt = c / vq, x = c % vq;
        if (base_col + x * 4 < p.dvp) cp_async16(dst + tt * cs + x * 4, p.s.v + ((blk * kBlock + tt) * p.H + h) * p.dvp + base_col + x * 4);
      }
      dst += kBlock * cs;
      if (threadIdx.x < kScal / 4) cp_async16(dst + threadIdx.x * 4, p.s.scal + (blk * p.H + h) * kScal + threadIdx.x * 4);
    }
    cp_async_commit();
  };

  float* gst = p.state + (static_cast<long long>(slot) * p.H + h) * p.dk * p.dv;
  StateSlice<NJ> st;
  st.load(gst, rg, col0, p.dk, p.dv, fresh);
  const long long ostep = static_cast<long long>(p.H) * p.dvp;
  float* orow = p.s.o + (static_cast<long long>(t0) * p.H + h) * p.dvp + col0 + (rg & 3);
  const bool writes = rg >= 4 && col0 + (rg & 3) < p.dv;

  const int stages = (blocks + kStageBlocks - 1) / kStageBlocks;
  fetch(0);
  for (int stage = 0; stage < stages; ++stage) {
    if (stage + 1 < stages) {
      fetch(stage + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const int n = min(kStageBlocks, blocks - stage * kStageBlocks);
    for (int i = 0; i < n; ++i) {
      const float* vec = sm + (stage & 1) * stage_floats + i * block_floats + rg * 4;
      const float* vrow = sm + (stage & 1) * stage_floats + i * block_floats + kVecs * DKP + wcol + (rg & 3);
      const float* sc = sm + (stage & 1) * stage_floats + i * block_floats + kVecs * DKP + kBlock * cs;
      // lane rg ends with S^T (P_t k_t) of column rg (rg < 4), or S^T (P_t q_t) of column rg - 4
      float w[kBlock];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) {
        f32x2 accA[4], accO[4];
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(vec + t * DKP + j * 32);
          const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(vec + (kBlock + t) * DKP + j * 32);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            accA[c] = j == 0 ? mul2(st.S[j][c][0], k2.x) : fma2(st.S[j][c][0], k2.x, accA[c]);
            accO[c] = j == 0 ? mul2(st.S[j][c][0], q2.x) : fma2(st.S[j][c][0], q2.x, accO[c]);
            accA[c] = fma2(st.S[j][c][1], k2.y, accA[c]);
            accO[c] = fma2(st.S[j][c][1], q2.y, accO[c]);
          }
        }
        float y[4], z[2];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float xa = hsum(accA[c]), xo = hsum(accO[c]);
          const float send = (rg & 4) ? xa : xo, keep = (rg & 4) ? xo : xa;
          y[c] = keep + __shfl_xor_sync(0xffffffffu, send, 4);
        }
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const float send = (rg & 2) ? y[c] : y[2 + c], keep = (rg & 2) ? y[2 + c] : y[c];
          z[c] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
        }
        const float send = (rg & 1) ? z[0] : z[1], keep = (rg & 1) ? z[1] : z[0];
        w[t] = keep + __shfl_xor_sync(0xffffffffu, send, 1);
      }
      // forward substitution (meaningful on the lanes rg < 4)
      const float4 beta = *reinterpret_cast<const float4*>(sc), kk0 = *reinterpret_cast<const float4*>(sc + 4);
      const float2 kk1 = *reinterpret_cast<const float2*>(sc + 8);
      float u[kBlock];
      u[0] = beta.x * (vrow[0] - w[0]);
      u[1] = beta.y * (vrow[cs] - w[1] - kk0.x * u[0]);
      u[2] = beta.z * (vrow[2 * cs] - w[2] - kk0.y * u[0] - kk0.z * u[1]);
      u[3] = beta.w * (vrow[3 * cs] - w[3] - kk0.w * u[0] - kk1.x * u[1] - kk1.y * u[2]);
      // S' = P_4 S + sum_j K_j u_j^T
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const ulonglong2 P = *reinterpret_cast<const ulonglong2*>(vec + 3 * kBlock * DKP + j * 32);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          st.S[j][c][0] = mul2(st.S[j][c][0], P.x);
          st.S[j][c][1] = mul2(st.S[j][c][1], P.y);
        }
      }
#pragma unroll
      for (int t = 0; t < kBlock; ++t) {
        f32x2 uu[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float x = __shfl_sync(0xffffffffu, u[t], (lane & 24) | c);
          uu[c] = pack2(x, x);
        }
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(vec + (2 * kBlock + t) * DKP + j * 32);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            st.S[j][c][0] = fma2(k2.x, uu[c], st.S[j][c][0]);
            st.S[j][c][1] = fma2(k2.y, uu[c], st.S[j][c][1]);
          }
        }
      }
      // outputs (lanes rg >= 4)
#pragma unroll
      for (int t = 0; t < kBlock; ++t) u[t] = __shfl_sync(0xffffffffu, u[t], (lane & 24) | (rg & 3));
      const int left = len - (stage * kStageBlocks + i) * kBlock;
#pragma unroll
      for (int t = 0; t < kBlock; ++t) {
        float o = w[t];
#pragma unroll
        for (int j = 0; j <= t; ++j) o = fmaf(sc[10 + t * (t + 1) / 2 + j], u[j], o);
        if (writes && t < left) orow[t * ostep] = o;
      }
      orow += kBlock * ostep;
    }
    __syncthreads();   // the stage may be refilled
  }
  pdl_launch_dependents();
  st.store(gst, rg, col0, p.dk, p.dv);
}

template <int R>
__global__ void __launch_bounds__(128, R <= 16 ? 4 : 2) mlstm_scan_kernel(const ScanParams p) {
  constexpr int DKP = 8 * R, NJ = R / 4;
  const int cs = (blockDim.x >> 5) * 16;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane & 7, cg = lane >> 3;
  const int h = blockIdx.y, b = blockIdx.z;
  const int base_col = blockIdx.x * cs;
  const int wcol = warp * 16 + cg * 4;
  const int col0 = base_col + wcol;
  extern __shared__ __align__(16) float sm[];
  const int stage_floats = kChunk * (2 * DKP + cs + 4);

  pdl_wait_prior_grids();
  const int t0 = p.cu_seqlens[b], len = p.cu_seqlens[b + 1] - t0;
  if (len <= 0) return;
  const int slot = p.slots[b];
  if (!slot_ok(slot, p.num_slots, p.status)) return;
  const bool fresh = p.past_seqlens[b] == 0;

  auto fetch = [&](int chunk) {
    float* st = sm + (chunk & 1) * stage_floats;
    const int first = chunk * kChunk, n = min(kChunk, len - first);
    for (int i = threadIdx.x; i < n * (2 * DKP / 4); i += blockDim.x) {
      const int tt = i / (2 * DKP / 4), c = i % (2 * DKP / 4);
      cp_async16(st + tt * 2 * DKP + c * 4, p.s.vec + ((static_cast<long long>(t0 + first + tt) * p.H + h) * 2 * DKP) + c * 4);
    }
    float* sv = st + kChunk * 2 * DKP;
    const int vq = cs / 4;
    for (int i = threadIdx.x; i < n * vq; i += blockDim.x) {
      const int tt = i / vq, c = i % vq;
      if (base_col + c * 4 < p.dvp) cp_async16(sv + tt * cs + c * 4, p.s.v + (static_cast<long long>(t0 + first + tt) * p.H + h) * p.dvp + base_col + c * 4);
    }
    float* sc = sv + kChunk * cs;
    for (int i = threadIdx.x; i < n; i += blockDim.x) cp_async16(sc + i * 4, p.s.scal + (static_cast<long long>(t0 + first + i) * p.H + h) * 4);
    cp_async_commit();
  };

  float* gst = p.state + (static_cast<long long>(slot) * p.H + h) * p.dk * p.dv;
  const float* gaux = p.aux + (static_cast<long long>(slot) * p.H + h) * (p.dk + 1);
  StateSlice<NJ> s;
  s.load(gst, rg, col0, p.dk, p.dv, fresh);
  constexpr int NR = DKP / 32;                     // every warp keeps n, lane l its rows l, l + 32, ...
  float nrm[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) nrm[i] = !fresh && i * 32 + lane < p.dk ? gaux[i * 32 + lane] : 0.f;
  float m = fresh ? 0.f : gaux[p.dk];
  float* orow = p.s.o + (static_cast<long long>(t0) * p.H + h) * p.dvp + col0;
  const long long ostep = static_cast<long long>(p.H) * p.dvp;

  const int chunks = (len + kChunk - 1) / kChunk;
  fetch(0);
  for (int ch = 0; ch < chunks; ++ch) {
    if (ch + 1 < chunks) {
      fetch(ch + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* st = sm + (ch & 1) * stage_floats;
    const float* sv = st + kChunk * 2 * DKP;
    const float* sc = sv + kChunk * cs;
    const int n = min(kChunk, len - ch * kChunk);
    for (int tt = 0; tt < n; ++tt) {
      const float* qr = st + tt * 2 * DKP;
      const float* kr = qr + DKP;
      const float4 vv = *reinterpret_cast<const float4*>(sv + tt * cs + wcol);
      const float2 gate = *reinterpret_cast<const float2*>(sc + tt * 4);
      const float m_new = fmaxf(gate.y + m, gate.x);
      const float fw = expf(gate.y + m - m_new), iw = expf(gate.x - m_new);
      m = m_new;
      const f32x2 f2 = pack2(fw, fw), i2 = pack2(iw, iw);
      const f32x2 v2[4] = {pack2(vv.x, vv.x), pack2(vv.y, vv.y), pack2(vv.z, vv.z), pack2(vv.w, vv.w)};
      f32x2 accO[4];
      float nq = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        nrm[i] = fmaf(nrm[i], fw, iw * kr[i * 32 + lane]);
        nq = fmaf(nrm[i], qr[i * 32 + lane], nq);
      }
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(qr + j * 32 + rg * 4);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(kr + j * 32 + rg * 4);
        const f32x2 ik0 = mul2(k2.x, i2), ik1 = mul2(k2.y, i2);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          s.S[j][c][0] = fma2(ik0, v2[c], mul2(s.S[j][c][0], f2));
          s.S[j][c][1] = fma2(ik1, v2[c], mul2(s.S[j][c][1], f2));
          accO[c] = j == 0 ? mul2(s.S[j][c][0], q2.x) : fma2(s.S[j][c][0], q2.x, accO[c]);
          accO[c] = fma2(s.S[j][c][1], q2.y, accO[c]);
        }
      }
#pragma unroll
      for (int off = 1; off <= 16; off <<= 1) nq += __shfl_xor_sync(0xffffffffu, nq, off);
      float x[4], y[2], w;
#pragma unroll
      for (int c = 0; c < 4; ++c) x[c] = hsum(accO[c]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float send = (rg & 2) ? x[i] : x[2 + i], keep = (rg & 2) ? x[2 + i] : x[i];
        y[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
      }
      {
        const float send = (rg & 1) ? y[0] : y[1], keep = (rg & 1) ? y[1] : y[0];
        w = keep + __shfl_xor_sync(0xffffffffu, send, 1);
      }
      w += __shfl_xor_sync(0xffffffffu, w, 4);
      if (rg < 4 && col0 + rg < p.dv) orow[rg] = w / (fmaxf(fabsf(nq), expf(-m)) + p.den_eps);
      orow += ostep;
    }
    __syncthreads();   // the stage may be refilled
  }
  pdl_launch_dependents();
  s.store(gst, rg, col0, p.dk, p.dv);
  // n and m: every block of a (head, sequence) computes the same values, and another block may still have to read the
  // old ones, so they leave through scratch and the post kernel moves them into the state
  if (blockIdx.x == 0 && warp == 0) {
    float* ao = p.s.aux_out + (static_cast<long long>(b) * p.H + h) * (p.dk + 1);
#pragma unroll
    for (int i = 0; i < NR; ++i)
      if (i * 32 + lane < p.dk) ao[i * 32 + lane] = nrm[i];
    if (lane == 0) ao[p.dk] = m;
  }
}

// ------------------------------------------------------------------------------------------------------------- post
struct PostParams {
  const float* o;          // [T, H, dvp]
  const float* norm;       // [dv] (norm_stride 0) or [H * dv] (norm_stride dv)
  const void* gate;        // row t at gate + t * gate_ld elements, H * dv entries
  void* out;               // [T, H * dv]
  long long gate_ld;
  int H, dv, dvp, norm_stride;
  float eps;
  // convolution inputs of the last `taps` tokens -> ring
  const void* conv_in;
  void* conv_state;
  int conv_ld, channels, taps;
  // n and m of the sequence -> state
  const float* aux_out;
  float* aux;
  int dk;
  const int* cu_seqlens;
  const int* past_seqlens;
  const int* slots;
  int B, num_slots;
  int vec;                 // gate, out and dv allow four-element accesses
};

template <typename T>
__device__ __forceinline__ void copy4(T* dst, const T* src) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(src);
  else *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(src);
}
template <typename T>
int post_vec(const PostParams& p) {
  return p.dv % 4 == 0 && p.gate_ld % 4 == 0 && ((reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out)) & (4 * sizeof(T) - 1)) == 0;
}

// One warp per (token, head); lane l holds the columns 4 l ... 4 l + 3 of every 128.
template <typename T>
__global__ void __launch_bounds__(256) recurrent_post_kernel(const PostParams p) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * 8 + warp;
  pdl_wait_prior_grids();
  pdl_launch_dependents();
  if (h < p.H) {
    const float* o = p.o + (static_cast<long long>(t) * p.H + h) * p.dvp;
    float x[kMaxHead / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxHead / 128; ++i) {
      const int d = i * 128 + lane * 4;
      const float4 v = d < p.dvp ? *reinterpret_cast<const float4*>(o + d) : make_float4(0.f, 0.f, 0.f, 0.f);   // rows padded to fours
      x[i * 4] = v.x;
      x[i * 4 + 1] = d + 1 < p.dv ? v.y : 0.f;
      x[i * 4 + 2] = d + 2 < p.dv ? v.z : 0.f;
      x[i * 4 + 3] = d + 3 < p.dv ? v.w : 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(x[i * 4 + e], x[i * 4 + e], ss);
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / p.dv + p.eps);
    const T* gate = static_cast<const T*>(p.gate) + t * p.gate_ld + h * p.dv;
    T* out = static_cast<T*>(p.out) + (static_cast<long long>(t) * p.H + h) * p.dv;
    const float* norm = p.norm + h * p.norm_stride;
#pragma unroll
    for (int i = 0; i < kMaxHead / 128; ++i) {
      const int d = i * 128 + lane * 4;
      if (p.vec) {
        if (d < p.dv) {
          __align__(16) T g[4], y[4];
          copy4(g, gate + d);
#pragma unroll
          for (int e = 0; e < 4; ++e) y[e] = from_float<T>(x[i * 4 + e] * r * norm[d + e] * act_sigmoid<T>(to_float<T>(g[e])));
          copy4(out + d, y);
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (d + e < p.dv) out[d + e] = from_float<T>(x[i * 4 + e] * r * norm[d + e] * act_sigmoid<T>(to_float<T>(gate[d + e])));
      }
    }
  }
  if (blockIdx.y != 0) return;
  const int b = sequence_of(p.cu_seqlens, p.B, t);
  const int end = p.cu_seqlens[b + 1];
  const int slot = p.slots[b];
  if (slot >= 0 && slot < p.num_slots) {
    if (p.conv_state && t >= end - p.taps) {
      const int pos = p.past_seqlens[b] + t - p.cu_seqlens[b];
      const T* src = static_cast<const T*>(p.conv_in) + static_cast<long long>(t) * p.conv_ld;
      T* dst = static_cast<T*>(p.conv_state) + (static_cast<long long>(slot) * p.taps + pos % p.taps) * p.channels;
      for (int c = threadIdx.x; c < p.channels; c += blockDim.x) dst[c] = src[c];
    }
    if (p.aux && t == end - 1) {
      const long long n = static_cast<long long>(p.H) * (p.dk + 1);
      for (int i = threadIdx.x; i < n; i += blockDim.x) p.aux[slot * n + i] = p.aux_out[b * n + i];
    }
  }
}

// ----------------------------------------------------------------------------------------------------------- decode
// One block per (head, sequence), one token.  Lane l of warp w holds rows w, w + 8, ... of four columns; RPW rows.
template <typename T, typename A, int RPW>
__global__ void __launch_bounds__(256) recurrent_decode_kernel(const A a) {
  constexpr bool DELTA = std::is_same<A, ortb200_gated_delta_args>::value;
  const int h = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = a.heads, dk = a.dk, dv = a.dv;
  __shared__ float sq[kMaxHead], sk[kMaxHead], sg[kMaxHead], sv[kMaxHead], so[kMaxHead];
  __shared__ float redA[8][128], redO[8][128], su[128];
  __shared__ float red[8], scal[4];
  __shared__ float4 red3[8];
  pdl_wait_prior_grids();
  const int slot = a.slots[b];
  if (!slot_ok(slot, a.num_slots, a.status)) return;
  const int pos = a.past_seqlens[b];
  const bool fresh = pos == 0;
  float* gst = a.state + (static_cast<long long>(slot) * H + h) * dk * dv;
  const bool vec = (dv & 3) == 0;

  float4 S[RPW];
  auto load_state = [&](int c0) {
    const int col = c0 + lane * 4;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + 8 * i;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && r < dk && col < dv) {
        const float* src = gst + static_cast<long long>(r) * dv + col;
        if (vec) {
          v = __ldcs(reinterpret_cast<const float4*>(src));
        } else {
          v.x = src[0];
          if (col + 1 < dv) v.y = src[1];
          if (col + 2 < dv) v.z = src[2];
          if (col + 3 < dv) v.w = src[3];
        }
      }
      S[i] = v;
    }
  };
  load_state(0);   // in flight while the inputs are prepared

  if constexpr (DELTA) {
    const int G = a.kv_heads, g = h / (H / G);
    const int channels = 2 * G * dk + H * dv;
    T* ring = static_cast<T*>(a.conv_state) + static_cast<long long>(slot) * a.taps * channels;
    T* ring_new = ring + static_cast<long long>(pos % a.taps) * channels;
    const T* x = static_cast<const T*>(a.qkvb) + static_cast<long long>(b) * a.ld;
    const T* low = static_cast<const T*>(a.low) + static_cast<long long>(b) * H * (dk + dv) + h * dk;
    const bool first_of_group = h % (H / G) == 0;
    float qq = 0.f, kk = 0.f, qk = 0.f;
    if (tid < dk) {
      const int cq = g * dk + tid, ck = (G + g) * dk + tid;
      const float q = conv_silu<T>(a, ring, channels, cq, b, pos, 0), k = conv_silu<T>(a, ring, channels, ck, b, pos, 0);
      sq[tid] = q;
      sk[tid] = k;
      qq = q * q;
      kk = k * k;
      qk = q * k;
      sg[tid] = expf(-expf(a.a_log[h]) * softplus_f(to_float<T>(low[tid]) + a.dt_bias[h * dk + tid]));
      if (first_of_group) {   // the ring entry of this position is read by nobody in this step
        ring_new[cq] = x[cq];
        ring_new[ck] = x[ck];
      }
    }
    if (tid < dv) {
      const int cv = 2 * G * dk + h * dv + tid;
      sv[tid] = conv_silu<T>(a, ring, channels, cv, b, pos, 0);
      ring_new[cv] = x[cv];
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    if (lane == 0) red3[warp] = make_float4(qq, kk, qk, 0.f);
    __syncthreads();
    qq = kk = qk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      qq += red3[w].x;
      kk += red3[w].y;
      qk += red3[w].z;
    }
    const float qs = 1.f / (sqrtf(qq + a.unit_eps) * sqrtf(static_cast<float>(dk))), ks = 1.f / sqrtf(kk + a.unit_eps);
    if (tid < dk) {
      sq[tid] *= qs;
      sk[tid] *= ks;
    }
    if (tid == 0) {
      scal[0] = sigmoid_f(to_float<T>(x[channels + h]));
      scal[1] = qk * qs * ks;
    }
  } else {
    const T* x = static_cast<const T*>(a.packed) + static_cast<long long>(b) * a.ld;
    float* aux = a.aux + (static_cast<long long>(slot) * H + h) * (dk + 1);
    const T* gates = x + 2 * H * (dk + dv);
    const float iv = a.gate_cap * tanhf((to_float<T>(gates[h]) + a.i_bias[h]) / a.gate_cap);
    const float fv = logsigmoid_f(a.gate_cap * tanhf((to_float<T>(gates[H + h]) + a.f_bias[h]) / a.gate_cap));
    const float m_old = fresh ? 0.f : aux[dk];
    const float m = fmaxf(fv + m_old, iv);
    const float fw = expf(fv + m_old - m), iw = expf(iv - m);
    float nq = 0.f;
    __syncthreads();   // every thread has read m before thread 0 replaces it
    if (tid < dk) {
      const float q = to_float<T>(x[h * dk + tid]) / sqrtf(static_cast<float>(dk));
      const float k = to_float<T>(x[(H + h) * dk + tid]) * iw;
      const float n = fmaf(fresh ? 0.f : aux[tid], fw, k);
      aux[tid] = n;
      sq[tid] = q;
      sk[tid] = k;
      nq = n * q;
    }
    if (tid < dv) sv[tid] = to_float<T>(x[2 * H * dk + h * dv + tid]);
    nq = block_sum_all(nq, red);
    if (tid == 0) {
      aux[dk] = m;
      scal[0] = fw;
      scal[1] = 1.f / (fmaxf(fabsf(nq), expf(-m)) + a.den_eps);
    }
  }
  __syncthreads();

  for (int c0 = 0; c0 < dv; c0 += 128) {
    if (c0 > 0) load_state(c0);
    const int col = c0 + lane * 4;
    float4 pa = make_float4(0.f, 0.f, 0.f, 0.f), po = pa;
    float4 v4 = pa;
    if (!DELTA) {
      if (col < dv) v4.x = sv[col];
      if (col + 1 < dv) v4.y = sv[col + 1];
      if (col + 2 < dv) v4.z = sv[col + 2];
      if (col + 3 < dv) v4.w = sv[col + 3];
    }
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + 8 * i;
      if (r >= dk) break;
      const float q = sq[r], k = sk[r];
      if (DELTA) {
        const float gr = sg[r];
        S[i].x *= gr; S[i].y *= gr; S[i].z *= gr; S[i].w *= gr;
        pa.x = fmaf(S[i].x, k, pa.x); pa.y = fmaf(S[i].y, k, pa.y); pa.z = fmaf(S[i].z, k, pa.z); pa.w = fmaf(S[i].w, k, pa.w);
      } else {
        const float f = scal[0];
        S[i].x = fmaf(k, v4.x, S[i].x * f); S[i].y = fmaf(k, v4.y, S[i].y * f);
        S[i].z = fmaf(k, v4.z, S[i].z * f); S[i].w = fmaf(k, v4.w, S[i].w * f);
      }
      po.x = fmaf(S[i].x, q, po.x); po.y = fmaf(S[i].y, q, po.y); po.z = fmaf(S[i].z, q, po.z); po.w = fmaf(S[i].w, q, po.w);
    }
    if (DELTA) *reinterpret_cast<float4*>(&redA[warp][lane * 4]) = pa;
    *reinterpret_cast<float4*>(&redO[warp][lane * 4]) = po;
    __syncthreads();
    if (tid < 128) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += redO[w][tid];
      const bool in = c0 + tid < dv;
      if (DELTA) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += redA[w][tid];
        const float u = in ? scal[0] * (sv[c0 + tid] - s) : 0.f;
        su[tid] = u;
        if (in) so[c0 + tid] = fmaf(scal[1], u, o);
      } else if (in) {
        so[c0 + tid] = o * scal[1];
      }
    }
    __syncthreads();
    float4 u4 = make_float4(0.f, 0.f, 0.f, 0.f);
    if (DELTA) u4 = *reinterpret_cast<const float4*>(&su[lane * 4]);
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + 8 * i;
      if (r >= dk || col >= dv) break;
      float4 v = S[i];
      if (DELTA) {
        const float k = sk[r];
        v.x = fmaf(k, u4.x, v.x); v.y = fmaf(k, u4.y, v.y); v.z = fmaf(k, u4.z, v.z); v.w = fmaf(k, u4.w, v.w);
      }
      float* dst = gst + static_cast<long long>(r) * dv + col;
      if (vec) {
        __stcs(reinterpret_cast<float4*>(dst), v);
      } else {
        dst[0] = v.x;
        if (col + 1 < dv) dst[1] = v.y;
        if (col + 2 < dv) dst[2] = v.z;
        if (col + 3 < dv) dst[3] = v.w;
      }
    }
    // redA / redO / su are rewritten by the next column pass only after its first barrier
    if (c0 + 128 < dv) __syncthreads();
  }
  pdl_launch_dependents();

  const float o = tid < dv ? so[tid] : 0.f;
  const float r = 1.f / sqrtf(block_sum_all(o * o, red) / dv + a.norm_eps);
  if (tid < dv) {
    float gate, w;
    if constexpr (DELTA) {
      gate = to_float<T>(static_cast<const T*>(a.low)[static_cast<long long>(b) * H * (dk + dv) + H * dk + h * dv + tid]);
      w = a.norm[tid];
    } else {
      gate = to_float<T>(static_cast<const T*>(a.packed)[static_cast<long long>(b) * a.ld + H * (2 * dk + dv) + h * dv + tid]);
      w = a.norm[h * dv + tid];
    }
    static_cast<T*>(a.out)[(static_cast<long long>(b) * H + h) * dv + tid] = from_float<T>(o * r * w * act_sigmoid<T>(gate));
  }
}

template <typename T, typename A>
int launch_decode(const A& a, cudaStream_t stream) {
  const dim3 grid(a.heads, a.B);
  const bool pdl = a.use_pdl != 0;
  if (a.dk <= 64) return launch_kernel(recurrent_decode_kernel<T, A, 8>, grid, 256, 0, stream, pdl, a);
  if (a.dk <= 128) return launch_kernel(recurrent_decode_kernel<T, A, 16>, grid, 256, 0, stream, pdl, a);
  return launch_kernel(recurrent_decode_kernel<T, A, 32>, grid, 256, 0, stream, pdl, a);
}

// Warps (16 columns each) per scan block: as many as share the staged rows without loading one SM more than another - all
// warps run from the first token to the last, so the fullest SM decides.
int scan_warps(int B, int H, int dv) {
  const int most = dv <= 16 ? 1 : (dv <= 32 ? 2 : 4);
  int warps = most;
  int64_t best = -1;
  for (int w = most; w >= 1; w /= 2) {
    const int64_t blocks = static_cast<int64_t>(B) * H * ((dv + w * 16 - 1) / (w * 16));
    const int64_t load = (blocks + 147) / 148 * w;
    if (best < 0 || load < best) {
      best = load;
      warps = w;
    }
  }
  return warps;
}

template <typename K>
int launch_scan(K kern, const ScanParams& p, int B, int warps, int smem, int* attr_smem, cudaStream_t stream, bool pdl) {
  if (smem > 48 * 1024 && smem > *attr_smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
    *attr_smem = smem;
  }
  const int cs = warps * 16;
  return launch_kernel(kern, dim3((p.dv + cs - 1) / cs, p.H, B), warps * 32, smem, stream, pdl, p);
}
template <int R>
int launch_delta_scan(const ScanParams& p, int B, cudaStream_t stream, bool pdl) {
  static int attr = 0;
  const int warps = scan_warps(B, p.H, p.dv);
  return launch_scan(delta_scan_kernel<R>, p, B, warps, 2 * kStageBlocks * (kVecs * 8 * R + kBlock * warps * 16 + kScal) * 4, &attr, stream, pdl);
}
template <int R>
int launch_mlstm_scan(const ScanParams& p, int B, cudaStream_t stream, bool pdl) {
  static int attr = 0;
  const int warps = scan_warps(B, p.H, p.dv);
  return launch_scan(mlstm_scan_kernel<R>, p, B, warps, 2 * kChunk * (2 * 8 * R + warps * 16 + 4) * 4, &attr, stream, pdl);
}

template <typename T, int TAPS>
int launch_delta_prep(const ortb200_gated_delta_args& a, const Scratch& s, int dkp, int dvp, cudaStream_t stream, bool pdl) {
  const dim3 grid(a.T / kPrepRun + a.B, (2 * a.heads + 7) / 8);   // every sequence has at most one partly filled run
  if (dkp == 64) return launch_kernel(delta_prep_kernel<T, TAPS, 2>, grid, 256, 0, stream, pdl, a, s, dkp, dvp);
  if (dkp == 128) return launch_kernel(delta_prep_kernel<T, TAPS, 4>, grid, 256, 0, stream, pdl, a, s, dkp, dvp);
  return launch_kernel(delta_prep_kernel<T, TAPS, 8>, grid, 256, 0, stream, pdl, a, s, dkp, dvp);
}

template <typename T>
int run_delta(const ortb200_gated_delta_args& a, cudaStream_t stream) {
  if (a.T == a.B) return launch_decode<T, ortb200_gated_delta_args>(a, stream);
  const bool pdl = a.use_pdl != 0;
  const int dkp = pad_dk(a.dk), dvp = pad4(a.dv);
  const Scratch s = split_scratch(a.workspace, delta_scratch(a.T, a.B, a.heads, dkp, dvp));
  int rc = a.taps == 4 ? launch_delta_prep<T, 4>(a, s, dkp, dvp, stream, pdl) : launch_delta_prep<T, 0>(a, s, dkp, dvp, stream, pdl);
  if (rc) return rc;
  ScanParams p{s, a.state, nullptr, a.cu_seqlens, a.past_seqlens, a.slots, a.heads, a.dk, a.dv, dvp, a.num_slots, 0.f, a.status};
  rc = dkp == 64 ? launch_delta_scan<8>(p, a.B, stream, pdl) : dkp == 128 ? launch_delta_scan<16>(p, a.B, stream, pdl) : launch_delta_scan<32>(p, a.B, stream, pdl);
  if (rc) return rc;
  PostParams q{};
  q.o = s.o; q.norm = a.norm; q.norm_stride = 0;
  q.gate = static_cast<const T*>(a.low) + static_cast<int64_t>(a.heads) * a.dk;
  q.gate_ld = static_cast<long long>(a.heads) * (a.dk + a.dv);
  q.out = a.out; q.H = a.heads; q.dv = a.dv; q.dvp = dvp; q.eps = a.norm_eps;
  q.conv_in = a.qkvb; q.conv_state = a.conv_state; q.conv_ld = a.ld;
  q.channels = 2 * a.kv_heads * a.dk + a.heads * a.dv; q.taps = a.taps;
  q.cu_seqlens = a.cu_seqlens; q.past_seqlens = a.past_seqlens; q.slots = a.slots; q.B = a.B; q.num_slots = a.num_slots;
  q.vec = post_vec<T>(q);
  return launch_kernel(recurrent_post_kernel<T>, dim3(a.T, (a.heads + 7) / 8), 256, 0, stream, pdl, q);
}

template <typename T>
int run_mlstm(const ortb200_mlstm_args& a, cudaStream_t stream) {
  if (a.T == a.B) return launch_decode<T, ortb200_mlstm_args>(a, stream);
  const bool pdl = a.use_pdl != 0;
  const int dkp = pad_dk(a.dk), dvp = pad4(a.dv);
  const Scratch s = split_scratch(a.workspace, mlstm_scratch(a.T, a.B, a.heads, a.dk, dkp, dvp));
  int rc = launch_kernel(mlstm_prep_kernel<T>, dim3(a.T, (a.heads + 7) / 8), 256, 0, stream, pdl, a, s, dkp, dvp);
  if (rc) return rc;
  ScanParams p{s, a.state, a.aux, a.cu_seqlens, a.past_seqlens, a.slots, a.heads, a.dk, a.dv, dvp, a.num_slots, a.den_eps, a.status};
  rc = dkp == 64 ? launch_mlstm_scan<8>(p, a.B, stream, pdl) : dkp == 128 ? launch_mlstm_scan<16>(p, a.B, stream, pdl) : launch_mlstm_scan<32>(p, a.B, stream, pdl);
  if (rc) return rc;
  PostParams q{};
  q.o = s.o; q.norm = a.norm; q.norm_stride = a.dv;
  q.gate = static_cast<const T*>(a.packed) + static_cast<int64_t>(a.heads) * (2 * a.dk + a.dv);
  q.gate_ld = a.ld;
  q.out = a.out; q.H = a.heads; q.dv = a.dv; q.dvp = dvp; q.eps = a.norm_eps;
  q.aux_out = s.aux_out; q.aux = a.aux; q.dk = a.dk;
  q.cu_seqlens = a.cu_seqlens; q.past_seqlens = a.past_seqlens; q.slots = a.slots; q.B = a.B; q.num_slots = a.num_slots;
  q.vec = post_vec<T>(q);
  return launch_kernel(recurrent_post_kernel<T>, dim3(a.T, (a.heads + 7) / 8), 256, 0, stream, pdl, q);
}

bool sizes_ok(int T, int B, int heads, int dk, int dv, int num_slots) {
  return T > 0 && B > 0 && B <= T && heads > 0 && dk > 0 && dk <= kMaxHead && dv > 0 && dv <= kMaxHead && num_slots > 0 && B <= 65535 &&
         heads <= 65535;
}

}  // namespace

}  // namespace ortb200

using namespace ortb200;

extern "C" int64_t ortb200_recurrent_workspace_bytes(int T, int B, int heads, int kv_heads, int dk, int dv) {
  if (T == B) return 0;
  (void)kv_heads;
  const int64_t delta = delta_scratch(T, B, heads, pad_dk(dk), pad4(dv)).total(), mem = mlstm_scratch(T, B, heads, dk, pad_dk(dk), pad4(dv)).total();
  return 4 * (delta > mem ? delta : mem);
}

extern "C" int ortb200_gated_delta(const ortb200_gated_delta_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->qkvb || !a->low || !a->conv || !a->a_log || !a->dt_bias || !a->norm || !a->conv_state || !a->state || !a->cu_seqlens ||
      !a->past_seqlens || !a->slots || !a->out)
    return -1;
  if (!sizes_ok(a->T, a->B, a->heads, a->dk, a->dv, a->num_slots) || a->kv_heads <= 0 || a->heads % a->kv_heads != 0) return -2;
  if (a->taps < 1 || a->taps > kMaxTaps || a->ld < 2 * a->kv_heads * a->dk + a->heads * (a->dv + 1)) return -2;
  if (a->T != a->B && (!a->workspace || a->workspace_bytes < ortb200_recurrent_workspace_bytes(a->T, a->B, a->heads, a->kv_heads, a->dk, a->dv)))
    return -5;
  if ((reinterpret_cast<uintptr_t>(a->workspace) | reinterpret_cast<uintptr_t>(a->state)) & 15) return -3;
  switch (a->dtype) {
    case ORTB200_F16: return run_delta<__half>(*a, stream);
    case ORTB200_BF16: return run_delta<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return run_delta<float>(*a, stream);
    default: return -4;
  }
}

extern "C" int ortb200_mlstm(const ortb200_mlstm_args* a, ortb200_stream_t stream_) {
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  if (!a || !a->packed || !a->i_bias || !a->f_bias || !a->norm || !a->state || !a->aux || !a->cu_seqlens || !a->past_seqlens || !a->slots ||
      !a->out)
    return -1;
  if (!sizes_ok(a->T, a->B, a->heads, a->dk, a->dv, a->num_slots) || a->gate_cap <= 0.f) return -2;
  if (a->ld < a->heads * (2 * a->dk + 2 * a->dv + 2)) return -2;
  if (a->T != a->B && (!a->workspace || a->workspace_bytes < ortb200_recurrent_workspace_bytes(a->T, a->B, a->heads, a->heads, a->dk, a->dv)))
    return -5;
  if ((reinterpret_cast<uintptr_t>(a->workspace) | reinterpret_cast<uintptr_t>(a->state)) & 15) return -3;
  switch (a->dtype) {
    case ORTB200_F16: return run_mlstm<__half>(*a, stream);
    case ORTB200_BF16: return run_mlstm<__nv_bfloat16>(*a, stream);
    case ORTB200_F32: return run_mlstm<float>(*a, stream);
    default: return -4;
  }
}
