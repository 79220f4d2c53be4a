// Shared by the flash-attention kernels (attn_prefill.cu, attn_split.cu).
#pragma once
#include <cuda_runtime.h>
#include "ortb200_kernels.h"

namespace ortb200 {

struct AttnParams {
  const int* seqlens_k;
  const int* key_mask;
  const void* head_sink;
  void* out;
  int B, S, N, Nk, kv_len;
  long long o_strides[3];
  int first_prompt, causal, window;
  float scale_log2, softcap, scale;
  int bf16;
  int* status;
  // packed queries over a paged cache (block_table given)
  const int* block_table;
  const int* cu_seqlens;
  const int* past_seqlens;
  int block_size, max_blocks, num_blocks;
  int chunk;             // > 0: keys of the query's own chunk only
};

// Packed queries over a paged cache, softmax weights as the sum of two 16-bit terms (the caller has checked the arguments).
int launch_attn_split(const ortb200_attn_prefill_args* a, cudaStream_t stream);

#ifdef __CUDACC__
__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float r;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}
__device__ __forceinline__ float ex2_approx(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
#endif

}  // namespace ortb200
