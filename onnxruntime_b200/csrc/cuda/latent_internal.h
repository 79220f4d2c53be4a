// Internal interface between the latent-attention dispatcher (latent.cu) and its tensor-core kernel (latent_decode_tc.cu).
#pragma once
#include <cuda_runtime.h>
#include "ortb200_kernels.h"

namespace ortb200 {

int launch_latent_decode_tc(const ortb200_latent_decode_args* a, cudaStream_t stream);

}  // namespace ortb200
