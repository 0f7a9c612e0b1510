// Internal declarations shared by the kernels of the scalar-decay state space recurrence (ssd.cu: fp32, position by position;
// ssd_chunk.cu: prompts of a bf16 engine on the tensor cores).
#pragma once
#include <cuda_runtime.h>

#include "blocks.h"

namespace asd {

struct SsdArgs {
    SeqIndex ix;
    const int* cu_q;
    const int* seq_slot;
    SsdInput in;
    SsdDims d;
    float* state;
    int ring, CH, v16;
    float* out;
};

__device__ __forceinline__ float softplus_step(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace asd
