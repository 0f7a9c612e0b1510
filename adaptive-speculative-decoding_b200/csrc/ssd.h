// Internal declarations shared by the kernels of the scalar-decay state space recurrence (ssd.cu: fp32, position by position;
// ssd_chunk.cu: prompts of a bf16 engine on the tensor cores).
#pragma once
#include <cuda_runtime.h>

#include "blocks.h"
#include "elem.cuh"

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
    int tail = 0;     // positions at the end of every sequence: only them (sequential kernel) or without them (chunks)
};

__device__ __forceinline__ float softplus_step(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// element i of x, b or c
__device__ __forceinline__ float ssd_in(const SsdArgs& a, const void* p, long long i) { return ldx(p, i, !a.in.bf16); }

// The positions of every sequence but the last a.tail on the tensor cores.  Returns 1 if these sizes are not taken, 0 after the
// launch, -1 on an error.
int launch_ssd_chunks(SsdArgs a, int nseq, cudaStream_t stream);

}  // namespace asd
