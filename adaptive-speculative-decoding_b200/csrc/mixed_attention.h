// Internal declarations shared by the kernels of the mixed-weights attention (mixed_attention.cu: CUDA cores, any sizes,
// both element types; mixed_attention_tc.cu: prompts of a bf16 engine on the tensor cores; steps of few tokens).
#pragma once
#include <cuda_runtime.h>

#include "blocks.h"
#include "elem.cuh"

namespace asd {

struct MixArgs {
    SeqIndex ix;
    const int* cu_q;
    const int* seq_slot;
    const float* q;
    long long ldq;
    MixDims d;
    const float* dist_bias;
    int far;
    const float* talk;
    const float* gate;
    long long ldg;
    PagedRows cache;
    void* out;
    int of32;
    long long ldo;
    float* stats;      // [2][shares][M][heads]: maximum, then sum of exponentials, of every key share
    float* part;       // [shares][M][heads * dv]
    float* scores;     // steps of few tokens: [M][heads][score_ld] scaled, biased scores of the visible keys
    long long score_ld;
    int QT, shares, gp, rag, dkp, dvp, vec;
};

// sigmoid of the gate of one result element (1 without a gate)
__device__ __forceinline__ float mix_gate(const MixArgs& a, long long m, int h, int col) {
    if (!a.gate) return 1.f;
    return 1.f / (1.f + expf(-a.gate[m * a.ldg + (a.d.gate_per_value ? h * a.d.dv + col : h)]));
}

// cap * tanh(v / cap) of a warp's scores: the Taylor series of tanh to the seventh power where all of them lie below a quarter
// of the cap, else 1 - 2 / (1 + e^(2a)) for those beyond it; relative error below 1e-6
template <int N>
__device__ __forceinline__ void cap_scores(float (&s)[N][4], float cap, float icap) {
    float top = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) top = fmaxf(top, fabsf(s[n][e]));
    const bool beyond = __any_sync(0xffffffffu, !(top * icap < 0.25f));
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float v = s[n][e], a = v * icap, a2 = a * a;
            float r = v * fmaf(a2, fmaf(a2, fmaf(a2, -17.f / 315.f, 2.f / 15.f), -1.f / 3.f), 1.f);
            if (beyond && fabsf(a) >= 0.25f) r = copysignf(cap * (1.f - __fdividef(2.f, 1.f + __expf(2.f * fabsf(a)))), v);
            s[n][e] = r;
        }
}

// Prompts and portions of a bf16 engine on the tensor cores (mma.sync, fp32 operands as two bf16 terms).  Returns 1 if
// these sizes are not taken (the caller then runs the CUDA-core kernels), 0 after the launches, -1 on an error.
int launch_mix_attention_tc(MixArgs a, int nseq, int max_qlen, int max_kv_len, const MixWork& ws, cudaStream_t stream);
// Steps of one token per sequence: scores once (kept in the workspace), then weights, mix and values.  Same returns.
int launch_mix_attention_decode(MixArgs a, int nseq, int max_kv_len, const MixWork& ws, cudaStream_t stream);
// The same with sigmoid weights (sigmoid_attention.cu): one pass.  Same returns.
int launch_sigmoid_attention_decode(MixArgs a, int max_kv_len, const MixWork& ws, cudaStream_t stream);
// Steps of few tokens on the tensor cores for bf16 cache rows, sigmoid or softmax weights without a head mix or distance bias
// (decode_attention_tc.cu).  Same returns.
int launch_attention_decode_tc(MixArgs a, int nseq, int max_qlen, int max_kv_len, const MixWork& ws,
                                       cudaStream_t stream);
// sums the key shares' partial results in index order, applies the gates, writes the engine's element type
int launch_mix_merge(const MixArgs& a, cudaStream_t stream, bool stats = false);

}  // namespace asd
