// Mixture-of-experts routing: fp32 softmax over all experts, the `top` largest probabilities kept as gates (as they
// are, or divided by their sum, which is the softmax over the chosen logits alone), or sigmoid scores chosen with a
// correction among the best groups of experts; then the (token, choice) pairs grouped by expert so that each expert's rows are contiguous
// for the grouped linear layers.  Which slot inside an expert's group a pair gets does not matter for the result: every
// slot is computed on its own and a token's choices are summed in choice order by the layer close.
#include <cuda_runtime.h>
#include <math.h>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"

namespace asd {

namespace {

struct RouteChoice {
    int top, renorm, sigmoid, groups, keep;
    const float* correction;
    float scale;
    int plain;             // sigmoid scores are the gates as they are
    float* slot_gate;      // optional [M * top]: the gate of each slot
};

// One warp chooses a token's experts from its logits z[E] and writes their indices and gates; counts take one each.
// pr: E floats of scratch; gr: c.groups floats of scratch (used with groups > 1 only).
__device__ void choose_experts(const float* z, int E, const RouteChoice& c, float* pr, float* gr, int* expert_of, float* gate,
                               int* counts, int lane) {
    const float TAKEN = -INFINITY;
    float inv = 1.f;
    if (c.sigmoid) {
        for (int e = lane; e < E; e += 32) pr[e] = 1.f / (1.f + expf(-z[e])) + (c.correction ? c.correction[e] : 0.f);
        __syncwarp();
        if (c.groups > 1) {
            const int n = E / c.groups;
            for (int g = lane; g < c.groups; g += 32) {
                float a = -INFINITY, b = -INFINITY;      // the two largest choice scores of the group
                for (int e = g * n; e < (g + 1) * n; ++e) {
                    const float v = pr[e];
                    if (v > a) {
                        b = a;
                        a = v;
                    } else if (v > b) {
                        b = v;
                    }
                }
                gr[g] = n > 1 ? a + b : a;
            }
            __syncwarp();
            // a group stays if fewer than `keep` groups stand before it (larger score, or equal and lower index)
            for (int g = lane; g < c.groups; g += 32) {
                int before = 0;
                for (int o = 0; o < c.groups; ++o) before += gr[o] > gr[g] || (gr[o] == gr[g] && o < g);
                if (before >= c.keep)
                    for (int e = g * n; e < (g + 1) * n; ++e) pr[e] = TAKEN;
            }
        }
    } else {
        float mx = -INFINITY;
        for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
        mx = warp_max(mx);
        float s = 0.f;
        for (int e = lane; e < E; e += 32) {
            const float v = expf(z[e] - mx);
            pr[e] = v;
            s += v;
        }
        inv = 1.f / warp_sum(s);
    }
    float chosen = 0.f;
    __syncwarp();
    for (int k = 0; k < c.top; ++k) {
        float best = TAKEN;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = pr[e];
            if (v > best) {        // increasing e per lane: the first maximum wins
                best = v;
                bi = e;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) {
                best = ob;
                bi = oi;
            }
        }
        if (bi >= E) bi = k;       // no comparable score is left (NaN logits): any expert, its gate is NaN as well
        if (lane == 0) {
            const float s = c.sigmoid ? 1.f / (1.f + expf(-z[bi])) : pr[bi];
            expert_of[k] = bi;
            gate[k] = s * inv;
            chosen += s;
            atomicAdd(&counts[bi], 1);
            pr[bi] = TAKEN;
        }
        __syncwarp();
    }
    if (lane == 0 && c.sigmoid) {
        const float r = c.plain ? c.scale : c.scale / (chosen + 1e-20f);
        for (int k = 0; k < c.top; ++k) gate[k] *= r;
    } else if (lane == 0 && c.renorm) {   // gates over the chosen alone: e^(z - max) / sum of the chosen e^(z - max)
        const float r = 1.f / (chosen * inv);
        for (int k = 0; k < c.top; ++k) gate[k] *= r;
    }
}

// one warp per token; probs of the token live in shared memory (E floats per warp).  With x != nullptr the warp first
// computes the token's router logits itself, z[e] = sum_d x[m][d] * wr[e][d] in fp32 (lane-strided partial sums in
// increasing d, then the fixed warp tree: the same for a token whatever else is in the batch), eight experts per pass
// over the row.
__global__ void moe_route_kernel(const float* logits, const void* x, int xf32, const void* wr, int wf32, int D, float* z_out,
                                 int M, int E, int zld, RouteChoice c, int* expert_of, float* gate, int* counts,
                                 const float* bias) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int m = blockIdx.x * (blockDim.x >> 5) + warp;
    if (m >= M) return;
    float* pr = sm + (size_t)warp * E;
    float* zs = sm + (size_t)(blockDim.x >> 5) * E + (size_t)warp * E;
    if (x) {
        for (int e0 = 0; e0 < E; e0 += 8) {
            float acc[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[j] = 0.f;
            for (int d = lane; d < D; d += 32) {
                const float xv = ldx(x, (long long)m * D + d, xf32);
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (e0 + j < E) acc[j] = fmaf(xv, ldx(wr, (long long)(e0 + j) * D + d, wf32), acc[j]);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float v = warp_sum(acc[j]);
                if (lane == 0 && e0 + j < E) {
                    const float zb = bias ? v + bias[e0 + j] : v;
                    zs[e0 + j] = zb;
                    if (z_out) z_out[(long long)m * E + e0 + j] = zb;
                }
            }
        }
        __syncwarp();
    }
    const float* z = x ? zs : logits + (long long)m * zld;
    choose_experts(z, E, c, pr, zs, expert_of + (long long)m * c.top, gate + (long long)m * c.top, counts, lane);
}

// Few tokens (M * top <= 4096): choice, group sizes, offsets and scatter in ONE CTA with shared-memory counters, so that a
// decode step spends two launches on routing (logits, then this) instead of five.
__global__ void __launch_bounds__(256) moe_route_small_kernel(const float* logits, int M, int E, int zld, RouteChoice c,
                                                              int* expert_of, float* gate, int* group_off, int* sorted_tok,
                                                              int* slot_of) {
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, top = c.top;
    const int per = E + (c.groups > 1 ? c.groups : 0);
    int* cnt = reinterpret_cast<int*>(sm + (size_t)nw * per);   // [E] group sizes, then fill counters
    int* off = cnt + E;                                          // [E + 1]
    for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    float* pr = sm + (size_t)warp * per;
    for (int m = warp; m < M; m += nw) {
        choose_experts(logits + (long long)m * zld, E, c, pr, pr + E, expert_of + (long long)m * top,
                       gate + (long long)m * top, cnt, lane);
        __syncwarp();
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int o = 0;
        for (int e = 0; e < E; ++e) {
            off[e] = o;
            group_off[e] = o;
            o += cnt[e];
            cnt[e] = 0;
        }
        off[E] = o;
        group_off[E] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < M * top; i += blockDim.x) {
        const int e = expert_of[i];
        const int slot = off[e] + atomicAdd(&cnt[e], 1);
        sorted_tok[slot] = i / top;
        slot_of[i] = slot;
        if (c.slot_gate) c.slot_gate[slot] = gate[i];
    }
}

// router logits, one CTA per token (or four): z[m][e] = sum_d x[m][d] * wr[e][d] in fp32.  Thread t sums blocks of four elements t, t + 128, ... in
// increasing order, then the fixed warp tree and the warps in index order: a token's logits do not depend on the batch.
// rows >= E: rows beyond the experts' are computed alike (no bias); z_out rows are `rows` floats.
// NJ rows of w and NTOK tokens share a pass (the sums and their order do not depend on either).
template <int NJ, int NTOK>
__global__ void __launch_bounds__(128) moe_logits_kernel(const void* x, int xf32, const void* wr, int wf32, int D, int M, int E,
                                                         int rows, float* z_out, const float* bias, int vec) {
    __shared__ float red[4][NTOK][NJ];
    const int m0 = blockIdx.x * NTOK, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int e0 = 0; e0 < rows; e0 += NJ) {
        float acc[NTOK][NJ];
#pragma unroll
        for (int t = 0; t < NTOK; ++t)
#pragma unroll
            for (int j = 0; j < NJ; ++j) acc[t][j] = 0.f;
        // four consecutive elements per load; a row that is no multiple of four ends element by element
        const int D4 = vec ? D >> 2 : 0;
#pragma unroll 2
        for (int i = threadIdx.x; i < D4; i += 128) {
            float xv[NTOK][4];
#pragma unroll
            for (int t = 0; t < NTOK; ++t) ldx4(x, (long long)(m0 + t < M ? m0 + t : m0) * D + 4 * i, xf32, xv[t]);
#pragma unroll
            for (int j = 0; j < NJ; ++j) {      // beyond the last row: its product again, not stored (no branch between loads)
                float w[4];
                ldx4(wr, (long long)min(e0 + j, rows - 1) * D + 4 * i, wf32, w);
#pragma unroll
                for (int t = 0; t < NTOK; ++t)
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[t][j] = fmaf(xv[t][e], w[e], acc[t][j]);
            }
        }
        for (int d = 4 * D4 + threadIdx.x; d < D; d += 128) {
#pragma unroll
            for (int t = 0; t < NTOK; ++t) {
                const float xv = ldx(x, (long long)(m0 + t < M ? m0 + t : m0) * D + d, xf32);
#pragma unroll
                for (int j = 0; j < NJ; ++j)
                    if (e0 + j < rows) acc[t][j] = fmaf(xv, ldx(wr, (long long)(e0 + j) * D + d, wf32), acc[t][j]);
            }
        }
        __syncthreads();
#pragma unroll
        for (int t = 0; t < NTOK; ++t)
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float v = warp_sum(acc[t][j]);
                if (lane == 0) red[warp][t][j] = v;
            }
        __syncthreads();
        const int t = threadIdx.x / NJ, j = threadIdx.x % NJ;
        if (t < NTOK && m0 + t < M && e0 + j < rows)
            z_out[(long long)(m0 + t) * rows + e0 + j] =
                (((red[0][t][j] + red[1][t][j]) + red[2][t][j]) + red[3][t][j]) + (bias && e0 + j < E ? bias[e0 + j] : 0.f);
    }
}

__global__ void moe_offsets_kernel(int* counters, int* group_off, int E) {
    if (threadIdx.x == 0) {
        int o = 0;
        for (int e = 0; e < E; ++e) {
            group_off[e] = o;
            o += counters[e];
            counters[E + e] = 0;   // fill counters of the scatter pass
        }
        group_off[E] = o;
    }
}

__global__ void moe_scatter_kernel(const int* expert_of, int n, int top, int E, const int* group_off, int* counters,
                                   int* sorted_tok, int* slot_of, const float* gate, float* slot_gate) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int e = expert_of[i];
    const int slot = group_off[e] + atomicAdd(&counters[E + e], 1);
    sorted_tok[slot] = i / top;
    slot_of[i] = slot;
    if (slot_gate) slot_gate[slot] = gate[i];
}

template <int NJ, int NTOK>
void launch_logits_as(const MoeRouterInput& in, int M, int E, int rows, cudaStream_t stream) {
    const uintptr_t at = reinterpret_cast<uintptr_t>(in.x) | reinterpret_cast<uintptr_t>(in.w);
    const int vec = in.D % 4 == 0 && (at & 15) == 0;
    moe_logits_kernel<NJ, NTOK><<<(M + NTOK - 1) / NTOK, 128, 0, stream>>>(in.x, in.x_f32, in.w, in.w_f32, in.D, M, E, rows,
                                                                         in.logits_out, in.bias, vec);
}
// the passes over a token's row are few and even
void launch_logits(const MoeRouterInput& in, int M, int E, int rows, cudaStream_t stream) {
    if (M >= 1024) {      // enough CTAs without one per token: each row of w is read for four tokens
        const int per = (rows + (rows + 11) / 12 - 1) / ((rows + 11) / 12);
        if (per <= 8) return launch_logits_as<8, 4>(in, M, E, rows, stream);
        if (per <= 10) return launch_logits_as<10, 4>(in, M, E, rows, stream);
        return launch_logits_as<12, 4>(in, M, E, rows, stream);
    }
    const int per = (rows + (rows + 15) / 16 - 1) / ((rows + 15) / 16);
    if (per <= 8) return launch_logits_as<8, 1>(in, M, E, rows, stream);
    if (per <= 10) return launch_logits_as<10, 1>(in, M, E, rows, stream);
    if (per <= 12) return launch_logits_as<12, 1>(in, M, E, rows, stream);
    return launch_logits_as<16, 1>(in, M, E, rows, stream);
}

}  // namespace

int launch_moe_route(const float* logits, const MoeRouterInput* in, int M, int E, int top, int* expert_of, float* gate,
                     int* counters, int* group_off, int* sorted_tok, int* slot_of, cudaStream_t stream) {
    if (M <= 0) return 0;
    if (E <= 0 || top <= 0 || top > E) return set_error("moe: need 0 < top <= experts (top %d, experts %d)", top, E);
    if ((size_t)E * 8 * sizeof(float) > 48 * 1024) return set_error("moe: more than 1536 experts");
    if (!logits && !in) return set_error("moe: neither logits nor router inputs");
    RouteChoice c{top, 0, 0, 1, 1, nullptr, 1.f, 0, nullptr};
    if (in)
        c = RouteChoice{top, in->renorm, in->sigmoid, in->groups, in->keep, in->correction, in->scale, in->plain_scores, in->slot_gate};
    if (c.sigmoid) {
        if (!in->logits_out) return set_error("moe: sigmoid scores need logits_out");
        if (c.groups < 1 || E % c.groups || c.keep < 1 || c.keep > c.groups || top > c.keep * (E / c.groups))
            return set_error("moe: %d experts in %d groups, %d kept, %d chosen", E, c.groups, c.keep, top);
    }
    const int zld = E + (in ? in->extra : 0);
    const size_t small_smem = (size_t)(8 * (E + (c.groups > 1 ? c.groups : 0)) + 2 * E + 1) * sizeof(float);
    if (in && in->logits_out && (long long)M * top <= 4096 && small_smem <= 48 * 1024) {
        launch_logits(*in, M, E, zld, stream);
        moe_route_small_kernel<<<1, 256, small_smem, stream>>>(in->logits_out, M, E, zld, c, expert_of, gate, group_off,
                                                               sorted_tok, slot_of);
        count_launch(2);
        ASD_CUDA(cudaGetLastError());
        return 0;
    }
    ASD_CUDA(cudaMemsetAsync(counters, 0, sizeof(int) * E, stream));
    if (in && in->logits_out) {          // a CTA per token for the logits: few tokens still spread over the GPU
        launch_logits(*in, M, E, zld, stream);
        count_launch(1);
        logits = in->logits_out;
        in = nullptr;
    }
    moe_route_kernel<<<(M + 3) / 4, 128, (size_t)E * 8 * sizeof(float), stream>>>(
        logits, in ? in->x : nullptr, in ? in->x_f32 : 0, in ? in->w : nullptr, in ? in->w_f32 : 0, in ? in->D : 0,
        nullptr, M, E, zld, c, expert_of, gate, counters, in ? in->bias : nullptr);
    moe_offsets_kernel<<<1, 32, 0, stream>>>(counters, group_off, E);
    const int n = M * top;
    moe_scatter_kernel<<<(n + 255) / 256, 256, 0, stream>>>(expert_of, n, top, E, group_off, counters, sorted_tok, slot_of,
                                                            gate, c.slot_gate);
    count_launch(3);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace asd
