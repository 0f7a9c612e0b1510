// Row kernels of sandwich-normed layers: scaled embedding, the close of a sublayer fused with the norm that follows
// (residual sum, norm after the sublayer, norm before the next one, optionally the concatenation a pass entry reads),
// plain / offset RMS norm of a slice of a row, the normalised cubic polynomial of a feed-forward row, the tanh cap of
// the logits; the normed embedding and the elementwise activations of plain and gated feed-forwards.  A norm may split
// its row into equal consecutive groups, each divided by its own root mean square.  One CTA per row; sums of squares,
// the residual stream and every norm are fp32 whatever the engine's type.
#include <cuda_bf16.h>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"

namespace asd {

namespace {

inline int row_threads(int D) { return D >= 2048 ? 512 : (D >= 1024 ? 256 : (D >= 256 ? 128 : 64)); }

__global__ void embed_scaled_kernel(SeqIndex ix, const void* embed, int wf32, float scale, float* x0, float* x, int D) {
    const int m = blockIdx.x;
    const long long src = (long long)ix.tokens[m] * D, dst = (long long)m * D;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        const float v = ldx(embed, src + d, wf32) * scale;
        x0[dst + d] = v;
        if (x) x[dst + d] = v;
    }
}

// x[m] = embed[token] * scale + (sin at even, cos at odd coordinates of position * freq[coordinate / 2]).  The angle is
// brought into one turn in fp64, so that a far position's angle is as exact as a near one's.
__global__ void embed_sinusoid_kernel(SeqIndex ix, const void* embed, int wf32, float scale, const double* freq, float* x,
                                      int D) {
    const int m = blockIdx.x;
    const long long src = (long long)ix.tokens[m] * D, dst = (long long)m * D;
    const double pos = (double)ix.positions[m];
    constexpr double TURN = 6.283185307179586476925;
    for (int i = threadIdx.x; 2 * i < D; i += blockDim.x) {
        const double a = pos * freq[i];
        float sn, cs;
        sincosf((float)(a - TURN * rint(a / TURN)), &sn, &cs);
        x[dst + 2 * i] = fmaf(ldx(embed, src + 2 * i, wf32), scale, sn);
        if (2 * i + 1 < D) x[dst + 2 * i + 1] = fmaf(ldx(embed, src + 2 * i + 1, wf32), scale, cs);
    }
}

constexpr int MAX_NORM_GROUPS = 64;   // parts a grouped norm may split a row into

template <int V>
__device__ __forceinline__ void loadv(const float* p, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
    } else {
        v[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void storev(float* p, const float (&v)[V]) {
    if constexpr (V == 4)
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else
        *p = v[0];
}
template <int V>
__device__ __forceinline__ void storevx(void* p, long long i, int f32, const float (&v)[V]) {
    if (V == 4 && !f32) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[V > 1 ? 1 : 0]), hi = __floats2bfloat162_rn(v[V > 2 ? 2 : 0], v[V - 1]);
        *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) =
            make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else if (f32) {
        storev<V>((float*)p + i, v);
    } else {
        stx(p, i, 0, v[0]);
    }
}

// dynamic shared memory: D floats (the row being built) + 33 for the block sums + MAX_NORM_GROUPS group factors.  V
// consecutive elements per thread and step: 4 where width, norm groups and addresses allow, else 1.
template <int V>
__global__ void row_close_kernel(RowClose c) {
    extern __shared__ __align__(16) float sm[];
    float* row = sm;
    float* red = sm + c.D;
    float* gs = red + 33;
    const int m = blockIdx.x, D = c.D, G = c.groups, Dg = D / G, step = blockDim.x * V, first = threadIdx.x * V;
    const long long base = (long long)m * D;
    const long long in_base = c.rows ? (long long)c.rows[m] * D : base;
    const float off = c.plain_w ? 0.f : 1.f;
    auto inv_rms = [&](const float* src) {
        float ss = 0.f;
        for (int d = first; d < D; d += step) {
            float v[V];
            loadv<V>(src + base + d, v);
#pragma unroll
            for (int e = 0; e < V; ++e) ss += v[e] * v[e];
        }
        return 1.f / sqrtf(block_sum(ss, red) / (float)D + c.eps);
    };
    const float post = c.y && c.post_w ? inv_rms(c.y) * c.y_scale : 1.f;
    const float post2 = c.y2 ? inv_rms(c.y2) * c.y_scale : 1.f;
    const float ff_gate = c.ff_gate ? 1.f / (1.f + expf(-c.ff_gate[(long long)m * c.ff_gate_ld])) : 1.f;
#pragma unroll(V == 4 ? 1 : 4)
    for (int d = first; d < D; d += step) {
        float v[V], xv[V], t[V], w[V];
#pragma unroll
        for (int e = 0; e < V; ++e) xv[e] = 0.f;
        if (c.x_in) loadv<V>(c.x_in + in_base + d, xv);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = c.mult == 1.f ? xv[e] : 0.f;
        if (c.y) {
            loadv<V>(c.y + base + d, t);
            if (c.post_w) {
                loadv<V>(c.post_w + d, w);
#pragma unroll
                for (int e = 0; e < V; ++e) t[e] = t[e] * post * (off + w[e]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] += t[e];
        }
        if (c.y2) {
            loadv<V>(c.y2 + base + d, t);
            loadv<V>(c.post_w2 + d, w);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] += t[e] * post2 * (off + w[e]);
        }
        if (c.ff) {
            loadv<V>(c.ff + base + d, t);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = fmaf(ff_gate, t[e], v[e]);
        }
        for (int k = 0; k < c.top; ++k) {   // routed experts' results in choice order
            const float g = c.gate[(long long)m * c.top + k];
            loadv<V>(c.expert_out + (long long)c.slot_of[(long long)m * c.top + k] * D + d, t);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = fmaf(g, t[e], v[e]);
        }
        if (c.bias) {
            loadv<V>(c.bias + d, t);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] += t[e];
        }
        if (c.mult != 1.f)
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = fmaf(c.mult, v[e], xv[e]);
        storev<V>(row + d, v);
        if (c.x_out) storev<V>(c.x_out + base + d, v);
    }
    if (c.next_w) {
        __syncthreads();
        float mean = 0.f;
        if (c.next_b) {
            float t = 0.f;
            for (int d = threadIdx.x; d < D; d += blockDim.x) t += row[d];
            mean = block_sum(t, red) / (float)D;
        }
        for (int g = 0; g < G; ++g) {
            float ss = 0.f;
            for (int d = g * Dg + threadIdx.x; d < (g + 1) * Dg; d += blockDim.x) ss += (row[d] - mean) * (row[d] - mean);
            const float t = block_sum(ss, red);
            if (threadIdx.x == 0) gs[g] = 1.f / sqrtf(t / (float)Dg + c.eps);
        }
        __syncthreads();
        for (int d = first; d < D; d += step) {
            float v[V], w[V];
            loadv<V>(row + d, v);
            loadv<V>(c.next_w + d, w);
            const float f = gs[d / Dg];      // V consecutive elements lie in one group
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = (v[e] - mean) * f * (off + w[e]);
            if (c.next_b) {
                loadv<V>(c.next_b + d, w);
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] += w[e];
            }
            storevx<V>(c.hn, base + d, c.hn_f32, v);
            if (c.hn_copy) storev<V>(c.hn_copy + base + d, v);
        }
    } else if (c.cat) {
        __syncthreads();
        for (int d = threadIdx.x; d < D; d += blockDim.x) {
            stx(c.hn, 2 * base + d, c.hn_f32, row[d]);
            stx(c.hn, 2 * base + D + d, c.hn_f32, c.cat[base + d]);
        }
    }
}

// Sublayer close of layers whose norms are tanh(alpha x) w + b: nothing is reduced over a row, so the elements are spread
// over the grid, V consecutive ones per thread.
template <int V>
__global__ void tanh_close_kernel(TanhClose c) {
    const int m = blockIdx.x, d = (blockIdx.y * blockDim.x + threadIdx.x) * V, D = c.D;
    if (d >= D) return;
    const long long base = (long long)m * D + d;
    float x[V], w[V], b[V];
    loadv<V>(c.x_in + (c.rows ? (long long)c.rows[m] * D + d : base), x);
    if (c.y || c.top > 0) {
        float s[V];
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] = 0.f;
        if (c.y) loadv<V>(c.y + base, s);
        for (int k = 0; k < c.top; ++k) {       // routed experts' results in choice order
            float t[V];
            loadv<V>(c.expert_out + (long long)c.slot_of[(long long)m * c.top + k] * D + d, t);
#pragma unroll
            for (int e = 0; e < V; ++e) s[e] += t[e];
        }
        const float alpha = *c.post.alpha;
        loadv<V>(c.post.w + d, w);
        loadv<V>(c.post.b + d, b);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = fmaf(c.mult, fmaf(tanhf(alpha * s[e]), w[e], b[e]), x[e]);
        if (c.x_out) storev<V>(c.x_out + base, x);
    }
    if (c.next.w) {
        const float alpha = *c.next.alpha;
        loadv<V>(c.next.w + d, w);
        loadv<V>(c.next.b + d, b);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = fmaf(tanhf(alpha * x[e]), w[e], b[e]);
        storevx<V>(c.hn, base, c.hn_f32, x);
    }
}

// x[m] = group_norm(embed[token]) * w, fp32 (dynamic shared memory as row_close_kernel)
__global__ void embed_normed_kernel(SeqIndex ix, const void* embed, int wf32, const float* w, int groups, float eps, float* x,
                                    int D) {
    extern __shared__ float sm[];
    float* row = sm;
    float* red = sm + D;
    float* gs = red + 33;
    const int m = blockIdx.x, Dg = D / groups;
    const long long src = (long long)ix.tokens[m] * D, dst = (long long)m * D;
    for (int d = threadIdx.x; d < D; d += blockDim.x) row[d] = ldx(embed, src + d, wf32);
    __syncthreads();
    for (int g = 0; g < groups; ++g) {
        float ss = 0.f;
        for (int d = g * Dg + threadIdx.x; d < (g + 1) * Dg; d += blockDim.x) ss += row[d] * row[d];
        const float t = block_sum(ss, red);
        if (threadIdx.x == 0) gs[g] = 1.f / sqrtf(t / (float)Dg + eps);
    }
    __syncthreads();
    for (int d = threadIdx.x; d < D; d += blockDim.x) x[dst + d] = row[d] * gs[d / Dg] * w[d];
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// out[r][f] = gelu_tanh(z[r][f]) (mode 0, z rows of F floats) or silu(z[r][f]) * z[r][F + f] (mode 1, rows of 2 F)
// mode 2: relu(z[r][f])^2.  bias (optional) is added to z first: [F], or [2 F] in mode 1.
__global__ void ff_act_kernel(const float* z, void* out, int of32, long long n, int F, int mode, const float* bias) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    if (mode != 1) {
        float v = z[i];
        if (bias) v += bias[(int)(i % F)];
        if (mode == 0) {
            stx(out, i, of32, gelu_tanh_f(v));
        } else {
            v = fmaxf(v, 0.f);
            stx(out, i, of32, v * v);
        }
    } else {
        const long long r = i / F;
        const int f = (int)(i - r * F);
        float g = z[r * 2 * F + f], u = z[r * 2 * F + F + f];
        if (bias) g += bias[f], u += bias[F + f];
        stx(out, i, of32, g / (1.f + expf(-g)) * u);
    }
}

// gated activations: z rows of 2 F floats (gate half, then up half), V consecutive results per thread
template <int V>
__global__ void gated_act_kernel(const float* z, void* out, int of32, long long rows, int F, GatedAct p) {
    const int per = F / V;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * per) return;
    const long long r = rows * per <= 0x7fffffffLL ? (long long)((unsigned)i / (unsigned)per) : i / per;
    const int f = (int)(i - r * per) * V;
    float g[V], u[V];
    loadv<V>(z + r * 2 * F + f, g);
    loadv<V>(z + r * 2 * F + F + f, u);
    const float k = p.row_factor ? p.row_factor[r] : 1.f;
#pragma unroll
    for (int e = 0; e < V; ++e) {
        const float ge = g[e] * k, ue = u[e] * k;
        if (p.kind == GATED_GELU_TANH) {
            g[e] = gelu_tanh_f(ge) * ue;
        } else {
            const float c = fminf(ge, p.limit);
            g[e] = c / (1.f + expf(-p.slope * c)) * (fminf(fmaxf(ue, -p.limit), p.limit) + 1.f);
        }
    }
    storevx<V>(out, r * F + f, of32, g);
}

__global__ void rms_rows_kernel(const float* in, long long ld_in, const float* w, int plus_one, float eps, void* out,
                                int of32, long long ld_out, int n) {
    __shared__ float red[33];
    const float* src = in + (long long)blockIdx.x * ld_in;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) ss += src[i] * src[i];
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        stx(out, (long long)blockIdx.x * ld_out + i, of32, src[i] * r * (plus_one ? 1.f + w[i] : w[i]));
}

// dynamic shared memory: the row (F floats, if it fits: `staged`) + 33 for the block sums
__global__ void polynorm_kernel(const float* z, const float* coeff, float eps, void* out, int of32, int F, int staged) {
    extern __shared__ float sm[];
    float* red = sm;
    float* row = sm + 33;
    const float* src = z + (long long)blockIdx.x * F;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int i = threadIdx.x; i < F; i += blockDim.x) {
        const float v = src[i], v2 = v * v, v3 = v2 * v;
        if (staged) row[i] = v;
        s2 += v2;
        s4 += v2 * v2;
        s6 += v3 * v3;
    }
    s2 = block_sum(s2, red);
    s4 = block_sum(s4, red);
    s6 = block_sum(s6, red);
    const float inv = 1.f / (float)F;
    const float a = coeff[0] / sqrtf(s2 * inv + eps), b = coeff[1] / sqrtf(s4 * inv + eps),
                c = coeff[2] / sqrtf(s6 * inv + eps), e = coeff[3];
    for (int i = threadIdx.x; i < F; i += blockDim.x) {
        const float v = staged ? row[i] : src[i], v2 = v * v;
        stx(out, (long long)blockIdx.x * F + i, of32, a * v + b * v2 + c * (v2 * v) + e);
    }
}

__global__ void softcap_kernel(float* logits, long long ld, int V, float cap) {
    float* row = logits + (long long)blockIdx.x * ld;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i < V) row[i] = cap * tanhf(row[i] / cap);
}

}  // namespace

int launch_embed_scaled(const SeqIndex& ix, const void* embed, int wf32, float scale, float* x0, float* x, int D,
                        cudaStream_t stream) {
    if (ix.M <= 0) return 0;
    embed_scaled_kernel<<<ix.M, row_threads(D), 0, stream>>>(ix, embed, wf32, scale, x0, x, D);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_embed_sinusoid(const SeqIndex& ix, const void* embed, int wf32, float scale, const double* freq, float* x, int D,
                          cudaStream_t stream) {
    if (ix.M <= 0) return 0;
    embed_sinusoid_kernel<<<ix.M, row_threads(D), 0, stream>>>(ix, embed, wf32, scale, freq, x, D);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_row_close(const RowClose& c, cudaStream_t stream) {
    if (c.M <= 0) return 0;
    if (c.D <= 0 || ((c.next_w || c.cat) && !c.hn)) return set_error("row_close: bad arguments");
    if (c.groups <= 0 || c.groups > MAX_NORM_GROUPS || c.D % c.groups)
        return set_error("row_close: %d norm groups do not divide width %d (at most %d)", c.groups, c.D, MAX_NORM_GROUPS);
    if (c.next_b && c.groups != 1) return set_error("row_close: a layer norm has no groups");
    if (c.y2 && !c.post_w2) return set_error("row_close: the second branch has no norm weight");
    if (c.top > 0 && (!c.expert_out || !c.slot_of || !c.gate)) return set_error("row_close: expert results missing");
    const size_t smem = (size_t)(c.D + 33 + MAX_NORM_GROUPS) * sizeof(float);
    if (smem > 200 * 1024) return set_error("row_close: width %d does not fit shared memory", c.D);
    static PerDeviceOnce once;
    if (once.need()) {
        ASD_CUDA(cudaFuncSetAttribute(row_close_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        ASD_CUDA(cudaFuncSetAttribute(row_close_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    }
    uintptr_t at = 0;
    for (const void* p : {(const void*)c.x_in, (const void*)c.y, (const void*)c.post_w, (const void*)c.bias, (const void*)c.x_out,
                          (const void*)c.next_w, (const void*)c.hn, (const void*)c.expert_out, (const void*)c.y2,
                          (const void*)c.post_w2, (const void*)c.ff, (const void*)c.next_b, (const void*)c.hn_copy})
        at |= reinterpret_cast<uintptr_t>(p);
    if (c.D % 4 == 0 && (c.D / c.groups) % 4 == 0 && (at & 15) == 0)
        row_close_kernel<4><<<c.M, row_threads(c.D), smem, stream>>>(c);
    else
        row_close_kernel<1><<<c.M, row_threads(c.D), smem, stream>>>(c);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_embed_normed(const SeqIndex& ix, const void* embed, int wf32, const float* w, int groups, float eps, float* x,
                        int D, cudaStream_t stream) {
    if (ix.M <= 0) return 0;
    if (groups <= 0 || groups > MAX_NORM_GROUPS || D % groups)
        return set_error("embed_normed: %d norm groups do not divide width %d (at most %d)", groups, D, MAX_NORM_GROUPS);
    const size_t smem = (size_t)(D + 33 + MAX_NORM_GROUPS) * sizeof(float);
    if (smem > 200 * 1024) return set_error("embed_normed: width %d does not fit shared memory", D);
    static PerDeviceOnce once;
    if (once.need()) ASD_CUDA(cudaFuncSetAttribute(embed_normed_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    embed_normed_kernel<<<ix.M, row_threads(D), smem, stream>>>(ix, embed, wf32, w, groups, eps, x, D);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_ff_act(const float* z, void* out, int of32, long long rows, int F, int gated, cudaStream_t stream,
                  const float* bias) {
    const long long n = rows * F;
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL) return set_error("ff_act: too many elements");
    ff_act_kernel<<<(unsigned)blocks, 256, 0, stream>>>(z, out, of32, n, F, gated, bias);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_gated_act(const float* z, void* out, int of32, long long rows, int F, const GatedAct& p, cudaStream_t stream) {
    if (rows <= 0 || F <= 0) return 0;
    if (p.kind == GATED_CLAMPED && !(p.limit > 0.f)) return set_error("gated_act: the limit must be positive");
    const bool four = F % 4 == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const long long blocks = (rows * (four ? F / 4 : F) + 255) / 256;
    if (blocks > 0x7fffffffLL) return set_error("gated_act: too many elements");
    if (four)
        gated_act_kernel<4><<<(unsigned)blocks, 256, 0, stream>>>(z, out, of32, rows, F, p);
    else
        gated_act_kernel<1><<<(unsigned)blocks, 256, 0, stream>>>(z, out, of32, rows, F, p);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_tanh_close(const TanhClose& c, cudaStream_t stream) {
    if (c.M <= 0) return 0;
    if (c.D <= 0 || !c.x_in || (c.next.w && !c.hn)) return set_error("tanh_close: bad arguments");
    if (c.top > 0 && (!c.expert_out || !c.slot_of)) return set_error("tanh_close: expert results missing");
    if ((c.y || c.top > 0) && (!c.post.w || !c.post.b || !c.post.alpha)) return set_error("tanh_close: the norm of the result is missing");
    if (c.next.w && (!c.next.b || !c.next.alpha)) return set_error("tanh_close: incomplete norm");
    uintptr_t at = 0;
    for (const void* p : {(const void*)c.x_in, (const void*)c.y, (const void*)c.expert_out, (const void*)c.post.w,
                          (const void*)c.post.b, (const void*)c.x_out, (const void*)c.next.w, (const void*)c.next.b,
                          (const void*)c.hn})
        at |= reinterpret_cast<uintptr_t>(p);
    const bool four = c.D % 4 == 0 && (at & 15) == 0;
    const int n = four ? c.D / 4 : c.D, threads = n >= 256 ? 256 : (n >= 128 ? 128 : 64);
    const dim3 grid(c.M, (n + threads - 1) / threads);
    if (four)
        tanh_close_kernel<4><<<grid, threads, 0, stream>>>(c);
    else
        tanh_close_kernel<1><<<grid, threads, 0, stream>>>(c);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_rms_rows(const float* in, long long ld_in, const float* w, int plus_one, float eps, void* out, int of32,
                    long long ld_out, int M, int n, cudaStream_t stream) {
    if (M <= 0 || n <= 0) return 0;
    rms_rows_kernel<<<M, row_threads(n), 0, stream>>>(in, ld_in, w, plus_one, eps, out, of32, ld_out, n);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_polynorm(const float* z, const float* coeff, float eps, void* out, int of32, int M, int F, cudaStream_t stream) {
    if (M <= 0 || F <= 0) return 0;
    const int staged = (size_t)F * sizeof(float) <= 96 * 1024;
    const size_t smem = (33 + (staged ? (size_t)F : 0)) * sizeof(float);
    static PerDeviceOnce once;
    if (once.need()) ASD_CUDA(cudaFuncSetAttribute(polynorm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    polynorm_kernel<<<M, row_threads(F), smem, stream>>>(z, coeff, eps, out, of32, F, staged);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

int launch_softcap(float* logits, long long ld, int n, int V, float cap, cudaStream_t stream) {
    if (n <= 0 || V <= 0 || !(cap > 0.f)) return 0;
    dim3 grid(n, (V + 255) / 256);
    softcap_kernel<<<grid, 256, 0, stream>>>(logits, ld, V, cap);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace asd
