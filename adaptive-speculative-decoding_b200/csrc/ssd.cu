// State space recurrence with one decay per head and position (Mamba-2).  Per head a state S [dk][dv] in fp32,
//   dt = softplus(raw + dt_bias);  S = exp(-exp(a_log) dt) S + dt B x^T;  y = S^T C + skip x,
// with B and C shared by the heads of a group.  Three kernels behind one launcher:
//   ssd_recurrence_kernel  position by position in fp32: a CTA owns 32 value columns of one (sequence, head), its warps slices
//                          of the key rows in registers; nothing of the state feeds back into what a position reads, so a
//                          chunk of staged positions runs without a barrier and its results are closed together;
//   ssd_step_kernel        one token per sequence: the state streams through once;
//   ssd_chunk_kernel       (ssd_chunk.cu) prompts of a bf16 engine, chunk by chunk on the tensor cores.
#include <cuda_bf16.h>
#include <math.h>

#include <algorithm>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"
#include "ssd.h"

namespace asd {

namespace {

__device__ __forceinline__ void stage4(float* dst, const float* src, bool valid) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(dst);
    const int sz = valid ? 4 : 0;       // 0: the destination is filled with zeros
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(addr), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void stage16(float* dst, const float* src) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(addr), "l"(src) : "memory");
}

constexpr int MAXC = 32;     // positions of a chunk: one lane each for the step sizes

// shared memory in floats: two buffers of { C [CH][dkp], B [CH][dkp], x [CH][32], dt [CH] }; then per chunk partial results
// [CH][RS][32] and per warp the decays and step sizes [RS][2][MAXC]
__host__ __device__ inline int buf_floats(int CH, int dkp) { return CH * (2 * dkp + 32 + 1); }
__host__ __device__ inline int total_floats(int CH, int dkp, int RS) {
    return 2 * ((buf_floats(CH, dkp) + 3) & ~3) + CH * RS * 32 + RS * 2 * MAXC;
}

template <int ROWS, int MAXT>
__global__ void __launch_bounds__(MAXT, 1) ssd_recurrence_kernel(SsdArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * 32;
    const int t1 = a.cu_q[seq + 1], t0 = a.tail > 0 ? max(a.cu_q[seq], t1 - a.tail) : a.cu_q[seq];
    if (t0 >= t1) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, RS = blockDim.x >> 5, nthr = blockDim.x;
    const int dk = a.d.dk, dv = a.d.dv, H = a.d.heads, CH = a.CH, ring = a.ring;
    const int grp = head / (H / a.d.groups);
    const int dkp = RS * ROWS, r0 = warp * ROWS;
    const int col = col0 + lane;
    const bool col_ok = col < dv;
    const int slot = a.seq_slot[seq];
    const int p0 = a.ix.positions[t0];
    const int buf = (buf_floats(CH, dkp) + 3) & ~3;
    float* red = sm + 2 * buf;
    float* fac = red + CH * RS * 32 + warp * 2 * MAXC;
    for (int i = threadIdx.x; i < 2 * buf; i += nthr) sm[i] = 0.f;   // rows beyond dk stay zero for good
    const size_t entry = (size_t)H * dk * dv;
    float* st = a.state + (size_t)slot * ring * entry + (size_t)head * dk * dv;
    float2 S[ROWS / 2];                   // rows in pairs: two of them per instruction
#pragma unroll
    for (int r = 0; r < ROWS / 2; ++r) S[r] = make_float2(0.f, 0.f);
    if (p0 > 0 && col_ok) {
        const float* src = st + (size_t)((p0 - 1) % ring) * entry;
#pragma unroll
        for (int r = 0; r < ROWS; r += 2) {
            if (r0 + r < dk) S[r >> 1].x = src[(size_t)(r0 + r) * dv + col];
            if (r0 + r + 1 < dk) S[r >> 1].y = src[(size_t)(r0 + r + 1) * dv + col];
        }
    }
    const float bias = a.in.dt_bias[head], rate = expf(a.in.a_log[head]), skip = a.in.skip[head];
    __syncthreads();
    auto fetch = [&](int b, int c0) {
        const int nt = min(CH, t1 - c0);
        float* cs = sm + b * buf;
        float* bs = cs + CH * dkp;
        float* xs = bs + CH * dkp;
        float* ds = xs + CH * 32;
        if (a.in.bf16) {
            for (int i = threadIdx.x; i < nt * dk; i += nthr) {
                const int t = i / dk, c = i - t * dk;
                const long long at = (long long)(c0 + t) * a.in.ld + (long long)grp * dk + c;
                cs[t * dkp + c] = ssd_in(a, a.in.c, at);
                bs[t * dkp + c] = ssd_in(a, a.in.b, at);
            }
        } else if (a.v16) {
            const int n4 = dk >> 2;
            for (int i = threadIdx.x; i < nt * n4; i += nthr) {
                const int t = i / n4, c = (i - t * n4) * 4;
                const long long at = (long long)(c0 + t) * a.in.ld + (long long)grp * dk + c;
                stage16(cs + t * dkp + c, static_cast<const float*>(a.in.c) + at);
                stage16(bs + t * dkp + c, static_cast<const float*>(a.in.b) + at);
            }
        } else {
            for (int i = threadIdx.x; i < nt * dk; i += nthr) {
                const int t = i / dk, c = i - t * dk;
                const long long at = (long long)(c0 + t) * a.in.ld + (long long)grp * dk + c;
                stage4(cs + t * dkp + c, static_cast<const float*>(a.in.c) + at, true);
                stage4(bs + t * dkp + c, static_cast<const float*>(a.in.b) + at, true);
            }
        }
        for (int i = threadIdx.x; i < nt * 32; i += nthr) {
            const int t = i >> 5, c = i & 31;
            const bool ok = col0 + c < dv;
            const long long at = ok ? (long long)(c0 + t) * a.in.ld + (long long)head * dv + col0 + c : 0;
            if (a.in.bf16)
                xs[i] = ok ? ssd_in(a, a.in.x, at) : 0.f;
            else
                stage4(xs + i, static_cast<const float*>(a.in.x) + at, ok);
        }
        for (int t = threadIdx.x; t < nt; t += nthr) stage4(ds + t, a.in.dt + (long long)(c0 + t) * a.in.ld_dt + head, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, t0);
    int it = 0;
    for (int c0 = t0; c0 < t1; c0 += CH, ++it) {
        const int nt = min(CH, t1 - c0);
        if (c0 + CH < t1) {
            fetch((it + 1) & 1, c0 + CH);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();   // this chunk's rows have landed for every thread
        const float* cs = sm + (it & 1) * buf;
        const float* bs = cs + CH * dkp;
        const float* xs = bs + CH * dkp;
        const float* ds = xs + CH * 32;
        if (lane < nt) {
            const float dt = softplus_step(ds[lane] + bias);
            fac[lane] = 1.f + expm1f(-rate * dt);       // a decay just below 1 is rounded once
            fac[MAXC + lane] = dt;
        }
        __syncwarp();
        auto position = [&](int t) {
            const float keep = fac[t];
            const float4* b4 = reinterpret_cast<const float4*>(bs + t * dkp + r0);
            const float4* c4 = reinterpret_cast<const float4*>(cs + t * dkp + r0);
            const float xv = fac[MAXC + t] * xs[t * 32 + lane];
            const float2 keep2 = make_float2(keep, keep), xv2 = make_float2(xv, xv);
            float2 oa = make_float2(0.f, 0.f), ob = make_float2(0.f, 0.f);
#pragma unroll
            for (int r = 0; r < ROWS; r += 4) {
                const float4 kk = b4[r >> 2], qq = c4[r >> 2];
                float2 &s0 = S[r >> 1], &s1 = S[(r >> 1) + 1];
                s0 = fma2(make_float2(kk.x, kk.y), xv2, mul2(keep2, s0));
                s1 = fma2(make_float2(kk.z, kk.w), xv2, mul2(keep2, s1));
                oa = fma2(s0, make_float2(qq.x, qq.y), oa);
                ob = fma2(s1, make_float2(qq.z, qq.w), ob);
            }
            red[(t * RS + warp) * 32 + lane] = (oa.x + oa.y) + (ob.x + ob.y);
        };
        const int plain = min(nt, max(0, t1 - ring - c0));      // positions that leave no state behind
#pragma unroll 2
        for (int t = 0; t < plain; ++t) position(t);
        for (int t = plain; t < nt; ++t) {
            position(t);
            if (!col_ok) continue;
            float* dst = st + (size_t)((p0 + (c0 + t - t0)) % ring) * entry;
#pragma unroll
            for (int r = 0; r < ROWS; r += 2) {
                if (r0 + r < dk) dst[(size_t)(r0 + r) * dv + col] = S[r >> 1].x;
                if (r0 + r + 1 < dk) dst[(size_t)(r0 + r + 1) * dv + col] = S[r >> 1].y;
            }
        }
        __syncthreads();   // the chunk's partial products are complete
#pragma unroll 4
        for (int t = warp; t < nt; t += RS) {
            float o = 0.f;
            for (int w = 0; w < RS; ++w) o += red[(t * RS + w) * 32 + lane];
            if (col_ok) a.out[(long long)(c0 + t) * H * dv + (long long)head * dv + col] = fmaf(skip, xs[t * 32 + lane], o);
        }
        __syncthreads();   // this buffer's x is read: it may be refilled
    }
}

// Steps of one token per sequence: the state is read and written once, so a CTA streams a (sequence, head)'s rows, four
// columns a thread and eight rows in flight, up to 128 columns wide.
constexpr int ST = 256, SCOLS = 128, SU = 8;
__global__ void __launch_bounds__(ST) ssd_step_kernel(SsdArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * SCOLS, tid = threadIdx.x;
    const int m = a.cu_q[seq];
    if (m >= a.cu_q[seq + 1]) return;
    const int dk = a.d.dk, dv = a.d.dv, H = a.d.heads, ring = a.ring, grp = head / (H / a.d.groups);
    const int L = (min(SCOLS, dv - col0)) >> 2, R = ST / L;      // threads per row, rows per pass
    const int rg = tid / L, c4 = (tid - rg * L) * 4;
    const int pos = a.ix.positions[m];
    const size_t entry = (size_t)H * dk * dv;
    float* slot = a.state + (size_t)a.seq_slot[seq] * ring * entry + (size_t)head * dk * dv + col0 + c4;
    const float* src = slot + (size_t)((pos + ring - 1) % ring) * entry;      // pos - 1, not read at position 0
    float* dst = slot + (size_t)(pos % ring) * entry;
    const bool old = pos > 0, live = rg < R;
    float* cs = sm;
    float* bs = cs + dk;
    float* red = bs + dk;             // [R][4 L] partial results
    float4 S[SU];
    auto load = [&](int r0) {
#pragma unroll
        for (int u = 0; u < SU; ++u) {
            const int r = r0 + u * R;
            S[u] = (live && old && r < dk) ? *reinterpret_cast<const float4*>(src + (size_t)r * dv)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    load(rg);
    const long long row = (long long)m * a.in.ld;
    for (int i = tid; i < dk; i += ST) {
        cs[i] = ssd_in(a, a.in.c, row + (long long)grp * dk + i);
        bs[i] = ssd_in(a, a.in.b, row + (long long)grp * dk + i);
    }
    const float dt = softplus_step(a.in.dt[(long long)m * a.in.ld_dt + head] + a.in.dt_bias[head]);
    const float keep = 1.f + expm1f(-expf(a.in.a_log[head]) * dt);
    const long long x_at = row + (long long)head * dv + col0;
    float xv[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
    if (live)
#pragma unroll
        for (int e = 0; e < 4; ++e) xv[e] = dt * ssd_in(a, a.in.x, x_at + c4 + e);
    __syncthreads();
    for (int r0 = rg; r0 < dk && live; r0 += SU * R) {
        if (r0 != rg) load(r0);
#pragma unroll
        for (int u = 0; u < SU; ++u) {
            const int r = r0 + u * R;
            if (r >= dk) break;
            const float kk = bs[r], qq = cs[r];
            float4 s = S[u];
            s.x = fmaf(kk, xv[0], keep * s.x), s.y = fmaf(kk, xv[1], keep * s.y);
            s.z = fmaf(kk, xv[2], keep * s.z), s.w = fmaf(kk, xv[3], keep * s.w);
            *reinterpret_cast<float4*>(dst + (size_t)r * dv) = s;
            o[0] = fmaf(s.x, qq, o[0]), o[1] = fmaf(s.y, qq, o[1]);
            o[2] = fmaf(s.z, qq, o[2]), o[3] = fmaf(s.w, qq, o[3]);
        }
    }
    if (live)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[rg * 4 * L + c4 + e] = o[e];
    __syncthreads();
    const float skip = a.in.skip[head];
    for (int c = tid; c < 4 * L; c += ST) {
        float t = 0.f;
        for (int r = 0; r < R; ++r) t += red[r * 4 * L + c];
        a.out[(long long)m * H * dv + (long long)head * dv + col0 + c] = fmaf(skip, ssd_in(a, a.in.x, x_at + c), t);
    }
}

}  // namespace

int launch_ssd_recurrence(const SeqIndex& ix, const int* cu_q, const int* seq_slot, int nseq, int max_qlen, const SsdInput& in,
                          const SsdDims& d, float* state, int ring, float* out, int mode, cudaStream_t stream) {
    if (ix.M <= 0 || nseq <= 0) return 0;
    if (d.heads <= 0 || d.groups <= 0 || d.heads % d.groups || d.dv <= 0 || d.dk <= 0 || d.dk > 1024)
        return set_error("ssd: %d heads in %d groups, state %d x %d", d.heads, d.groups, d.dk, d.dv);
    if (ring <= 0 || !state) return set_error("ssd: no state");
    if (!in.x || !in.b || !in.c || !in.dt || !in.dt_bias || !in.a_log || !in.skip) return set_error("ssd: missing inputs");
    if (d.heads > 65535) return set_error("ssd: too many heads");
    SsdArgs a;
    a.ix = ix, a.cu_q = cu_q, a.seq_slot = seq_slot, a.in = in, a.d = d, a.state = state, a.ring = ring, a.CH = 1;
    a.v16 = 0, a.out = out;
    if (max_qlen == 1 && d.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0) {
        const size_t smem = (size_t)(2 * d.dk + 4 * ST) * sizeof(float);
        ssd_step_kernel<<<dim3(nseq, d.heads, (d.dv + SCOLS - 1) / SCOLS), ST, smem, stream>>>(a);
        count_launch(1);
        ASD_CUDA(cudaGetLastError());
        return 0;
    }
    if (mode == 0 && in.bf16 && max_qlen >= 16) {
        // chunks leave the state after their last position; the states of the ring's other entries come from a sequential
        // pass over the last positions
        a.tail = ring - 1;
        const int rc = launch_ssd_chunks(a, nseq, stream);
        if (rc < 0) return -1;
        if (rc == 0 && ring == 1) return 0;
        if (rc == 1) a.tail = 0;
    }
    int rows = 4;
    while (rows < 32 && rows * 4 < d.dk) rows *= 2;     // four warps up to key size 128, then more
    const int RS = (d.dk + rows - 1) / rows, dkp = RS * rows;
    int ch = MAXC;   // positions per staged chunk; steps of few tokens stage (and clear) no more than they use
    const long long positions = a.tail > 0 ? std::min<long long>(ix.M, (long long)nseq * a.tail) : ix.M;
    while (ch > 1 && (long long)(ch / 2) * nseq >= positions) ch >>= 1;
    auto need = [&](int c) { return (size_t)total_floats(c, dkp, RS) * sizeof(float); };
    while (ch > 1 && need(ch) > 112 * 1024) ch >>= 1;
    const size_t smem = need(ch);
    if (smem > 220 * 1024) return set_error("ssd: state size %d does not fit shared memory", d.dk);
    const dim3 grid(nseq, d.heads, (d.dv + 31) / 32);
    if (grid.z > 65535) return set_error("ssd: too many value columns");
    a.CH = ch;
    const uintptr_t at = reinterpret_cast<uintptr_t>(in.c) | reinterpret_cast<uintptr_t>(in.b);
    a.v16 = (d.dk % 4 == 0 && in.ld % 4 == 0 && (at & 15) == 0) ? 1 : 0;
#define ASD_SSD_CASE(R, T)                                                                                            \
    {                                                                                                                 \
        auto fn = ssd_recurrence_kernel<R, T>;                                                                        \
        static PerDeviceOnce once;                                                                                    \
        if (once.need()) ASD_CUDA(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)); \
        fn<<<grid, RS * 32, smem, stream>>>(a);                                                                       \
    }
    if (RS > 8) ASD_SSD_CASE(32, 1024)
    else if (rows == 4) ASD_SSD_CASE(4, 256)
    else if (rows == 8) ASD_SSD_CASE(8, 256)
    else if (rows == 16) ASD_SSD_CASE(16, 256)
    else ASD_SSD_CASE(32, 256)
#undef ASD_SSD_CASE
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace asd
