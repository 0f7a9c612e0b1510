// Matrix memory with exponential gates (mLSTM).  Per head a state S [dk][dv] and a normaliser n [dk], both kept relative to
// a running maximum M of the gates' logarithms so that every exponential stays at most 1:
//   M' = max(f + M, i);  S = exp(f + M - M') S + exp(i - M') k v^T;  n = exp(f + M - M') n + exp(i - M') k;
//   o = S^T q / (max(|n . q|, exp(-M')) + 1e-6).
// Nothing of the state feeds back into the gates, so a chunk of staged positions runs without a barrier: a CTA owns 32
// value columns of one (sequence, head), its warps slices of the key rows in registers; each warp leaves its partial
// products of a position in shared memory and the chunk's results are closed together.  The gate factors of a chunk come
// from a scan over its positions (M -> max(a + M, b) composes to the same form), done by every warp for itself.
#include <cuda_bf16.h>
#include <math.h>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"

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

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

constexpr int MAXC = 32;     // positions of a chunk: one lane each in the gate scan

struct MlstmArgs {
    SeqIndex ix;
    const int* cu_q;
    const int* seq_slot;
    MlstmInput in;
    MlstmDims d;
    float* state;
    int ring, CH, v16;
    float* out;
};

// every block of 32 value columns keeps its own copy of n and M, so that CTAs share no state
__host__ __device__ inline size_t entry_elems(const MlstmDims& d) {
    return ((size_t)d.heads * ((size_t)d.dk * d.dv + (size_t)((d.dv + 31) / 32) * (d.dk + 1)) + 3) & ~(size_t)3;
}

// shared memory in floats: two buffers of { q [CH][dkp], k [CH][dkp], v [CH][32], zi [CH], zf [CH] }; then per chunk
// partial results [CH][RS][32], partial normaliser products [CH][RS][32], gate factors per warp [RS][3][MAXC]
__host__ __device__ inline int buf_floats(int CH, int dkp) { return CH * (2 * dkp + 32 + 2); }
__host__ __device__ inline int total_floats(int CH, int dkp, int RS) {
    return 2 * ((buf_floats(CH, dkp) + 3) & ~3) + 2 * CH * RS * 32 + RS * 3 * MAXC;
}

template <int ROWS, int MAXT>
__global__ void __launch_bounds__(MAXT, 1) mlstm_recurrence_kernel(MlstmArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * 32;
    const int t0 = a.cu_q[seq], t1 = a.cu_q[seq + 1];
    if (t0 >= t1) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, RS = blockDim.x >> 5, nthr = blockDim.x;
    const int dk = a.d.dk, dv = a.d.dv, H = a.d.heads, CH = a.CH, ring = a.ring;
    const int dkp = RS * ROWS, r0 = warp * ROWS;
    const int col = col0 + lane;
    const bool col_ok = col < dv;
    const int slot = a.seq_slot[seq];
    const int p0 = a.ix.positions[t0];
    const int buf = (buf_floats(CH, dkp) + 3) & ~3;
    float* red = sm + 2 * buf;
    float* redn = red + CH * RS * 32;
    float* gates = redn + CH * RS * 32 + warp * 3 * MAXC;      // keep, put, floor of this warp
    for (int i = threadIdx.x; i < 2 * buf; i += nthr) sm[i] = 0.f;   // key rows beyond dk stay zero for good
    const size_t entry = entry_elems(a.d);
    float* st_slot = a.state + (size_t)slot * ring * entry;
    const size_t st_S = (size_t)head * dk * dv,
                 st_n = (size_t)H * dk * dv + ((size_t)head * gridDim.z + blockIdx.z) * (dk + 1), st_m = st_n + dk;
    float2 S[ROWS / 2];                   // rows in pairs: two of them per instruction
#pragma unroll
    for (int r = 0; r < ROWS / 2; ++r) S[r] = make_float2(0.f, 0.f);
    float n = 0.f, mrun = 0.f;            // lane r of a warp holds row r0 + r of the normaliser
    const bool n_ok = lane < ROWS && r0 + lane < dk;
    if (p0 > 0) {
        const float* src = st_slot + (size_t)((p0 - 1) % ring) * entry;
        if (col_ok) {
#pragma unroll
            for (int r = 0; r < ROWS; r += 2) {
                if (r0 + r < dk) S[r >> 1].x = src[st_S + (size_t)(r0 + r) * dv + col];
                if (r0 + r + 1 < dk) S[r >> 1].y = src[st_S + (size_t)(r0 + r + 1) * dv + col];
            }
        }
        if (n_ok) n = src[st_n + r0 + lane];
        mrun = src[st_m];
    }
    const float bi = a.in.bias_i ? a.in.bias_i[head] : 0.f, bf = a.in.bias_f ? a.in.bias_f[head] : 0.f;
    __syncthreads();
    auto fetch = [&](int b, int c0) {
        const int nt = min(CH, t1 - c0);
        float* qs = sm + b * buf;
        float* ks = qs + CH * dkp;
        float* vs = ks + CH * dkp;
        float* zs = vs + CH * 32;
        if (a.v16) {
            const int n4 = dk >> 2;
            for (int i = threadIdx.x; i < nt * n4; i += nthr) {
                const int t = i / n4, c = (i - t * n4) * 4;
                const long long at = (long long)(c0 + t) * a.in.ld + (long long)head * dk + c;
                stage16(qs + t * dkp + c, a.in.q + at);
                stage16(ks + t * dkp + c, a.in.k + at);
            }
        } else {
            for (int i = threadIdx.x; i < nt * dk; i += nthr) {
                const int t = i / dk, c = i - t * dk;
                const long long at = (long long)(c0 + t) * a.in.ld + (long long)head * dk + c;
                stage4(qs + t * dkp + c, a.in.q + at, true);
                stage4(ks + t * dkp + c, a.in.k + at, true);
            }
        }
        for (int i = threadIdx.x; i < nt * 32; i += nthr) {
            const int t = i >> 5, c = i & 31;
            const bool ok = col0 + c < dv;
            stage4(vs + i, a.in.v + (ok ? (long long)(c0 + t) * a.in.ld + (long long)head * dv + col0 + c : 0), ok);
        }
        for (int t = threadIdx.x; t < nt; t += nthr) {
            stage4(zs + t, a.in.zi + (long long)(c0 + t) * a.in.ld + head, true);
            stage4(zs + CH + t, a.in.zf + (long long)(c0 + t) * a.in.ld + head, true);
        }
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
        const float* qs = sm + (it & 1) * buf;
        const float* ks = qs + CH * dkp;
        const float* vs = ks + CH * dkp;
        const float* zs = vs + CH * 32;
        float mlane;       // the running maximum after position `lane` of the chunk
        {
            const float cap = a.d.cap;
            const bool ok = lane < nt;
            const float li = ok ? cap * tanhf((zs[lane] + bi) / cap) : -INFINITY;
            const float lf = ok ? log_sigmoid(cap * tanhf((zs[CH + lane] + bf) / cap)) : 0.f;
            float sa = lf, sb = li;          // M -> max(sa + M, sb) over positions up to this lane's
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pa = __shfl_up_sync(0xffffffffu, sa, o), pb = __shfl_up_sync(0xffffffffu, sb, o);
                if (lane >= o) {
                    sb = fmaxf(sa + pb, sb);
                    sa = sa + pa;
                }
            }
            mlane = fmaxf(sa + mrun, sb);
            float prev = __shfl_up_sync(0xffffffffu, mlane, 1);
            if (lane == 0) prev = mrun;
            if (ok) {
                gates[lane] = expf(lf + prev - mlane);
                gates[MAXC + lane] = expf(li - mlane);
                gates[2 * MAXC + lane] = expf(-mlane);
            }
            mrun = __shfl_sync(0xffffffffu, mlane, nt - 1);
            __syncwarp();
        }
        auto position = [&](int t) {
            const float keep = gates[t], put = gates[MAXC + t];
            const float4* k4 = reinterpret_cast<const float4*>(ks + t * dkp + r0);
            const float4* q4 = reinterpret_cast<const float4*>(qs + t * dkp + r0);
            const float pv = put * vs[t * 32 + lane];
            const float2 keep2 = make_float2(keep, keep), pv2 = make_float2(pv, pv);
            float2 oa = make_float2(0.f, 0.f), ob = make_float2(0.f, 0.f);
#pragma unroll
            for (int r = 0; r < ROWS; r += 4) {
                const float4 kk = k4[r >> 2], qq = q4[r >> 2];
                float2 &s0 = S[r >> 1], &s1 = S[(r >> 1) + 1];
                s0 = fma2(make_float2(kk.x, kk.y), pv2, mul2(keep2, s0));
                s1 = fma2(make_float2(kk.z, kk.w), pv2, mul2(keep2, s1));
                oa = fma2(s0, make_float2(qq.x, qq.y), oa);
                ob = fma2(s1, make_float2(qq.z, qq.w), ob);
            }
            red[(t * RS + warp) * 32 + lane] = (oa.x + oa.y) + (ob.x + ob.y);
            float nq = 0.f;
            if (lane < ROWS) {
                n = fmaf(ks[t * dkp + r0 + lane], put, keep * n);
                nq = n * qs[t * dkp + r0 + lane];
            }
            redn[(t * RS + warp) * 32 + lane] = nq;
        };
        const int plain = min(nt, max(0, t1 - ring - c0));      // positions that leave no state behind
#pragma unroll 2
        for (int t = 0; t < plain; ++t) position(t);
        for (int t = plain; t < nt; ++t) {
            position(t);
            float* dst = st_slot + (size_t)((p0 + (c0 + t - t0)) % ring) * entry;
            if (col_ok) {
#pragma unroll
                for (int r = 0; r < ROWS; r += 2) {
                    if (r0 + r < dk) dst[st_S + (size_t)(r0 + r) * dv + col] = S[r >> 1].x;
                    if (r0 + r + 1 < dk) dst[st_S + (size_t)(r0 + r + 1) * dv + col] = S[r >> 1].y;
                }
            }
            if (n_ok) dst[st_n + r0 + lane] = n;
            const float mt = __shfl_sync(0xffffffffu, mlane, t);
            if (threadIdx.x == 0) dst[st_m] = mt;
        }
        __syncthreads();   // the chunk's partial products are complete (and its buffer may be refilled)
#pragma unroll 4
        for (int t = warp; t < nt; t += RS) {
            float nq = 0.f, o = 0.f;
            for (int w = 0; w < RS; ++w) {
                o += red[(t * RS + w) * 32 + lane];
                nq += redn[(t * RS + w) * 32 + lane];
            }
            nq = warp_sum(nq) * a.d.q_scale;
            const float den = fmaxf(fabsf(nq), gates[2 * MAXC + t]) + 1e-6f;
            if (col_ok) a.out[(long long)(c0 + t) * H * dv + (long long)head * dv + col] = o * a.d.q_scale / den;
        }
    }
}

// Steps of one token per sequence: the state is read and written once, so a CTA streams a (sequence, head)'s rows, four
// columns a thread and eight rows in flight, up to 128 columns wide.
constexpr int ST = 256, SCOLS = 128, SU = 8;
__global__ void __launch_bounds__(ST) mlstm_step_kernel(MlstmArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * SCOLS, tid = threadIdx.x;
    const int m = a.cu_q[seq];
    if (m >= a.cu_q[seq + 1]) return;
    const int dk = a.d.dk, dv = a.d.dv, H = a.d.heads, ring = a.ring;
    const int L = (min(SCOLS, dv - col0)) >> 2, R = ST / L;      // threads per row, rows per pass
    const int rg = tid / L, c4 = (tid - rg * L) * 4;
    const int pos = a.ix.positions[m];
    const size_t entry = entry_elems(a.d);
    float* slot = a.state + (size_t)a.seq_slot[seq] * ring * entry;
    const float* src = slot + (size_t)((pos + ring - 1) % ring) * entry;      // pos - 1, not read at position 0
    float* dst = slot + (size_t)(pos % ring) * entry;
    const size_t st_S = (size_t)head * dk * dv + col0 + c4;
    const bool old = pos > 0, live = rg < R;
    float* qs = sm;
    float* ks = qs + dk;
    float* red = ks + dk;             // [R][4 L] partial results, then 33 for a block sum
    float4 S[SU];
    auto load = [&](int r0) {
#pragma unroll
        for (int u = 0; u < SU; ++u) {
            const int r = r0 + u * R;
            S[u] = (live && old && r < dk) ? *reinterpret_cast<const float4*>(src + st_S + (size_t)r * dv)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    load(rg);
    const long long row = (long long)m * a.in.ld;
    for (int i = tid; i < dk; i += ST) {
        qs[i] = a.in.q[row + (long long)head * dk + i];
        ks[i] = a.in.k[row + (long long)head * dk + i];
    }
    const int nb = (dv + 31) / 32, b0 = col0 / 32, b1 = min(nb, b0 + SCOLS / 32);
    const size_t st_n = (size_t)H * dk * dv + ((size_t)head * nb) * (dk + 1);
    const float mold = old ? src[st_n + (size_t)b0 * (dk + 1) + dk] : 0.f;
    const float cap = a.d.cap;
    const float li = cap * tanhf((a.in.zi[row + head] + (a.in.bias_i ? a.in.bias_i[head] : 0.f)) / cap);
    const float lf = log_sigmoid(cap * tanhf((a.in.zf[row + head] + (a.in.bias_f ? a.in.bias_f[head] : 0.f)) / cap));
    const float mnew = fmaxf(lf + mold, li);
    const float keep = expf(lf + mold - mnew), put = expf(li - mnew), flr = expf(-mnew);
    float pv[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
    if (live)
#pragma unroll
        for (int e = 0; e < 4; ++e) pv[e] = put * a.in.v[row + (long long)head * dv + col0 + c4 + e];
    __syncthreads();
    for (int r0 = rg; r0 < dk && live; r0 += SU * R) {
        if (r0 != rg) load(r0);
#pragma unroll
        for (int u = 0; u < SU; ++u) {
            const int r = r0 + u * R;
            if (r >= dk) break;
            const float kk = ks[r], qq = qs[r];
            float4 s = S[u];
            s.x = fmaf(kk, pv[0], keep * s.x), s.y = fmaf(kk, pv[1], keep * s.y);
            s.z = fmaf(kk, pv[2], keep * s.z), s.w = fmaf(kk, pv[3], keep * s.w);
            *reinterpret_cast<float4*>(dst + st_S + (size_t)r * dv) = s;
            o[0] = fmaf(s.x, qq, o[0]), o[1] = fmaf(s.y, qq, o[1]);
            o[2] = fmaf(s.z, qq, o[2]), o[3] = fmaf(s.w, qq, o[3]);
        }
    }
    float nq = 0.f;
    for (int i = tid; i < (b1 - b0) * dk; i += ST) {      // the copies of n that belong to these columns
        const int j = i / dk, r = i - j * dk;
        const size_t at = st_n + (size_t)(b0 + j) * (dk + 1) + r;
        const float n = fmaf(ks[r], put, old ? keep * src[at] : 0.f);
        dst[at] = n;
        if (j == 0) nq = fmaf(n, qs[r], nq);
    }
    if (live)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[rg * 4 * L + c4 + e] = o[e];
    nq = block_sum(nq, red + R * 4 * L) * a.d.q_scale;     // its barriers also complete red, and every read of M
    if (tid < b1 - b0) dst[st_n + (size_t)(b0 + tid) * (dk + 1) + dk] = mnew;
    const float inv = a.d.q_scale / (fmaxf(fabsf(nq), flr) + 1e-6f);
    for (int c = tid; c < 4 * L; c += ST) {
        float t = 0.f;
        for (int r = 0; r < R; ++r) t += red[r * 4 * L + c];
        a.out[(long long)m * H * dv + (long long)head * dv + col0 + c] = t * inv;
    }
}

}  // namespace

size_t mlstm_state_elems(const MlstmDims& d) { return entry_elems(d); }

int launch_mlstm_recurrence(const SeqIndex& ix, const int* cu_q, const int* seq_slot, int nseq, int max_qlen,
                            const MlstmInput& in, const MlstmDims& d, float* state, int ring, float* out, cudaStream_t stream) {
    if (ix.M <= 0 || nseq <= 0) return 0;
    if (d.heads <= 0 || d.dv <= 0 || d.dk <= 0 || d.dk > 1024) return set_error("mlstm: key size %d outside 1..1024", d.dk);
    if (!(d.cap > 0.f)) return set_error("mlstm: the gate cap must be positive");
    if (ring <= 0 || !state) return set_error("mlstm: no state");
    if (!in.q || !in.k || !in.v || !in.zi || !in.zf) return set_error("mlstm: missing inputs");
    if (max_qlen == 1 && d.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0 && d.heads <= 65535) {
        MlstmArgs a;
        a.ix = ix, a.cu_q = cu_q, a.seq_slot = seq_slot, a.in = in, a.d = d, a.state = state, a.ring = ring, a.CH = 1;
        a.v16 = 0, a.out = out;
        const size_t smem = (size_t)(2 * d.dk + 4 * ST + 33) * sizeof(float);
        mlstm_step_kernel<<<dim3(nseq, d.heads, (d.dv + SCOLS - 1) / SCOLS), ST, smem, stream>>>(a);
        count_launch(1);
        ASD_CUDA(cudaGetLastError());
        return 0;
    }
    int rows = 4;
    while (rows < 32 && rows * 4 < d.dk) rows *= 2;     // four warps up to key size 128, then more
    const int RS = (d.dk + rows - 1) / rows, dkp = RS * rows;
    int ch = MAXC;   // positions per staged chunk; steps of few tokens stage (and clear) no more than they use
    while (ch > 1 && (long long)(ch / 2) * nseq >= ix.M) ch >>= 1;
    auto need = [&](int c) { return (size_t)total_floats(c, dkp, RS) * sizeof(float); };
    while (ch > 1 && need(ch) > 112 * 1024) ch >>= 1;
    const size_t smem = need(ch);
    if (smem > 220 * 1024) return set_error("mlstm: key size %d does not fit shared memory", d.dk);
    dim3 grid(nseq, d.heads, (d.dv + 31) / 32);
    if (grid.y > 65535 || grid.z > 65535) return set_error("mlstm: too many heads or value columns");
    MlstmArgs a;
    a.ix = ix, a.cu_q = cu_q, a.seq_slot = seq_slot, a.in = in, a.d = d, a.state = state, a.ring = ring, a.CH = ch, a.out = out;
    const uintptr_t at = reinterpret_cast<uintptr_t>(in.q) | reinterpret_cast<uintptr_t>(in.k);
    a.v16 = (d.dk % 4 == 0 && in.ld % 4 == 0 && (at & 15) == 0) ? 1 : 0;
#define ASD_ML_CASE(R, T)                                                                                             \
    {                                                                                                                 \
        auto fn = mlstm_recurrence_kernel<R, T>;                                                                      \
        static PerDeviceOnce once;                                                                                    \
        if (once.need()) ASD_CUDA(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)); \
        fn<<<grid, RS * 32, smem, stream>>>(a);                                                                       \
    }
    if (RS > 8) ASD_ML_CASE(32, 1024)
    else if (rows == 4) ASD_ML_CASE(4, 256)
    else if (rows == 8) ASD_ML_CASE(8, 256)
    else if (rows == 16) ASD_ML_CASE(16, 256)
    else ASD_ML_CASE(32, 256)
#undef ASD_ML_CASE
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace asd
