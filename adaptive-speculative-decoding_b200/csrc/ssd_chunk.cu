// Scalar-decay state space recurrence (ssd.cu) chunk by chunk on the tensor cores (mma.sync m16n8k16, bf16 operands, fp32
// accumulation), for prompts whose x, B and C are bf16.  With the logarithms of the decays summed up inside a chunk,
// c_t = sum_(s <= t) -exp(a_log) dt_s, a chunk of 64 positions is four products:
//   W[t][s] = (C_t . B_s) exp(c_t - c_s) dt_s  (s <= t),        y = W x + exp(c_t) C_t S + skip x,
//   S <- exp(c_last) S + sum_s exp(c_last - c_s) dt_s B_s x_s^T.
// A CTA owns up to 64 value columns of one (sequence, head) for the whole run of new positions, warp w the columns
// 16 w .. 16 w + 15.  The state is kept transposed, [columns][dk], in the accumulators of the product that updates it, from
// where it enters the product with C as an operand without leaving the registers.  Everything that is not bf16 by nature
// (state, W, the scaled x of the update) enters a product as two bf16 terms; decays, step sizes and the state are fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"
#include "mma_sync.cuh"
#include "ssd.h"

namespace asd {

namespace {

typedef __nv_bfloat16 bf16;
constexpr int NW = 4, NT = NW * 32;
constexpr int CL = 64;             // positions of a chunk
constexpr int PB = NW * 16;        // value columns of a CTA
constexpr int XS = PB + 8, WS = CL + 8;

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// two fp32 values as two bf16 pairs: the rounded values and what the rounding left
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = pack_bf16(a - __low2float(h), b - __high2float(h));
}

// bytes: two buffers of { C [CL][DS], B [CL][DS], x [CL][XS] } bf16, W as two terms [2][CL][WS] bf16, two sets of
// { c [CL], dt [CL] } fp32
__host__ __device__ inline int buf_elems(int DS) { return CL * (2 * DS + XS); }
__host__ __device__ inline int chunk_smem(int DS) { return 2 * buf_elems(DS) * 2 + 2 * CL * WS * 2 + 4 * CL * 4; }

template <int NK>      // dk <= 16 NK
__global__ void __launch_bounds__(NT) ssd_chunk_kernel(SsdArgs a) {
    extern __shared__ __align__(16) unsigned char smraw[];
    constexpr int DKP = 16 * NK, DS = DKP + 8;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, lr = lane & 7, mat = lane >> 3;
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * PB;
    const int t0 = a.cu_q[seq], t1 = a.cu_q[seq + 1] - a.tail;      // the last `tail` positions are another kernel's
    if (t0 >= t1) return;
    const int dk = a.d.dk, dv = a.d.dv, H = a.d.heads, ring = a.ring, grp = head / (H / a.d.groups);
    const int slot = a.seq_slot[seq], p0 = a.ix.positions[t0];
    const bf16* xg = static_cast<const bf16*>(static_cast<const void*>(a.in.x)) + (long long)head * dv + col0;
    const bf16* bg = static_cast<const bf16*>(static_cast<const void*>(a.in.b)) + (long long)grp * dk;
    const bf16* cg = static_cast<const bf16*>(static_cast<const void*>(a.in.c)) + (long long)grp * dk;
    bf16* bufs = reinterpret_cast<bf16*>(smraw);
    bf16* Wh = bufs + 2 * buf_elems(DS);
    bf16* Wl = Wh + CL * WS;
    float* fac = reinterpret_cast<float*>(Wl + CL * WS);
    const size_t entry = (size_t)H * dk * dv;
    float* st = a.state + (size_t)slot * ring * entry + (size_t)head * dk * dv;
    const float bias = a.in.dt_bias[head], rate = expf(a.in.a_log[head]), skip = a.in.skip[head];
    const int ncol = min(PB, dv - col0);
    const bool mine = warp * 16 < ncol;          // this warp has value columns (it helps with W in any case)
    const int pr[2] = {warp * 16 + g, warp * 16 + g + 8};

    auto fetch = [&](int which, int c0) {
        const int nt = min(CL, t1 - c0);
        bf16* cs = bufs + which * buf_elems(DS);
        bf16* bs = cs + CL * DS;
        bf16* xs = bs + CL * DS;
        if (a.v16) {
            constexpr int n8 = DKP / 8;
            for (int i = tid; i < CL * n8; i += NT) {
                const int t = i / n8, d = (i - t * n8) * 8;
                const bool live = t < nt && d < dk;
                const long long at = live ? (long long)(c0 + t) * a.in.ld + d : 0;
                cp_async16(smem_at(cs + t * DS + d), cg + at, live);
                cp_async16(smem_at(bs + t * DS + d), bg + at, live);
            }
            for (int i = tid; i < CL * (PB / 8); i += NT) {
                const int t = i / (PB / 8), d = (i % (PB / 8)) * 8;
                const bool live = t < nt && d < ncol;
                cp_async16(smem_at(xs + t * XS + d), xg + (live ? (long long)(c0 + t) * a.in.ld + d : 0), live);
            }
        } else {
            const bf16 zero = __float2bfloat16(0.f);
            for (int i = tid; i < CL * DKP; i += NT) {
                const int t = i / DKP, d = i % DKP;
                const bool live = t < nt && d < dk;
                const long long at = (long long)(c0 + t) * a.in.ld + d;
                cs[t * DS + d] = live ? cg[at] : zero;
                bs[t * DS + d] = live ? bg[at] : zero;
            }
            for (int i = tid; i < CL * PB; i += NT) {
                const int t = i / PB, d = i % PB;
                xs[t * XS + d] = t < nt && d < ncol ? xg[(long long)(c0 + t) * a.in.ld + d] : zero;
            }
        }
        cp_async_commit();
    };
    // raw step sizes of the positions 2 lane, 2 lane + 1 of a chunk (warp 0)
    auto raw_dt = [&](int c0, float (&z)[2]) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int m = c0 + 2 * lane + e;
            z[e] = m < t1 ? a.in.dt[(long long)m * a.in.ld_dt + head] : 0.f;
        }
    };

    float S[2 * NK][4];            // S^T: rows pr[], columns n * 8 + 2 t4 + e
    {
        const float* src = st + (size_t)((p0 + ring - 1) % ring) * entry;
#pragma unroll
        for (int n = 0; n < 2 * NK; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = n * 8 + 2 * t4 + (e & 1), p = pr[e >> 1];
                S[n][e] = (p0 > 0 && d < dk && p < ncol) ? src[(size_t)d * dv + col0 + p] : 0.f;
            }
    }
    float z[2] = {0.f, 0.f};
    if (warp == 0) raw_dt(t0, z);
    fetch(0, t0);
    int it = 0;
    for (int c0 = t0; c0 < t1; c0 += CL, ++it) {
        float* cum = fac + (it & 1) * 2 * CL;
        float* dts = cum + CL;
        if (warp == 0) {
            float d[2], l[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                d[e] = c0 + 2 * lane + e < t1 ? softplus_step(z[e] + bias) : 0.f;    // beyond the end: no decay, nothing written
                l[e] = -rate * d[e];
            }
            float run = l[0] + l[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run += up;
            }
            cum[2 * lane] = run - l[1], cum[2 * lane + 1] = run;
            dts[2 * lane] = d[0], dts[2 * lane + 1] = d[1];
            if (c0 + CL < t1) raw_dt(c0 + CL, z);
        }
        cp_async_wait<0>();
        __syncthreads();           // the chunk has landed; every warp is done with the one before
        if (c0 + CL < t1) fetch((it + 1) & 1, c0 + CL);
        const bf16* cs = bufs + (it & 1) * buf_elems(DS);
        const bf16* bs = cs + CL * DS;
        const bf16* xs = bs + CL * DS;
        {   // W: positions t = 16 warp + .., every s up to the warp's last position
            float w[CL / 8][4];
#pragma unroll
            for (int n = 0; n < CL / 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) w[n][e] = 0.f;
            const uint32_t a_at = smem_at(cs + (warp * 16 + lr + (mat & 1) * 8) * DS + (mat >> 1) * 8);
            const uint32_t b_at = smem_at(bs + (lr + (mat >> 1) * 8) * DS + (mat & 1) * 8);
#pragma unroll
            for (int kk = 0; kk < NK; ++kk) {
                uint32_t ca[4];
                ldsm_x4(a_at + kk * 32, ca);
#pragma unroll
                for (int n2 = 0; n2 < CL / 16; ++n2) {
                    if (n2 > warp) break;
                    uint32_t bb[4];
                    ldsm_x4(b_at + (n2 * 16 * DS + kk * 16) * 2, bb);
                    mma_bf16(w[2 * n2], ca, bb[0], bb[1]);
                    mma_bf16(w[2 * n2 + 1], ca, bb[2], bb[3]);
                }
            }
            const float ct[2] = {cum[pr[0]], cum[pr[1]]};
#pragma unroll
            for (int n = 0; n < CL / 8; ++n) {
                if (n > 2 * warp + 1) break;
                const int s = n * 8 + 2 * t4;
                const float2 cc = *reinterpret_cast<const float2*>(cum + s), dd = *reinterpret_cast<const float2*>(dts + s);
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const int t = pr[x];
                    const float w0 = s <= t ? w[n][2 * x] * expf(ct[x] - cc.x) * dd.x : 0.f;
                    const float w1 = s + 1 <= t ? w[n][2 * x + 1] * expf(ct[x] - cc.y) * dd.y : 0.f;
                    uint32_t hi, lo;
                    split2(w0, w1, hi, lo);
                    *reinterpret_cast<uint32_t*>(Wh + t * WS + s) = hi;
                    *reinterpret_cast<uint32_t*>(Wl + t * WS + s) = lo;
                }
            }
        }
        __syncthreads();           // W is complete
        if (!mine) continue;
        float y[CL / 8][4];        // rows: columns of x; columns: positions
#pragma unroll
        for (int n = 0; n < CL / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[n][e] = 0.f;
        {   // what the state from before the chunk gives: S^T C^T
            const uint32_t c_at = smem_at(cs + (lr + (mat >> 1) * 8) * DS + (mat & 1) * 8);
#pragma unroll
            for (int kk = 0; kk < NK; ++kk) {
                uint32_t sh[4], sl[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) split2(S[2 * kk + (u >> 1)][(u & 1) * 2], S[2 * kk + (u >> 1)][(u & 1) * 2 + 1], sh[u], sl[u]);
#pragma unroll
                for (int n2 = 0; n2 < CL / 16; ++n2) {
                    uint32_t cb[4];
                    ldsm_x4(c_at + (n2 * 16 * DS + kk * 16) * 2, cb);
                    mma_bf16(y[2 * n2], sh, cb[0], cb[1]);
                    mma_bf16(y[2 * n2 + 1], sh, cb[2], cb[3]);
                    mma_bf16(y[2 * n2], sl, cb[0], cb[1]);
                    mma_bf16(y[2 * n2 + 1], sl, cb[2], cb[3]);
                }
            }
#pragma unroll
            for (int n = 0; n < CL / 8; ++n) {
                const float2 cc = *reinterpret_cast<const float2*>(cum + n * 8 + 2 * t4);
                const float e0 = expf(cc.x), e1 = expf(cc.y);
                y[n][0] *= e0, y[n][1] *= e1, y[n][2] *= e0, y[n][3] *= e1;
            }
        }
        const float last = cum[CL - 1];
        const float keep = expf(last);
#pragma unroll
        for (int n = 0; n < 2 * NK; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[n][e] *= keep;
        const uint32_t x_at = smem_at(xs + (lr + (mat >> 1) * 8) * XS + warp * 16 + (mat & 1) * 8);
        const uint32_t w_at = smem_at(Wh + (lr + (mat >> 1) * 8) * WS + (mat & 1) * 8);
        const uint32_t wl_off = CL * WS * 2;
        const uint32_t b_at = smem_at(bs + (lr + (mat & 1) * 8) * DS + (mat >> 1) * 8);
#pragma unroll
        for (int ks = 0; ks < CL / 16; ++ks) {
            uint32_t xa[4];                     // x^T: rows columns of x, k = positions s
            ldsm_x4_t(x_at + ks * 16 * XS * 2, xa);
            // positions t from this block of s on
#pragma unroll
            for (int n2 = ks; n2 < CL / 16; ++n2) {
                uint32_t wh[4], wl[4];
                ldsm_x4(w_at + (n2 * 16 * WS + ks * 16) * 2, wh);
                ldsm_x4(w_at + wl_off + (n2 * 16 * WS + ks * 16) * 2, wl);
                mma_bf16(y[2 * n2], xa, wh[0], wh[1]);
                mma_bf16(y[2 * n2 + 1], xa, wh[2], wh[3]);
                mma_bf16(y[2 * n2], xa, wl[0], wl[1]);
                mma_bf16(y[2 * n2 + 1], xa, wl[2], wl[3]);
            }
            // the state takes the block: x scaled by exp(c_last - c_s) dt_s, as two terms
            uint32_t xh[4], xl[4];
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int s = ks * 16 + hf * 8 + 2 * t4;
                const float2 cc = *reinterpret_cast<const float2*>(cum + s), dd = *reinterpret_cast<const float2*>(dts + s);
                const float f0 = expf(last - cc.x) * dd.x, f1 = expf(last - cc.y) * dd.y;
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const uint32_t r = xa[2 * hf + x];
                    split2(__uint_as_float(r << 16) * f0, __uint_as_float(r & 0xffff0000u) * f1, xh[2 * hf + x], xl[2 * hf + x]);
                }
            }
#pragma unroll
            for (int n = 0; n < 2 * NK; n += 2) {
                uint32_t bb[4];
                ldsm_x4_t(b_at + (ks * 16 * DS + n * 8) * 2, bb);
                mma_bf16(S[n], xh, bb[0], bb[1]);
                mma_bf16(S[n + 1], xh, bb[2], bb[3]);
                mma_bf16(S[n], xl, bb[0], bb[1]);
                mma_bf16(S[n + 1], xl, bb[2], bb[3]);
            }
        }
        const int nt = min(CL, t1 - c0);
#pragma unroll
        for (int n = 0; n < CL / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = n * 8 + 2 * t4 + (e & 1), p = pr[e >> 1];
                if (t < nt && p < ncol)
                    a.out[(long long)(c0 + t) * H * dv + (long long)head * dv + col0 + p] =
                        fmaf(skip, __bfloat162float(xs[t * XS + p]), y[n][e]);
            }
    }
    if (!mine) return;
    float* dst = st + (size_t)((p0 + (t1 - 1 - t0)) % ring) * entry;
#pragma unroll
    for (int n = 0; n < 2 * NK; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = n * 8 + 2 * t4 + (e & 1), p = pr[e >> 1];
            if (d < dk && p < ncol) dst[(size_t)d * dv + col0 + p] = S[n][e];
        }
}

template <int NK>
int launch_nk(const SsdArgs& a, dim3 grid, cudaStream_t stream) {
    const int smem = chunk_smem(16 * NK + 8);
    static PerDeviceOnce once;
    if (once.need()) ASD_CUDA(cudaFuncSetAttribute(ssd_chunk_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    ssd_chunk_kernel<NK><<<grid, NT, smem, stream>>>(a);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace

int launch_ssd_chunks(SsdArgs a, int nseq, cudaStream_t stream) {
    if (!a.in.bf16 || a.d.dk > 128 || a.d.heads > 65535) return 1;
    const uintptr_t at = reinterpret_cast<uintptr_t>(a.in.x) | reinterpret_cast<uintptr_t>(a.in.b) | reinterpret_cast<uintptr_t>(a.in.c);
    a.v16 = (a.d.dk % 8 == 0 && a.d.dv % 8 == 0 && a.in.ld % 8 == 0 && (at & 15) == 0) ? 1 : 0;
    const dim3 grid(nseq, a.d.heads, (a.d.dv + PB - 1) / PB);
    if (grid.z > 65535) return 1;
    return a.d.dk <= 32 ? launch_nk<2>(a, grid, stream)
                        : (a.d.dk <= 64 ? launch_nk<4>(a, grid, stream)
                                        : (a.d.dk <= 96 ? launch_nk<6>(a, grid, stream) : launch_nk<8>(a, grid, stream)));
}

}  // namespace asd
