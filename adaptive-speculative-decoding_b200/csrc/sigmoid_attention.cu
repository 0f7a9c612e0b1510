// Steps of few tokens of the grouped-query attention with sigmoid weights,
//   o_h = sum over the visible keys j of sigmoid(scale * q_h . k_j + head_bias[h]) v_j.
// The weights are not normalised over the keys, so one pass suffices and key shares simply add.  A CTA owns one token, one
// key share and up to eight query heads of one key/value group.  Per block of 64 keys it issues its value loads first
// (they do not depend on the scores), then eight lanes share a key row against the queries in shared memory, the weights go
// through shared memory, and every warp multiplies the value rows it already holds in registers.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include <algorithm>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"
#include "mixed_attention.h"

namespace asd {

namespace {

constexpr int NT = 256, NW = NT / 32;
constexpr int KB = 64;      // keys of a block
constexpr int HB = 8;       // query heads of a CTA

// N consecutive elements of a cache row as floats, N = 4 or 8 (vec: 8- or 16-byte loads; else element by element with zeros
// from `n` on, d = place of the first element)
template <typename T, int N>
__device__ __forceinline__ void load_row(const T* src, int d, int n, int vec, float (&v)[N]) {
    if (vec && d + N <= n) {
        if constexpr (sizeof(T) == 4) {
#pragma unroll
            for (int e = 0; e < N; e += 4) {
                const float4 f = *reinterpret_cast<const float4*>(src + e);
                v[e] = f.x, v[e + 1] = f.y, v[e + 2] = f.z, v[e + 3] = f.w;
            }
        } else {
            uint32_t raw[N / 2];
            if constexpr (N == 8) {
                const uint4 r = *reinterpret_cast<const uint4*>(src);
                raw[0] = r.x, raw[1] = r.y, raw[2] = r.z, raw[3] = r.w;
            } else {
                const uint2 r = *reinterpret_cast<const uint2*>(src);
                raw[0] = r.x, raw[1] = r.y;
            }
#pragma unroll
            for (int e = 0; e < N / 2; ++e) {
                v[2 * e] = __uint_as_float(raw[e] << 16);
                v[2 * e + 1] = __uint_as_float(raw[e] & 0xffff0000u);
            }
        }
    } else {
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] = d + e < n ? ldf(src + e) : 0.f;
    }
}

// dynamic shared memory (floats): queries [HB][dkp], weights [2][HB][KB], sums [NW][HB][dvp], 64-bit row offsets [2][KB]
__host__ __device__ inline int sig_floats(int dkp, int dvp) { return HB * dkp + 2 * HB * KB + NW * HB * dvp + 4 * KB; }

template <typename T, int VC>
__global__ void __launch_bounds__(NT) sigmoid_decode_kernel(MixArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l8 = lane & 7, sub = lane >> 3;
    const int H = a.d.heads, G = a.d.kv_heads, rep = H / G, dk = a.d.dk, dv = a.d.dv, dkp = a.dkp, dvp = a.dvp;
    const int nhb = (rep + HB - 1) / HB, c = blockIdx.z / nhb, x0 = (blockIdx.z % nhb) * HB;
    const int nx = min(HB, rep - x0), h0 = c * rep + x0;
    const int m = blockIdx.y, share = blockIdx.x, M = a.ix.M;
    float* qs = sm;
    float* Ws = qs + HB * dkp;
    float* red = Ws + 2 * HB * KB;
    long long* rowoff = reinterpret_cast<long long*>(red + NW * HB * dvp);
    const int pos = a.ix.positions[m], slot = a.ix.token_slot[m];
    const int kmin = a.d.chunk > 0 ? (pos / a.d.chunk) * a.d.chunk : 0;
    const int n = pos - kmin + 1, nblk = (n + KB - 1) / KB, per = (nblk + a.shares - 1) / a.shares;
    const int b0 = share * per, b1 = min(nblk, b0 + per);
    const T* pool = static_cast<const T*>(a.cache.pool);
    const int row_elems = G * (dk + dv), psz = a.cache.page_size;
    auto block_rows = [&](int b, long long* ro) {
        if (tid < KB) {
            const int j = b * KB + tid;
            long long off = 0;
            if (j < n) {
                const int p = kmin + j;
                off = ((long long)a.cache.page_table[(long long)slot * a.cache.max_pages + p / psz] * psz + p % psz) * row_elems;
            }
            ro[tid] = off;      // beyond the last key: row 0, read but weighted by zero
        }
    };
    for (int idx = tid; idx < HB * dkp; idx += NT) {
        const int x = idx / dkp, d = idx - x * dkp;
        qs[idx] = (x < nx && d < dk) ? a.q[(long long)m * a.ldq + (long long)(h0 + x) * dk + d] : 0.f;
    }
    if (b0 < b1) block_rows(b0, rowoff + (b0 & 1) * KB);
    float acc[HB][VC];
#pragma unroll
    for (int x = 0; x < HB; ++x)
#pragma unroll
        for (int e = 0; e < VC; ++e) acc[x][e] = 0.f;
    const bool col_ok = VC * lane < dv;
    const int npiece = dkp >> 3, voff = G * dk + c * dv + VC * lane;
    __syncthreads();
    for (int b = b0; b < b1; ++b) {
        const long long* ro = rowoff + (b & 1) * KB;
        float* W = Ws + (b & 1) * HB * KB;
        const int nk = min(KB, n - b * KB);
        float v[KB / NW][VC];
        if (col_ok) {
#pragma unroll
            for (int u = 0; u < KB / NW; ++u) load_row<T, VC>(pool + ro[warp + u * NW] + voff, VC * lane, dv, a.vec, v[u]);
        }
#pragma unroll
        for (int half = 0; half < KB / (4 * NW); ++half) {
            const int ki = half * 4 * NW + warp * 4 + sub;
            const T* kr = pool + ro[ki] + c * dk;
            float s[HB];
#pragma unroll
            for (int x = 0; x < HB; ++x) s[x] = 0.f;
            for (int p = l8; p < npiece; p += 8) {
                float kk[8];
                load_row<T, 8>(kr + 8 * p, 8 * p, dk, a.gp, kk);
#pragma unroll
                for (int x = 0; x < HB; ++x) {
                    if (x >= nx) break;
                    const float4 q0 = *reinterpret_cast<const float4*>(qs + x * dkp + 8 * p);
                    const float4 q1 = *reinterpret_cast<const float4*>(qs + x * dkp + 8 * p + 4);
                    s[x] = fmaf(q0.x, kk[0], s[x]);
                    s[x] = fmaf(q0.y, kk[1], s[x]);
                    s[x] = fmaf(q0.z, kk[2], s[x]);
                    s[x] = fmaf(q0.w, kk[3], s[x]);
                    s[x] = fmaf(q1.x, kk[4], s[x]);
                    s[x] = fmaf(q1.y, kk[5], s[x]);
                    s[x] = fmaf(q1.z, kk[6], s[x]);
                    s[x] = fmaf(q1.w, kk[7], s[x]);
                }
            }
#pragma unroll
            for (int x = 0; x < HB; ++x) {
                if (x >= nx) break;
                float t = s[x];
                t += __shfl_xor_sync(0xffffffffu, t, 1);
                t += __shfl_xor_sync(0xffffffffu, t, 2);
                t += __shfl_xor_sync(0xffffffffu, t, 4);
                if (l8 == 0) {
                    t = fmaf(t, a.d.scale, a.d.head_bias ? a.d.head_bias[h0 + x] : 0.f);
                    W[x * KB + ki] = ki < nk ? 1.f / (1.f + expf(-t)) : 0.f;
                }
            }
        }
        if (b + 1 < b1) block_rows(b + 1, rowoff + ((b + 1) & 1) * KB);
        __syncthreads();   // weights of this block and row offsets of the next; the block after next reuses the buffers
        if (col_ok) {
#pragma unroll
            for (int u = 0; u < KB / NW; ++u) {
                if (warp + u * NW >= nk) break;
#pragma unroll
                for (int x = 0; x < HB; ++x) {
                    if (x >= nx) break;
                    const float w = W[x * KB + warp + u * NW];
#pragma unroll
                    for (int e = 0; e < VC; ++e) acc[x][e] = fmaf(w, v[u][e], acc[x][e]);
                }
            }
        }
    }
    if (col_ok) {
#pragma unroll
        for (int x = 0; x < HB; ++x) {
            if (x >= nx) break;
#pragma unroll
            for (int e = 0; e < VC; ++e) red[(warp * HB + x) * dvp + VC * lane + e] = acc[x][e];
        }
    }
    __syncthreads();
    for (int idx = tid; idx < nx * dv; idx += NT) {      // the warps' sums in index order
        const int x = idx / dv, col = idx - x * dv, h = h0 + x;
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) t += red[(w * HB + x) * dvp + col];
        if (a.shares == 1) {
            const float gate = mix_gate(a, m, h, col);
            stx(a.out, (long long)m * a.ldo + (long long)h * dv + col, a.of32, t * gate);
        } else {
            a.part[((long long)share * M + m) * H * dv + (long long)h * dv + col] = t;
        }
    }
}

template <typename T, int VC>
int launch_sig(const MixArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
    static PerDeviceOnce once;
    if (once.need())
        ASD_CUDA(cudaFuncSetAttribute(sigmoid_decode_kernel<T, VC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    sigmoid_decode_kernel<T, VC><<<grid, NT, smem, stream>>>(a);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

}  // namespace

int launch_sigmoid_attention_decode(MixArgs a, int max_kv_len, const MixWork& ws, cudaStream_t stream) {
    const int H = a.d.heads, G = a.d.kv_heads, rep = H / G, M = a.ix.M, dv = a.d.dv;
    if (dv > 256 || a.dist_bias) return 1;
    const int vc = dv <= 128 ? 4 : 8;
    a.dkp = (a.d.dk + 7) & ~7, a.dvp = (dv + vc - 1) / vc * vc;
    const size_t smem = (size_t)sig_floats(a.dkp, a.dvp) * sizeof(float);
    if (smem > 200 * 1024 || M > 65535) return 1;
    const int units = G * ((rep + HB - 1) / HB), blocks = (max_kv_len + KB - 1) / KB;
    // shares of the keys: about four CTAs per SM, two blocks of keys at least
    int shares = (int)std::min<long long>((592 + (long long)M * units - 1) / ((long long)M * units), std::max(1, blocks / 2));
    shares = std::max(1, std::min(shares, 64));
    while (shares > 1 && (!ws.part || (long long)shares * M * H * dv > ws.part_elems)) --shares;
    a.shares = shares;
    const int wide = a.cache.f32 ? 4 : 8;                                   // elements of a 16-byte load
    a.gp = (a.d.dk % wide == 0 && dv % wide == 0) ? 1 : 0;                  // key pieces
    a.vec = vc == 4 ? (a.d.dk % 4 == 0 && dv % 4 == 0 ? 1 : 0) : a.gp;      // value columns
    if (a.gp && (reinterpret_cast<uintptr_t>(a.cache.pool) & 15)) a.gp = a.vec = 0;
    const dim3 grid(shares, M, units);
    int rc;
    if (a.cache.f32)
        rc = vc == 4 ? launch_sig<float, 4>(a, grid, smem, stream) : launch_sig<float, 8>(a, grid, smem, stream);
    else
        rc = vc == 4 ? launch_sig<__nv_bfloat16, 4>(a, grid, smem, stream) : launch_sig<__nv_bfloat16, 8>(a, grid, smem, stream);
    if (rc) return -1;
    if (shares > 1 && launch_mix_merge(a, stream)) return -1;
    return 0;
}

}  // namespace asd
