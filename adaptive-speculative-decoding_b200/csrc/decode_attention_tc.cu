// Steps of few tokens of attention with sigmoid or softmax weights on the tensor cores (bf16 cache rows; mma.sync m16n8k16, fp32 accumulation).
// A CTA owns one sequence, one key/value group, up to sixteen (token, head) rows and one key share.  Its warps work on
// 16-key tiles of their own, staged by cp.async in a ring per warp, so nothing but the end meets at a barrier: scores of the
// sixteen rows against a tile, weights in registers (they already stand in the layout of the next product's operand),
// values.  Queries and weights enter as two bf16 terms each, so that scores and sums keep fp32 accuracy against the cache's
// bf16 rows.  Sigmoid weights are not normalised, so the warps' sums and the key shares simply add, in index order.  Softmax:
// every warp keeps a running maximum per row, against which its sums stand; the warps' sums are brought to their common
// maximum at the end, and the key shares' sums by the merge.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include <algorithm>

#include "asd_internal.h"
#include "blocks.h"
#include "elem.cuh"
#include "mixed_attention.h"
#include "mma_sync.cuh"

namespace asd {

namespace {

constexpr int NW = 4, NT = NW * 32;
constexpr int KT = 16;      // keys of a tile
typedef __nv_bfloat16 bf16;

__device__ __forceinline__ uint32_t smem_at(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// bytes: queries (two terms) [2][16][dkp + 8], then NW x NS tiles { keys [16][dkp + 8], values [16][dvp + 8] }; the warps'
// sums fp32 [NW][16][dvp] take the tiles' place at the end
__host__ __device__ inline int tile_elems(int dkp, int dvp) { return KT * (dkp + 8 + dvp + 8); }
__host__ __device__ inline int smem_bytes(int dkp, int dvp, int NS) {
    const int tiles = NW * NS * tile_elems(dkp, dvp) * 2, red = NW * 16 * dvp * 4;
    return 2 * 16 * (dkp + 8) * 2 + (tiles > red ? tiles : red);
}

enum { D_SIGMOID = 0, D_SOFTMAX = 1, D_SOFTMAX_CAP = 2 };
template <int NDV, int NS, int MODE>
__global__ void __launch_bounds__(NT) decode_tc_kernel(MixArgs a) {
    constexpr bool SOFT = MODE != D_SIGMOID;
    extern __shared__ __align__(16) unsigned char smraw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int H = a.d.heads, G = a.d.kv_heads, rep = H / G, dk = a.d.dk, dv = a.d.dv, M = a.ix.M;
    constexpr int DVP = NDV * 8, VS = DVP + 8;
    const int dkp = a.dkp, DS = dkp + 8;
    const int b = blockIdx.y, share = blockIdx.x, c = blockIdx.z % G, rb = blockIdx.z / G;
    const int q0 = a.cu_q[b], qlen = a.cu_q[b + 1] - q0;
    const int nrows = min(16, qlen * rep - rb * 16);      // rows of this block: (token, head of the group), token major
    if (nrows <= 0) return;
    const int p0 = a.ix.positions[q0], slot = a.seq_slot[b];
    const int last = p0 + (rb * 16 + nrows - 1) / rep;    // last position any row sees
    // chunked mask: keys from the first row's chunk on
    const int chunk = a.d.chunk, kmin = chunk > 0 ? (p0 + rb * 16 / rep) / chunk * chunk : 0;
    const int ntile = (last - kmin) / KT + 1, per = (ntile + a.shares - 1) / a.shares;
    const int t0 = share * per, t1 = min(ntile, t0 + per);
    bf16* Qh = reinterpret_cast<bf16*>(smraw);
    bf16* Ql = Qh + 16 * DS;
    bf16* ring = Ql + 16 * DS + (size_t)warp * NS * tile_elems(dkp, DVP);
    const bf16* pool = static_cast<const bf16*>(a.cache.pool);
    const int row_elems = G * (dk + dv), psz = a.cache.page_size;

    for (int idx = tid; idx < 16 * dkp; idx += NT) {
        const int r = idx / dkp, d = idx - r * dkp;
        float v = 0.f;
        if (r < nrows && d < dk) {
            const int gr = rb * 16 + r;
            v = a.q[(long long)(q0 + gr / rep) * a.ldq + (long long)(c * rep + gr % rep) * dk + d];
        }
        const bf16 hi = __float2bfloat16(v);
        Qh[r * DS + d] = hi;
        Ql[r * DS + d] = __float2bfloat16(v - __bfloat162float(hi));
    }
    if (dk != dkp)      // key columns beyond dk meet zero queries: they must hold numbers
        for (int i = lane; i < NS * KT * 8; i += 32) {
            const int s = i / (KT * 8), k = (i / 8) % KT, d = dkp - 8 + i % 8;
            if (d >= dk) ring[s * tile_elems(dkp, DVP) + k * DS + d] = __float2bfloat16(0.f);
        }

    int posr[2], lor[2];
    float hb[2], mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
    const float icap = MODE == D_SOFTMAX_CAP ? 1.f / a.d.softcap : 0.f;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int r = g + 8 * x, gr = rb * 16 + r;
        posr[x] = r < nrows ? p0 + gr / rep : -1;
        lor[x] = chunk > 0 ? posr[x] / chunk * chunk : 0;
        hb[x] = (r < nrows && a.d.head_bias) ? a.d.head_bias[c * rep + gr % rep] : 0.f;
    }
    float O[NDV][4];
#pragma unroll
    for (int n = 0; n < NDV; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) O[n][e] = 0.f;
    __syncthreads();

    // tile of this warp's step i: t0 + warp + NW * i; the cache row of its key `lane` (lanes 0 - 15), -1 beyond the last key
    auto rows_of = [&](int i) {
        const int t = t0 + warp + NW * i, j = kmin + t * KT + (lane & 15);
        if (t >= t1 || j > last) return -1;
        return a.cache.page_table[(long long)slot * a.cache.max_pages + j / psz] * psz + j % psz;
    };
    const int l8 = lane & 7, sub = lane >> 3;
    auto fetch = [&](int i, int rows) {       // eight lanes copy a key's row in 16-byte pieces
        bf16* kt = ring + (i % NS) * tile_elems(dkp, DVP);
        bf16* vt = kt + KT * DS;
#pragma unroll
        for (int u = 0; u < KT / 4; ++u) {
            const int key = sub + 4 * u;
            const int row = __shfl_sync(0xffffffffu, rows, key);
            const bool live = row >= 0;
            const bf16* src = pool + (live ? (long long)row * row_elems : 0);
            for (int p = l8 * 8; p < dk; p += 64) cp_async16(smem_at(kt + key * DS + p), src + c * dk + p, live);
            for (int p = l8 * 8; p < dv; p += 64) cp_async16(smem_at(vt + key * VS + p), src + G * dk + c * dv + p, live);
        }
    };
    const int nmine = t1 > t0 + warp ? (t1 - t0 - warp + NW - 1) / NW : 0;
    int rows = rows_of(0);
#pragma unroll
    for (int i = 0; i < NS - 1; ++i) {
        if (i < nmine) fetch(i, rows);
        cp_async_commit();
        rows = rows_of(i + 1);
    }
    const int lr = lane & 7, mat = lane >> 3;
    const uint32_t qh_at = smem_at(Qh + (lr + (mat & 1) * 8) * DS + (mat >> 1) * 8);
    const uint32_t ql_at = smem_at(Ql + (lr + (mat & 1) * 8) * DS + (mat >> 1) * 8);
    for (int i = 0; i < nmine; ++i) {
        cp_async_wait<NS - 2>();
        __syncwarp();          // the tile's pieces of all lanes; and every lane is done with the tile whose place comes next
        if (i + NS - 1 < nmine) fetch(i + NS - 1, rows);
        cp_async_commit();
        rows = rows_of(i + NS);
        const bf16* kt = ring + (i % NS) * tile_elems(dkp, DVP);
        const bf16* vt = kt + KT * DS;
        const uint32_t k_at = smem_at(kt + (lr + (mat >> 1) * 8) * DS + (mat & 1) * 8);
        const uint32_t v_at = smem_at(vt + (lr + (mat & 1) * 8) * VS + (mat >> 1) * 8);
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        for (int ks = 0; ks < dkp; ks += 16) {
            uint32_t ah[4], al[4], bq[4];
            ldsm_x4(qh_at + ks * 2, ah);
            ldsm_x4(ql_at + ks * 2, al);
            ldsm_x4(k_at + ks * 2, bq);
            mma_bf16(s[0], ah, bq[0], bq[1]);
            mma_bf16(s[1], ah, bq[2], bq[3]);
            mma_bf16(s[0], al, bq[0], bq[1]);
            mma_bf16(s[1], al, bq[2], bq[3]);
        }
        const int j0 = kmin + (t0 + warp + NW * i) * KT;
        uint32_t ph[4], pl[4];
        if (SOFT) {
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] *= a.d.scale;
            if (MODE == D_SOFTMAX_CAP) cap_scores(s, a.d.softcap, icap);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                float mx = -INFINITY;
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int j = j0 + n * 8 + 2 * t4 + e;
                        const float v = j <= posr[x] && j >= lor[x] ? s[n][2 * x + e] : -INFINITY;
                        s[n][2 * x + e] = v;
                        mx = fmaxf(mx, v);
                    }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float mnew = fmaxf(mrun[x], mx), ref = mnew > -INFINITY ? mnew : 0.f;
                const float keep = __expf(mrun[x] - ref);
                float sum = 0.f;           // this thread's part of the row's sum; the quad's parts are added at the end
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        s[n][2 * x + e] = __expf(s[n][2 * x + e] - ref);
                        sum += s[n][2 * x + e];
                    }
                lrun[x] = fmaf(lrun[x], keep, sum);
                mrun[x] = mnew;
                if (__any_sync(0xffffffffu, keep != 1.f))
#pragma unroll
                    for (int n = 0; n < NDV; ++n) O[n][2 * x] *= keep, O[n][2 * x + 1] *= keep;
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int x = u & 1, n = u >> 1;
            float w[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (SOFT) {
                    w[e] = s[n][2 * x + e];
                } else {
                    const float z = fmaf(s[n][2 * x + e], a.d.scale, hb[x]);
                    const int j = j0 + n * 8 + 2 * t4 + e;
                    w[e] = j <= posr[x] && j >= lor[x] ? __fdividef(1.f, 1.f + __expf(-z)) : 0.f;
                }
            }
            const bf16 h0 = __float2bfloat16(w[0]), h1 = __float2bfloat16(w[1]);
            ph[u] = (uint32_t)__bfloat16_as_ushort(h0) | ((uint32_t)__bfloat16_as_ushort(h1) << 16);
            pl[u] = pack_bf16(w[0] - __bfloat162float(h0), w[1] - __bfloat162float(h1));
        }
#pragma unroll
        for (int n = 0; n < NDV; n += 2) {
            uint32_t bv[4];
            ldsm_x4_t(v_at + n * 16, bv);
            mma_bf16(O[n], ph, bv[0], bv[1]);
            mma_bf16(O[n + 1], ph, bv[2], bv[3]);
            mma_bf16(O[n], pl, bv[0], bv[1]);
            mma_bf16(O[n + 1], pl, bv[2], bv[3]);
        }
    }
    cp_async_wait<0>();
    __syncthreads();          // every warp is done with its tiles: their place takes the sums
    float* red = reinterpret_cast<float*>(Ql + 16 * DS);
    float* stat = reinterpret_cast<float*>(Qh);       // [NW][16] maxima, then sums, in the queries' place
    if (SOFT)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            lrun[x] += __shfl_xor_sync(0xffffffffu, lrun[x], 1);
            lrun[x] += __shfl_xor_sync(0xffffffffu, lrun[x], 2);
            if (t4 == 0) stat[warp * 16 + g + 8 * x] = mrun[x], stat[NW * 16 + warp * 16 + g + 8 * x] = lrun[x];
        }
#pragma unroll
    for (int n = 0; n < NDV; ++n)
#pragma unroll
        for (int x = 0; x < 2; ++x)
            *reinterpret_cast<float2*>(red + ((size_t)warp * 16 + g + 8 * x) * DVP + n * 8 + 2 * t4) =
                make_float2(O[n][2 * x], O[n][2 * x + 1]);
    __syncthreads();
    for (int idx = tid; idx < nrows * dv; idx += NT) {
        const int r = idx / dv, col = idx - r * dv, gr = rb * 16 + r;
        const int m = q0 + gr / rep, h = c * rep + gr % rep;
        float v = 0.f;
        if (SOFT) {
            float mm = -INFINITY, l = 0.f;
#pragma unroll
            for (int w = 0; w < NW; ++w) mm = fmaxf(mm, stat[w * 16 + r]);
#pragma unroll
            for (int w = 0; w < NW; ++w) {
                const float f = mm > -INFINITY ? expf(stat[w * 16 + r] - mm) : 0.f;
                l = fmaf(f, stat[NW * 16 + w * 16 + r], l);
                v = fmaf(f, red[((size_t)w * 16 + r) * DVP + col], v);
            }
            if (a.shares == 1) {
                v = l > 0.f ? v / l : 0.f;
            } else if (col == 0) {
                a.stats[((long long)share * M + m) * H + h] = mm;
                a.stats[((long long)(a.shares + share) * M + m) * H + h] = l;
            }
        } else {
#pragma unroll
            for (int w = 0; w < NW; ++w) v += red[((size_t)w * 16 + r) * DVP + col];
        }
        if (a.shares == 1) {
            stx(a.out, (long long)m * a.ldo + (long long)h * dv + col, a.of32, v * mix_gate(a, m, h, col));
        } else {
            a.part[((long long)share * M + m) * H * dv + (long long)h * dv + col] = v;
        }
    }
}

template <int NDV, int NS, int MODE>
int launch_mode(const MixArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
    auto kernel = decode_tc_kernel<NDV, NS, MODE>;
    static PerDeviceOnce once;
    if (once.need()) ASD_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    kernel<<<grid, NT, smem, stream>>>(a);
    count_launch(1);
    ASD_CUDA(cudaGetLastError());
    return 0;
}

template <int NDV, int NS>
int launch_ns(const MixArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
    if (a.d.sigmoid) return launch_mode<NDV, NS, D_SIGMOID>(a, grid, smem, stream);
    return a.d.softcap > 0.f ? launch_mode<NDV, NS, D_SOFTMAX_CAP>(a, grid, smem, stream)
                             : launch_mode<NDV, NS, D_SOFTMAX>(a, grid, smem, stream);
}

template <int NDV>
int launch_ndv(const MixArgs& a, dim3 grid, cudaStream_t stream) {
    // ring depth: as deep as two CTAs per SM leave room for
    const int s4 = smem_bytes(a.dkp, NDV * 8, 4), s3 = smem_bytes(a.dkp, NDV * 8, 3), s2 = smem_bytes(a.dkp, NDV * 8, 2);
    if (s4 <= 112 * 1024) return launch_ns<NDV, 4>(a, grid, s4, stream);
    if (s3 <= 112 * 1024) return launch_ns<NDV, 3>(a, grid, s3, stream);
    return launch_ns<NDV, 2>(a, grid, s2, stream);
}

}  // namespace

int launch_attention_decode_tc(MixArgs a, int nseq, int max_qlen, int max_kv_len, const MixWork& ws, cudaStream_t stream) {
    const int H = a.d.heads, G = a.d.kv_heads, rep = H / G, M = a.ix.M, dk = a.d.dk, dv = a.d.dv;
    if (a.cache.f32 || a.dist_bias || a.talk || (a.d.sigmoid && a.d.softcap > 0.f) || dv > 256 || dk % 8 || dv % 8 || nseq > 65535) return 1;
    if (reinterpret_cast<uintptr_t>(a.cache.pool) & 15) return 1;
    const int ndv = dv <= 32 ? 4 : (dv <= 64 ? 8 : (dv <= 96 ? 12 : (dv <= 128 ? 16 : 32)));
    a.dkp = (dk + 15) & ~15, a.dvp = ndv * 8;
    if (smem_bytes(a.dkp, a.dvp, 2) > 200 * 1024) return 1;
    const int keys = a.d.chunk > 0 ? std::min(max_kv_len, a.d.chunk + max_qlen - 1) : max_kv_len;     // at most, of a block
    const int blocks = (max_qlen * rep + 15) / 16, ntile = (keys + KT - 1) / KT;
    const long long base = (long long)nseq * G * blocks;
    if ((long long)G * blocks > 65535) return 1;
    // key shares: a few CTAs for each of the two places an SM has, four tiles per warp at least
    int shares = (int)std::min<long long>((888 + base - 1) / base, std::max(1, ntile / (4 * NW)));
    shares = std::max(1, std::min(shares, 64));
    while (shares > 1 && (!ws.part || (long long)shares * M * H * dv > ws.part_elems ||
                          (!a.d.sigmoid && (long long)2 * shares * M * H > ws.stats_elems)))
        --shares;
    a.shares = shares;
    const dim3 grid(shares, nseq, G * blocks);
    const int rc = ndv == 4    ? launch_ndv<4>(a, grid, stream)
                   : ndv == 8  ? launch_ndv<8>(a, grid, stream)
                   : ndv == 12 ? launch_ndv<12>(a, grid, stream)
                   : ndv == 16 ? launch_ndv<16>(a, grid, stream)
                               : launch_ndv<32>(a, grid, stream);
    if (rc) return -1;
    if (shares > 1 && launch_mix_merge(a, stream, !a.d.sigmoid)) return -1;
    return 0;
}

}  // namespace asd
