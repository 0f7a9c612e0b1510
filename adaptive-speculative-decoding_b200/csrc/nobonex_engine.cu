// Nobonex family forward engine: one opaque handle per model.  asd_nobonex_forward runs, on the caller's stream and with
// no host synchronisation,
//   scaled embedding -> for every layer [ norm, mixer, norm, residual; norm, feed-forward, norm, residual ] -> final norm of
//   the wanted rows, head.
// Every norm is a dynamic tanh (nothing is reduced over a row), so a sublayer's close and the next one's norm are one
// elementwise pass.  A layer's mixer is grouped-query attention over convolved queries and keys that also serve as
// values, a scalar-decay state space recurrence (Mamba-2), or chunked attention with capped scores and an output gate,
// which may read another layer's keys and values.  The feed-forward is a gated layer or routed experts whose weight
// multiplies their input, or absent.  Every step is a building block of blocks.h that takes its sizes from the layer's
// configuration; dense bf16 projections go to the tcgen05 GEMMs when their shape fits.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <string.h>

#include <algorithm>
#include <string>
#include <unordered_map>
#include <vector>

#include "../../include/asd_b200.h"
#include "asd_internal.h"
#include "blocks.h"
#include "dense.h"
#include "prof.h"

struct asd_nobonex_engine {};

namespace asd {

enum NbType { NB_CONV_ATTN = 0, NB_SSD = 1, NB_CHUNK_ATTN = 2 };
enum NbFf { NB_FF_NONE = 0, NB_FF_DENSE = 1, NB_FF_MOE = 2 };

struct NbLayer {
    asd_nobonex_layer_config c;
    std::unordered_map<std::string, const void*> t;   // weights by engine tensor name
    int n_in = 0, ld_in = 0;   // rows of the stacked input projection; floats between its result's rows
    int cache_row = 0;         // cached elements per position (0: none of its own)
    int conv_ch = 0, conv_ring = 0;
    size_t conv_elems = 0;     // carried inputs of the convolution per sequence
    size_t state_elems = 0;    // recurrent state per (sequence, ring entry)
    double* freq = nullptr;    // device: rotation frequencies
    float rot_mag = 1.f;
    size_t cache_off = 0;      // elements from the pool start (a sharing layer: its source's)
    size_t conv_off = 0, state_off = 0;   // floats from the state start
    const void* w(const char* name) const {
        auto it = t.find(name);
        return it == t.end() ? nullptr : it->second;
    }
    const float* f(const char* name) const { return static_cast<const float*>(w(name)); }
};

struct NbEngine : asd_nobonex_engine {
    asd_nobonex_config c;
    std::vector<NbLayer> layers;
    std::unordered_map<std::string, const void*> g;   // global weights
    int f32 = 0, esz = 2, ssd_mode = 0;
    char* pool = nullptr;
    const int* page_table = nullptr;
    int num_pages = 0, max_seqs = 0, max_pages = 0;
    float* state = nullptr;
    // owned activations
    float *x = nullptr, *y = nullptr, *proj = nullptr, *conv = nullptr, *orec = nullptr, *up = nullptr, *eout = nullptr,
          *rlog = nullptr, *rgate = nullptr, *sgate = nullptr;
    void *hn = nullptr, *mixed = nullptr, *act = nullptr, *xsel = nullptr;
    int *expert_of = nullptr, *counters = nullptr, *group_off = nullptr, *sorted_tok = nullptr, *slot_of = nullptr;
    std::vector<void*> owned;
    DenseRunner dn;
    EventProfiler prof;
    MixWork attn_ws;
    int* dev_error = nullptr;
    int device = 0;
    const void* gw(const char* name) const {
        auto it = g.find(name);
        return it == g.end() ? nullptr : it->second;
    }
    const float* gf(const char* name) const { return static_cast<const float*>(gw(name)); }
};

template <typename T>
static int dev_alloc(NbEngine* e, T** p, size_t n) {
    void* q = nullptr;
    ASD_CUDA(cudaMalloc(&q, (n ? n : 1) * sizeof(T)));
    e->owned.push_back(q);
    *p = (T*)q;
    return 0;
}

enum NbProf { NB_DENSE = 0, NB_ATTN, NB_RECUR, NB_EXPERTS, NB_ROUTER, NB_ACT, NB_GLUE, NB_HEAD, NB_NCLASS };
#define NB_PROF(cls) ProfRegion _region(e->prof, cls, s)

static int linear(NbEngine* e, const SimtLinear& L, cudaStream_t s) {
    if (!e->f32 && e->dn.tc_linear && tc_linear_supports(L)) return launch_tc_linear(L, e->dev_error, s);
    return launch_simt_linear(L, s);
}

struct Batch {
    SeqIndex ix;
    const int* cu_q;
    const int* seq_slot;
    int nseq, max_qlen, max_kv_len;
};

static MixDims attn_dims(const asd_nobonex_layer_config& c) {
    MixDims d{c.heads, c.kv_heads, c.dim, c.vdim, c.type == NB_CHUNK_ATTN ? c.chunk : 0, c.scale};
    if (c.type == NB_CHUNK_ATTN) d.softcap = c.softcap, d.gate_per_value = 1;
    return d;
}

// what both attention mixers share: norms, rotation and append of qkv rows (ld floats apart), attention, output projection
static int attend(NbEngine* e, const NbLayer& ly, int li, const Batch& b, float* qkv, long long ld, MixPost p, const float* gate,
                  cudaStream_t s) {
    const asd_nobonex_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width, f32 = e->f32, na = c.heads * c.vdim;
    const MixDims md = attn_dims(c);
    const PagedRows cache{e->pool + ly.cache_off * e->esz, f32, e->page_table, e->max_pages, e->c.page_size};
    p.q_norm = ly.f("q_norm"), p.k_norm = ly.f("k_norm"), p.eps = e->c.eps;
    p.rot_freq = ly.freq, p.rot_dims = c.rot_dims, p.rot_interleaved = c.type == NB_CONV_ATTN, p.rot_mag = ly.rot_mag;
    {
        NB_PROF(NB_GLUE);
        if (launch_mix_post(b.ix, qkv, ld, md, p, cache, s)) return -1;
    }
    {
        NB_PROF(NB_ATTN);
        if (launch_mix_attention(b.ix, b.cu_q, b.seq_slot, b.nseq, b.max_qlen, b.max_kv_len, qkv, ld, md, nullptr, 0, nullptr,
                                 gate, ly.ld_in, cache, e->mixed, f32, na, e->attn_ws, s))
            return -1;
    }
    NB_PROF(NB_DENSE);
    return e->dn.run(e->mixed, ly.w("w_o"), e->y, M, D, na, D, li * 16 + 1, s);
}

// every mixer: hn [M][width] (engine type) -> y
static int mix_conv_attention(NbEngine* e, const NbLayer& ly, int li, const Batch& b, cudaStream_t s) {
    const int M = b.ix.M, D = e->c.width;
    {   // q | k
        NB_PROF(NB_DENSE);
        if (e->dn.run(e->hn, ly.w("w_in"), e->proj, M, ly.n_in, D, ly.ld_in, li * 16 + 0, s)) return -1;
    }
    {
        NB_PROF(NB_GLUE);
        if (launch_carried_conv(b.ix, b.cu_q, b.nseq, b.max_qlen, e->proj, ly.ld_in, ly.f("conv_w"), ly.c.conv, ly.conv_ch,
                                e->state + ly.conv_off, ly.conv_ring, CONV_PLAIN, e->conv, 1, s))
            return -1;
    }
    MixPost p;
    p.norm_whole = 1, p.v_from_k = 1;
    return attend(e, ly, li, b, e->conv, ly.conv_ch, p, nullptr, s);
}

static int mix_chunk_attention(NbEngine* e, const NbLayer& ly, int li, const Batch& b, cudaStream_t s) {
    const asd_nobonex_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width;
    {   // q | k | v | gate, or q | gate beside another layer's keys and values
        NB_PROF(NB_DENSE);
        if (e->dn.run(e->hn, ly.w("w_in"), e->proj, M, ly.n_in, D, ly.ld_in, li * 16 + 0, s)) return -1;
    }
    MixPost p;
    p.bias = ly.f("in_bias"), p.q_only = c.kv_from >= 0;
    return attend(e, ly, li, b, e->proj, ly.ld_in, p, e->proj + ly.n_in - c.heads * c.vdim, s);
}

static int mix_ssd(NbEngine* e, const NbLayer& ly, int li, const Batch& b, cudaStream_t s) {
    const asd_nobonex_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width, inner = c.heads * c.vdim, bc = c.groups * c.state;
    {   // z | x | B | C | dt
        NB_PROF(NB_DENSE);
        if (e->dn.run(e->hn, ly.w("w_in"), e->proj, M, ly.n_in, D, ly.ld_in, li * 16 + 0, s)) return -1;
    }
    {
        NB_PROF(NB_GLUE);
        if (launch_carried_conv(b.ix, b.cu_q, b.nseq, b.max_qlen, e->proj + inner, ly.ld_in, ly.f("conv_w"), c.conv, ly.conv_ch,
                                e->state + ly.conv_off, ly.conv_ring, CONV_SILU, e->conv, e->f32, s, ly.f("conv_b")))
            return -1;
    }
    {
        NB_PROF(NB_RECUR);
        SsdInput in;
        char* cv = reinterpret_cast<char*>(e->conv);
        in.x = cv, in.b = cv + (size_t)inner * e->esz, in.c = cv + (size_t)(inner + bc) * e->esz, in.ld = ly.conv_ch;
        in.bf16 = !e->f32;
        in.dt = e->proj + inner + ly.conv_ch, in.ld_dt = ly.ld_in;
        in.dt_bias = ly.f("dt_bias"), in.a_log = ly.f("a_log"), in.skip = ly.f("skip");
        if (launch_ssd_recurrence(b.ix, b.cu_q, b.seq_slot, b.nseq, b.max_qlen, in, SsdDims{c.heads, c.groups, c.state, c.vdim},
                                  e->state + ly.state_off, e->c.ring, e->orec, e->ssd_mode, s))
            return -1;
    }
    {
        NB_PROF(NB_GLUE);
        HeadNormGate ng;
        ng.gate = e->proj, ng.ldg = ly.ld_in, ng.w = ly.f("out_norm"), ng.w_per_head = 1, ng.gate_act = 2, ng.gate_first = 1;
        ng.eps = e->c.eps;
        if (launch_head_norm_gate(e->orec, ng, e->mixed, e->f32, inner, M, c.norm_groups, inner / c.norm_groups, s)) return -1;
    }
    NB_PROF(NB_DENSE);
    return e->dn.run(e->mixed, ly.w("w_o"), e->y, M, D, inner, D, li * 16 + 1, s);
}

// feed-forward of hn; its result is added by the close
static int feed_forward(NbEngine* e, const NbLayer& ly, int li, const Batch& b, TanhClose& C, cudaStream_t s) {
    const asd_nobonex_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width, f32 = e->f32;
    if (c.ff_kind == NB_FF_DENSE) {
        {
            NB_PROF(NB_DENSE);
            if (e->dn.run(e->hn, ly.w("w_gu"), e->up, M, 2 * c.ff, D, 2 * c.ff, li * 16 + 3, s)) return -1;
        }
        {
            NB_PROF(NB_ACT);
            if (launch_gated_act(e->up, e->act, f32, M, c.ff, GatedAct(), s)) return -1;
        }
        NB_PROF(NB_DENSE);
        C.y = e->y;
        return e->dn.run(e->act, ly.w("w_down"), e->y, M, D, c.ff, D, li * 16 + 4, s);
    }
    {   // router logits in fp32 on the CUDA cores in both modes
        NB_PROF(NB_ROUTER);
        MoeRouterInput in{e->hn, f32, ly.w("router"), 1, D, e->rlog};
        in.sigmoid = 1, in.plain_scores = 1, in.slot_gate = e->sgate;
        if (launch_moe_route(nullptr, &in, M, c.experts, c.top, e->expert_of, e->rgate, e->counters, e->group_off,
                             e->sorted_tok, e->slot_of, s))
            return -1;
    }
    {
        NB_PROF(NB_EXPERTS);
        SimtLinear U;   // gate | up of every chosen (token, expert) pair
        U.a = e->hn, U.a_f32 = f32, U.lda = D;
        U.w = ly.w("w_egu"), U.w_f32 = f32, U.ldw = D, U.w_zs = (long long)2 * c.expert_ff * D;
        U.c = e->up, U.c_f32 = 1, U.ldc = 2 * c.expert_ff;
        U.M = M, U.N = 2 * c.expert_ff, U.K = D, U.Z = c.experts;
        U.group_off = e->group_off, U.gather = e->sorted_tok;
        if (linear(e, U, s)) return -1;
    }
    {   // the weight of an expert's input goes through its bias-free products: it multiplies their results
        NB_PROF(NB_ACT);
        GatedAct ga;
        ga.kind = GATED_CLAMPED, ga.limit = c.limit, ga.row_factor = e->sgate;
        if (launch_gated_act(e->up, e->act, f32, (long long)M * c.top, c.expert_ff, ga, s)) return -1;
    }
    {
        NB_PROF(NB_EXPERTS);
        SimtLinear W;
        W.a = e->act, W.a_f32 = f32, W.lda = c.expert_ff;
        W.w = ly.w("w_edown"), W.w_f32 = f32, W.ldw = c.expert_ff, W.w_zs = (long long)D * c.expert_ff;
        W.c = e->eout, W.c_f32 = 1, W.ldc = D;
        W.M = M, W.N = D, W.K = c.expert_ff, W.Z = c.experts;
        W.group_off = e->group_off;
        if (linear(e, W, s)) return -1;
    }
    C.expert_out = e->eout, C.slot_of = e->slot_of, C.top = c.top;
    return 0;
}

static TanhNorm norm_of(const NbLayer& ly, const char* w, const char* b, const char* alpha) {
    return TanhNorm{ly.f(w), ly.f(b), ly.f(alpha)};
}

static int forward(NbEngine* e, const Batch& b, const int* logit_rows, int n_rows, float* logits, long long ld,
                   float* layer_out, cudaStream_t s) {
    const int D = e->c.width, M = b.ix.M, f32 = e->f32;
    const int L = (int)e->layers.size();
    auto base_close = [&]() {
        TanhClose C;
        C.x_in = e->x, C.x_out = e->x, C.mult = e->c.residual_mult, C.M = M, C.D = D;
        return C;
    };
    auto open_next = [&](int l, TanhClose& C) {   // hn: what layer l's mixer reads
        if (l < L) C.next = norm_of(e->layers[l], "norm1", "norm1_b", "norm1_alpha"), C.hn = e->hn, C.hn_f32 = f32;
    };
    {
        NB_PROF(NB_GLUE);
        if (launch_embed_scaled(b.ix, e->gw("embed"), f32, e->c.embed_scale, e->x, nullptr, D, s)) return -1;
        if (L) {
            TanhClose C = base_close();
            open_next(0, C);
            if (launch_tanh_close(C, s)) return -1;
        }
    }
    for (int l = 0; l < L; ++l) {
        const NbLayer& ly = e->layers[l];
        if (ly.c.type == NB_CONV_ATTN ? mix_conv_attention(e, ly, l, b, s)
                                      : (ly.c.type == NB_SSD ? mix_ssd(e, ly, l, b, s) : mix_chunk_attention(e, ly, l, b, s)))
            return -1;
        {   // x += mult * norm1b(mixer); then what the feed-forward (or the next layer) reads
            NB_PROF(NB_GLUE);
            TanhClose C = base_close();
            C.y = e->y, C.post = norm_of(ly, "norm1b", "norm1b_b", "norm1b_alpha");
            if (ly.c.ff_kind != NB_FF_NONE)
                C.next = norm_of(ly, "norm2", "norm2_b", "norm2_alpha"), C.hn = e->hn, C.hn_f32 = f32;
            else
                open_next(l + 1, C);
            if (launch_tanh_close(C, s)) return -1;
        }
        if (ly.c.ff_kind != NB_FF_NONE) {
            TanhClose C = base_close();
            if (feed_forward(e, ly, l, b, C, s)) return -1;
            NB_PROF(NB_GLUE);
            C.post = norm_of(ly, "norm2b", "norm2b_b", "norm2b_alpha");
            open_next(l + 1, C);
            if (launch_tanh_close(C, s)) return -1;
        }
        if (layer_out)
            ASD_CUDA(cudaMemcpyAsync(layer_out + (size_t)l * M * D, e->x, sizeof(float) * M * D, cudaMemcpyDeviceToDevice, s));
    }
    if (n_rows > 0) {
        NB_PROF(NB_HEAD);
        TanhClose C = base_close();
        C.x_out = nullptr, C.rows = logit_rows, C.hn = e->xsel, C.hn_f32 = f32, C.M = n_rows;
        C.next = TanhNorm{e->gf("final_norm"), e->gf("final_norm_b"), e->gf("final_norm_alpha")};
        if (launch_tanh_close(C, s)) return -1;
        const int V = e->c.vocab;
        if (e->dn.run(e->xsel, e->gw("head"), logits, n_rows, V, D, ld ? (int)ld : V, L * 16 + 2, s)) return -1;
    }
    return 0;
}

// elements one layer's rows take in the pool, rounded up so that every layer starts on a 16-byte boundary
static size_t pool_elems(const NbEngine* e, const NbLayer& ly, int num_pages) {
    const size_t n = (size_t)num_pages * e->c.page_size * ly.cache_row;
    return (n + 7) & ~(size_t)7;
}

// the parts of one layer's carried state, floats per sequence slot count; every part starts on a 16-byte boundary
static size_t up4(size_t n) { return (n + 3) & ~(size_t)3; }
static size_t conv_floats(const NbLayer& ly, int max_seqs) { return up4((size_t)max_seqs * ly.conv_elems); }
static size_t state_floats(const NbEngine* e, const NbLayer& ly, int max_seqs) {
    return up4((size_t)max_seqs * e->c.ring * ly.state_elems);
}

static const char* const kLayerNames[] = {
    "norm1", "norm1_b", "norm1_alpha", "norm1b", "norm1b_b", "norm1b_alpha", "norm2", "norm2_b", "norm2_alpha", "norm2b",
    "norm2b_b", "norm2b_alpha", "w_in", "w_o", "in_bias", "q_norm", "k_norm", "conv_w", "conv_b", "a_log", "dt_bias", "skip",
    "out_norm", "w_gu", "w_down", "router", "w_egu", "w_edown"};
static const char* const kGlobalNames[] = {"embed", "final_norm", "final_norm_b", "final_norm_alpha", "head"};

static std::vector<const char*> required(const NbLayer& ly) {
    std::vector<const char*> n = {"norm1", "norm1_b", "norm1_alpha", "norm1b", "norm1b_b", "norm1b_alpha", "w_in", "w_o"};
    if (ly.c.type == NB_CONV_ATTN)
        n.insert(n.end(), {"q_norm", "k_norm", "conv_w"});
    else if (ly.c.type == NB_SSD)
        n.insert(n.end(), {"conv_w", "conv_b", "a_log", "dt_bias", "skip", "out_norm"});
    else
        n.insert(n.end(), {"in_bias", "q_norm"});
    if (ly.c.type == NB_CHUNK_ATTN && ly.c.kv_from < 0) n.push_back("k_norm");
    if (ly.c.ff_kind != NB_FF_NONE)
        n.insert(n.end(), {"norm2", "norm2_b", "norm2_alpha", "norm2b", "norm2b_b", "norm2b_alpha"});
    if (ly.c.ff_kind == NB_FF_DENSE) n.insert(n.end(), {"w_gu", "w_down"});
    if (ly.c.ff_kind == NB_FF_MOE) n.insert(n.end(), {"router", "w_egu", "w_edown"});
    return n;
}

// Rotation frequencies base^(-2i/dims); with YaRN scaling (factor > 0) the pairs that turn fast over the original length keep
// theirs, the slow ones are divided by the factor, a linear ramp over the pair index in between, and cos and sin grow by
// 0.1 ln(factor) + 1.
static std::vector<double> rotation(const asd_nobonex_layer_config& c, float* mag) {
    const int n = c.rot_dims;
    std::vector<double> f(n / 2);
    for (int i = 0; i < n / 2; ++i) f[i] = pow(c.rot_base, -2.0 * i / n);
    *mag = 1.f;
    if (c.yarn_factor > 0.0) {
        auto pair_of = [&](double turns) {
            return n * log(c.yarn_original / (2.0 * 3.14159265358979323846 * turns)) / (2.0 * log(c.rot_base));
        };
        const double lo = std::max(floor(pair_of(c.yarn_fast)), 0.0), hi = std::min(ceil(pair_of(c.yarn_slow)), n - 1.0);
        for (int i = 0; i < n / 2; ++i) {
            const double r = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f[i] = f[i] / c.yarn_factor * r + f[i] * (1.0 - r);
        }
        *mag = (float)(0.1 * log(c.yarn_factor) + 1.0);
    }
    return f;
}

}  // namespace asd

using namespace asd;

extern "C" {

asd_nobonex_engine_t* asd_nobonex_create(const asd_nobonex_config* cfg, const asd_nobonex_layer_config* layers) {
    if (!cfg || (cfg->n_layers > 0 && !layers)) {
        set_error("asd_nobonex_create: NULL config");
        return nullptr;
    }
    if (cfg->width <= 0 || cfg->vocab <= 0 || cfg->n_layers < 0 || cfg->max_tokens <= 0 || cfg->page_size <= 0 ||
        cfg->ring <= 0 || (cfg->dtype != 0 && cfg->dtype != 1)) {
        set_error("asd_nobonex_create: bad sizes");
        return nullptr;
    }
    NbEngine* e = new NbEngine();
    e->c = *cfg;
    e->f32 = e->dn.f32 = cfg->dtype;
    e->esz = cfg->dtype ? 4 : 2;
    cudaGetDevice(&e->device);
    const size_t MT = cfg->max_tokens, D = cfg->width;
    size_t ld_in = 4, conv = 1, inner = 1, mixw = 1, attn_heads = 0, upw = 1, actw = 1, E = 1, top = 1;
    auto fail = [&](const char* what, int l) {
        set_error("asd_nobonex_create: %s (layer %d)", what, l);
        asd_nobonex_destroy(e);
        return nullptr;
    };
    for (int l = 0; l < cfg->n_layers; ++l) {
        NbLayer ly;
        ly.c = layers[l];
        auto& c = ly.c;
        if (c.type == NB_SSD) {
            if (c.heads <= 0 || c.vdim <= 0 || c.state <= 0 || c.state > 1024 || c.groups <= 0 || c.heads % c.groups ||
                c.norm_groups <= 0 || (c.heads * c.vdim) % c.norm_groups || c.conv <= 0)
                return fail("bad state space sizes", l);
            const int in = c.heads * c.vdim;
            ly.conv_ch = in + 2 * c.groups * c.state;
            ly.n_in = in + ly.conv_ch + c.heads;
            ly.state_elems = (size_t)c.heads * c.state * c.vdim;
            inner = std::max(inner, (size_t)in);
            mixw = std::max(mixw, (size_t)in);
        } else if (c.type == NB_CONV_ATTN || c.type == NB_CHUNK_ATTN) {
            if (mix_attention_check(attn_dims(c), 0)) {
                asd_nobonex_destroy(e);
                return nullptr;
            }
            if (c.rot_dims < 0 || c.rot_dims % 2 || c.rot_dims > c.dim || (c.rot_dims > 0 && !(c.rot_base > 0.0)))
                return fail("bad rotation", l);
            if (c.yarn_factor > 0.0 && !(c.yarn_original > 0.0 && c.yarn_fast > 0.0 && c.yarn_slow > 0.0 && c.rot_base != 1.0))
                return fail("bad rotation scaling", l);
            const int nq = c.heads * c.dim, nk = c.kv_heads * c.dim, nv = c.kv_heads * c.vdim;
            if (c.type == NB_CONV_ATTN) {
                if (c.vdim != c.dim || c.conv <= 0 || c.kv_from >= 0) return fail("bad convolved attention", l);
                ly.n_in = ly.conv_ch = nq + nk;
            } else {
                if (c.kv_from >= 0) {
                    if (c.kv_from >= l || layers[c.kv_from].type != NB_CHUNK_ATTN || layers[c.kv_from].kv_from >= 0 ||
                        layers[c.kv_from].kv_heads != c.kv_heads || layers[c.kv_from].dim != c.dim ||
                        layers[c.kv_from].vdim != c.vdim)
                        return fail("kv_from names no earlier layer with keys and values of these sizes", l);
                } else if (c.kv_from < -1) {
                    return fail("bad kv_from", l);
                }
                ly.n_in = nq + (c.kv_from < 0 ? nk + nv : 0) + c.heads * c.vdim;
            }
            if (c.kv_from < 0) ly.cache_row = nk + nv;
            attn_heads = std::max(attn_heads, (size_t)c.heads);
            mixw = std::max(mixw, (size_t)c.heads * c.vdim);
        } else {
            return fail("unknown mixer type", l);
        }
        if (ly.conv_ch > 0) {
            // inputs of the last taps - 1 positions, for each of the `ring` positions a forward may start after
            ly.conv_ring = c.conv > 1 ? c.conv - 1 + cfg->ring - 1 : 0;
            ly.conv_elems = (size_t)ly.conv_ring * ly.conv_ch;
            conv = std::max(conv, (size_t)ly.conv_ch);
        }
        if (c.ff_kind == NB_FF_DENSE) {
            if (c.ff <= 0) return fail("bad feed-forward size", l);
            upw = std::max(upw, (size_t)2 * c.ff);
            actw = std::max(actw, (size_t)c.ff);
        } else if (c.ff_kind == NB_FF_MOE) {
            if (c.experts <= 0 || c.expert_ff <= 0 || c.top <= 0 || c.top > c.experts || !(c.limit > 0.f))
                return fail("bad expert sizes", l);
            upw = std::max(upw, (size_t)c.top * 2 * c.expert_ff);
            actw = std::max(actw, (size_t)c.top * c.expert_ff);
            E = std::max(E, (size_t)c.experts);
            top = std::max(top, (size_t)c.top);
        } else if (c.ff_kind != NB_FF_NONE) {
            return fail("unknown feed-forward kind", l);
        }
        ly.ld_in = (ly.n_in + 3) & ~3;
        ld_in = std::max(ld_in, (size_t)ly.ld_in);
        e->layers.push_back(ly);
    }
    int rc = 0;
    for (NbLayer& ly : e->layers) {
        if (ly.c.type == NB_SSD || ly.c.rot_dims == 0) continue;
        const std::vector<double> f = rotation(ly.c, &ly.rot_mag);
        rc |= dev_alloc(e, &ly.freq, f.size());
        if (!rc && cudaMemcpy(ly.freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice) != cudaSuccess) rc = -1;
    }
    rc |= dev_alloc(e, &e->x, MT * D);
    rc |= dev_alloc(e, &e->y, MT * D);
    rc |= dev_alloc(e, &e->proj, MT * ld_in);
    rc |= dev_alloc(e, &e->conv, MT * conv);
    rc |= dev_alloc(e, &e->orec, MT * inner);
    rc |= dev_alloc(e, &e->up, MT * upw);
    rc |= dev_alloc(e, &e->eout, MT * top * D);
    rc |= dev_alloc(e, &e->rlog, MT * E);
    rc |= dev_alloc(e, &e->rgate, MT * top);
    rc |= dev_alloc(e, &e->sgate, MT * top);
    rc |= dev_alloc(e, (char**)&e->hn, MT * D * e->esz);
    rc |= dev_alloc(e, (char**)&e->mixed, MT * mixw * e->esz);
    rc |= dev_alloc(e, (char**)&e->act, MT * actw * e->esz);
    rc |= dev_alloc(e, (char**)&e->xsel, MT * D * e->esz);
    rc |= dev_alloc(e, &e->expert_of, MT * top);
    rc |= dev_alloc(e, &e->counters, 2 * E + 1);
    rc |= dev_alloc(e, &e->group_off, E + 1);
    rc |= dev_alloc(e, &e->sorted_tok, MT * top);
    rc |= dev_alloc(e, &e->slot_of, MT * top);
    if (attn_heads) {   // statistics of a pass over the keys, and of key shares with their partial results (few tokens)
        const size_t rows = std::max<size_t>(MT, 2048);
        e->attn_ws.stats_elems = (long long)(2 * rows * attn_heads);
        rc |= dev_alloc(e, &e->attn_ws.stats, (size_t)e->attn_ws.stats_elems);
        e->attn_ws.part_elems = (long long)(2048 * mixw);
        rc |= dev_alloc(e, &e->attn_ws.part, (size_t)e->attn_ws.part_elems);
        e->attn_ws.score_elems = 4ll << 20;      // scores of single-token steps that stay on the CUDA cores
        rc |= dev_alloc(e, &e->attn_ws.scores, (size_t)e->attn_ws.score_elems);
    }
    rc |= dev_alloc(e, &e->dev_error, 1);
    if (!rc && cudaMemset(e->dev_error, 0, sizeof(int)) != cudaSuccess) rc = -1;
    if (rc) {
        asd_nobonex_destroy(e);
        return nullptr;
    }
    return e;
}

void asd_nobonex_destroy(asd_nobonex_engine_t* h) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e) return;
    for (void* p : e->owned) cudaFree(p);
    delete e;
}

int asd_nobonex_set_tensor(asd_nobonex_engine_t* h, int layer, const char* name, const void* data) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e || !name || !data) return set_error("asd_nobonex_set_tensor: NULL argument");
    if (layer >= (int)e->layers.size() || layer < -1) return set_error("asd_nobonex_set_tensor: bad layer %d", layer);
    bool known = false;
    if (layer < 0) {
        for (const char* n : kGlobalNames) known |= !strcmp(n, name);
        if (known) e->g[name] = data;
    } else {
        for (const char* n : kLayerNames) known |= !strcmp(n, name);
        if (known) e->layers[layer].t[name] = data;
    }
    if (!known) return set_error("asd_nobonex_set_tensor: unknown tensor %s (layer %d)", name, layer);
    e->dn.clear();
    return 0;
}

size_t asd_nobonex_cache_bytes(const asd_nobonex_engine_t* h, int num_pages) {
    const NbEngine* e = static_cast<const NbEngine*>(h);
    if (!e) return 0;
    size_t n = 0;
    for (const NbLayer& ly : e->layers) n += pool_elems(e, ly, num_pages);
    return n * e->esz;
}

size_t asd_nobonex_state_bytes(const asd_nobonex_engine_t* h, int max_seqs) {
    const NbEngine* e = static_cast<const NbEngine*>(h);
    if (!e) return 0;
    size_t n = 0;
    for (const NbLayer& ly : e->layers) n += conv_floats(ly, max_seqs) + state_floats(e, ly, max_seqs);
    return n * sizeof(float);
}

int asd_nobonex_set_cache(asd_nobonex_engine_t* h, void* pool, int num_pages, const int32_t* page_table, int max_seqs,
                          int max_pages_per_seq, float* state) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e || !pool || !page_table || !state || num_pages <= 0 || max_seqs <= 0 || max_pages_per_seq <= 0)
        return set_error("asd_nobonex_set_cache: bad arguments");
    e->pool = static_cast<char*>(pool);
    e->num_pages = num_pages, e->page_table = page_table, e->max_seqs = max_seqs, e->max_pages = max_pages_per_seq;
    e->state = state;
    size_t off = 0, soff = 0;
    for (NbLayer& ly : e->layers) {
        ly.cache_off = off;
        off += pool_elems(e, ly, num_pages);
        ly.conv_off = soff;
        soff += conv_floats(ly, max_seqs);
        ly.state_off = soff;
        soff += state_floats(e, ly, max_seqs);
    }
    for (NbLayer& ly : e->layers)
        if (ly.c.type == NB_CHUNK_ATTN && ly.c.kv_from >= 0) ly.cache_off = e->layers[ly.c.kv_from].cache_off;
    return 0;
}

int asd_nobonex_set_option(asd_nobonex_engine_t* h, const char* name, int value) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e || !name) return set_error("asd_nobonex_set_option: NULL argument");
    if (!strcmp(name, "tc_linear")) {
        e->dn.tc_linear = value;
        return 0;
    }
    if (!strcmp(name, "tc_min_rows")) {
        e->dn.tc_min_rows = value > 0 ? value : 1 << 30;
        e->dn.clear();
        return 0;
    }
    if (!strcmp(name, "attn_general")) {
        e->attn_ws.mode = value;
        return 0;
    }
    if (!strcmp(name, "ssd_mode")) {
        e->ssd_mode = value;
        return 0;
    }
    if (!strcmp(name, "profile")) {
        e->prof.on = value;
        e->prof.reset();
        return 0;
    }
    return set_error("asd_nobonex_set_option: unknown option %s", name);
}

int asd_nobonex_forward(asd_nobonex_engine_t* h, const int32_t* tokens, const int32_t* positions,
                        const int32_t* token_slot, int M, const int32_t* cu_q, const int32_t* seq_slot, int nseq,
                        int max_qlen, int max_kv_len, const int32_t* logit_rows, int n_logit_rows, float* logits_out,
                        long long logits_ld, float* layer_out, void* stream) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e) return set_error("asd_nobonex_forward: NULL engine");
    if (M <= 0 || M > e->c.max_tokens) return set_error("asd_nobonex_forward: M = %d outside 1..%d", M, e->c.max_tokens);
    if (!e->pool) return set_error("asd_nobonex_forward: cache not set");
    for (const char* n : kGlobalNames)
        if (!e->gw(n)) return set_error("asd_nobonex_forward: tensor %s not set", n);
    for (size_t l = 0; l < e->layers.size(); ++l)
        for (const char* n : required(e->layers[l]))
            if (!e->layers[l].w(n)) return set_error("asd_nobonex_forward: layer %d has no tensor %s", (int)l, n);
    if (!tokens || !positions || !token_slot || !cu_q || !seq_slot || nseq <= 0 || max_qlen <= 0)
        return set_error("asd_nobonex_forward: bad index arguments");
    if (max_kv_len > e->max_pages * e->c.page_size)
        return set_error("asd_nobonex_forward: length bound %d exceeds the page table", max_kv_len);
    if (n_logit_rows > 0 && !logits_out) return set_error("asd_nobonex_forward: logits_out is NULL");
    if (n_logit_rows > e->c.max_tokens) return set_error("asd_nobonex_forward: too many logit rows");
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev != e->device) return set_error("asd_nobonex_forward: called on device %d, engine lives on %d", dev, e->device);
    const Batch b{SeqIndex{tokens, positions, token_slot, M}, cu_q, seq_slot, nseq, max_qlen, max_kv_len};
    return forward(e, b, logit_rows, logit_rows ? n_logit_rows : (n_logit_rows > 0 ? M : 0), logits_out, logits_ld,
                   layer_out, static_cast<cudaStream_t>(stream));
}

int asd_nobonex_profile_read(asd_nobonex_engine_t* h, float* ms_by_class, int* launches_by_class, int nclass) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e || !ms_by_class || nclass < NB_NCLASS) return set_error("asd_nobonex_profile_read: bad argument");
    ASD_CUDA(e->prof.read(ms_by_class, launches_by_class, nclass));
    return 0;
}

int asd_nobonex_device_error(asd_nobonex_engine_t* h) {
    NbEngine* e = static_cast<NbEngine*>(h);
    if (!e) return set_error("asd_nobonex_device_error: NULL engine");
    int v = 0;
    ASD_CUDA(cudaMemcpy(&v, e->dev_error, sizeof(int), cudaMemcpyDeviceToHost));
    if (v) return set_error("a Nobonex kernel gave up a bounded wait (tcgen05 linear)");
    return 0;
}

}  // extern "C"
