// Dikopel family forward engine: one opaque handle per model.  asd_dikopel_forward runs, on the caller's stream and with
// no host synchronisation,
//   scaled embedding + sinusoids of the position -> for every layer [ layer norm, input convolution of what the mixer
//   reads, mixer and feed-forward side by side, residual ] -> final layer norm of the wanted rows, head.
// A layer's mixer is either a matrix memory with exponential gates ("mlstm"), or two mixers on the same input
// ("parallel"): grouped-query attention with sigmoid weights and the gated delta rule with one decay per head, whose
// results are RMS-normed each and averaged.  The feed-forward is a gated layer or routed gated experts (sigmoid scores,
// choice within the best groups of experts) plus a shared one behind a gate of its own, or absent.  A layer may use
// another layer's weights; every layer has a cache or state of its own.  Every step is a building block of blocks.h that
// takes its sizes from the layer's configuration; dense bf16 projections go to the tcgen05 GEMMs when their shape fits.
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

struct asd_dikopel_engine {};

namespace asd {

enum DkType { DK_MLSTM = 0, DK_PARALLEL = 1 };
enum DkFf { DK_FF_NONE = 0, DK_FF_DENSE = 1, DK_FF_MOE = 2 };

struct DkLayer {
    asd_dikopel_layer_config c;
    std::unordered_map<std::string, const void*> t;   // weights by engine tensor name
    int n_in = 0, ld_in = 0;   // rows of the stacked input projection; floats between its result's rows
    int cache_row = 0;         // cached elements per position (0: none)
    int conv_ch = 0, conv_ring = 0;
    size_t conv_elems = 0;     // carried inputs of the mixer's convolutions per sequence
    size_t state_elems = 0;    // recurrent state per (sequence, ring entry)
    const void* w(const char* name) const {
        auto it = t.find(name);
        return it == t.end() ? nullptr : it->second;
    }
    const float* f(const char* name) const { return static_cast<const float*>(w(name)); }
};

struct DkRun {
    int layer;                 // the layer whose weights (and sizes) this execution uses
    size_t cache_off = 0;      // elements from the pool start
    size_t input_off = 0;      // floats from the state start: carried inputs of the layer's own convolution
    size_t conv_off = 0;
    size_t state_off = 0;
};

struct DkEngine : asd_dikopel_engine {
    asd_dikopel_config c;
    std::vector<DkLayer> layers;
    std::vector<DkRun> runs;   // one per layer
    std::unordered_map<std::string, const void*> g;   // global weights
    int f32 = 0, esz = 2;
    char* pool = nullptr;
    const int* page_table = nullptr;
    int num_pages = 0, max_seqs = 0, max_pages = 0;
    float* state = nullptr;
    int input_ring = 0;        // carried rows of the input convolution per sequence
    // owned activations
    double* freq = nullptr;
    float *x = nullptr, *hf = nullptr, *y = nullptr, *y2 = nullptr, *yf = nullptr, *proj = nullptr, *conv = nullptr,
          *rv = nullptr, *sc = nullptr, *orec = nullptr, *up = nullptr, *eout = nullptr, *rlog = nullptr, *rgate = nullptr;
    void *hn = nullptr, *hc = nullptr, *mixed = nullptr, *mixed2 = nullptr, *act = nullptr, *xsel = nullptr;
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
static int dev_alloc(DkEngine* e, T** p, size_t n) {
    void* q = nullptr;
    ASD_CUDA(cudaMalloc(&q, (n ? n : 1) * sizeof(T)));
    e->owned.push_back(q);
    *p = (T*)q;
    return 0;
}

enum DkProf { DK_DENSE = 0, DK_ATTN, DK_RECUR, DK_EXPERTS, DK_ROUTER, DK_ACT, DK_GLUE, DK_HEAD, DK_NCLASS };
#define DK_PROF(cls) ProfRegion _region(e->prof, cls, s)

static int linear(DkEngine* e, const SimtLinear& L, cudaStream_t s) {
    if (!e->f32 && e->dn.tc_linear && tc_linear_supports(L)) return launch_tc_linear(L, e->dev_error, s);
    return launch_simt_linear(L, s);
}

struct Batch {
    SeqIndex ix;
    const int* cu_q;
    const int* seq_slot;
    int nseq, max_qlen, max_kv_len;
};

static MlstmDims mlstm_dims(const asd_dikopel_layer_config& c) {
    return MlstmDims{c.heads, c.dim, c.vdim, c.gate_cap, 1.f / sqrtf((float)c.dim)};
}

// mixer input hc [M][D] (engine type) -> y (the close reads it as it is)
static int mix_mlstm(DkEngine* e, const DkLayer& ly, const DkRun& run, int li, const Batch& b, cudaStream_t s) {
    const asd_dikopel_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width;
    const int nk = c.heads * c.dim, nv = c.heads * c.vdim;
    {   // q | k | v | output gate | input gate | forget gate in one projection
        DK_PROF(DK_DENSE);
        if (e->dn.run(e->hc, ly.w("w_in"), e->proj, M, ly.n_in, D, ly.ld_in, li * 16 + 0, s)) return -1;
    }
    {
        DK_PROF(DK_RECUR);
        MlstmInput in;
        in.q = e->proj, in.k = e->proj + nk, in.v = e->proj + 2 * nk, in.zi = e->proj + 2 * (nk + nv), in.zf = in.zi + c.heads;
        in.ld = ly.ld_in, in.bias_i = ly.f("i_bias"), in.bias_f = ly.f("f_bias");
        if (launch_mlstm_recurrence(b.ix, b.cu_q, b.seq_slot, b.nseq, b.max_qlen, in, mlstm_dims(c),
                                    e->state + run.state_off, e->c.ring, e->orec, s))
            return -1;
    }
    {
        DK_PROF(DK_GLUE);
        HeadNormGate ng;
        ng.gate = e->proj + 2 * nk + nv, ng.ldg = ly.ld_in, ng.w = ly.f("out_norm"), ng.w_per_head = 1, ng.gate_act = 1;
        ng.eps = e->c.eps;
        if (launch_head_norm_gate(e->orec, ng, e->mixed, e->f32, nv, M, c.heads, c.vdim, s)) return -1;
    }
    DK_PROF(DK_DENSE);
    return e->dn.run(e->mixed, ly.w("w_o"), e->y, M, D, nv, D, li * 16 + 1, s);
}

// -> y (left) and y2 (right); the close norms and averages them
static int mix_parallel(DkEngine* e, const DkLayer& ly, const DkRun& run, int li, const Batch& b, cudaStream_t s) {
    const asd_dikopel_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width, f32 = e->f32;
    const int nl = c.a_heads * c.a_dim + c.a_kv_heads * (c.a_dim + c.a_vdim), na = c.a_heads * c.a_vdim;
    const int nk = c.r_kv_heads * c.r_dim, nv = c.r_heads * c.r_vdim;
    {   // left q | k | v, right q | k | v | gate | beta | decay in one projection
        DK_PROF(DK_DENSE);
        if (e->dn.run(e->hc, ly.w("w_in"), e->proj, M, ly.n_in, D, ly.ld_in, li * 16 + 0, s)) return -1;
    }
    MixDims md{c.a_heads, c.a_kv_heads, c.a_dim, c.a_vdim, 0, c.scale};
    md.sigmoid = 1, md.head_bias = ly.f("head_bias");
    const PagedRows cache{e->pool + run.cache_off * e->esz, f32, e->page_table, e->max_pages, e->c.page_size};
    {
        DK_PROF(DK_GLUE);
        if (launch_mix_post(b.ix, e->proj, ly.ld_in, md, MixPost(), cache, s)) return -1;
    }
    {
        DK_PROF(DK_ATTN);
        if (launch_mix_attention(b.ix, b.cu_q, b.seq_slot, b.nseq, b.max_qlen, b.max_kv_len, e->proj, ly.ld_in, md, nullptr, 0,
                                 nullptr, nullptr, 0, cache, e->mixed, f32, na, e->attn_ws, s))
            return -1;
    }
    {
        DK_PROF(DK_DENSE);
        if (e->dn.run(e->mixed, ly.w("w_o"), e->y, M, D, na, D, li * 16 + 1, s)) return -1;
    }
    float* r = e->proj + nl;
    {
        DK_PROF(DK_GLUE);
        if (launch_carried_conv(b.ix, b.cu_q, b.nseq, b.max_qlen, r, ly.ld_in, ly.f("conv_w"), c.conv, ly.conv_ch,
                                e->state + run.conv_off, ly.conv_ring, 0, e->conv, 1, s))
            return -1;
        DeltaPrep dp;
        dp.q = e->conv, dp.k = e->conv + nk, dp.ld = ly.conv_ch, dp.rv = e->rv, dp.sc = e->sc;
        dp.heads = c.r_heads, dp.kv_heads = c.r_kv_heads, dp.dk = c.r_dim, dp.general = 2;
        dp.q_scale = 1.f / sqrtf((float)c.r_dim);
        dp.beta = r + ly.conv_ch + nv, dp.ld_beta = ly.ld_in;
        dp.rate = dp.beta + c.r_heads, dp.ld_rate = ly.ld_in, dp.rate_bias = ly.f("dt_bias"), dp.head_log_rate = ly.f("a_log");
        if (launch_delta_prep(dp, M, s)) return -1;
    }
    {
        DK_PROF(DK_RECUR);
        if (launch_delta_recurrence(b.ix, b.cu_q, b.seq_slot, b.nseq, e->rv, e->sc, 2, e->conv + 2 * nk, ly.conv_ch, c.r_heads,
                                    c.r_dim, c.r_vdim, e->state + run.state_off, e->c.ring, e->orec, s))
            return -1;
    }
    {
        DK_PROF(DK_GLUE);
        HeadNormGate ng;
        ng.gate = r + ly.conv_ch, ng.ldg = ly.ld_in, ng.w = ly.f("out_norm"), ng.gate_act = 2, ng.eps = e->c.eps;
        if (launch_head_norm_gate(e->orec, ng, e->mixed2, f32, nv, M, c.r_heads, c.r_vdim, s)) return -1;
    }
    DK_PROF(DK_DENSE);
    return e->dn.run(e->mixed2, ly.w("w_o2"), e->y2, M, D, nv, D, li * 16 + 2, s);
}

// feed-forward of hn (the layer's normed input before its convolution); its result is added by the close
static int feed_forward(DkEngine* e, const DkLayer& ly, int li, const Batch& b, RowClose& C, cudaStream_t s) {
    const asd_dikopel_layer_config& c = ly.c;
    const int M = b.ix.M, D = e->c.width, f32 = e->f32;
    auto gated = [&](const char* gu, const char* down, int F, int key) {   // W_down (silu(W_gate h) * W_up h) -> yf
        {
            DK_PROF(DK_DENSE);
            if (e->dn.run(e->hn, ly.w(gu), e->up, M, 2 * F, D, 2 * F, li * 16 + key, s)) return -1;
        }
        {
            DK_PROF(DK_ACT);
            if (launch_ff_act(e->up, e->act, f32, M, F, 1, s)) return -1;
        }
        DK_PROF(DK_DENSE);
        return e->dn.run(e->act, ly.w(down), e->yf, M, D, F, D, li * 16 + key + 1, s);
    };
    if (c.ff_kind == DK_FF_DENSE) {
        C.ff = e->yf;
        return gated("w_gu", "w_down", c.ff, 3);
    }
    const int zld = c.experts + (c.shared_ff > 0 ? 1 : 0);
    {   // router logits (and the shared expert's gate) in fp32 on the CUDA cores in both modes
        DK_PROF(DK_ROUTER);
        MoeRouterInput in{e->hn, f32, ly.w("router"), 1, D, e->rlog};
        in.sigmoid = 1, in.correction = ly.f("correction"), in.groups = c.groups, in.keep = c.keep, in.scale = c.router_scale;
        in.extra = zld - c.experts;
        if (launch_moe_route(nullptr, &in, M, c.experts, c.top, e->expert_of, e->rgate, e->counters, e->group_off,
                             e->sorted_tok, e->slot_of, s))
            return -1;
    }
    {
        DK_PROF(DK_EXPERTS);
        SimtLinear U;   // gate | up of every chosen (token, expert) pair
        U.a = e->hn, U.a_f32 = f32, U.lda = D;
        U.w = ly.w("w_egu"), U.w_f32 = f32, U.ldw = D, U.w_zs = (long long)2 * c.expert_ff * D;
        U.c = e->up, U.c_f32 = 1, U.ldc = 2 * c.expert_ff;
        U.M = M, U.N = 2 * c.expert_ff, U.K = D, U.Z = c.experts;
        U.group_off = e->group_off, U.gather = e->sorted_tok;
        if (linear(e, U, s)) return -1;
    }
    {
        DK_PROF(DK_ACT);
        if (launch_ff_act(e->up, e->act, f32, (long long)M * c.top, c.expert_ff, 1, s)) return -1;
    }
    {
        DK_PROF(DK_EXPERTS);
        SimtLinear W;
        W.a = e->act, W.a_f32 = f32, W.lda = c.expert_ff;
        W.w = ly.w("w_edown"), W.w_f32 = f32, W.ldw = c.expert_ff, W.w_zs = (long long)D * c.expert_ff;
        W.c = e->eout, W.c_f32 = 1, W.ldc = D;
        W.M = M, W.N = D, W.K = c.expert_ff, W.Z = c.experts;
        W.group_off = e->group_off;
        if (linear(e, W, s)) return -1;
    }
    C.expert_out = e->eout, C.slot_of = e->slot_of, C.gate = e->rgate, C.top = c.top;
    if (c.shared_ff > 0) {
        C.ff = e->yf, C.ff_gate = e->rlog + c.experts, C.ff_gate_ld = zld;
        return gated("w_sgu", "w_sdown", c.shared_ff, 5);
    }
    return 0;
}

static int forward(DkEngine* e, const Batch& b, const int* logit_rows, int n_rows, float* logits, long long ld,
                   float* layer_out, cudaStream_t s) {
    const int D = e->c.width, M = b.ix.M, f32 = e->f32;
    const int nruns = (int)e->runs.size();
    auto base_close = [&]() {
        RowClose C;
        C.x_in = e->x, C.x_out = e->x, C.eps = e->c.eps, C.M = M, C.D = D, C.plain_w = 1;
        return C;
    };
    auto open_next = [&](int r, RowClose& C) {   // hn and hf: what layer r's feed-forward and input convolution read
        if (r >= nruns) return;
        const DkLayer& ly = e->layers[e->runs[r].layer];
        C.next_w = ly.f("norm1"), C.next_b = ly.f("norm1_b"), C.hn = e->hn, C.hn_f32 = f32;
        C.hn_copy = f32 ? nullptr : e->hf;       // an fp32 engine's hn is fp32 already
    };
    const float* hf = f32 ? static_cast<const float*>(e->hn) : e->hf;
    {
        DK_PROF(DK_GLUE);
        if (launch_embed_sinusoid(b.ix, e->gw("embed"), f32, e->c.embed_scale, e->freq, e->x, D, s)) return -1;
        if (nruns) {
            RowClose C = base_close();
            C.x_out = nullptr;
            open_next(0, C);
            if (launch_row_close(C, s)) return -1;
        }
    }
    for (int r = 0; r < nruns; ++r) {
        const DkRun& run = e->runs[r];
        const DkLayer& ly = e->layers[run.layer];
        const int li = run.layer;
        {   // what the mixer reads: h + its causal convolution
            DK_PROF(DK_GLUE);
            if (launch_carried_conv(b.ix, b.cu_q, b.nseq, b.max_qlen, hf, D, ly.f("input_conv"), e->c.input_taps, D,
                                    e->state + run.input_off, e->input_ring, 1, e->hc, f32, s))
                return -1;
        }
        if (ly.c.type == DK_MLSTM ? mix_mlstm(e, ly, run, li, b, s) : mix_parallel(e, ly, run, li, b, s)) return -1;
        RowClose C = base_close();
        C.mult = e->c.residual_mult;
        C.y = e->y;
        if (ly.c.type == DK_PARALLEL) {
            C.post_w = ly.f("out_left"), C.y2 = e->y2, C.post_w2 = ly.f("out_right");
            C.y_scale = 0.5f;
        }
        if (ly.c.ff_kind != DK_FF_NONE && feed_forward(e, ly, li, b, C, s)) return -1;
        {   // x += mult * (mixer + feed-forward); then what the next layer reads
            DK_PROF(DK_GLUE);
            open_next(r + 1, C);
            if (launch_row_close(C, s)) return -1;
        }
        if (layer_out)
            ASD_CUDA(cudaMemcpyAsync(layer_out + (size_t)r * M * D, e->x, sizeof(float) * M * D, cudaMemcpyDeviceToDevice, s));
    }
    if (n_rows > 0) {
        DK_PROF(DK_HEAD);
        RowClose C = base_close();
        C.x_out = nullptr, C.rows = logit_rows, C.next_w = e->gf("final_norm"), C.next_b = e->gf("final_norm_b");
        C.hn = e->xsel, C.hn_f32 = f32, C.M = n_rows;
        if (launch_row_close(C, s)) return -1;
        const int V = e->c.vocab;
        if (e->dn.run(e->xsel, e->gw("head"), logits, n_rows, V, D, ld ? (int)ld : V, (int)e->layers.size() * 16 + 2, s))
            return -1;
    }
    return 0;
}

// elements one layer's rows take in the pool, rounded up so that every layer starts on a 16-byte boundary
static size_t pool_elems(const DkEngine* e, const DkRun& r, int num_pages) {
    const size_t n = (size_t)num_pages * e->c.page_size * e->layers[r.layer].cache_row;
    return (n + 7) & ~(size_t)7;
}

// the parts of one layer's carried state, floats per sequence slot count; every part starts on a 16-byte boundary
static size_t up4(size_t n) { return (n + 3) & ~(size_t)3; }
static size_t input_floats(const DkEngine* e, int max_seqs) { return up4((size_t)max_seqs * e->input_ring * e->c.width); }
static size_t conv_floats(const DkLayer& ly, int max_seqs) { return up4((size_t)max_seqs * ly.conv_elems); }
static size_t state_floats(const DkEngine* e, const DkLayer& ly, int max_seqs) {
    return up4((size_t)max_seqs * e->c.ring * ly.state_elems);
}

static const char* const kLayerNames[] = {"norm1", "norm1_b", "input_conv", "w_in", "w_o", "w_o2", "i_bias", "f_bias",
                                          "out_norm", "head_bias", "conv_w", "a_log", "dt_bias", "out_left", "out_right",
                                          "w_gu", "w_down", "router", "correction", "w_egu", "w_edown", "w_sgu", "w_sdown"};
static const char* const kGlobalNames[] = {"embed", "final_norm", "final_norm_b", "head"};

static std::vector<const char*> required(const DkLayer& ly) {
    std::vector<const char*> n = {"norm1", "norm1_b", "input_conv", "w_in", "w_o", "out_norm"};
    if (ly.c.type == DK_MLSTM)
        n.insert(n.end(), {"i_bias", "f_bias"});
    else
        n.insert(n.end(), {"w_o2", "head_bias", "conv_w", "a_log", "dt_bias", "out_left", "out_right"});
    if (ly.c.ff_kind == DK_FF_DENSE) n.insert(n.end(), {"w_gu", "w_down"});
    if (ly.c.ff_kind == DK_FF_MOE) {
        n.insert(n.end(), {"router", "correction", "w_egu", "w_edown"});
        if (ly.c.shared_ff > 0) n.insert(n.end(), {"w_sgu", "w_sdown"});
    }
    return n;
}

}  // namespace asd

using namespace asd;

extern "C" {

asd_dikopel_engine_t* asd_dikopel_create(const asd_dikopel_config* cfg, const asd_dikopel_layer_config* layers) {
    if (!cfg || (cfg->n_layers > 0 && !layers)) {
        set_error("asd_dikopel_create: NULL config");
        return nullptr;
    }
    if (cfg->width <= 0 || cfg->vocab <= 0 || cfg->n_layers < 0 || cfg->max_tokens <= 0 || cfg->page_size <= 0 ||
        cfg->ring <= 0 || cfg->input_taps <= 0 || (cfg->dtype != 0 && cfg->dtype != 1)) {
        set_error("asd_dikopel_create: bad sizes");
        return nullptr;
    }
    DkEngine* e = new DkEngine();
    e->c = *cfg;
    e->f32 = e->dn.f32 = cfg->dtype;
    e->esz = cfg->dtype ? 4 : 2;
    cudaGetDevice(&e->device);
    const size_t MT = cfg->max_tokens, D = cfg->width;
    size_t ld_in = 4, conv = 1, nv = 1, rvn = 1, heads = 1, mixw = 1, mixw2 = 1, upw = 1, actw = 1, E = 1, top = 1;
    bool attn = false;
    auto fail = [&](const char* what, int l) {
        set_error("asd_dikopel_create: %s (layer %d)", what, l);
        asd_dikopel_destroy(e);
        return nullptr;
    };
    // inputs of the last taps - 1 positions, for each of the `ring` positions a forward may start after
    auto carried = [&](int taps) { return taps > 1 ? taps - 1 + cfg->ring - 1 : 0; };
    e->input_ring = carried(cfg->input_taps);
    for (int l = 0; l < cfg->n_layers; ++l) {
        DkLayer ly;
        ly.c = layers[l];
        auto& c = ly.c;
        if (c.weights_of < -1 || c.weights_of >= cfg->n_layers || c.weights_of == l) return fail("bad weights_of", l);
        int own = l;
        for (int hops = 0; layers[own].weights_of >= 0; ++hops) {
            own = layers[own].weights_of;
            if (own >= cfg->n_layers || hops > cfg->n_layers) return fail("weights_of names no layer with weights", l);
        }
        e->runs.push_back(DkRun{own});
        if (c.type == DK_MLSTM) {
            if (c.heads <= 0 || c.dim <= 0 || c.dim > 1024 || c.vdim <= 0 || !(c.gate_cap > 0.f)) return fail("bad mlstm sizes", l);
            ly.n_in = 2 * c.heads * (c.dim + c.vdim) + 2 * c.heads;
            ly.state_elems = mlstm_state_elems(mlstm_dims(c));
            mixw = std::max(mixw, (size_t)c.heads * c.vdim);
            nv = std::max(nv, (size_t)c.heads * c.vdim);
        } else if (c.type == DK_PARALLEL) {
            MixDims md{c.a_heads, c.a_kv_heads, c.a_dim, c.a_vdim, 0, c.scale};
            md.sigmoid = 1;
            if (mix_attention_check(md, 0)) {
                asd_dikopel_destroy(e);
                return nullptr;
            }
            if (c.r_heads <= 0 || c.r_kv_heads <= 0 || c.r_heads % c.r_kv_heads || c.r_dim <= 0 || c.r_dim > 1024 ||
                c.r_vdim <= 0 || c.conv <= 0)
                return fail("bad gated delta rule sizes", l);
            ly.cache_row = c.a_kv_heads * (c.a_dim + c.a_vdim);
            ly.conv_ch = 2 * c.r_kv_heads * c.r_dim + c.r_heads * c.r_vdim;
            ly.n_in = c.a_heads * c.a_dim + ly.cache_row + ly.conv_ch + c.r_heads * c.r_vdim + 2 * c.r_heads;
            ly.conv_ring = carried(c.conv);
            ly.conv_elems = (size_t)ly.conv_ring * ly.conv_ch;
            ly.state_elems = (size_t)c.r_heads * c.r_dim * c.r_vdim;
            attn = true;
            mixw = std::max(mixw, (size_t)c.a_heads * c.a_vdim);
            mixw2 = std::max(mixw2, (size_t)c.r_heads * c.r_vdim);
            nv = std::max(nv, (size_t)c.r_heads * c.r_vdim);
            conv = std::max(conv, (size_t)ly.conv_ch);
            rvn = std::max(rvn, (size_t)c.r_heads * 2 * c.r_dim);
            heads = std::max(heads, (size_t)c.r_heads);
        } else {
            return fail("unknown mixer type", l);
        }
        if (c.ff_kind == DK_FF_DENSE) {
            if (c.ff <= 0) return fail("bad feed-forward size", l);
            upw = std::max(upw, (size_t)2 * c.ff);
            actw = std::max(actw, (size_t)c.ff);
        } else if (c.ff_kind == DK_FF_MOE) {
            if (c.experts <= 0 || c.expert_ff <= 0 || c.shared_ff < 0 || c.groups <= 0 || c.experts % c.groups || c.keep <= 0 ||
                c.keep > c.groups || c.top <= 0 || c.top > c.keep * (c.experts / c.groups))
                return fail("bad expert sizes", l);
            upw = std::max(upw, std::max((size_t)c.top * 2 * c.expert_ff, (size_t)2 * c.shared_ff));
            actw = std::max(actw, std::max((size_t)c.top * c.expert_ff, (size_t)c.shared_ff));
            E = std::max(E, (size_t)c.experts);
            top = std::max(top, (size_t)c.top);
        } else if (c.ff_kind != DK_FF_NONE) {
            return fail("unknown feed-forward kind", l);
        }
        ly.ld_in = (ly.n_in + 3) & ~3;
        ld_in = std::max(ld_in, (size_t)ly.ld_in);
        e->layers.push_back(ly);
    }
    for (size_t l = 0; l < e->layers.size(); ++l) {   // a shared layer's sizes are its owner's
        asd_dikopel_layer_config a = e->layers[l].c, o = e->layers[e->runs[l].layer].c;
        a.weights_of = o.weights_of = -1;
        if (memcmp(&a, &o, sizeof(a))) return fail("differs from the layer whose weights it uses", (int)l);
    }
    int rc = 0;
    std::vector<double> freq((D + 1) / 2);
    for (size_t i = 0; i < freq.size(); ++i) freq[i] = pow(10000.0, -2.0 * (double)i / (double)D);
    rc |= dev_alloc(e, &e->freq, freq.size());
    if (!rc && cudaMemcpy(e->freq, freq.data(), freq.size() * sizeof(double), cudaMemcpyHostToDevice) != cudaSuccess) rc = -1;
    rc |= dev_alloc(e, &e->x, MT * D);
    if (!e->f32) rc |= dev_alloc(e, &e->hf, MT * D);
    rc |= dev_alloc(e, &e->y, MT * D);
    rc |= dev_alloc(e, &e->y2, MT * D);
    rc |= dev_alloc(e, &e->yf, MT * D);
    rc |= dev_alloc(e, &e->proj, MT * ld_in);
    rc |= dev_alloc(e, &e->conv, MT * conv);
    rc |= dev_alloc(e, &e->rv, MT * rvn);
    rc |= dev_alloc(e, &e->sc, MT * heads * 4);
    rc |= dev_alloc(e, &e->orec, MT * nv);
    rc |= dev_alloc(e, &e->up, MT * upw);
    rc |= dev_alloc(e, &e->eout, MT * top * D);
    rc |= dev_alloc(e, &e->rlog, MT * (E + 1));
    rc |= dev_alloc(e, &e->rgate, MT * top);
    rc |= dev_alloc(e, (char**)&e->hn, MT * D * e->esz);
    rc |= dev_alloc(e, (char**)&e->hc, MT * D * e->esz);
    rc |= dev_alloc(e, (char**)&e->mixed, MT * mixw * e->esz);
    rc |= dev_alloc(e, (char**)&e->mixed2, MT * mixw2 * e->esz);
    rc |= dev_alloc(e, (char**)&e->act, MT * actw * e->esz);
    rc |= dev_alloc(e, (char**)&e->xsel, MT * D * e->esz);
    rc |= dev_alloc(e, &e->expert_of, MT * top);
    rc |= dev_alloc(e, &e->counters, 2 * E + 1);
    rc |= dev_alloc(e, &e->group_off, E + 1);
    rc |= dev_alloc(e, &e->sorted_tok, MT * top);
    rc |= dev_alloc(e, &e->slot_of, MT * top);
    if (attn) {   // partial results of key shares (steps of few tokens)
        e->attn_ws.part_elems = (long long)(2048 * mixw);
        rc |= dev_alloc(e, &e->attn_ws.part, (size_t)e->attn_ws.part_elems);
    }
    rc |= dev_alloc(e, &e->dev_error, 1);
    if (!rc && cudaMemset(e->dev_error, 0, sizeof(int)) != cudaSuccess) rc = -1;
    if (rc) {
        asd_dikopel_destroy(e);
        return nullptr;
    }
    return e;
}

void asd_dikopel_destroy(asd_dikopel_engine_t* h) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e) return;
    for (void* p : e->owned) cudaFree(p);
    delete e;
}

int asd_dikopel_set_tensor(asd_dikopel_engine_t* h, int layer, const char* name, const void* data) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e || !name || !data) return set_error("asd_dikopel_set_tensor: NULL argument");
    if (layer >= (int)e->layers.size() || layer < -1) return set_error("asd_dikopel_set_tensor: bad layer %d", layer);
    bool known = false;
    if (layer < 0) {
        for (const char* n : kGlobalNames) known |= !strcmp(n, name);
        if (known) e->g[name] = data;
    } else {
        for (const char* n : kLayerNames) known |= !strcmp(n, name);
        if (known) e->layers[layer].t[name] = data;
    }
    if (!known) return set_error("asd_dikopel_set_tensor: unknown tensor %s (layer %d)", name, layer);
    e->dn.clear();
    return 0;
}

size_t asd_dikopel_cache_bytes(const asd_dikopel_engine_t* h, int num_pages) {
    const DkEngine* e = static_cast<const DkEngine*>(h);
    if (!e) return 0;
    size_t n = 0;
    for (const DkRun& r : e->runs) n += pool_elems(e, r, num_pages);
    return n * e->esz;
}

size_t asd_dikopel_state_bytes(const asd_dikopel_engine_t* h, int max_seqs) {
    const DkEngine* e = static_cast<const DkEngine*>(h);
    if (!e) return 0;
    size_t n = 0;
    for (const DkRun& r : e->runs) {
        const DkLayer& ly = e->layers[r.layer];
        n += input_floats(e, max_seqs) + conv_floats(ly, max_seqs) + state_floats(e, ly, max_seqs);
    }
    return n * sizeof(float);
}

int asd_dikopel_set_cache(asd_dikopel_engine_t* h, void* pool, int num_pages, const int32_t* page_table, int max_seqs,
                          int max_pages_per_seq, float* state) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e || !pool || !page_table || !state || num_pages <= 0 || max_seqs <= 0 || max_pages_per_seq <= 0)
        return set_error("asd_dikopel_set_cache: bad arguments");
    e->pool = static_cast<char*>(pool);
    e->num_pages = num_pages, e->page_table = page_table, e->max_seqs = max_seqs, e->max_pages = max_pages_per_seq;
    e->state = state;
    size_t off = 0, soff = 0;
    for (DkRun& r : e->runs) {
        const DkLayer& ly = e->layers[r.layer];
        r.cache_off = off;
        off += pool_elems(e, r, num_pages);
        r.input_off = soff;
        soff += input_floats(e, max_seqs);
        r.conv_off = soff;
        soff += conv_floats(ly, max_seqs);
        r.state_off = soff;
        soff += state_floats(e, ly, max_seqs);
    }
    return 0;
}

int asd_dikopel_set_option(asd_dikopel_engine_t* h, const char* name, int value) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e || !name) return set_error("asd_dikopel_set_option: NULL argument");
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
    if (!strcmp(name, "profile")) {
        e->prof.on = value;
        e->prof.reset();
        return 0;
    }
    return set_error("asd_dikopel_set_option: unknown option %s", name);
}

int asd_dikopel_forward(asd_dikopel_engine_t* h, const int32_t* tokens, const int32_t* positions,
                        const int32_t* token_slot, int M, const int32_t* cu_q, const int32_t* seq_slot, int nseq,
                        int max_qlen, int max_kv_len, const int32_t* logit_rows, int n_logit_rows, float* logits_out,
                        long long logits_ld, float* layer_out, void* stream) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e) return set_error("asd_dikopel_forward: NULL engine");
    if (M <= 0 || M > e->c.max_tokens) return set_error("asd_dikopel_forward: M = %d outside 1..%d", M, e->c.max_tokens);
    if (!e->pool) return set_error("asd_dikopel_forward: cache not set");
    for (const char* n : kGlobalNames)
        if (!e->gw(n)) return set_error("asd_dikopel_forward: tensor %s not set", n);
    for (const DkRun& r : e->runs)
        for (const char* n : required(e->layers[r.layer]))
            if (!e->layers[r.layer].w(n)) return set_error("asd_dikopel_forward: layer %d has no tensor %s", r.layer, n);
    if (!tokens || !positions || !token_slot || !cu_q || !seq_slot || nseq <= 0 || max_qlen <= 0)
        return set_error("asd_dikopel_forward: bad index arguments");
    if (max_kv_len > e->max_pages * e->c.page_size)
        return set_error("asd_dikopel_forward: length bound %d exceeds the page table", max_kv_len);
    if (n_logit_rows > 0 && !logits_out) return set_error("asd_dikopel_forward: logits_out is NULL");
    if (n_logit_rows > e->c.max_tokens) return set_error("asd_dikopel_forward: too many logit rows");
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev != e->device) return set_error("asd_dikopel_forward: called on device %d, engine lives on %d", dev, e->device);
    const Batch b{SeqIndex{tokens, positions, token_slot, M}, cu_q, seq_slot, nseq, max_qlen, max_kv_len};
    return forward(e, b, logit_rows, logit_rows ? n_logit_rows : (n_logit_rows > 0 ? M : 0), logits_out, logits_ld,
                   layer_out, static_cast<cudaStream_t>(stream));
}

int asd_dikopel_profile_read(asd_dikopel_engine_t* h, float* ms_by_class, int* launches_by_class, int nclass) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e || !ms_by_class || nclass < DK_NCLASS) return set_error("asd_dikopel_profile_read: bad argument");
    ASD_CUDA(e->prof.read(ms_by_class, launches_by_class, nclass));
    return 0;
}

int asd_dikopel_device_error(asd_dikopel_engine_t* h) {
    DkEngine* e = static_cast<DkEngine*>(h);
    if (!e) return set_error("asd_dikopel_device_error: NULL engine");
    int v = 0;
    ASD_CUDA(cudaMemcpy(&v, e->dev_error, sizeof(int), cudaMemcpyDeviceToHost));
    if (v) return set_error("a Dikopel kernel gave up a bounded wait (tcgen05 linear)");
    return 0;
}

}  // extern "C"
