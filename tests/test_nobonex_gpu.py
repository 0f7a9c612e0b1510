"""GPU: the Nobonex engine against the plain restatement in oracle/nobonex_oracle.py (fp64, whole sequences, no cache).
Every test makes its own small configuration and random weights.  The fp32 engine is held to 2e-4 of the logits'
spread, which a single key missed or double-counted among hundreds, a lost state or convolution input, a wrong expert or
a stale page all exceed; the bf16 engine to what its roundings allow."""
import copy
import json
import os
import struct
import subprocess
import sys

import pytest
import torch

pytestmark = pytest.mark.gpu

from oracle import nobonex_oracle as O  # noqa: E402


# ------------------------------------------------------------------------------------------------ configurations
def dense(ff=48):
    return {"kind": "dense", "ff": ff} if ff else None


def moe(experts=7, top=2, ff=40, limit=1.5):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def att(heads=6, kv_heads=2, dim=24, scale=0.2, conv=3, rot=12, base=5000.0, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                                                       "scale": scale, "conv": conv, "rot": {"dims": rot, "base": base}}}


def ssd(heads=4, vdim=24, state=20, groups=2, norm_groups=3, conv=3, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                    "norm_groups": norm_groups, "conv": conv}}


YARN = {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 2.0}


def chk(heads=4, kv_heads=2, dim=32, vdim=24, scale=0.2, chunk=24, cap=20.0, rot=16, base=9000.0, yarn=YARN, of=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
         "softcap": cap, "rot": {"dims": rot, "base": base}}
    if yarn:
        m["rot"]["scaling"] = dict(yarn)
    if of is not None:
        m["kv_from"] = of
    return {"type": "attention_2", "mlp": mlp, "mixer": m}


def config(layers, width=104, vocab=120, eps=1e-5, scale=1.5, mult=0.5):
    return {"architecture": "Nobonex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": layers}


# every mixer and feed-forward kind, a layer that reads another one's keys and values (with more query heads, its own chunk)
SMALL = config([att(mlp=dense(72)), ssd(mlp=moe()), chk(mlp=moe(5, 3, 24, 0.8)), chk(heads=8, chunk=40, of=2),
                ssd(heads=3, vdim=40, state=16, groups=1, norm_groups=1, conv=4, mlp=dense(30))])
# sizes that are multiples of nothing; one tap and many; one key head per query head and one for all; whole-head rotation and
# none; no scaling of the rotation; two sources, read out of order
ODD = config([chk(heads=5, kv_heads=5, dim=10, vdim=7, scale=0.4, chunk=7, cap=3.0, rot=10, base=77.0, mlp=moe(7, 7, 9, 0.5)),
              ssd(heads=6, vdim=7, state=10, groups=3, norm_groups=6, conv=1, mlp=dense(50)),
              chk(heads=6, kv_heads=1, dim=14, vdim=34, scale=0.3, chunk=19, cap=50.0, rot=2, yarn=None, mlp=moe(4, 1, 21, 3.0)),
              att(heads=6, kv_heads=1, dim=18, scale=0.5, conv=6, rot=18, base=300.0),
              chk(heads=10, kv_heads=5, dim=10, vdim=7, scale=0.2, chunk=11, cap=8.0, rot=10, base=77.0, of=0, mlp=dense(9)),
              chk(heads=3, kv_heads=1, dim=14, vdim=34, scale=0.6, chunk=1000, cap=5.0, rot=2, yarn=None, of=2),
              att(heads=3, kv_heads=3, dim=11, scale=0.3, conv=1, rot=0, mlp=moe(3, 2, 5, 1.0))],
             width=72, vocab=101, eps=1e-3, scale=0.7, mult=1.0)
PLAIN = config([att(conv=5), ssd(), chk()], mult=0.25)        # no feed-forward at all


def make_engine(cfg_dict, w, dtype=torch.float32, max_tokens=64, max_seq_len=512, page_size=16, num_pages=None,
                max_seqs=4, ring=1, tc=1, ssd_mode=0):
    from asd_b200.engine import NobonexEngine
    from asd_b200.models.nobonex import NobonexConfig
    eng = NobonexEngine(NobonexConfig.from_dict(cfg_dict), max_seqs=max_seqs, max_seq_len=max_seq_len, max_tokens=max_tokens,
                        page_size=page_size, dtype=dtype, dynamic_pages=True, num_pages=num_pages, ring=ring)
    eng.load_weights(w)
    eng.set_option("tc_linear", tc)
    eng.set_option("ssd_mode", ssd_mode)
    return eng


def close(eng):
    """no kernel of the engine gave up a wait"""
    eng.check_device()
    eng.close()


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel_err(got, want):
    got, want = got.double().cpu(), want.double()
    return ((got - want).norm() / want.norm()).item(), ((got - want).abs().max() / want.std()).item()


def feed(eng, slot, ids, cuts, start=0):
    """feeds ids in portions of the given sizes (the rest in one go), all logits wanted"""
    out, a = [], 0
    sizes = list(cuts)
    while a < len(ids):
        n = sizes.pop(0) if sizes else len(ids) - a
        n = min(n, len(ids) - a)
        eng.reserve(slot, start + a + n)
        out.append(eng.forward_ragged([(slot, start + a, ids[a:a + n], list(range(n)))]))
        a += n
    return torch.cat(out, 0)


def run_cuts(cfg_dict, w, ids, cuts=(), **kw):
    eng = make_engine(cfg_dict, w, **kw)
    slot = eng.open_sequence()
    got = feed(eng, slot, ids, cuts)
    close(eng)
    return got


def oracle(cfg_dict, w, ids, streams=None):
    return O.forward(cfg_dict, w, ids, layers_out=streams)


def changed(cfg, w, ids, ref, **tensors):
    """how far the oracle's logits move when these tensors (names with __ for .) are replaced"""
    w2 = dict(w)
    w2.update({k.replace("__", "."): v for k, v in tensors.items()})
    return rel_err(oracle(cfg, w2, ids).float(), ref)[1]


# ------------------------------------------------------------------------------------------------ whole prompts
@pytest.mark.parametrize("cfg_dict", [SMALL, ODD, PLAIN], ids=["small", "odd", "plain"])
def test_whole_prompt_logits_and_every_layer(cfg_dict):
    w = O.random_model(cfg_dict, seed=1)
    ids = tokens(45, cfg_dict["vocab"], 2)
    streams = []
    ref = oracle(cfg_dict, w, ids, streams)
    eng = make_engine(cfg_dict, w)
    slot = eng.open_sequence()
    eng.reserve(slot, len(ids))
    got, st = eng.forward_ragged([(slot, 0, ids, list(range(len(ids))))], layer_out=True)
    st = torch.cat(st, 1).cpu().double()
    assert st.shape[0] == len(cfg_dict["layers"]) == len(streams)
    for i in range(st.shape[0]):           # the first layer that differs names the mechanism
        assert (st[i] - streams[i]).abs().max() <= 2e-4 * streams[i].abs().max(), f"stream leaving layer {i}"
    assert rel_err(got, ref)[1] < 2e-4
    close(eng)


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("width,scale", [(40, 3.0), (41, 0.3), (128, 1.0)])
def test_scaled_embedding_and_final_norm_alone(width, scale):
    """no layers: logits = head . (w tanh(alpha embed scale) + b)"""
    cfg = config([], width=width, vocab=50, scale=scale)
    w = O.random_model(cfg, seed=3)
    ids = tokens(300, 50, 4)
    ref = oracle(cfg, w, ids)
    assert rel_err(run_cuts(cfg, w, ids, [150]), ref)[1] < 1e-4
    assert changed(cfg, w, ids, ref, final__norm__b=torch.zeros(width)) > 1e-2
    assert changed(cfg, w, ids, ref, final__norm__alpha=torch.tensor(1.3)) > 1e-2


def silence_mixer(cfg, w, i=0):
    """layer i's mixer gives nothing but its norm's bias, which is taken away as well"""
    for k in (f"l{i}.mix.o", f"l{i}.norm1b.b"):
        w[k] = torch.zeros_like(w[k])


def test_four_norms_and_the_residual_multiplier():
    for mult in (0.3, 1.0, 1.7):
        cfg = config([ssd(mlp=dense(56)), chk()], mult=mult)
        w = O.random_model(cfg, seed=5, scale=2.0)
        ids = tokens(33, 120, 6)
        ref = oracle(cfg, w, ids)
        assert rel_err(run_cuts(cfg, w, ids), ref)[1] < 2e-4
    assert rel_err(oracle(dict(cfg, residual_mult=1.6), w, ids).float(), ref)[1] > 1e-2
    for n in ("l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l1.norm1", "l1.norm1b"):
        for part in (".alpha", ".b", ""):
            k = n + part
            assert rel_err(oracle(cfg, dict(w, **{k: w[k] + 0.5}), ids).float(), ref)[1] > 1e-2, k


@pytest.mark.parametrize("ff", [8, 33, 128])
def test_gated_feed_forward_alone(ff):
    cfg = config([ssd(mlp=dense(ff))])
    w = O.random_model(cfg, seed=7, scale=2.0)
    silence_mixer(cfg, w)
    ids = tokens(50, 120, 8)
    assert rel_err(run_cuts(cfg, w, ids), oracle(cfg, w, ids))[1] < 2e-4


@pytest.mark.parametrize("experts,top,ff,limit", [(7, 2, 40, 1.5), (12, 1, 17, 0.3), (5, 5, 8, 2.0), (40, 3, 12, 7.0), (2, 1, 64, 1.0),
                                                  (70, 4, 8, 0.7), (1, 1, 24, 1.0)])
def test_routed_experts_alone(experts, top, ff, limit):
    """the weight goes in front of the clamped activations, where it is not the same as behind them; scores are not divided
    by their sum; the clamps are reached on both sides"""
    cfg = config([ssd(mlp=moe(experts, top, ff, limit))])
    w = O.random_model(cfg, seed=9, scale=2.0)
    silence_mixer(cfg, w)
    ids = tokens(50, 120, 10)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 50):
        assert rel_err(run_cuts(cfg, w, ids, cuts), ref)[1] < 2e-4
    c2 = copy.deepcopy(cfg)
    c2["layers"][0]["mlp"]["expert"]["limit"] = limit * 1.5
    assert rel_err(oracle(c2, w, ids).float(), ref)[1] > (1e-2 if limit < 3 else 0)
    assert changed(cfg, w, ids, ref, l0__mlp__router=w["l0.mlp.router"] * 0) > 1e-2


def test_expert_weight_multiplies_the_input(monkeypatch):
    cfg = config([ssd(mlp=moe(6, 2, 32, 1.0))])
    w = O.random_model(cfg, seed=11, scale=2.0)
    silence_mixer(cfg, w)
    ids = tokens(40, 120, 12)
    ref = oracle(cfg, w, ids)
    assert rel_err(run_cuts(cfg, w, ids), ref)[1] < 2e-4

    def behind(h, ww, f):
        s = torch.sigmoid(h @ ww["router"].T)
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            for e in s[t].topk(f["router"]["top"]).indices.tolist():
                out[t] += s[t, e] * O.expert(h[t:t + 1], O.sub(ww, f"e{e}."), f["expert"]["limit"])[0]
        return out
    monkeypatch.setattr(O, "feed_forward", behind)
    assert rel_err(oracle(cfg, w, ids).float(), ref)[1] > 1e-2


def test_many_tokens_take_the_other_routing_kernel():
    cfg = config([ssd(heads=1, vdim=8, state=4, groups=1, norm_groups=1, conv=1, mlp=moe(16, 4, 24, 1.0))])
    w = O.random_model(cfg, seed=13, scale=2.0)
    silence_mixer(cfg, w)
    ids = tokens(1400, 120, 14)
    assert rel_err(run_cuts(cfg, w, ids, max_tokens=2048, max_seq_len=2048), oracle(cfg, w, ids))[1] < 2e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim,taps,rot", [(6, 2, 24, 3, 12), (4, 4, 32, 1, 32), (8, 1, 64, 2, 0), (20, 4, 16, 7, 4), (12, 1, 40, 4, 40),
                                                   (5, 5, 10, 5, 6), (2, 1, 136, 3, 64), (34, 1, 16, 4, 8), (3, 1, 200, 2, 2), (24, 2, 128, 4, 96), (2, 1, 256, 4, 64)])
def test_convolved_attention_alone(heads, kv, dim, taps, rot, dtype):
    """every kernel: prompts, portions of a few tokens, single tokens; sizes that fill a load and that do not; more than
    eight and sixteen query heads per key head; a large oldest tap makes a lost or misplaced carried row show"""
    cfg = config([att(heads, kv, dim, 1.5 / dim ** 0.5, taps, rot, 700.0)])
    w = O.random_model(cfg, seed=15)
    for n in ("q", "k"):
        t = w[f"l0.mix.{n}.conv"].float()
        t[:, 0] *= 3
        w[f"l0.mix.{n}.conv"] = t.to(torch.bfloat16)
    ids = tokens(210, 120, 16)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [130] + [1] * 80, [2] * 105, [3, 64, 5, 7, 33, 4, 2, 1]):
        got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=256)
        assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 5e-2), cuts
    for n in ("q.norm", "k.norm", "k.conv"):
        assert rel_err(oracle(cfg, dict(w, **{f"l0.mix.{n}": w[f"l0.mix.{n}"].flip(0)}), ids).float(), ref)[1] > 1e-2
    if rot:
        c2 = copy.deepcopy(cfg)
        c2["layers"][0]["mixer"]["rot"]["base"] = 900.0
        assert rot == 2 or rel_err(oracle(c2, w, ids).float(), ref)[1] > 1e-3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim,vdim,chunk,cap,rot,factor", [
    (4, 2, 32, 24, 24, 20.0, 16, 4.0), (4, 4, 32, 64, 64, 2.0, 32, 1.0), (8, 1, 64, 128, 33, 50.0, 8, 2.0), (20, 4, 16, 16, 200, 1.0, 4, 0.0),
    (12, 1, 40, 24, 1000, 5.0, 40, 40.0), (5, 5, 10, 6, 7, 3.0, 6, 8.0), (2, 1, 136, 200, 1, 30.0, 64, 1.5), (34, 1, 16, 16, 17, 10.0, 8, 3.0),
    (3, 1, 8, 130, 16, 4.0, 2, 4.0), (24, 3, 128, 128, 100, 15.0, 64, 4.0), (4, 2, 256, 256, 50, 9.0, 128, 2.0)])
def test_chunked_attention_alone(heads, kv, dim, vdim, chunk, cap, rot, factor, dtype):
    """biases, norms per head, rotation with scaled frequencies, capped scores, chunks that end inside pages, tiles and
    portions, the output gate"""
    yarn = {"factor": factor, "original": 100, "fast": 8.0, "slow": 1.0} if factor else None
    cfg = config([chk(heads, kv, dim, vdim, 2.0 / dim ** 0.5, chunk, cap, rot, 700.0, yarn)])
    w = O.random_model(cfg, seed=17)
    ids = tokens(210, 120, 18)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [130] + [1] * 80, [2] * 105, [3, 64, 5, 7, 33, 4, 2, 1]):
        got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=256)
        assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 5e-2), cuts
    for n in ("v.b", "g") + (("q.b", "k.b", "q.norm", "k.norm") if chunk > 1 else ()):       # a chunk of one has one weight
        assert rel_err(oracle(cfg, dict(w, **{f"l0.mix.{n}": w[f"l0.mix.{n}"] + 0.5}), ids).float(), ref)[1] > 1e-3, n
    c2 = copy.deepcopy(cfg)
    c2["layers"][0]["mixer"].update(softcap=cap * 1.5, mask={"size": chunk + 1})
    assert rel_err(oracle(c2, w, ids).float(), ref)[1] > 1e-3


@pytest.mark.parametrize("scaling", [{"factor": 2.0, "original": 64, "fast": 4.0, "slow": 0.5}, {"factor": 16.0, "original": 1000, "fast": 32.0, "slow": 1.0},
                                     {"factor": 3.0, "original": 4, "fast": 300.0, "slow": 200.0}, {"factor": 8.0, "original": 10 ** 6, "fast": 2.0, "slow": 1.0}])
def test_scaled_rotation_alone(scaling):
    """the ramp between kept and divided frequencies inside the pairs, before the first one, and beyond the last one"""
    cfg = config([chk(4, 2, 32, 24, 0.6, 500, 30.0, 24, 50.0, scaling)])
    w = O.random_model(cfg, seed=19)
    ids = tokens(120, 120, 20)
    ref = oracle(cfg, w, ids)
    assert rel_err(run_cuts(cfg, w, ids, [70] + [1] * 50, max_tokens=128), ref)[1] < 2e-4
    c2 = copy.deepcopy(cfg)
    del c2["layers"][0]["mixer"]["rot"]["scaling"]
    assert rel_err(oracle(c2, w, ids).float(), ref)[1] > 1e-2


def test_rotation_stays_exact_at_far_positions():
    """one key and one query far along: the angles are those of positions in the thousands"""
    cfg = config([chk(2, 1, 16, 16, 1.0, 1 << 20, 50.0, 16, 3.0, None), att(2, 1, 16, 0.5, 1, 16, 3.0)])
    w = O.random_model(cfg, seed=21)
    ids = tokens(2900, 120, 22)
    ref = oracle(cfg, w, ids)
    got = run_cuts(cfg, w, ids, [1400, 1400], max_tokens=1536, max_seq_len=4096)
    assert rel_err(got[-64:], ref[-64:])[1] < 2e-4


def test_attention_kernels_agree():
    """bf16 cache rows: the tensor-core kernels and the general CUDA-core kernel read the same cache and the same queries,
    so they differ by fp32 roundings only (option 2: few tokens on the CUDA cores, prompts on the tensor cores); prompts,
    portions that end inside a tile, few tokens and single ones"""
    for i, (heads, kv, dim, vdim, chunk) in enumerate(((4, 4, 32, 16, 50), (6, 2, 16, 32, 128), (8, 1, 64, 128, 30), (16, 4, 48, 64, 1000), (3, 1, 80, 24, 3),
                                                       (32, 8, 32, 32, 64), (24, 3, 16, 64, 100), (18, 9, 16, 16, 33), (20, 1, 48, 96, 250))):
        for layer in (chk(heads, kv, dim, vdim, 2.0 / dim ** 0.5, chunk, 4.0, 8), att(heads, kv, dim, 1.5 / dim ** 0.5, 3, 8)):
            cfg = config([layer])
            w = O.random_model(cfg, seed=55 + i)
            ids = tokens(330, 120, 56)
            ref = oracle(cfg, w, ids)
            for cuts in ((), [200, 64, 9, 1, 1, 2, 53], [300] + [1] * 30, [17] * 20, [310, 4, 3, 2, 4, 4, 3]):
                got = []
                for general in (0, 2, 1):
                    eng = make_engine(cfg, w, dtype=torch.bfloat16, max_tokens=512, page_size=8)
                    eng.set_option("attn_general", general)
                    slot = eng.open_sequence()
                    got.append(feed(eng, slot, ids, cuts))
                    close(eng)
                    assert rel_err(got[-1], ref)[0] < 5e-2, (heads, kv, cuts, general)
                for other in got[1:]:
                    assert rel_err(got[0], other.cpu())[0] < 3e-3, (heads, kv, cuts)


def test_shared_keys_and_values():
    """two layers read the first one's cache with queries, head counts, chunks, scales and caps of their own"""
    cfg = config([chk(heads=2, chunk=30), chk(heads=6, chunk=9, scale=0.4, cap=4.0, of=0, mlp=dense(40)), ssd(),
                  chk(heads=4, chunk=600, of=0)])
    w = O.random_model(cfg, seed=23)
    assert "l1.mix.k" not in w and "l3.mix.v.b" not in w
    ids = tokens(90, 120, 24)
    ref = oracle(cfg, w, ids)
    for dtype in (torch.float32, torch.bfloat16):
        for cuts in ((), [40] + [1] * 50, [7, 2, 2, 11], [2] * 45):
            got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=128, page_size=8)
            assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 5e-2), cuts
    assert changed(cfg, w, ids, ref, l0__mix__k=w["l0.mix.k"].flip(0)) > 1e-2


@pytest.mark.parametrize("heads,vdim,state,groups,norm_groups,conv", [
    (4, 24, 20, 2, 3, 3), (1, 64, 64, 1, 1, 4), (6, 16, 128, 3, 2, 2), (2, 130, 33, 2, 1, 1), (3, 40, 16, 1, 5, 7), (5, 5, 3, 5, 1, 4),
    (2, 20, 300, 1, 2, 3), (8, 64, 96, 2, 1, 4), (1, 200, 10, 1, 10, 2)])
def test_state_space_recurrence_alone(heads, vdim, state, groups, norm_groups, conv):
    cfg = config([ssd(heads, vdim, state, groups, norm_groups, conv)])
    w = O.random_model(cfg, seed=25)
    t = w["l0.mix.conv"].float()
    t[:, 0] *= 2
    w["l0.mix.conv"] = t.to(torch.bfloat16)
    w["l0.mix.dt_bias"] = torch.linspace(-5.0, 1.0, heads).to(torch.bfloat16)      # states that live long, and not
    ids = tokens(150, 120, 26)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 150, [2] * 75, [33, 3, 1, 1, 2], [32, 64, 31, 1], [64, 70]):
        assert rel_err(run_cuts(cfg, w, ids, cuts, max_tokens=256), ref)[1] < 2e-4, cuts
    for n in ("dt_bias", "A_log", "D", "conv.b", "norm"):
        assert rel_err(oracle(cfg, dict(w, **{f"l0.mix.{n}": w[f"l0.mix.{n}"] + 0.7}), ids).float(), ref)[1] > 1e-3, n


@pytest.mark.parametrize("heads,vdim,state,groups,ring", [(4, 24, 20, 2, 1), (2, 64, 128, 1, 1), (6, 32, 48, 3, 5), (3, 72, 64, 1, 2), (5, 5, 3, 5, 3),
                                                          (2, 130, 96, 2, 70), (2, 16, 150, 1, 2), (8, 64, 128, 2, 6)])
def test_recurrence_kernels_agree(heads, vdim, state, groups, ring):
    """bf16 engine: chunks on the tensor cores against position by position, from the same bf16 inputs; chunks that end inside
    a portion, portions that continue a state, states left for every entry of the ring"""
    cfg = config([ssd(heads, vdim, state, groups, 1, 4)])
    w = O.random_model(cfg, seed=27)
    w["l0.mix.dt_bias"] = torch.linspace(-6.0, 2.0, heads).to(torch.bfloat16)
    ids = tokens(300, 120, 28)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [64, 64, 128], [200, 63, 1, 1, 2, 33], [17] * 17, [100] + [1] * 5 + [65, 130]):
        got = [run_cuts(cfg, w, ids, cuts, dtype=torch.bfloat16, max_tokens=512, ring=ring, ssd_mode=mode) for mode in (0, 1)]
        assert rel_err(got[0], ref)[0] < 3e-2 and rel_err(got[0], got[1].cpu())[0] < 3e-3, cuts
    tail = tokens(20, 120, 29)
    for back in sorted({0, ring // 2, ring - 1}):        # any of the last `ring` positions may be followed by other tokens
        eng = make_engine(cfg, w, dtype=torch.bfloat16, max_tokens=512, ring=ring)
        slot = eng.open_sequence()
        feed(eng, slot, ids, [130, 170])
        got = feed(eng, slot, tail, [1, 19], start=300 - back)
        assert rel_err(got, oracle(cfg, w, ids[:300 - back] + tail)[300 - back:])[0] < 3e-2, back
        close(eng)


# ------------------------------------------------------------------------------------------------ cache and state
@pytest.mark.parametrize("cfg_dict", [SMALL, ODD, PLAIN], ids=["small", "odd", "plain"])
@pytest.mark.parametrize("page_size", [4, 16])
def test_prefill_then_decode_and_portions(cfg_dict, page_size):
    w = O.random_model(cfg_dict, seed=25)
    ids = tokens(61, cfg_dict["vocab"], 26)
    ref = oracle(cfg_dict, w, ids)
    for cuts in ([1] * 61, [40] + [1] * 21, [2] * 30, [3, 17, 2, 1, 1, 5, 2, 30], [16, 16, 16], [15, 17, 1, 16]):
        assert rel_err(run_cuts(cfg_dict, w, ids, cuts, page_size=page_size), ref)[1] < 2e-4, cuts


def test_forward_larger_than_the_engine_step_is_cut_inside():
    w = O.random_model(SMALL, seed=27)
    ids = tokens(100, 120, 28)
    assert rel_err(run_cuts(SMALL, w, ids, max_tokens=24), oracle(SMALL, w, ids))[1] < 2e-4


def test_batch_of_unequal_requests_equals_each_alone():
    w = O.random_model(SMALL, seed=29)
    seqs = [tokens(n, 120, 20 + n) for n in (31, 5, 1, 18)]
    refs = [oracle(SMALL, w, s) for s in seqs]
    for dtype in (torch.float32, torch.bfloat16):
        eng = make_engine(SMALL, w, max_tokens=32, dtype=dtype)
        slots = [eng.open_sequence() for _ in seqs]
        first = [12, 5, 1, 2]
        for sl, s in zip(slots, seqs):
            eng.reserve(sl, len(s))
        a = eng.forward_ragged([(sl, 0, s[:f], list(range(f))) for sl, s, f in zip(slots, seqs, first)])
        b = eng.forward_ragged([(sl, f, s[f:], list(range(len(s) - f))) for sl, s, f in zip(slots, seqs, first) if len(s) > f])
        oa = ob = 0
        for s, f, ref in zip(seqs, first, refs):
            got = a[oa:oa + f]
            oa += f
            if len(s) > f:
                got = torch.cat([got, b[ob:ob + len(s) - f]], 0)
                ob += len(s) - f
            assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 8e-2)
        close(eng)


def test_batched_single_token_and_few_token_steps():
    """decoding several sequences of unequal length together, then steps of two and of unequal few tokens"""
    for dtype in (torch.float32, torch.bfloat16):
        w = O.random_model(SMALL, seed=31)
        seqs = [tokens(n, 120, 40 + n) for n in (90, 47, 61, 34)]
        refs = [oracle(SMALL, w, s) for s in seqs]
        eng = make_engine(SMALL, w, max_tokens=256, dtype=dtype, page_size=8)
        slots = [eng.open_sequence() for _ in seqs]
        for sl, s in zip(slots, seqs):
            eng.reserve(sl, len(s))
        at = [len(s) - 26 for s in seqs]
        eng.forward_ragged([(sl, 0, s[:a], []) for sl, s, a in zip(slots, seqs, at)])
        got = [[] for _ in seqs]
        for sizes in ([1, 1, 1, 1],) * 12 + ([2, 2, 2, 2],) * 2 + ([4, 1, 3, 2], [1, 4, 2, 3], [3, 3, 3, 3], [2, 2, 2, 2]):
            out = eng.forward_ragged([(sl, a, s[a:a + n], list(range(n))) for sl, s, a, n in zip(slots, seqs, at, sizes)])
            o = 0
            for i, n in enumerate(sizes):
                got[i].append(out[o:o + n])
                o += n
                at[i] += n
        for g, s, ref, a in zip(got, seqs, refs, at):
            g = torch.cat(g, 0)
            r = ref[a - g.shape[0]:a]
            assert (rel_err(g, r)[1] < 2e-4) if dtype == torch.float32 else (rel_err(g, r)[0] < 8e-2)
        close(eng)


def test_prompt_beside_single_tokens_and_short_portions():
    """one step brings a long prompt, a long portion that continues a state, single tokens and two tokens; the step after
    it single tokens of all four"""
    w = O.random_model(SMALL, seed=32)
    seqs = [tokens(n, 120, 50 + n) for n in (90, 130, 41, 30)]
    refs = [oracle(SMALL, w, s) for s in seqs]
    for dtype in (torch.float32, torch.bfloat16):
        eng = make_engine(SMALL, w, max_tokens=256, dtype=dtype, page_size=8)
        slots = [eng.open_sequence() for _ in seqs]
        for sl, s in zip(slots, seqs):
            eng.reserve(sl, len(s))
        eng.forward_ragged([(slots[1], 0, seqs[1][:50], []), (slots[2], 0, seqs[2][:38], []), (slots[3], 0, seqs[3][:25], [])])
        at = [0, 50, 38, 25]
        for sizes in ((85, 75, 1, 2), (1, 1, 1, 1), (4, 4, 1, 2)):
            out = eng.forward_ragged([(sl, a, s[a:a + n], list(range(n))) for sl, s, a, n in zip(slots, seqs, at, sizes)])
            o = 0
            for i, n in enumerate(sizes):
                g, r = out[o:o + n], refs[i][at[i]:at[i] + n]
                o, at[i] = o + n, at[i] + n
                assert (rel_err(g, r)[1] < 2e-4) if dtype == torch.float32 else (rel_err(g, r)[0] < 8e-2), (i, sizes)
        close(eng)


def test_pages_slots_and_state_freed_and_used_again():
    """a pool with room for one request at a time: the second request gets the first one's slot, pages, carried inputs
    and states with the old contents still in them"""
    w = O.random_model(SMALL, seed=33)
    eng = make_engine(SMALL, w, page_size=4, num_pages=12, max_seqs=1, max_seq_len=48)
    for seed, n in ((30, 44), (31, 47), (32, 9), (33, 48), (34, 1), (35, 2)):
        ids = tokens(n, 120, seed)
        ref = oracle(SMALL, w, ids)
        slot = eng.open_sequence()
        assert slot == 0
        assert rel_err(feed(eng, slot, ids, [7, 1, 1, 13, 2] if n > 2 else [1]), ref)[1] < 2e-4
        eng.close_sequence(slot)
        assert eng.pages.pages_in_use() == 0
    from asd_b200._lib import AsdError
    slot = eng.open_sequence()
    with pytest.raises(AsdError):
        eng.reserve(slot, 49)
    close(eng)


def test_refeeding_recent_positions_finds_their_state():
    """rings of states and of carried inputs: after 30 tokens the last three are taken back and other tokens follow, as a
    verification step does after a rejected tail"""
    w = O.random_model(SMALL, seed=35)
    ids = tokens(30, 120, 36)
    new_tail = tokens(9, 120, 37)
    for cuts in ([11, 1, 6], [11, 1, 6, 8, 1, 1, 1, 1]):
        eng = make_engine(SMALL, w, ring=4)
        slot = eng.open_sequence()
        feed(eng, slot, ids, cuts)
        got = feed(eng, slot, new_tail, [4, 1], start=27)
        ref = oracle(SMALL, w, ids[:27] + new_tail)
        assert rel_err(got, ref[27:])[1] < 2e-4, cuts
        close(eng)


def test_refeeding_recent_positions_in_the_bf16_engine():
    """a prompt long enough for the chunked recurrence, then other tokens after each of the last positions"""
    w = O.random_model(SMALL, seed=37)
    ids = tokens(100, 120, 38)
    for back in (0, 1, 3):
        eng = make_engine(SMALL, w, ring=4, dtype=torch.bfloat16, max_tokens=128)
        slot = eng.open_sequence()
        feed(eng, slot, ids, [70, 30])
        tail = tokens(6, 120, 39)
        got = feed(eng, slot, tail, [2, 1, 3], start=100 - back)
        assert rel_err(got, oracle(SMALL, w, ids[:100 - back] + tail)[100 - back:])[0] < 8e-2, back
        close(eng)


def test_long_decoding_keeps_the_recurrent_state():
    """slow decays and one token with a large step size: what it wrote at position 0 is still in the state after hundreds of
    single-token steps"""
    cfg = config([ssd(2, 24, 16, 1, 1, 3), chk(chunk=50)])
    w = O.random_model(cfg, seed=39)
    w["l0.mix.dt_bias"] = torch.full_like(w["l0.mix.dt_bias"], -6.0)
    w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -1.0)
    sign = torch.randn(104, generator=torch.Generator().manual_seed(3)).sign()
    w["embed"][119] = (3 * sign).to(torch.bfloat16)
    w["l0.mix.in"][-2:] = (sign * 8 / 104).to(torch.bfloat16)
    ids = [119] + tokens(419, 119, 40)
    ref = oracle(cfg, w, ids)
    assert rel_err(oracle(cfg, w, [5] + ids[1:])[-1:].float(), ref[-1:])[1] > 5e-3      # the first token still matters
    assert rel_err(run_cuts(cfg, w, ids, [5] + [1] * 415, page_size=8), ref)[1] < 2e-4
    for cuts in ([400], [20] + [1] * 400):
        assert rel_err(run_cuts(cfg, w, ids, cuts, dtype=torch.bfloat16, max_tokens=512), ref)[0] < 5e-2


# ------------------------------------------------------------------------------------------------ standout keys
def plant(cfg, w, pairs, at=0, keys_at=0):
    """Gives every pair (key token, query token) a coordinate of its own in layer `at`: its queries hold the one's component
    there, the keys of layer `keys_at` the other's.  All other tokens share a large component that goes to a key coordinate
    no query looks at, so the norm of the keys leaves them small where queries look.  The coordinates lie beyond the
    rotated ones and the convolutions pass through."""
    m, D = cfg["layers"][at]["mixer"], cfg["width"]
    H, G, dk, r = m["heads"], m["kv_heads"], m["dim"], m["rot"]["dims"]
    g = torch.Generator().manual_seed(77)
    basis = torch.linalg.qr(torch.randn(D, D, generator=g))[0] * D ** 0.5           # columns with elements of order one
    V = cfg["vocab"]
    e = 0.3 * torch.randn(V, D, generator=g) + basis[:, 0]
    k, q = torch.zeros(G, dk, D), torch.zeros(H, dk, D)
    k[:, r] = basis[:, 0] / D
    for i, (kt, qt) in enumerate(pairs):
        u, v = basis[:, 2 * i + 1], basis[:, 2 * i + 2]
        e[kt], e[qt] = 2 * u, 2 * v + basis[:, 0]
        k[:, r + 1 + i] = u / D
        q[:, r + 1 + i] = v / D
    w["embed"] = (e / cfg["embedding"]["scale"]).to(torch.bfloat16)
    w[f"l{keys_at}.mix.k"], w[f"l{at}.mix.q"] = k.reshape(G * dk, D).to(torch.bfloat16), q.reshape(H * dk, D).to(torch.bfloat16)
    w[f"l{at}.mix.q.norm"] = torch.full_like(w[f"l{at}.mix.q.norm"], 4.0)
    w[f"l{keys_at}.mix.k.norm"] = torch.ones_like(w[f"l{keys_at}.mix.k.norm"])
    for i, n in ((at, "q"), (keys_at, "k")):
        for leaf in (".b", ".conv"):
            t = w.get(f"l{i}.mix.{n}{leaf}")
            if t is not None:
                w[f"l{i}.mix.{n}{leaf}"] = torch.zeros_like(t)
                if leaf == ".conv":
                    w[f"l{i}.mix.{n}{leaf}"][:, -1] = 1.0
    for i in {at, keys_at}:
        w[f"l{i}.norm1.alpha"] = torch.tensor(0.0625).to(torch.bfloat16)            # close to the identity
        w[f"l{i}.norm1"], w[f"l{i}.norm1.b"] = torch.full((D,), 16.0).to(torch.bfloat16), torch.zeros(D).to(torch.bfloat16)


def standout(cfg, w, where, n, dtype, page_size, cuts_list, pairs, moved=0.2):
    V = cfg["vocab"]
    ids = [t % (V - 2 * len(pairs)) for t in tokens(n, V, 42)]
    for (kt, qt), (kp, qp, _) in zip(pairs, where):
        ids[kp], ids[qp] = kt, qt
    ref = oracle(cfg, w, ids)
    for (kp, qp, seen) in where:        # the oracle says that the key decides the answer there, or is out of sight
        gone = list(ids)
        gone[kp] = 5
        d = rel_err(oracle(cfg, w, gone)[qp:qp + 1].float(), ref[qp:qp + 1])[1]
        assert (d > moved) == seen, (kp, qp, d)
    for cuts in cuts_list:
        got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=1024, max_seq_len=1024, page_size=page_size)
        if dtype == torch.float32:
            assert rel_err(got, ref)[1] < 1e-3
        for _, qp, _ in where:
            assert rel_err(got[qp:qp + 1], ref[qp:qp + 1])[1] < (1e-3 if dtype == torch.float32 else 0.1), (cuts, qp)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("page_size", [4, 16])
def test_standout_keys_far_back_and_at_page_borders(page_size, dtype):
    """one key with a weight near one among hundreds near zero: the sequence's first tokens, the last of a page, the first
    of the next, the query's neighbour; in a prompt, in portions and while decoding"""
    cfg = config([att(heads=4, kv_heads=2, dim=48, scale=0.25, conv=3, rot=16)], scale=2.0, mult=2.0)
    w = O.random_model(cfg, seed=41)
    V = cfg["vocab"]
    pairs = [(V - 1 - 2 * i, V - 2 - 2 * i) for i in range(7)]
    plant(cfg, w, pairs)
    where = [(0, 600, True), (20 * page_size - 1, 603, True), (20 * page_size, 606, True), (610, 611, True), (63, 613, True),
             (64, 616, True), (1, 619, True)]
    standout(cfg, w, where, 640, dtype, page_size, ((), [590] + [1] * 50, [37] * 18, [2] * 320, [598, 3, 4, 2, 4, 3]), pairs)


@pytest.mark.parametrize("shared", [False, True], ids=["own", "shared"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("chunk", [48, 70, 256])
def test_standout_keys_just_inside_and_outside_a_chunk(chunk, dtype, shared):
    """the first key of the query's chunk decides the answer, the last one of the chunk before is out of sight; queries at
    a chunk's last and inner positions, in prompts and while decoding, chunks counted from position 0 whatever the portions"""
    if shared:      # the second layer's mask decides; the first one's, which is wider or narrower, does not
        layers = [chk(4, 2, 32, 16, 0.25, chunk + 13, 20.0, 8), chk(8, 2, 32, 16, 0.25, chunk, 20.0, 8, of=0)]
    else:
        layers = [chk(4, 2, 32, 16, 0.25, chunk, 20.0, 8)]
    cfg = config(layers, scale=2.0, mult=2.0)
    w = O.random_model(cfg, seed=43)
    if shared:
        silence_mixer(cfg, w, 0)
    V = cfg["vocab"]
    pairs = [(V - 1 - 2 * i, V - 2 - 2 * i) for i in range(6)]
    plant(cfg, w, pairs, at=len(layers) - 1)
    c1, c2 = (560 // chunk) * chunk, (560 // chunk - 1) * chunk
    where = [(c1, c1 + 20, True), (c1 - 1, c1 + 22, False), (c2, c1 - 3, True), (c2 - 1, c1 - 5, False), (c2 + 7, c2 + chunk - 8, True),
             (c1 - 2, c1 + 1, False)]
    standout(cfg, w, where, c1 + 30, dtype, 16, ((), [c1 - 10] + [1] * 40, [37] * 20, [2] * 320, [c2 + 5, chunk - 3, 3, 4, 2, 9]), pairs)


def test_single_token_steps_with_key_shares_over_several_ctas():
    """few sequences and many keys: steps of one, two and four tokens cut the keys into shares for several CTAs and merge
    their results; two sequences of unequal length"""
    cfg = config([att(heads=4, kv_heads=2, dim=32, scale=0.3), chk(4, 2, 32, 40, 0.3, 700, 6.0)])
    w = O.random_model(cfg, seed=47)
    a, b = tokens(900, 120, 48), tokens(300, 120, 49)
    ra, rb = oracle(cfg, w, a), oracle(cfg, w, b)
    for dtype in (torch.float32, torch.bfloat16):
        for n in (1, 2, 4):
            eng = make_engine(cfg, w, dtype=dtype, max_tokens=1024, max_seq_len=1024)
            sa, sb = eng.open_sequence(), eng.open_sequence()
            eng.reserve(sa, 900), eng.reserve(sb, 300)
            eng.forward_ragged([(sa, 0, a[:868], []), (sb, 0, b[:268], [])])
            ga, gb = [], []
            for i in range(8):
                out = eng.forward_ragged([(sa, 868 + n * i, a[868 + n * i:868 + n * (i + 1)], list(range(n))),
                                          (sb, 268 + n * i, b[268 + n * i:268 + n * (i + 1)], list(range(n)))])
                ga.append(out[:n]), gb.append(out[n:])
            for got, ref in ((torch.cat(ga), ra[868:868 + 8 * n]), (torch.cat(gb), rb[268:268 + 8 * n])):
                assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 5e-2), n
            close(eng)


# ------------------------------------------------------------------------------------------------ random configurations
def random_config(seed):
    """layers in any order and number with sizes drawn at random (multiples of 16 and of nothing), shared keys"""
    g = torch.Generator().manual_seed(seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for i in range(pick([2, 3, 4, 5])):
        E = pick([1, 3, 8, 20])
        mlp = pick([None, dense(pick([24, 64, 100])), moe(E, pick([k for k in (1, 2, 3) if k <= E]), pick([16, 40, 64]), pick([0.5, 2.0, 7.0]))])
        kind, kv, dim = pick(["a", "s", "c", "c"]), pick([1, 2, 4]), pick([8, 16, 32, 48, 128])
        rot = pick([r for r in (0, 2, 8, 16, 32) if r <= dim])
        if kind == "a":
            layers.append(att(kv * pick([1, 2, 4]), kv, dim, pick([0.09, 0.3]), pick([1, 2, 4, 5]), rot, pick([50.0, 1e4, 1e6]), mlp))
        elif kind == "s":
            grp, v, H = pick([1, 2, 3]), pick([8, 16, 40, 64]), pick([1, 2, 4])
            layers.append(ssd(grp * H, v, pick([8, 16, 48, 72, 128]), grp, pick([n for n in (1, 2, 4) if grp * H * v % n == 0]), pick([1, 2, 4, 5]), mlp))
        else:
            own = [j for j in range(i) if layers[j]["type"] == "attention_2" and "kv_from" not in layers[j]["mixer"]]
            j = pick(own) if own else None
            if j is not None and pick([True, False]):
                e = copy.deepcopy(layers[j])
                e["mlp"] = mlp
                e["mixer"].update(kv_from=j, heads=e["mixer"]["kv_heads"] * pick([1, 2, 4]), mask={"size": pick([5, 32, 1000])})
                layers.append(e)
            else:
                yarn = pick([None, YARN, {"factor": 2.5, "original": 2000, "fast": 24.0, "slow": 1.5}])
                layers.append(chk(kv * pick([1, 2, 4]), kv, dim, pick([8, 16, 32, 64, 128, 20]), pick([0.09, 0.3]), pick([3, 16, 40, 64]),
                                  pick([2.0, 30.0]), rot, pick([50.0, 1e4, 1e6]), yarn, None, mlp))
    return config(layers, width=pick([48, 64, 80, 120, 128]), vocab=pick([50, 96, 257]), eps=pick([1e-5, 1e-6]),
                  scale=pick([0.4, 1.0, 3.0]), mult=pick([1.0, 0.5, 0.3]))


@pytest.mark.parametrize("seed", list(range(12)))
def test_configurations_drawn_at_random(seed):
    """what a checkpoint's config.json may say, drawn at random: whole prompt, prompt then single tokens, portions"""
    cfg = random_config(100 + seed)
    w = O.random_model(cfg, seed=200 + seed)
    ids = tokens(75, cfg["vocab"], 300 + seed)
    ref = oracle(cfg, w, ids)
    for dtype in (torch.float32, torch.bfloat16):
        for cuts in ((), [50] + [1] * 25, [37, 2, 3, 1, 1, 14, 2]):
            got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=128, page_size=8)
            if dtype == torch.float32:
                assert rel_err(got, ref)[1] < 3e-4, (cfg, cuts)
            else:       # a close choice of experts may fall the other way after bf16 roundings, at a few positions
                rows = (got.double().cpu() - ref).norm(dim=-1) / ref.norm(dim=-1)
                assert rows.median() < 4e-2 and rel_err(got, ref)[0] < 0.2, (cfg, cuts)


# ------------------------------------------------------------------------------------------------ bf16 engine
@pytest.mark.parametrize("tc", [1, 0], ids=["tcgen05", "cuda-cores"])
@pytest.mark.parametrize("cfg_dict", [SMALL, ODD], ids=["small", "odd"])
def test_bf16_engine_both_linear_paths(cfg_dict, tc):
    w = O.random_model(cfg_dict, seed=51)
    ids = tokens(90, cfg_dict["vocab"], 52)
    ref = oracle(cfg_dict, w, ids)
    for cuts in ((), [50] + [1] * 40, [7] * 13):
        got = run_cuts(cfg_dict, w, ids, cuts, dtype=torch.bfloat16, max_tokens=128, tc=tc).double().cpu()
        # a router choice between two near-equal scores may fall the other way after bf16 roundings and move that
        # position by more than rounding does: the bulk of the positions is held tighter than the whole
        rows = (got - ref).norm(dim=-1) / ref.norm(dim=-1)
        assert rows.median() < 3e-2 and rel_err(got, ref)[0] < 8e-2


def test_bf16_engine_on_sizes_that_fill_tensor_core_tiles():
    """multiples of 64: every projection and the expert layers take the tcgen05 kernels; 300 tokens take the
    tensor-bound CTA-pair GEMM"""
    cfg = config([att(4, 2, 64, 0.125, 4, 32, 1e4, moe(8, 2, 128, 2.0)), ssd(8, 64, 64, 1, 1, 4, dense(256)),
                  chk(4, 1, 128, 128, 0.09, 128, 30.0, 64, 1e5, YARN, None, dense(256)), ssd(4, 128, 128, 2, 2, 4)],
                 width=320, vocab=512)
    w = O.random_model(cfg, seed=53)
    ids = tokens(300, 512, 54)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [280] + [1] * 20, [150, 97, 40, 2, 2]):
        assert rel_err(run_cuts(cfg, w, ids, cuts, dtype=torch.bfloat16, max_tokens=512), ref)[0] < 5e-2


# ------------------------------------------------------------------------------------------------ entry points
def test_greedy_generation_through_stage_and_scheduler():
    """Stage.generate (byte tokenizer, ragged prefill, the step loop and the fused sampler at temperature 0) against
    greedy decoding with the oracle"""
    from asd_b200.models.nobonex import NobonexConfig
    from asd_b200.models.stage import Stage
    cfg_dict = copy.deepcopy(SMALL)
    cfg_dict["vocab"] = 256
    w = O.random_model(cfg_dict, seed=61)
    w["head"] = (w["head"].float() * 4).to(torch.bfloat16)          # spread logits: no near ties between arg-maxima
    st = Stage("unused", "nobonex-test", config=NobonexConfig.from_dict(cfg_dict), weights=w, max_batch=3, max_model_len=128, k=0)
    assert st.get_model_info()["family"] == "nobonex"
    prompts = ["abc", "hello world, this is longer", "z"]
    texts, _, stats = st.generate(prompts, max_tokens=12, temperature=0.0)
    assert stats["decode_steps"] >= 11
    ids = [list(p.encode()) for p in prompts]
    toks = st._generate_ids(ids, 12, 0.0)[0]
    for p, t, new in zip(ids, texts, toks):
        assert st.tokenizer.decode(new) == t and len(new) == 12
        # teacher-forced on the engine's own tokens: each one is the oracle's arg-max, or within bf16 noise of it
        lg = oracle(cfg_dict, w, p + new)
        for j, tok in enumerate(new):
            row = lg[len(p) + j - 1]
            assert row[tok] >= row.max() - 0.03 * row.std(), (j, tok, int(row.argmax()))
        assert sum(int(lg[len(p) + j - 1].argmax()) == tok for j, tok in enumerate(new)) >= 10


def test_speculative_decoding_with_a_nobonex_draft_equals_plain_greedy():
    """draft and target both carry recurrent states and convolution inputs; a rejected tail is re-fed from the rings"""
    from asd_b200.engine import NobonexEngine, SpecDecoder
    from asd_b200.models.nobonex import NobonexConfig
    tcfg = copy.deepcopy(SMALL)
    dcfg = config([ssd(1, 16, 8, 1, 1, 2), att(2, 1, 8, 0.3, 3, 4), chk(2, 1, 8, 8, 0.3, 10, 5.0, 4)])
    wt, wd = O.random_model(tcfg, seed=63), O.random_model(dcfg, seed=64)
    wt["head"] = (wt["head"].float() * 4).to(torch.bfloat16)
    prompts = [tokens(9, 120, 65), tokens(15, 120, 66)]

    def run(with_draft):
        kw = dict(max_seqs=2, max_seq_len=96, max_tokens=64, dtype=torch.float32, ring=6)     # fp32: no near ties
        mk = lambda c, w: NobonexEngine(NobonexConfig.from_dict(c), **kw).load_weights(w)
        t = mk(tcfg, wt)
        d = mk(dcfg, wd) if with_draft else None
        return SpecDecoder(t, d, 2, 3, temperature=0.0).generate(prompts, 16)[0].tolist()

    plain = run(False)
    assert run(True) == plain
    lg = oracle(tcfg, wt, prompts[0] + plain[0])
    assert sum(int(lg[len(prompts[0]) + j - 1].argmax()) == t for j, t in enumerate(plain[0])) >= 14


def write_checkpoint(path, cfg_dict, w):
    """config.json + model.safetensors (8-byte little-endian header length, JSON header, raw data)"""
    path.mkdir()
    (path / "config.json").write_text(json.dumps(cfg_dict))
    header, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    hj = json.dumps(header).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_command_on_a_checkpoint_directory(tmp_path, dtype):
    """the command-line runner end to end: registry by config.json, safetensors loader, page table with two requests one
    after the other (the second reuses the first one's slot, pages and state), portions down to one token, wanted rows only"""
    import numpy as np
    w = {k: v.to(torch.bfloat16) for k, v in O.random_model(ODD, seed=71).items()}
    write_checkpoint(tmp_path / "model", ODD, w)
    a, b = tokens(41, ODD["vocab"], 72), tokens(23, ODD["vocab"], 73)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:33], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[33:], "want": [7, 3]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [22]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype",
                        dtype, "--out", str(out), "--max-tokens", "48"], input="\n".join(json.dumps(x) for x in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(5)]
    ra, rb = oracle(ODD, w, a), oracle(ODD, w, b)
    want = {0: ra[[0, 29]], 2: ra[[32]], 3: ra[[40, 36]], 4: rb[[22]]}
    assert not (out / "1.f32").exists()
    for step, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(ref.shape[0], -1).copy())
        if dtype == "float32":
            assert rel_err(got, ref)[1] < 2e-4, step
        else:
            assert rel_err(got, ref)[0] < 5e-2, step
