"""GPU: the Dikopel engine against the plain restatement in oracle/dikopel_oracle.py (fp64, whole sequences, no cache).
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

from oracle import dikopel_oracle as O  # noqa: E402


# ------------------------------------------------------------------------------------------------ configurations
def dense(ff=48):
    return {"kind": "dense", "ff": ff} if ff else None


def moe(experts=9, top=3, ff=40, shared=24, count=3, keep=2, scale=1.5):
    f = {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale},
         "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def mlstm(heads=3, dim=24, vdim=40, cap=9.0, mlp=None, of=None):
    e = {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}
    if of is not None:
        e["weights_of"] = of
    return e


def par(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.25, r_heads=4, r_kv_heads=2, r_dim=16, r_vdim=24, conv=3, mlp=None,
        of=None):
    e = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale},
        "right": {"heads": r_heads, "kv_heads": r_kv_heads, "dim": r_dim, "vdim": r_vdim, "conv": conv}}}
    if of is not None:
        e["weights_of"] = of
    return e


def config(layers, width=104, vocab=120, eps=1e-5, scale=7.0, mult=0.6, taps=3):
    return {"architecture": "Dikopel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "canon": {"taps": taps}, "layers": layers}


# both mixers, every feed-forward kind, a layer that uses another one's weights on both sides
SMALL = config([mlstm(mlp=moe()), par(mlp=dense(72)), par(heads=2, kv_heads=2, dim=16, vdim=40, conv=4),
                mlstm(mlp=moe(), of=0), par(mlp=dense(72), of=1)])
# sizes that are multiples of nothing; weights of a later layer; one key head per query head and one for all; a single tap
# in both kinds of convolution; one group of experts, and groups of one
ODD = config([mlstm(heads=2, dim=10, vdim=7, cap=2.0, mlp=dense(50), of=3),
              par(heads=5, kv_heads=5, dim=10, vdim=6, scale=0.4, r_heads=3, r_kv_heads=3, r_dim=22, r_vdim=5, conv=1,
                  mlp=moe(7, 3, 9, 11, 7, 4, 1.0)),
              par(heads=6, kv_heads=1, dim=12, vdim=34, scale=0.5, r_heads=6, r_kv_heads=1, r_dim=6, r_vdim=70, conv=6,
                  mlp=moe(4, 2, 21, 0, 1, 1, 0.7)),
              mlstm(heads=2, dim=10, vdim=7, cap=2.0, mlp=dense(50)),
              mlstm(heads=1, dim=66, vdim=34, cap=30.0, mlp=moe(6, 1, 5, 3, 2, 1, 3.0))],
             width=72, vocab=101, eps=1e-3, scale=1.0, mult=1.0, taps=1)
PLAIN = config([par(), mlstm()], taps=5, mult=0.25)        # no feed-forward at all


def make_engine(cfg_dict, w, dtype=torch.float32, max_tokens=64, max_seq_len=512, page_size=16, num_pages=None,
                max_seqs=4, ring=1, tc=1):
    from asd_b200.engine import DikopelEngine
    from asd_b200.models.dikopel import DikopelConfig
    eng = DikopelEngine(DikopelConfig.from_dict(cfg_dict), max_seqs=max_seqs, max_seq_len=max_seq_len, max_tokens=max_tokens,
                        page_size=page_size, dtype=dtype, dynamic_pages=True, num_pages=num_pages, ring=ring)
    eng.load_weights(w)
    eng.set_option("tc_linear", tc)
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
@pytest.mark.parametrize("width,scale", [(40, 3.0), (41, 0.0), (128, 1.0)])
def test_embedding_sinusoids_and_final_layer_norm_alone(width, scale):
    """no layers: logits = head . norm(embed * scale + sinusoids), also at positions in the thousands"""
    cfg = config([], width=width, vocab=50, scale=scale)
    w = O.random_model(cfg, seed=3)
    ids = tokens(3000, 50, 4)
    ref = oracle(cfg, w, ids)
    got = run_cuts(cfg, w, ids, [1500], max_tokens=2048, max_seq_len=4096)
    assert rel_err(got[:64], ref[:64])[1] < 1e-4 and rel_err(got[-64:], ref[-64:])[1] < 1e-4
    assert changed(cfg, w, ids, ref, final__norm__b=torch.zeros(width)) > 1e-2
    shifted = oracle(cfg, w, ids[1:] + ids[:1])
    assert rel_err(shifted[100:101].float(), ref[101:102])[1] > 1e-2           # the same token one position earlier


def silence_mixer(cfg, w, i=0):
    for k in list(w):
        if k.startswith(f"l{i}.mix.") and k.rsplit(".", 1)[-1] == "o":
            w[k] = torch.zeros_like(w[k])


def test_gated_feed_forward_alone_and_residual_multiplier():
    for mult in (0.3, 1.0, 1.7):
        cfg = config([mlstm(mlp=dense(56))], mult=mult)
        w = O.random_model(cfg, seed=5, scale=2.0)
        silence_mixer(cfg, w)
        ids = tokens(33, 120, 6)
        ref = oracle(cfg, w, ids)
        assert rel_err(run_cuts(cfg, w, ids), ref)[1] < 2e-4
    c2 = dict(cfg, residual_mult=1.6)
    assert rel_err(oracle(c2, w, ids).float(), ref)[1] > 1e-2


@pytest.mark.parametrize("experts,top,ff,shared,count,keep,scale", [
    (9, 3, 40, 24, 3, 2, 1.5), (8, 2, 17, 0, 2, 1, 2.5), (9, 9, 8, 5, 3, 3, 1.0), (40, 3, 12, 7, 8, 2, 0.5), (2, 1, 64, 64, 1, 1, 1.0),
    (6, 2, 16, 16, 6, 3, 1.2), (64, 6, 9, 5, 4, 4, 2.0), (70, 4, 8, 3, 35, 2, 1.0)])
def test_routed_experts_alone(experts, top, ff, shared, count, keep, scale):
    """the correction decides who is chosen and stays out of the weights; choice scores may be negative; the shared
    expert has a gate of its own"""
    cfg = config([mlstm(mlp=moe(experts, top, ff, shared, count, keep, scale))])
    w = O.random_model(cfg, seed=7, scale=2.0)
    silence_mixer(cfg, w)
    g = torch.Generator().manual_seed(experts)
    w["l0.mlp.correction"] = (torch.randn(experts, generator=g) * 0.7 - 1.5).to(torch.bfloat16)
    ids = tokens(50, 120, 8)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 50):
        assert rel_err(run_cuts(cfg, w, ids, cuts), ref)[1] < 2e-4
    if top < experts:
        assert changed(cfg, w, ids, ref, l0__mlp__correction=torch.zeros(experts)) > 1e-2
    if keep < count and experts > count:          # groups of one expert exclude nobody who would be chosen
        c2 = copy.deepcopy(cfg)
        c2["layers"][0]["mlp"]["router"]["groups"]["keep"] = count
        assert rel_err(oracle(c2, w, ids).float(), ref)[1] > 1e-2
    if shared:
        assert changed(cfg, w, ids, ref, **{"l0__mlp__shared__sg": torch.zeros(1, 104)}) > 1e-2


def test_many_tokens_take_the_other_routing_kernel():
    cfg = config([mlstm(mlp=moe(16, 4, 24, 16, 4, 2, 1.5))])
    w = O.random_model(cfg, seed=9, scale=2.0)
    silence_mixer(cfg, w)
    ids = tokens(1400, 120, 10)
    assert rel_err(run_cuts(cfg, w, ids, max_tokens=2048, max_seq_len=2048), oracle(cfg, w, ids))[1] < 2e-4


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_input_convolution_alone_feeds_the_mixer_only(taps):
    """the mixer reads h + conv(h), the feed-forward h; a large oldest tap makes a lost or misplaced carried row show"""
    cfg = config([mlstm(mlp=dense(40)), par(mlp=dense(40))], taps=taps)
    w = O.random_model(cfg, seed=11)
    for i in range(2):
        t = w[f"l{i}.canon1"].float()
        t[:, 0] *= 4
        w[f"l{i}.canon1"] = t.to(torch.bfloat16)
    ids = tokens(40, 120, 12)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 40, [2] * 20, [taps, 1, taps, 3]):
        assert rel_err(run_cuts(cfg, w, ids, cuts), ref)[1] < 2e-4, cuts
    late = w["l0.canon1"].roll(1, 1) if taps > 1 else torch.zeros_like(w["l0.canon1"])
    assert changed(cfg, w, ids, ref, l0__canon1=late) > 1e-2


@pytest.mark.parametrize("heads,dim,vdim,cap", [(3, 24, 40, 9.0), (1, 64, 32, 15.0), (2, 130, 33, 1.5), (4, 16, 128, 30.0), (1, 300, 20, 5.0),
                                                (5, 5, 3, 15.0), (2, 32, 200, 4.0)])
def test_matrix_memory_alone(heads, dim, vdim, cap):
    cfg = config([mlstm(heads, dim, vdim, cap)])
    w = O.random_model(cfg, seed=13)
    # input gates of very different size: the running maximum jumps, decays back and stays, and the floor of the
    # denominator matters where the gates are small
    w["l0.mix.i"] = w["l0.mix.i"] * 4
    w["l0.mix.i.b"] = torch.linspace(-3.0, 3.0, heads).to(torch.bfloat16)
    ids = tokens(150, 120, 14)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 150, [2] * 75, [33, 3, 1, 1, 2], [32, 64, 31, 1], [64, 70]):
        assert rel_err(run_cuts(cfg, w, ids, cuts, max_tokens=256), ref)[1] < 2e-4, cuts
    assert changed(cfg, w, ids, ref, l0__mix__f__b=torch.full((heads,), -2.0)) > 1e-2


def test_matrix_memory_floor_and_first_maximum(monkeypatch):
    """small input gates: the denominator is its floor exp(-M), and M starts at 0; both show in the answer"""
    cfg = config([mlstm(2, 24, 16, 12.0)])
    w = O.random_model(cfg, seed=15)
    w["l0.mix.i.b"] = torch.tensor([-6.0, -9.0]).to(torch.bfloat16)
    w["l0.mix.norm"] = w["l0.mix.norm"] * 3
    ids = tokens(40, 120, 16)
    cfg["norm"]["eps"] = 1e-2                      # large beside the small results: their size reaches the answer
    ref = oracle(cfg, w, ids)
    assert rel_err(run_cuts(cfg, w, ids), ref)[1] < 2e-4
    assert rel_err(run_cuts(cfg, w, ids, [1] * 40), ref)[1] < 2e-4
    core = O.mlstm_core

    def no_floor(q, k, v, i, f):
        return core(q, k, v, i + 40.0, f)          # every gate far up: the floor never matters
    monkeypatch.setattr(O, "mlstm_core", no_floor)
    assert rel_err(oracle(cfg, w, ids).float(), ref)[1] > 1e-2


def silence(w, side):
    for k in list(w):
        if f".mix.{side}.out" in k:
            w[k] = torch.zeros_like(w[k])


@pytest.mark.parametrize("r_heads,r_kv,dim,vdim,conv", [(4, 2, 16, 24, 3), (3, 3, 20, 12, 2), (4, 1, 64, 40, 4), (2, 2, 130, 33, 1),
                                                        (1, 1, 300, 20, 7), (2, 1, 32, 130, 5)])
def test_gated_delta_rule_alone(r_heads, r_kv, dim, vdim, conv):
    cfg = config([par(r_heads=r_heads, r_kv_heads=r_kv, r_dim=dim, r_vdim=vdim, conv=conv)])
    w = O.random_model(cfg, seed=17)
    silence(w, "left")
    ids = tokens(70, 120, 18)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [1] * 70, [2] * 35, [33, 3, 1, 1, 2]):
        assert rel_err(run_cuts(cfg, w, ids, cuts, max_tokens=128), ref)[1] < 2e-4, cuts
    assert changed(cfg, w, ids, ref, l0__mix__right__A_log=torch.full((r_heads,), -6.0)) > 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("heads,kv,dim,vdim", [(6, 2, 24, 16), (4, 4, 32, 64), (8, 1, 64, 128), (20, 4, 16, 16), (12, 1, 40, 24),
                                               (24, 2, 16, 8), (5, 5, 10, 6), (2, 1, 136, 200), (34, 1, 16, 16), (3, 1, 8, 130)])
def test_sigmoid_attention_alone(heads, kv, dim, vdim, dtype):
    """every kernel: prompts, portions of a few tokens, single tokens; key and value sizes that fill a load and that do
    not; more than eight and more than sixteen query heads per key head"""
    cfg = config([par(heads, kv, dim, vdim, scale=1.5 / dim ** 0.5)])
    w = O.random_model(cfg, seed=19)
    silence(w, "right")
    w["l0.mix.left.pb"] = torch.linspace(-5.0, 1.0, heads).to(torch.bfloat16)
    ids = tokens(210, 120, 20)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [130] + [1] * 80, [2] * 105, [3, 64, 5, 7, 33, 4, 2, 1]):
        got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=256)
        assert (rel_err(got, ref)[1] < 2e-4) if dtype == torch.float32 else (rel_err(got, ref)[0] < 5e-2), cuts
    assert changed(cfg, w, ids, ref, l0__mix__left__pb=torch.zeros(heads)) > 1e-2


def test_attention_kernels_agree():
    """bf16 cache rows: the tensor-core kernels and the general CUDA-core kernel read the same cache and the same queries,
    so they differ by fp32 roundings only (option 2: few tokens on the CUDA cores, prompts on the tensor cores); prompts, portions that end inside a tile, few tokens and single ones"""
    for heads, kv, dim, vdim in ((4, 4, 32, 16), (6, 2, 16, 32), (8, 1, 64, 128), (16, 4, 48, 64), (3, 1, 80, 24), (32, 8, 32, 32),
                                 (24, 3, 16, 64), (18, 9, 16, 16), (20, 1, 48, 96)):
        cfg = config([par(heads, kv, dim, vdim, scale=1.0 / dim ** 0.5)])
        w = O.random_model(cfg, seed=55)
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
                assert rel_err(got[0], other.cpu())[0] < 2e-3, (heads, kv, cuts)


def test_two_branches_are_normed_and_averaged():
    cfg = config([par(mlp=dense(30))])
    w = O.random_model(cfg, seed=21)
    w["l0.mix.right.o"] = w["l0.mix.right.o"] * 30          # its norm takes the size away again
    ids = tokens(30, 120, 22)
    ref = oracle(cfg, w, ids)
    assert rel_err(run_cuts(cfg, w, ids), ref)[1] < 2e-4
    assert changed(cfg, w, ids, ref, l0__mix__left__out=w["l0.mix.left.out"] * 2) > 1e-2


def test_shared_weights_have_a_state_of_their_own():
    """the same tensors four times over: every layer keeps its own cache, carried inputs and states"""
    for entry in (mlstm(mlp=moe()), par(mlp=dense(40))):
        cfg = config([entry] + [dict(copy.deepcopy(entry), weights_of=j) for j in (0, 0, 2)])
        w = O.random_model(cfg, seed=23)
        assert not any(k.startswith("l1.") or k.startswith("l3.") for k in w)
        ids = tokens(50, 120, 24)
        ref = oracle(cfg, w, ids)
        for cuts in ((), [20] + [1] * 30, [7, 2, 2, 11]):
            assert rel_err(run_cuts(cfg, w, ids, cuts), ref)[1] < 2e-4, cuts


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


def test_long_decoding_keeps_the_recurrent_states():
    """slow decays: what the first tokens wrote is still in both states after hundreds of single-token steps"""
    cfg = config([mlstm(2, 24, 16), par(r_heads=2, r_kv_heads=1)])
    w = O.random_model(cfg, seed=39)
    w["l0.mix.f.b"] = torch.full_like(w["l0.mix.f.b"], 7.0)
    w["l0.mix.f"] = w["l0.mix.f"] * 0.1
    w["l1.mix.right.dt_bias"] = torch.full_like(w["l1.mix.right.dt_bias"], -7.0)
    ids = tokens(420, 120, 40)
    ref = oracle(cfg, w, ids)
    cut = [(ids[0] + 1) % 120] + ids[1:]
    other = oracle(cfg, w, cut)
    assert rel_err(other[-1:].float(), ref[-1:])[1] > 1e-3      # the first token still matters
    assert rel_err(run_cuts(cfg, w, ids, [5] + [1] * 415, page_size=8), ref)[1] < 2e-4
    got = run_cuts(cfg, w, ids, [400], dtype=torch.bfloat16, max_tokens=512)
    assert rel_err(got, ref)[0] < 5e-2


# ------------------------------------------------------------------------------------------------ standout keys
def plant(cfg, w, pairs, strength=9.0):
    """Gives every pair (key token, query token) a direction of its own: the first layer's keys hold the one's component,
    its queries the other's, in one coordinate, so their score stands out by tens among scores near zero; the head bias
    lies so low that only such a key has any weight."""
    m, D = cfg["layers"][0]["mixer"]["left"], cfg["width"]
    H, G, dk = m["heads"], m["kv_heads"], m["dim"]
    g = torch.Generator().manual_seed(77)
    basis = torch.linalg.qr(torch.randn(D, D, generator=g))[0]
    basis = basis - basis.mean(0, keepdim=True)
    k = torch.zeros(G, dk, D)
    q = torch.zeros(H, dk, D)
    for i, (kt, qt) in enumerate(pairs):
        u, v = basis[:, 2 * i] / basis[:, 2 * i].norm(), basis[:, 2 * i + 1] / basis[:, 2 * i + 1].norm()
        w["embed"][kt] = (u * D ** 0.5 * 4).to(torch.bfloat16)
        w["embed"][qt] = (v * D ** 0.5 * 4).to(torch.bfloat16)
        k[:, i] += u
        q[:, i] += v * strength / D / m["scale"] * 2
    w["l0.mix.left.k"], w["l0.mix.left.q"] = k.reshape(G * dk, D).to(torch.bfloat16), q.reshape(H * dk, D).to(torch.bfloat16)
    w["l0.mix.left.pb"] = torch.full((H,), -10.0).to(torch.bfloat16)
    w["l0.canon1"] = torch.zeros_like(w["l0.canon1"])
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(D).to(torch.bfloat16), torch.zeros(D).to(torch.bfloat16)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
@pytest.mark.parametrize("page_size", [4, 16])
def test_standout_keys_far_back_and_at_page_borders(page_size, dtype):
    """one key with a weight near one among hundreds near zero: the sequence's first token, the last of a page, the first
    of the next, the query's neighbour and the query itself; in a prompt, in portions and while decoding"""
    cfg = config([par(heads=4, kv_heads=2, dim=48, vdim=16, scale=0.25)], scale=2.0, mult=8.0)
    w = O.random_model(cfg, seed=41)
    silence(w, "right")
    V, n = cfg["vocab"], 640
    pairs = [(V - 1 - 2 * i, V - 2 - 2 * i) for i in range(6)]
    plant(cfg, w, pairs)
    ids = [t % (V - 12) for t in tokens(n, V, 42)]
    where = [(0, 600), (20 * page_size - 1, 603), (20 * page_size, 606), (610, 611), (63, 613), (64, 616)]
    for (kt, qt), (kp, qp) in zip(pairs, where):
        ids[kp], ids[qp] = kt, qt
    ref = oracle(cfg, w, ids)
    for (kt, qt), (kp, qp) in zip(pairs, where):        # the oracle says that the key decides the answer there
        gone = list(ids)
        gone[kp] = 5
        assert rel_err(oracle(cfg, w, gone)[qp:qp + 1].float(), ref[qp:qp + 1])[1] > 0.2, (kp, qp)
    for cuts in ((), [590] + [1] * 50, [37] * 18, [2] * 320, [598, 3, 4, 2, 4, 3]):
        got = run_cuts(cfg, w, ids, cuts, dtype=dtype, max_tokens=1024, max_seq_len=1024, page_size=page_size)
        if dtype == torch.float32:
            assert rel_err(got, ref)[1] < 1e-3
        for _, qp in where:
            assert rel_err(got[qp:qp + 1], ref[qp:qp + 1])[1] < (1e-3 if dtype == torch.float32 else 0.1), (cuts, qp)


def test_single_token_steps_with_key_shares_over_several_ctas():
    """few sequences and many keys: steps of one, two and four tokens cut the keys into shares for several CTAs and add
    their results; two sequences of unequal length"""
    cfg = config([par(heads=4, kv_heads=2, dim=32, vdim=40, scale=0.3)])
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
    """layers in any order and number with sizes drawn at random (multiples of 16 and of nothing), shared weights"""
    g = torch.Generator().manual_seed(seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    n = pick([2, 3, 4, 5])
    layers = []
    for i in range(n):
        own = [j for j in range(i) if "weights_of" not in layers[j]]
        if own and pick([True, False, False]):
            j = pick(own)
            layers.append(dict(copy.deepcopy(layers[j]), weights_of=j))
            continue
        count = pick([1, 2, 4])
        per = pick([1, 2, 3, 5])
        keep = pick(list(range(1, count + 1)))
        mlp = pick([None, dense(pick([24, 64, 100])),
                    moe(count * per, pick(list(range(1, keep * per + 1))), pick([16, 40, 64]), pick([0, 32, 50]), count, keep,
                        pick([1.0, 2.5]))])
        if pick([True, False]):
            layers.append(mlstm(pick([1, 2, 4, 5]), pick([8, 16, 48, 72, 128]), pick([8, 16, 32, 40, 64, 96]), pick([3.0, 15.0, 40.0]), mlp))
        else:
            kv, rk = pick([1, 2, 4]), pick([1, 2, 3])
            dim = pick([8, 16, 32, 48, 128])
            layers.append(par(kv * pick([1, 2, 4]), kv, dim, pick([8, 16, 32, 64, 128, 20]), pick([0.09, 0.3]), rk * pick([1, 2, 4]), rk,
                              pick([8, 16, 40, 64]), pick([8, 16, 40, 64]), pick([1, 2, 4, 5]), mlp))
    return config(layers, width=pick([48, 64, 80, 120, 128]), vocab=pick([50, 96, 257]), eps=pick([1e-5, 1e-6]),
                  scale=pick([1.0, 5.0, 11.3]), mult=pick([1.0, 0.5, 0.3]), taps=pick([1, 2, 4, 5]))


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
    cfg = config([mlstm(4, 64, 64, 15.0, moe(8, 2, 128, 128, 2, 1, 1.0)),
                  par(4, 2, 64, 64, 0.125, 4, 2, 64, 64, 4, dense(256)), mlstm(2, 128, 128, 15.0, dense(256))],
                 width=256, vocab=512, taps=4)
    w = O.random_model(cfg, seed=53)
    ids = tokens(300, 512, 54)
    ref = oracle(cfg, w, ids)
    for cuts in ((), [280] + [1] * 20, [150, 97, 40, 2, 2]):
        assert rel_err(run_cuts(cfg, w, ids, cuts, dtype=torch.bfloat16, max_tokens=512), ref)[0] < 5e-2


# ------------------------------------------------------------------------------------------------ entry points
def test_greedy_generation_through_stage_and_scheduler():
    """Stage.generate (byte tokenizer, ragged prefill, the step loop and the fused sampler at temperature 0) against
    greedy decoding with the oracle"""
    from asd_b200.models.dikopel import DikopelConfig
    from asd_b200.models.stage import Stage
    cfg_dict = copy.deepcopy(SMALL)
    cfg_dict["vocab"] = 256
    w = O.random_model(cfg_dict, seed=61)
    w["head"] = (w["head"].float() * 4).to(torch.bfloat16)          # spread logits: no near ties between arg-maxima
    st = Stage("unused", "dikopel-test", config=DikopelConfig.from_dict(cfg_dict), weights=w, max_batch=3, max_model_len=128, k=0)
    assert st.get_model_info()["family"] == "dikopel"
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


def test_speculative_decoding_with_a_dikopel_draft_equals_plain_greedy():
    """draft and target both carry recurrent states and convolution inputs; a rejected tail is re-fed from the rings"""
    from asd_b200.engine import DikopelEngine, SpecDecoder
    from asd_b200.models.dikopel import DikopelConfig
    tcfg = copy.deepcopy(SMALL)
    dcfg = config([mlstm(1, 16, 8), par(heads=2, kv_heads=1, dim=8, vdim=8, r_heads=1, r_kv_heads=1, r_dim=8, r_vdim=8)])
    wt, wd = O.random_model(tcfg, seed=63), O.random_model(dcfg, seed=64)
    wt["head"] = (wt["head"].float() * 4).to(torch.bfloat16)
    prompts = [tokens(9, 120, 65), tokens(15, 120, 66)]

    def run(with_draft):
        kw = dict(max_seqs=2, max_seq_len=96, max_tokens=64, dtype=torch.float32, ring=6)     # fp32: no near ties
        mk = lambda c, w: DikopelEngine(DikopelConfig.from_dict(c), **kw).load_weights(w)
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
        raw = t.to(torch.bfloat16).contiguous().view(torch.uint8).numpy().tobytes()
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
