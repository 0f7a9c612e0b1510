"""CPU: the Nobonex family's configuration, registry entry, tensor packing and shared keys, and the plain restatement's
own mechanisms on inputs made by hand (so that the oracle the GPU tests lean on is itself pinned)."""
import json
import math

import pytest
import torch

from oracle import nobonex_oracle as O

F64 = torch.float64


def t64(x):
    return torch.tensor(x, dtype=F64)


def test_config_round_trip_and_registry(tmp_path):
    from asd_b200.models import registry
    from asd_b200.models.nobonex import NobonexConfig, sized_config, tensor_shapes, tiny_config
    for cfg in (tiny_config(), sized_config(256, 7, 4, vocab=64, dim=32, experts=4)):
        d = cfg.to_dict()
        assert d["architecture"] == "Nobonex"
        assert NobonexConfig.from_dict(json.loads(json.dumps(d)), name=cfg.name) == cfg
        assert O.tensor_shapes(d) == tensor_shapes(cfg)
        fam = registry.family_of_dict(d)
        assert fam.name == "nobonex" and "nobonex" in fam.components and set(fam.dtypes) == {"bfloat16", "float32"}
        assert registry.family_of_config(cfg).name == "nobonex"
    (tmp_path / "config.json").write_text(json.dumps(d))
    fam2, cfg2 = registry.read_config(str(tmp_path))
    assert fam2.name == "nobonex" and cfg2.layers == cfg.layers


def test_defaults_of_absent_keys_and_refusals():
    from asd_b200.models.nobonex import NobonexConfig, tiny_config
    d = tiny_config().to_dict()
    m = [e["mixer"] for e in d["layers"]]
    del m[0]["kv_heads"], m[0]["vdim"], m[0]["rot"], m[1]["norm_groups"], m[2]["rot"]["scaling"]
    d["layers"] = d["layers"][:3]
    d["layers"][2]["mlp"] = None
    l = NobonexConfig.from_dict(d).layers
    assert l[0].kv_heads == l[0].heads and l[0].vdim == l[0].dim and l[0].rot_dims == 0 and l[0].kv_from == -1
    assert l[1].norm_groups == 1 and l[2].yarn is None and l[2].ff_kind is None

    def mixer(i, **kw):
        return lambda b: b["layers"][i]["mixer"].update(kw)
    for change in (lambda b: b["layers"][0].update(type="convolution"), lambda b: b["layers"][1]["mlp"].update(kind="sparse"),
                   mixer(0, vdim=8), mixer(3, kv_from=0), mixer(3, kv_from=1), mixer(3, kv_from=3), mixer(3, kv_from=9),
                   mixer(2, kv_from=3), mixer(3, dim=16), mixer(3, kv_heads=4), mixer(3, vdim=32)):
        bad = json.loads(json.dumps(tiny_config().to_dict()))
        change(bad)
        with pytest.raises(ValueError):
            NobonexConfig.from_dict(bad)


def test_a_layer_that_reads_another_cache_has_no_keys_of_its_own():
    from dataclasses import replace

    from asd_b200.models.nobonex import tensor_shapes, tiny_config
    own = tiny_config().layers[2]
    one, two = tiny_config(layers=[own]), tiny_config(layers=[own, replace(own, kv_from=0), replace(own, kv_from=0, heads=8)])
    assert two.kv_bytes_per_token() == one.kv_bytes_per_token() > 0
    names = {k for k in tensor_shapes(two) if k.startswith("l1.mix.")}
    assert names == {"l1.mix." + n for n in ("q", "q.b", "q.norm", "g", "o")}
    assert two.layers[2].in_rows == 8 * (own.dim + own.vdim) and own.in_rows == 4 * (own.dim + own.vdim) + own.cache_row


def test_packing_stacks_projections_and_experts():
    from asd_b200.models.nobonex import pack, random_weights, tensor_shapes, tiny_config
    cfg = tiny_config()
    w = random_weights(cfg, seed=1)
    p = pack(w, cfg, "cpu", torch.float32)
    a, s, c, r = cfg.layers
    for i, l in enumerate(cfg.layers):
        assert p[(i, "w_in")].shape == (l.in_rows, cfg.width)
        assert p[(i, "norm1_alpha")].shape == (1,) and p[(i, "norm1b")].shape == (cfg.width,)
    nq = a.heads * a.dim
    assert torch.equal(p[(0, "w_in")][nq:], w["l0.mix.k"].float()) and p[(0, "conv_w")].shape == (a.conv_channels, a.conv)
    assert torch.equal(p[(1, "w_in")], w["l1.mix.in"].float()) and p[(1, "conv_b")].shape == (s.conv_channels,)
    nq = c.heads * c.dim
    assert torch.equal(p[(2, "w_in")][-c.heads * c.vdim:], w["l2.mix.g"].float())
    assert torch.equal(p[(2, "in_bias")], torch.cat([w[f"l2.mix.{n}.b"] for n in "qkv"]).float())
    assert torch.equal(p[(3, "in_bias")], w["l3.mix.q.b"].float()) and (3, "k_norm") not in p
    assert p[(1, "w_egu")].shape == (s.experts, 2 * s.expert_ff, cfg.width)
    assert torch.equal(p[(1, "w_egu")][3, s.expert_ff:], w["l1.mlp.e3.up"].float())
    assert torch.equal(p[(0, "w_gu")][:a.ff], w["l0.mlp.gate"].float())
    assert (3, "w_gu") not in p and (3, "norm2") not in p
    bad = dict(w)
    bad["l1.mix.D"] = torch.zeros(s.heads + 1)
    with pytest.raises(ValueError):
        pack(bad, cfg, "cpu", torch.float32)
    del bad["l1.mix.D"]
    with pytest.raises(KeyError):
        pack(bad, cfg, "cpu", torch.float32)
    assert set(tensor_shapes(cfg)) == set(w)


def test_library_components_of_the_family():
    import importlib.util
    import os
    here = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "adaptive-speculative-decoding_b200", "build.py")
    spec = importlib.util.spec_from_file_location("asd_build", here)
    b = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(b)
    names = {os.path.basename(s) for s in b.sources(("nobonex",))}
    assert {"nobonex_engine.cu", "ssd.cu", "ssd_chunk.cu", "delta_rule.cu", "decode_attention_tc.cu", "moe.cu", "gemm.cu"} <= names
    assert not names & {"engine.cu", "dikopel_engine.cu", "mlstm.cu", "talking_attention.cu", "sampler.cu"}


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_oracle_dynamic_tanh_by_hand():
    w = {"n": t64([1.0, 2.0, 3.0]), "n.b": t64([0.0, 0.5, 0.0]), "n.alpha": t64(0.5)}
    got = O.dynamic_tanh(t64([[2.0, -4.0, 1e9]]), w, "n")
    assert torch.allclose(got, t64([[math.tanh(1.0), 0.5 - 2 * math.tanh(2.0), 3.0]]))


def test_oracle_convolution_weighs_the_current_position_last():
    x = t64([[1.0], [10.0], [100.0], [1000.0]])
    assert O.causal_conv(x, t64([[3.0, 2.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0, 123.0, 1230.0]
    assert O.causal_conv(x[:2], t64([[5.0, 4.0, 3.0, 2.0, 1.0]]), t64([7.0]))[:, 0].tolist() == [8.0, 19.0]


def test_oracle_rotation_of_both_layouts():
    x = torch.arange(1.0, 7.0, dtype=F64).reshape(1, 1, 6).repeat(3, 1, 1)
    rot = {"dims": 4, "base": 100.0}
    inter, half = O.rotate(x, rot, True), O.rotate(x, rot, False)
    for p in range(3):
        for i, (a, b, u, v) in enumerate(((0, 1, 1.0, 2.0), (2, 3, 3.0, 4.0))):
            c, s = math.cos(p * 100.0 ** (-i / 2)), math.sin(p * 100.0 ** (-i / 2))
            assert torch.allclose(inter[p, 0, [a, b]], t64([u * c - v * s, v * c + u * s]))
        for i, (a, b, u, v) in enumerate(((0, 2, 1.0, 3.0), (1, 3, 2.0, 4.0))):
            c, s = math.cos(p * 100.0 ** (-i / 2)), math.sin(p * 100.0 ** (-i / 2))
            assert torch.allclose(half[p, 0, [a, b]], t64([u * c - v * s, v * c + u * s]))
    assert inter[2, 0, 4:].tolist() == half[2, 0, 4:].tolist() == [5.0, 6.0]
    assert torch.equal(O.rotate(x, None, True), x)


def test_oracle_scaled_frequencies_by_hand():
    """base e^2 over 8 dims: a pair turns t times in n positions at index 2 ln(n / (2 pi t))"""
    base, n = math.exp(2.0), 2 * math.pi * math.exp(1.75)
    freq = [base ** (-2 * i / 8) for i in range(4)]
    out, mag = O.yarn(freq, base, 8, {"factor": 5.0, "original": n, "fast": math.exp(0.9), "slow": 1.0})
    # fast at 1.7 -> 1, slow at 3.5 -> 4: the ramp runs over the indices 1 .. 4
    want = [freq[0], freq[1], freq[2] * (2 / 3 + 1 / 15), freq[3] * (1 / 3 + 2 / 15)]
    assert torch.allclose(t64(out), t64(want)) and math.isclose(mag, 0.1 * math.log(5.0) + 1)
    out, _ = O.yarn(freq, base, 8, {"factor": 5.0, "original": 1e9, "fast": 2.0, "slow": 1.0})     # all pairs turn fast
    assert torch.allclose(t64(out), t64(freq))


def test_oracle_visibility():
    assert O.visible(4, 0).long().sum(1).tolist() == [1, 2, 3, 4]
    assert O.visible(7, 3).long().sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1]
    assert O.visible(7, 3)[4].tolist() == [False, False, False, True, True, False, False]


def test_oracle_softmax_attention_by_hand():
    q, k, v = t64([[[2.0], [4.0]], [[1.0], [-1.0]]]), t64([[[1.0]], [[3.0]]]), t64([[[10.0]], [[20.0]]])
    got = O.softmax_attention(q, k, v, 0.5, O.visible(2, 0), 2.0)
    assert got[0].tolist() == [10.0, 10.0]
    for h, qv in enumerate((1.0, -1.0)):
        e = [math.exp(2 * math.tanh(qv * kv * 0.5 / 2)) for kv in (1.0, 3.0)]
        assert math.isclose(got[1, h].item(), (10 * e[0] + 20 * e[1]) / sum(e))


def test_oracle_values_are_the_convolved_keys():
    """one head, two coordinates, one visible position: the answer is the key before its norm"""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "conv": 1}
    w = {"q": torch.eye(2, dtype=F64), "k": t64([[2.0, 0.0], [0.0, 3.0]]), "o": torch.eye(2, dtype=F64), "q.norm": t64([1.0, 1.0]),
         "k.norm": t64([9.0, 9.0]), "q.conv": t64([[1.0], [1.0]]), "k.conv": t64([[10.0], [100.0]])}
    assert torch.allclose(O.conv_attention(t64([[1.0, 1.0]]), w, m, 0.0), t64([[20.0, 300.0]]))


def test_oracle_gate_and_shared_keys():
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 5}, "softcap": 9.0}
    one = t64([[1.0]])
    w = {n: one for n in ("q", "k", "v", "o")} | {n + ".b": t64([0.5]) for n in "qkv"} | {"q.norm": t64([1.0]), "k.norm": t64([1.0]), "g": 2 * one}
    y, kv = O.chunk_attention(3 * one, w, m, 0.0)
    assert math.isclose(y.item(), 3.5 / (1 + math.exp(-6.0))) and kv[0].item() == 1.0 and kv[1].item() == 3.5
    y, _ = O.chunk_attention(3 * one, {k: t for k, t in w.items() if k[0] not in "kv"}, m, 0.0, (kv[0], 2 * kv[1]))
    assert math.isclose(y.item(), 7.0 / (1 + math.exp(-6.0)))


def test_oracle_state_space_recurrence_by_hand():
    """one channel: S <- exp(-e^A dt) S + dt B x, y = C S + D x"""
    one = torch.ones(3, 1, 1, dtype=F64)
    A, dt = math.log(math.log(2.0)), torch.ones(3, 1, dtype=F64)          # the state halves in every step
    y = O.ssd_core(8 * one, one, 2 * one, dt, t64([A]), t64([0.5]))
    assert torch.allclose(y[:, 0, 0], t64([20.0, 28.0, 32.0]))
    y = O.ssd_core(8 * one, one, 2 * one, 2 * dt, t64([A]), t64([0.0]))
    assert torch.allclose(y[:, 0, 0], t64([32.0, 40.0, 42.0]))
    x = t64([[[1.0], [1.0], [1.0], [1.0]]])                                # four heads over two groups
    y = O.ssd_core(x, t64([[[1.0], [2.0]]]), t64([[[1.0], [3.0]]]), torch.ones(1, 4, dtype=F64), torch.zeros(4, dtype=F64), torch.zeros(4, dtype=F64))
    assert y[0, :, 0].tolist() == [1.0, 1.0, 6.0, 6.0]


def test_oracle_gate_comes_before_the_grouped_norm():
    m = {"heads": 2, "vdim": 1, "state": 1, "groups": 1, "norm_groups": 2, "conv": 1}
    # z = (1, 2), x = (3, 4), B = C = 0 before silu, dt = 0: y = D x with D = 1
    w = {"in": t64([[1.0], [2.0], [3.0], [4.0], [0.0], [0.0], [0.0], [0.0]]), "conv": torch.ones(4, 1, dtype=F64), "conv.b": torch.zeros(4, dtype=F64),
         "dt_bias": torch.zeros(2, dtype=F64), "A_log": torch.zeros(2, dtype=F64), "D": torch.ones(2, dtype=F64), "norm": t64([5.0, 7.0]),
         "o": torch.eye(2, dtype=F64)}
    assert torch.allclose(O.mamba2_mixer(t64([[1.0]]), w, m, 0.0), t64([[5.0, 7.0]]))           # parts of one: everything becomes its sign
    got = O.mamba2_mixer(t64([[1.0]]), w, dict(m, norm_groups=1), 0.0)
    sl = lambda v: v / (1 + math.exp(-v))
    v = t64([sl(3.0) * sl(1.0), sl(4.0) * sl(2.0)])
    assert torch.allclose(got[0], v / (v * v).mean().sqrt() * t64([5.0, 7.0]))


def test_oracle_expert_clamps_and_weighted_input():
    w = {"gate": t64([[2.0]]), "up": t64([[-3.0]]), "down": t64([[10.0]])}
    sg = lambda v: 1 / (1 + math.exp(-v))
    assert math.isclose(O.expert(t64([[0.5]]), w, 7.0).item(), 10 * sg(1.702) * (1 - 1.5))
    assert math.isclose(O.expert(t64([[5.0]]), w, 2.0).item(), 10 * 2 * sg(3.404) * (1 - 2.0))         # both clamped
    assert math.isclose(O.expert(t64([[-5.0]]), w, 2.0).item(), 10 * -10 * sg(-17.02) * 3.0)           # the gate only from above
    f = {"kind": "moe", "router": {"experts": 2, "top": 1}, "expert": {"ff": 1, "limit": 7.0}}
    ws = {"router": t64([[1.0], [-1.0]])} | {f"e{i}.{k}": t * (1 + i) for i in range(2) for k, t in w.items()}
    got = O.feed_forward(t64([[0.5], [-0.5]]), ws, f)
    assert math.isclose(got[0].item(), O.expert(t64([[0.5 * sg(0.5)]]), w, 7.0).item())
    assert math.isclose(got[1].item(), O.expert(t64([[-0.5 * sg(0.5)]]), {k: 2 * t for k, t in w.items()}, 7.0).item())


def test_oracle_layer_norms_before_and_after_each_sublayer():
    cfg = {"width": 4, "vocab": 5, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0}, "residual_mult": 0.5,
           "layers": [{"type": "mamba2", "mixer": {"heads": 1, "vdim": 2, "state": 3, "groups": 1, "norm_groups": 1, "conv": 2},
                       "mlp": {"kind": "dense", "ff": 6}}]}
    w = {k: t.to(F64) for k, t in O.random_model(cfg, seed=2).items()}
    ids, streams = [1, 4, 2], []
    O.forward(cfg, w, ids, layers_out=streams)
    x, n = w["embed"][ids] * 2.0, O.sub(w, "l0.")
    x = x + 0.5 * O.dynamic_tanh(O.mamba2_mixer(O.dynamic_tanh(x, n, "norm1"), O.sub(n, "mix."), cfg["layers"][0]["mixer"], 1e-5), n, "norm1b")
    x = x + 0.5 * O.dynamic_tanh(O.gated_ff(O.dynamic_tanh(x, n, "norm2"), O.sub(n, "mlp.")), n, "norm2b")
    assert torch.allclose(streams[0], x)
