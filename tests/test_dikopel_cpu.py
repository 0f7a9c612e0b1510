"""CPU: the Dikopel family's configuration, registry entry, tensor packing and shared layer weights, and the plain
restatement's own mechanisms on inputs made by hand (so that the oracle the GPU tests lean on is itself pinned)."""
import json
import math

import pytest
import torch

from oracle import dikopel_oracle as O

F64 = torch.float64


def t64(x):
    return torch.tensor(x, dtype=F64)


def test_config_round_trip_and_registry(tmp_path):
    from asd_b200.models import registry
    from asd_b200.models.dikopel import DikopelConfig, tensor_shapes, tiny_config
    cfg = tiny_config()
    d = cfg.to_dict()
    assert d["architecture"] == "Dikopel"
    assert DikopelConfig.from_dict(json.loads(json.dumps(d)), name="tiny") == cfg
    fam = registry.family_of_dict(d)
    assert fam.name == "dikopel" and "dikopel" in fam.components and set(fam.dtypes) == {"bfloat16", "float32"}
    assert registry.family_of_config(cfg).name == "dikopel"
    assert O.tensor_shapes(d) == tensor_shapes(cfg)
    (tmp_path / "config.json").write_text(json.dumps(d))
    fam2, cfg2 = registry.read_config(str(tmp_path))
    assert fam2.name == "dikopel" and cfg2.layers == cfg.layers


def test_defaults_of_absent_keys_and_refusals():
    from asd_b200.models.dikopel import DikopelConfig, tiny_config
    d = tiny_config().to_dict()
    d["layers"] = d["layers"][:3]
    m = d["layers"][1]["mixer"]
    del m["left"]["kv_heads"], m["left"]["vdim"], m["right"]["kv_heads"], m["right"]["vdim"], d["layers"][0]["mixer"]["vdim"]
    del d["layers"][0]["mlp"]["router"]["groups"], d["layers"][0]["mlp"]["shared"]
    cfg = DikopelConfig.from_dict(d)
    l = cfg.layers[1]
    assert l.a_kv_heads == l.a_heads and l.a_vdim == l.a_dim and l.r_kv_heads == l.r_heads and l.r_vdim == l.r_dim
    assert cfg.layers[0].vdim == cfg.layers[0].dim and (cfg.layers[0].groups, cfg.layers[0].keep, cfg.layers[0].shared_ff) == (1, 1, 0)
    assert cfg.layers[2].ff_kind is None and cfg.layers[2].weights_of == -1
    for change in (lambda b: b["layers"][0].update(type="convolution"), lambda b: b["layers"][1]["mlp"].update(kind="sparse"),
                   lambda b: b["layers"][3].update(weights_of=4), lambda b: b["layers"][3].update(weights_of=3),
                   lambda b: b["layers"][3].update(weights_of=1), lambda b: b["layers"][0].update(weights_of=3)):
        bad = json.loads(json.dumps(tiny_config().to_dict()))
        change(bad)
        with pytest.raises(ValueError):
            DikopelConfig.from_dict(bad)


def test_a_shared_layer_has_no_tensors_and_a_cache_of_its_own():
    from dataclasses import replace

    from asd_b200.models.dikopel import tensor_shapes, tiny_config
    cfg = tiny_config()
    par = cfg.layers[1]
    two = tiny_config(layers=[par, replace(par, weights_of=0), replace(par, weights_of=1)])
    assert two.runs() == [(0, -1)] * 3 and [O.owner(two.to_dict(), i) for i in range(3)] == [0, 0, 0]
    one = tiny_config(layers=[par])
    assert tensor_shapes(two) == tensor_shapes(one)
    assert two.kv_bytes_per_token() == 3 * one.kv_bytes_per_token()
    assert cfg.runs() == [(0, -1), (1, -1), (2, -1), (0, -1)]


def test_packing_stacks_projections_and_experts():
    from asd_b200.models.dikopel import pack, random_weights, tensor_shapes, tiny_config
    cfg = tiny_config()
    w = random_weights(cfg, seed=1)
    p = pack(w, cfg, "cpu", torch.float32)
    a, b, _, _ = cfg.layers
    nk, nv = a.heads * a.dim, a.heads * a.vdim
    assert p[(0, "w_in")].shape == (2 * nk + 2 * nv + 2 * a.heads, cfg.width)
    assert torch.equal(p[(0, "w_in")][2 * nk + nv:2 * (nk + nv)], w["l0.mix.g"].float())
    assert torch.equal(p[(0, "w_in")][-a.heads:], w["l0.mix.f"].float())
    nl = b.a_heads * b.a_dim + b.a_kv_heads * (b.a_dim + b.a_vdim)
    assert p[(1, "w_in")].shape == (nl + b.conv_channels + b.r_heads * b.r_vdim + 2 * b.r_heads, cfg.width)
    assert torch.equal(p[(1, "w_in")][nl:nl + b.r_kv_heads * b.r_dim], w["l1.mix.right.q"].float())
    assert torch.equal(p[(1, "w_in")][-b.r_heads:], w["l1.mix.right.a"].float())
    assert p[(1, "conv_w")].shape == (b.conv_channels, b.conv)
    assert p[(0, "router")].shape == (a.experts + 1, cfg.width)
    assert torch.equal(p[(0, "router")][-1:], w["l0.mlp.shared.sg"].float())
    assert p[(0, "w_egu")].shape == (a.experts, 2 * a.expert_ff, cfg.width)
    assert torch.equal(p[(0, "w_egu")][3, a.expert_ff:], w["l0.mlp.e3.up"].float())
    assert torch.equal(p[(1, "w_gu")][:b.ff], w["l1.mlp.gate"].float())
    assert not any(layer == 3 for layer, _ in p) and (2, "w_gu") not in p
    bad = dict(w)
    bad["l1.mix.left.pb"] = torch.zeros(b.a_heads + 1)
    with pytest.raises(ValueError):
        pack(bad, cfg, "cpu", torch.float32)
    del bad["l1.mix.left.pb"]
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
    names = {os.path.basename(s) for s in b.sources(("dikopel",))}
    assert {"dikopel_engine.cu", "mlstm.cu", "delta_rule.cu", "sigmoid_attention.cu", "moe.cu", "gemm.cu"} <= names
    assert not names & {"engine.cu", "mavipel_engine.cu", "lukopel_engine.cu", "talking_attention.cu", "sampler.cu"}


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_oracle_layer_norm_by_hand():
    got = O.layer_norm(t64([[1.0, 3.0, 5.0, 7.0]]), t64([1.0, 2.0, 1.0, 1.0]), t64([0.0, 0.0, 10.0, 0.0]), 0.0)
    s = math.sqrt(5.0)
    assert torch.allclose(got, t64([[-3 / s, -2 / s, 10 + 1 / s, 3 / s]]))


def test_oracle_sinusoids_alternate():
    x = O.sinusoids(torch.tensor([0, 7]), 6, F64)
    assert x[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0, 1.0]
    for i in range(3):
        ang = 7 * 10000.0 ** (-2 * i / 6)
        assert math.isclose(x[1, 2 * i], math.sin(ang)) and math.isclose(x[1, 2 * i + 1], math.cos(ang))
    e = O.embedding(torch.tensor([1]), torch.tensor([7]), t64([[0.0] * 6, [2.0] * 6]), 3.0)
    assert torch.allclose(e[0], 6.0 + x[1])


def test_oracle_convolution_weighs_the_current_position_last():
    x = t64([[1.0], [10.0], [100.0], [1000.0]])
    taps = t64([[3.0, 2.0, 1.0]])
    assert O.causal_conv(x, taps)[:, 0].tolist() == [1.0, 12.0, 123.0, 1230.0]
    assert O.input_conv(x, taps)[:, 0].tolist() == [2.0, 22.0, 223.0, 2230.0]
    assert O.causal_conv(x[:2], t64([[5.0, 4.0, 3.0, 2.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0]


def test_oracle_matrix_memory_by_hand_and_without_the_running_maximum():
    """the running maximum changes nothing but the range: S and n with plain exponentials and a floor of one"""
    g = torch.Generator().manual_seed(3)
    T, H, dk, dv = 9, 2, 3, 4
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    q, k, v, i, f = r(T, H, dk), r(T, H, dk), r(T, H, dv), 2 * r(T, H), torch.nn.functional.logsigmoid(r(T, H))
    got = O.mlstm_core(q, k, v, i, f)
    for h in range(H):
        S, n = torch.zeros(dk, dv, dtype=F64), torch.zeros(dk, dtype=F64)
        for t in range(T):
            S = f[t, h].exp() * S + i[t, h].exp() * torch.outer(k[t, h], v[t, h])
            n = f[t, h].exp() * n + i[t, h].exp() * k[t, h]
            want = (S.T @ q[t, h]) / max(abs(n @ q[t, h]).item(), 1.0)
            assert torch.allclose(got[t, h], want, rtol=1e-4)      # up to the 1e-6 beside the floor
    one = torch.ones(1, 1, 1, dtype=F64)
    out = O.mlstm_core(2 * one, 3 * one, 5 * one, t64([[1.0]]), t64([[-0.5]]))   # M = max(-0.5, 1) = 1, S = 15, n = 3
    assert math.isclose(out.item(), 30.0 / (6.0 + 1e-6))
    out = O.mlstm_core(2 * one, 3 * one, 5 * one, t64([[-4.0]]), t64([[-0.5]]))  # M = -0.5: the floor is exp(0.5)
    p = math.exp(-3.5)
    assert math.isclose(out.item(), 30.0 * p / (max(6 * p, math.exp(0.5)) + 1e-6))


def test_oracle_sigmoid_attention_by_hand():
    m = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.5}
    w = {"q": t64([[1.0], [2.0]]), "k": t64([[1.0]]), "v": t64([[10.0]]), "pb": t64([0.3, -0.4]), "o": torch.eye(2, dtype=F64)}
    h = t64([[1.0], [3.0]])
    sg = lambda z: 1 / (1 + math.exp(-z))
    got = O.sigmoid_attention(h, w, m)
    want = [[10 * sg(0.5 * a + b) for a, b in ((1.0, 0.3), (2.0, -0.4))],
            [10 * sg(0.5 * 3 * c + b) + 30 * sg(0.5 * 9 * c + b) for c, b in ((1.0, 0.3), (2.0, -0.4))]]
    assert torch.allclose(got, t64(want))


def test_oracle_gated_delta_rule_by_hand():
    """one head, one key and value channel, k = q = 1: S <- g S + beta (v - g S), o = S"""
    one = torch.ones(3, 1, 1, dtype=F64)
    out = O.gated_delta_core(one, one, 8.0 * one, torch.full((3, 1), 0.5, dtype=F64), torch.full((3, 1), 0.5, dtype=F64))
    assert out[:, 0, 0].tolist() == [4.0, 5.0, 5.25]
    # two query heads share a key head
    q = torch.ones(1, 1, 1, dtype=F64)
    out = O.gated_delta_core(q, q, t64([[[2.0], [6.0]]]), t64([[1.0, 0.5]]), t64([[1.0, 1.0]]))
    assert out[0, :, 0].tolist() == [2.0, 3.0]


def test_oracle_choice_by_corrected_scores_within_the_best_groups():
    z = t64([0.0, 4.0, 1.0, 1.5, -3.0, 2.0])           # sigmoids .5 .98 .73 .82 .05 .88
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0}
    corr = t64([-0.9, -0.9, 0.0, 0.0, -1.0, -0.2])     # group sums -.3, 1.55, -.27
    idx, g = O.choose_experts(z, corr, router)
    assert idx.tolist() == [3, 2]
    s = torch.sigmoid(z[[3, 2]])
    assert torch.allclose(g, 2.0 * s / s.sum())        # the correction is no part of the weights
    router["groups"]["keep"] = 2                       # group 2 (-.27) beats group 0 (-.3): expert 0's and 1's stay out
    router["top"] = 4
    assert O.choose_experts(z, corr, router)[0].tolist() == [3, 2, 5, 4]
    router["groups"]["keep"] = 3
    assert O.choose_experts(z, corr, router)[0].tolist() == [3, 2, 5, 1]


def test_oracle_shared_expert_has_its_own_gate():
    one = torch.ones(1, 1, dtype=F64)
    f = {"kind": "moe", "router": {"experts": 1, "top": 1, "scale": 1.0}, "expert": {"ff": 1}, "shared": {"ff": 1}}
    w = {"router": one, "correction": t64([0.0]), "e0.gate": 50 * one, "e0.up": one, "e0.down": one / 50, "shared.gate": 50 * one,
         "shared.up": one, "shared.down": one * 2 / 50, "shared.sg": 3.0 * one}
    got = O.feed_forward(torch.ones(1, 1, dtype=F64), w, f)
    assert math.isclose(got.item(), 1.0 + 2.0 / (1 + math.exp(-3.0)), rel_tol=1e-6)


def test_oracle_layer_adds_both_sublayers_times_the_multiplier():
    cfg = {"width": 4, "vocab": 5, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0}, "residual_mult": 0.5, "canon": {"taps": 2},
           "layers": [{"type": "mlstm", "mixer": {"heads": 1, "dim": 2, "vdim": 3, "gate_cap": 5.0}, "mlp": {"kind": "dense", "ff": 6}}]}
    w = {k: t.to(F64) for k, t in O.random_model(cfg, seed=2).items()}
    ids = torch.tensor([1, 4, 2])
    streams = []
    O.forward(cfg, w, ids, layers_out=streams)
    x = O.embedding(ids, torch.arange(3), w["embed"], 2.0)
    h = O.layer_norm(x, w["l0.norm1"], w["l0.norm1.b"], 1e-5)
    mix = O.mlstm_mixer(O.input_conv(h, w["l0.canon1"]), O.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5)
    assert torch.allclose(streams[0], x + 0.5 * (mix + O.gated_ff(h, O.sub(w, "l0.mlp."))))
