"""Dikopel family: configuration (read from a checkpoint's ``config.json``), tensor names, random initialisation and
the packing of a named state dict into the buffers ``asd_dikopel_set_tensor`` expects (include/asd_b200.h).

A Dikopel layer has ONE layer norm (weight and bias) whose result h both sublayers read side by side:
x <- x + r (mixer(h + conv(h)) + ff(h)), conv a causal convolution over time on every channel, r a constant.  The input is
a scaled embedding plus sinusoids of the position.  A layer names ONE of two mixers.  "mlstm": a matrix memory per head
with exponential input and forget gates, a normaliser and a running maximum that keeps the exponentials in range.
"parallel": two mixers on the same input whose results are RMS-normed and averaged: grouped-query causal attention whose
weights are sigmoids of the scores plus a bias per head (no softmax, no positions), and the gated delta rule with short
convolutions and one decay per head and position.  The feed-forward is a gated silu layer, or routed gated experts (sigmoid
scores, a correction that only enters the choice, choice within the best groups of experts) plus a shared expert behind a
gate of its own, or absent.  A layer may use another layer's tensors, with a cache and state of its own.  The reference
project has no model code of its own (its stages are vLLM checkpoints, src/serving/real_model_pipeline.py:98-108); this
family runs behind the same ``Stage`` seam."""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field, replace
from typing import Dict, List, Optional, Tuple

import torch

ARCHITECTURE = "Dikopel"
MIXERS = ("mlstm", "parallel")
FF_KINDS = (None, "dense", "moe")


@dataclass(frozen=True)
class DikopelLayer:
    type: str
    # mlstm
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    gate_cap: float = 0.0
    # parallel, left: sigmoid attention
    a_heads: int = 0
    a_kv_heads: int = 0
    a_dim: int = 0
    a_vdim: int = 0
    scale: float = 1.0
    # parallel, right: gated delta rule
    r_heads: int = 0
    r_kv_heads: int = 0
    r_dim: int = 0
    r_vdim: int = 0
    conv: int = 1
    # feed-forward
    ff_kind: Optional[str] = None
    ff: int = 0
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    shared_ff: int = 0
    groups: int = 1
    keep: int = 1
    router_scale: float = 1.0
    weights_of: int = -1         # the layer whose tensors this one uses; -1: its own

    @property
    def cache_row(self) -> int:
        """cached elements per position (paged); the recurrent states are per sequence, not per position"""
        return self.a_kv_heads * (self.a_dim + self.a_vdim) if self.type == "parallel" else 0

    @property
    def state_elems(self) -> int:
        """floats of recurrent state per sequence (and ring entry)"""
        if self.type == "mlstm":
            return (self.heads * (self.dim * self.vdim + (self.vdim + 31) // 32 * (self.dim + 1)) + 3) // 4 * 4
        return self.r_heads * self.r_dim * self.r_vdim

    @property
    def conv_channels(self) -> int:
        return 2 * self.r_kv_heads * self.r_dim + self.r_heads * self.r_vdim if self.type == "parallel" else 0


@dataclass(frozen=True)
class DikopelConfig:
    width: int
    vocab_size: int
    layers: List[DikopelLayer] = field(default_factory=list)
    eps: float = 1e-5
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    input_taps: int = 1
    name: str = "dikopel"

    architecture = ARCHITECTURE
    build_components = ("dikopel",)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    def owner(self, i: int) -> int:
        """the layer whose tensors layer i uses"""
        seen = set()
        while self.layers[i].weights_of >= 0:
            if i in seen:
                raise ValueError(f"layer {i}: weights_of names no layer with tensors of its own")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def runs(self) -> List[Tuple[int, int]]:
        """(layer whose tensors are used, -1) of every layer execution in order"""
        return [(self.owner(i), -1) for i in range(len(self.layers))]

    @classmethod
    def from_dict(cls, d: dict, name: str = "dikopel") -> "DikopelConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            t = e.get("type")
            if t not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {t!r} (have {MIXERS})")
            m, f = e["mixer"], e.get("mlp")
            kw = dict(type=t)
            if t == "mlstm":
                kw.update(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m.get("vdim", m["dim"])),
                          gate_cap=float(m["gate_cap"]))
            else:
                a, r = m["left"], m["right"]
                kw.update(a_heads=int(a["heads"]), a_kv_heads=int(a.get("kv_heads", a["heads"])), a_dim=int(a["dim"]),
                          a_vdim=int(a.get("vdim", a["dim"])), scale=float(a["scale"]), r_heads=int(r["heads"]),
                          r_kv_heads=int(r.get("kv_heads", r["heads"])), r_dim=int(r["dim"]),
                          r_vdim=int(r.get("vdim", r["dim"])), conv=int(r.get("conv", 1)))
            if f is not None:
                kind = f.get("kind", "dense")
                if kind == "dense":
                    kw.update(ff_kind="dense", ff=int(f["ff"]))
                elif kind == "moe":
                    r, g = f["router"], f["router"].get("groups") or {}
                    kw.update(ff_kind="moe", experts=int(r["experts"]), top=int(r["top"]), expert_ff=int(f["expert"]["ff"]),
                              shared_ff=int((f.get("shared") or {}).get("ff", 0)), groups=int(g.get("count", 1)),
                              keep=int(g.get("keep", 1)), router_scale=float(r.get("scale", 1.0)))
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
            j = e.get("weights_of")
            if j is not None:
                if not 0 <= int(j) < len(d["layers"]) or int(j) == i:
                    raise ValueError(f"layer {i}: weights_of {j!r} names no other layer")
                kw["weights_of"] = int(j)
            layers.append(DikopelLayer(**kw))
        cfg = cls(width=int(d["width"]), vocab_size=int(d["vocab"]), layers=layers,
                  eps=float((d.get("norm") or {}).get("eps", 1e-5)),
                  embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                  residual_mult=float(d.get("residual_mult", 1.0)), input_taps=int((d.get("canon") or {}).get("taps", 1)),
                  name=name)
        for i, l in enumerate(layers):
            o = layers[cfg.owner(i)]
            if replace(l, weights_of=-1) != replace(o, weights_of=-1):
                raise ValueError(f"layer {i} differs from layer {cfg.owner(i)}, whose weights it uses")
        return cfg

    def to_dict(self) -> dict:
        """the ``config.json`` form (inverse of ``from_dict``)"""
        out = []
        for l in self.layers:
            if l.type == "mlstm":
                m = {"heads": l.heads, "dim": l.dim, "vdim": l.vdim, "gate_cap": l.gate_cap}
            else:
                m = {"left": {"heads": l.a_heads, "kv_heads": l.a_kv_heads, "dim": l.a_dim, "vdim": l.a_vdim, "scale": l.scale},
                     "right": {"heads": l.r_heads, "kv_heads": l.r_kv_heads, "dim": l.r_dim, "vdim": l.r_vdim, "conv": l.conv}}
            if l.ff_kind == "dense":
                f = {"kind": "dense", "ff": l.ff}
            elif l.ff_kind == "moe":
                f = {"kind": "moe", "expert": {"ff": l.expert_ff},
                     "router": {"experts": l.experts, "top": l.top, "groups": {"count": l.groups, "keep": l.keep},
                                "scale": l.router_scale}}
                if l.shared_ff:
                    f["shared"] = {"ff": l.shared_ff}
            else:
                f = None
            e = {"type": l.type, "mixer": m, "mlp": f}
            if l.weights_of >= 0:
                e["weights_of"] = l.weights_of
            out.append(e)
        return {"architecture": ARCHITECTURE, "width": self.width, "vocab": self.vocab_size, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult,
                "canon": {"taps": self.input_taps}, "layers": out}

    @property
    def params(self) -> int:
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    def streamed_bytes(self, elem: int = 2) -> int:
        """weight bytes one decode step of ONE token reads: every matrix once per layer that uses it (of the experts
        only the chosen ones), the head"""
        shapes = tensor_shapes(self)
        n = self.vocab_size * self.width
        for i, _ in self.runs():
            l = self.layers[i]
            for k, s in shapes.items():
                if not k.startswith(f"l{i}.") or len(s) != 2:
                    continue
                if ".mlp.e" in k:
                    n += math.prod(s) * l.top / l.experts
                else:
                    n += math.prod(s)
        return int(n * elem)

    def kv_bytes_per_token(self, elem: int = 2) -> int:
        return sum(l.cache_row for l in self.layers) * elem


def tensor_shapes(cfg: DikopelConfig) -> Dict[str, tuple]:
    """every tensor of a checkpoint, by name"""
    D, V = cfg.width, cfg.vocab_size
    s = {"embed": (V, D), "final.norm": (D,), "final.norm.b": (D,), "head": (V, D)}
    for i, l in enumerate(cfg.layers):
        if l.weights_of >= 0:
            continue
        p = f"l{i}."
        s.update({p + "norm1": (D,), p + "norm1.b": (D,), p + "canon1": (D, cfg.input_taps)})
        if l.type == "mlstm":
            m, nk, nv = p + "mix.", l.heads * l.dim, l.heads * l.vdim
            s.update({m + "q": (nk, D), m + "k": (nk, D), m + "v": (nv, D), m + "g": (nv, D), m + "o": (D, nv),
                      m + "norm": (nv,), m + "i": (l.heads, D), m + "i.b": (l.heads,), m + "f": (l.heads, D),
                      m + "f.b": (l.heads,)})
        else:
            a, r = p + "mix.left.", p + "mix.right."
            na = l.a_heads * l.a_vdim
            s.update({a + "q": (l.a_heads * l.a_dim, D), a + "k": (l.a_kv_heads * l.a_dim, D),
                      a + "v": (l.a_kv_heads * l.a_vdim, D), a + "pb": (l.a_heads,), a + "o": (D, na), a + "out": (D,)})
            nk, nv = l.r_kv_heads * l.r_dim, l.r_heads * l.r_vdim
            s.update({r + "q": (nk, D), r + "q.conv": (nk, l.conv), r + "k": (nk, D), r + "k.conv": (nk, l.conv),
                      r + "v": (nv, D), r + "v.conv": (nv, l.conv), r + "b": (l.r_heads, D), r + "A_log": (l.r_heads,),
                      r + "norm": (l.r_vdim,), r + "a": (l.r_heads, D), r + "dt_bias": (l.r_heads,), r + "g": (nv, D),
                      r + "o": (D, nv), r + "out": (D,)})
        f = p + "mlp."
        if l.ff_kind == "dense":
            s.update({f + "gate": (l.ff, D), f + "up": (l.ff, D), f + "down": (D, l.ff)})
        elif l.ff_kind == "moe":
            s.update({f + "router": (l.experts, D), f + "correction": (l.experts,)})
            for e in range(l.experts):
                s.update({f + f"e{e}.gate": (l.expert_ff, D), f + f"e{e}.up": (l.expert_ff, D),
                          f + f"e{e}.down": (D, l.expert_ff)})
            if l.shared_ff:
                s.update({f + "shared.gate": (l.shared_ff, D), f + "shared.up": (l.shared_ff, D),
                          f + "shared.down": (D, l.shared_ff), f + "shared.sg": (1, D)})
    return s


def tiny_config(**kw) -> DikopelConfig:
    """one small layer of every kind, unequal sizes, a layer that uses another one's weights (tests, smoke runs)"""
    ml = DikopelLayer(type="mlstm", heads=3, dim=24, vdim=40, gate_cap=9.0, ff_kind="moe", experts=9, top=3, expert_ff=40,
                      shared_ff=24, groups=3, keep=2, router_scale=1.5)
    par = DikopelLayer(type="parallel", a_heads=6, a_kv_heads=2, a_dim=24, a_vdim=16, scale=0.25, r_heads=4, r_kv_heads=2,
                       r_dim=16, r_vdim=24, conv=3, ff_kind="dense", ff=72)
    layers = [ml, par, replace(par, ff_kind=None, ff=0, a_heads=2, a_kv_heads=2), replace(ml, weights_of=0)]
    base = dict(width=104, vocab_size=120, layers=layers, eps=1e-5, embed_scale=7.0, residual_mult=0.6, input_taps=3,
                name="tiny")
    base.update(kw)
    return DikopelConfig(**base)


def sized_config(width: int, n_layers: int, heads: int, vocab: int = 32768, dim: int = 128, ff: Optional[int] = None,
                 experts: int = 0, top: int = 2, name: str = "dikopel-sized") -> DikopelConfig:
    """layers of a realistic size for throughput measurements (random weights): two matrix-memory layers, then a parallel
    one, in turn; dense feed-forwards of width ff (3 x width by default), or `experts` experts of ff / (top + 1)"""
    ff = ff if ff is not None else 3 * width
    if experts:
        fe = max(64, ff // (top + 1))
        f = dict(ff_kind="moe", experts=experts, top=top, expert_ff=fe, shared_ff=fe, groups=2 if experts % 2 == 0 else 1,
                 keep=1, router_scale=1.0)
    else:
        f = dict(ff_kind="dense", ff=ff)
    ml = DikopelLayer(type="mlstm", heads=heads, dim=dim, vdim=dim, gate_cap=15.0, **f)
    par = DikopelLayer(type="parallel", a_heads=heads, a_kv_heads=max(1, heads // 4), a_dim=dim, a_vdim=dim,
                       scale=1.0 / math.sqrt(dim), r_heads=max(1, heads // 2), r_kv_heads=max(1, heads // 4), r_dim=dim,
                       r_vdim=dim, conv=4, **f)
    return DikopelConfig(width=width, vocab_size=vocab, layers=[(ml, ml, par)[i % 3] for i in range(n_layers)],
                         embed_scale=math.sqrt(width), residual_mult=0.5, input_taps=4, name=name)


def random_weights(cfg: DikopelConfig, seed: int, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Named state dict with variance-preserving random matrices, norm weights near one, gates and decays that keep a
    state alive for tens of tokens (throughput runs and smoke tests; nothing trained)."""
    g = torch.Generator(device=device).manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        rnd = lambda: torch.randn(shape, generator=g, device=device)
        if leaf in ("norm1", "norm", "out"):
            t = 1.0 + 0.1 * rnd()
        elif leaf in ("conv", "canon1"):
            t = 0.4 * rnd()
        elif name.endswith("f.b"):
            t = 3.0 + 0.5 * rnd()
        elif leaf == "pb":
            t = -3.0 + 0.5 * rnd()
        elif leaf in ("A_log", "correction"):
            t = 0.3 * rnd()
        elif leaf == "dt_bias":
            t = -2.0 + rnd()
        elif leaf == "b" and len(shape) == 1:
            t = 0.2 * rnd()
        else:
            t = rnd() / math.sqrt(shape[-1])
        w[name] = t.to(dtype)
    return w


def pack(w: Dict[str, torch.Tensor], cfg: DikopelConfig, device, dtype) -> Dict[Tuple[int, str], torch.Tensor]:
    """checkpoint names -> engine buffers keyed (layer or -1, engine tensor name).  Matrices that read the same input
    are stacked into one; an expert's gate and up matrices are stacked and the experts laid out back to back; the shared
    expert's gate row follows the router's rows.  Matrices take the engine's element type, everything that enters 32-bit
    arithmetic directly (norm weights, biases, convolution taps, decay parameters, router) stays fp32."""
    want = tensor_shapes(cfg)
    for k, shape in want.items():
        if k not in w:
            raise KeyError(f"checkpoint lacks tensor {k}")
        if tuple(w[k].shape) != tuple(shape):
            raise ValueError(f"tensor {k} has shape {tuple(w[k].shape)}, the configuration says {tuple(shape)}")
    mat = lambda t: t.to(device=device, dtype=dtype).contiguous()
    vec = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    cat = lambda names, dim=0: torch.cat([w[n] for n in names], dim)
    out = {(-1, "embed"): mat(w["embed"]), (-1, "final_norm"): vec(w["final.norm"]),
           (-1, "final_norm_b"): vec(w["final.norm.b"]), (-1, "head"): mat(w["head"])}
    for i, l in enumerate(cfg.layers):
        if l.weights_of >= 0:
            continue
        p = f"l{i}."
        out[(i, "norm1")], out[(i, "norm1_b")] = vec(w[p + "norm1"]), vec(w[p + "norm1.b"])
        out[(i, "input_conv")] = vec(w[p + "canon1"])
        if l.type == "mlstm":
            m = p + "mix."
            out[(i, "w_in")] = mat(cat([m + x for x in ("q", "k", "v", "g", "i", "f")]))
            out[(i, "i_bias")], out[(i, "f_bias")] = vec(w[m + "i.b"]), vec(w[m + "f.b"])
            out[(i, "out_norm")], out[(i, "w_o")] = vec(w[m + "norm"]), mat(w[m + "o"])
        else:
            a, r = p + "mix.left.", p + "mix.right."
            out[(i, "w_in")] = mat(cat([a + x for x in ("q", "k", "v")] + [r + x for x in ("q", "k", "v", "g", "b", "a")]))
            out[(i, "head_bias")] = vec(w[a + "pb"])
            out[(i, "conv_w")] = vec(cat([r + x for x in ("q.conv", "k.conv", "v.conv")]))
            out[(i, "a_log")], out[(i, "dt_bias")] = vec(w[r + "A_log"]), vec(w[r + "dt_bias"])
            out[(i, "out_norm")] = vec(w[r + "norm"])
            out[(i, "w_o")], out[(i, "w_o2")] = mat(w[a + "o"]), mat(w[r + "o"])
            out[(i, "out_left")], out[(i, "out_right")] = vec(w[a + "out"]), vec(w[r + "out"])
        f = p + "mlp."
        if l.ff_kind == "dense":
            out[(i, "w_gu")], out[(i, "w_down")] = mat(cat([f + "gate", f + "up"])), mat(w[f + "down"])
        elif l.ff_kind == "moe":
            out[(i, "router")] = vec(cat([f + "router"] + ([f + "shared.sg"] if l.shared_ff else [])))
            out[(i, "correction")] = vec(w[f + "correction"])
            out[(i, "w_egu")] = mat(torch.stack([cat([f + f"e{e}.gate", f + f"e{e}.up"]) for e in range(l.experts)]))
            out[(i, "w_edown")] = mat(torch.stack([w[f + f"e{e}.down"] for e in range(l.experts)]))
            if l.shared_ff:
                out[(i, "w_sgu")] = mat(cat([f + "shared.gate", f + "shared.up"]))
                out[(i, "w_sdown")] = mat(w[f + "shared.down"])
    return out


def load_config_dir(path: str) -> DikopelConfig:
    with open(os.path.join(path, "config.json")) as f:
        return DikopelConfig.from_dict(json.load(f), name=os.path.basename(os.path.normpath(path)) or "dikopel")
