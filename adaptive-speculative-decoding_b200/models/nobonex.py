"""Nobonex family: configuration (read from a checkpoint's ``config.json``), tensor names, random initialisation and
the packing of a named state dict into the buffers ``asd_nobonex_set_tensor`` expects (include/asd_b200.h).

A Nobonex layer norms before and after each sublayer, x <- x + r norm1b(mixer(norm1(x))), x <- x + r norm2b(ff(norm2(x))),
with norms that reduce nothing over a row: tanh(alpha x) w + b.  A layer names ONE of three mixers.  "attention": queries
and keys pass a short causal convolution; a convolved key serves as value as it is, and as key after an RMS norm over the
whole projection and a rotation of interleaved pairs (queries alike); causal softmax attention.  "mamba2": the scalar-decay state space recurrence, gated
before its norm in groups.  "attention_2": biased projections, an RMS norm per head, a rotation of half-split pairs with YaRN
scaling, capped scores inside chunks of positions, an output gate per element; it may read the keys and values of an earlier
such layer.  The feed-forward is a gated layer, or routed experts with clamped activations whose weight multiplies their
input, or absent.  The reference project has no model code of its own (its stages are vLLM checkpoints,
src/serving/real_model_pipeline.py:98-108); this family runs behind the same ``Stage`` seam."""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field, replace
from typing import Dict, List, Optional, Tuple

import torch

ARCHITECTURE = "Nobonex"
MIXERS = ("attention", "mamba2", "attention_2")
FF_KINDS = (None, "dense", "moe")


@dataclass(frozen=True)
class NobonexLayer:
    type: str
    heads: int = 0
    vdim: int = 0
    # attention kinds
    kv_heads: int = 0
    dim: int = 0
    scale: float = 1.0
    rot_dims: int = 0
    rot_base: float = 10000.0
    yarn: Optional[Tuple[float, float, float, float]] = None     # factor, original length, fast, slow
    chunk: int = 0               # attention_2; 0: every earlier position is visible
    softcap: float = 0.0         # attention_2; 0: scores are not capped
    kv_from: int = -1            # attention_2: the layer whose keys and values are used; -1: its own
    # short convolution (attention, mamba2)
    conv: int = 1
    # mamba2
    state: int = 0
    groups: int = 1
    norm_groups: int = 1
    # feed-forward
    ff_kind: Optional[str] = None
    ff: int = 0
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    limit: float = 0.0

    @property
    def cache_row(self) -> int:
        """cached elements per position (paged); recurrent states are per sequence, not per position"""
        return self.kv_heads * (self.dim + self.vdim) if self.type != "mamba2" and self.kv_from < 0 else 0

    @property
    def state_elems(self) -> int:
        """floats of recurrent state per sequence (and ring entry)"""
        return self.heads * self.state * self.vdim if self.type == "mamba2" else 0

    @property
    def conv_channels(self) -> int:
        if self.type == "mamba2":
            return self.heads * self.vdim + 2 * self.groups * self.state
        return (self.heads + self.kv_heads) * self.dim if self.type == "attention" else 0

    @property
    def in_rows(self) -> int:
        """rows of the stacked projection that reads the mixer input"""
        if self.type == "mamba2":
            return self.heads * self.vdim + self.conv_channels + self.heads
        if self.type == "attention":
            return self.conv_channels
        return self.heads * self.dim + self.cache_row + self.heads * self.vdim


@dataclass(frozen=True)
class NobonexConfig:
    width: int
    vocab_size: int
    layers: List[NobonexLayer] = field(default_factory=list)
    eps: float = 1e-6
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    name: str = "nobonex"

    architecture = ARCHITECTURE
    build_components = ("nobonex",)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    def runs(self) -> List[Tuple[int, int]]:
        """(layer, -1) of every layer execution in order"""
        return [(i, -1) for i in range(len(self.layers))]

    @classmethod
    def from_dict(cls, d: dict, name: str = "nobonex") -> "NobonexConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            t = e.get("type")
            if t not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {t!r} (have {MIXERS})")
            m, f = e["mixer"], e.get("mlp")
            kw = dict(type=t, heads=int(m["heads"]))
            if t == "mamba2":
                kw.update(vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m.get("groups", 1)),
                          norm_groups=int(m.get("norm_groups", 1)), conv=int(m.get("conv", 1)))
            else:
                kw.update(kv_heads=int(m.get("kv_heads", m["heads"])), dim=int(m["dim"]), vdim=int(m.get("vdim", m["dim"])),
                          scale=float(m["scale"]))
                rot = m.get("rot") or {}
                if rot.get("dims"):
                    kw.update(rot_dims=int(rot["dims"]), rot_base=float(rot["base"]))
                    y = rot.get("scaling")
                    if y:
                        kw.update(yarn=(float(y["factor"]), float(y["original"]), float(y["fast"]), float(y["slow"])))
                if t == "attention":
                    kw.update(conv=int(m.get("conv", 1)))
                    if kw["vdim"] != kw["dim"]:
                        raise ValueError(f"layer {i}: values that are the keys have size {kw['dim']}, not {kw['vdim']}")
                else:
                    kw.update(chunk=int((m.get("mask") or {}).get("size", 0)), softcap=float(m.get("softcap") or 0.0))
                    if m.get("kv_from") is not None:
                        kw["kv_from"] = int(m["kv_from"])
            if f is not None:
                kind = f.get("kind", "dense")
                if kind == "dense":
                    kw.update(ff_kind="dense", ff=int(f["ff"]))
                elif kind == "moe":
                    kw.update(ff_kind="moe", experts=int(f["router"]["experts"]), top=int(f["router"]["top"]),
                              expert_ff=int(f["expert"]["ff"]), limit=float(f["expert"]["limit"]))
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
            layers.append(NobonexLayer(**kw))
        for i, l in enumerate(layers):
            if l.kv_from < 0:
                continue
            o = layers[l.kv_from] if l.kv_from < i else None
            if o is None or o.type != l.type or o.kv_from >= 0:
                raise ValueError(f"layer {i}: kv_from {l.kv_from} names no earlier layer with keys and values of its own")
            if (o.kv_heads, o.dim, o.vdim) != (l.kv_heads, l.dim, l.vdim):
                raise ValueError(f"layer {i}: its key/value heads differ from layer {l.kv_from}'s, whose keys it uses")
        return cls(width=int(d["width"]), vocab_size=int(d["vocab"]), layers=layers,
                   eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), name=name)

    def to_dict(self) -> dict:
        """the ``config.json`` form (inverse of ``from_dict``)"""
        out = []
        for l in self.layers:
            if l.type == "mamba2":
                m = {"heads": l.heads, "vdim": l.vdim, "state": l.state, "groups": l.groups, "norm_groups": l.norm_groups,
                     "conv": l.conv}
            else:
                m = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale}
                if l.rot_dims:
                    m["rot"] = {"dims": l.rot_dims, "base": l.rot_base}
                    if l.yarn:
                        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), l.yarn))
                if l.type == "attention":
                    m["conv"] = l.conv
                else:
                    m.update(mask={"size": l.chunk}, softcap=l.softcap)
                    if l.kv_from >= 0:
                        m["kv_from"] = l.kv_from
            if l.ff_kind == "dense":
                f = {"kind": "dense", "ff": l.ff}
            elif l.ff_kind == "moe":
                f = {"kind": "moe", "expert": {"ff": l.expert_ff, "limit": l.limit},
                     "router": {"experts": l.experts, "top": l.top}}
            else:
                f = None
            out.append({"type": l.type, "mixer": m, "mlp": f})
        return {"architecture": ARCHITECTURE, "width": self.width, "vocab": self.vocab_size, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult, "layers": out}

    @property
    def params(self) -> int:
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    def streamed_bytes(self, elem: int = 2) -> int:
        """weight bytes one decode step of ONE token reads: every matrix once (of the experts only the chosen ones), the
        head"""
        n = self.vocab_size * self.width
        for k, s in tensor_shapes(self).items():
            if not k.startswith("l") or len(s) != 2:
                continue
            l = self.layers[int(k[1:k.index(".")])]
            n += math.prod(s) * (l.top / l.experts if ".mlp.e" in k else 1)
        return int(n * elem)

    def kv_bytes_per_token(self, elem: int = 2) -> int:
        return sum(l.cache_row for l in self.layers) * elem


def norm_names(l: NobonexLayer) -> Tuple[str, ...]:
    return ("norm1", "norm1b") + (("norm2", "norm2b") if l.ff_kind else ())


def tensor_shapes(cfg: NobonexConfig) -> Dict[str, tuple]:
    """every tensor of a checkpoint, by name"""
    D, V = cfg.width, cfg.vocab_size
    s = {"embed": (V, D), "head": (V, D)}

    def norm(name):
        s.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})
    norm("final.norm")
    for i, l in enumerate(cfg.layers):
        for n in norm_names(l):
            norm(f"l{i}.{n}")
        m, f, H = f"l{i}.mix.", f"l{i}.mlp.", l.heads
        if l.type == "mamba2":
            ch, inner = l.conv_channels, H * l.vdim
            s.update({m + "in": (l.in_rows, D), m + "conv": (ch, l.conv), m + "conv.b": (ch,), m + "dt_bias": (H,),
                      m + "A_log": (H,), m + "D": (H,), m + "norm": (inner,), m + "o": (D, inner)})
        else:
            nq, nk, nv, no = H * l.dim, l.kv_heads * l.dim, l.kv_heads * l.vdim, H * l.vdim
            s.update({m + "q": (nq, D), m + "o": (D, no)})
            if l.type == "attention":
                s.update({m + "k": (nk, D), m + "q.norm": (nq,), m + "k.norm": (nk,), m + "q.conv": (nq, l.conv),
                          m + "k.conv": (nk, l.conv)})
            else:
                s.update({m + "q.b": (nq,), m + "q.norm": (l.dim,), m + "g": (no, D)})
                if l.kv_from < 0:
                    s.update({m + "k": (nk, D), m + "k.b": (nk,), m + "k.norm": (l.dim,), m + "v": (nv, D), m + "v.b": (nv,)})
        if l.ff_kind == "dense":
            s.update({f + "gate": (l.ff, D), f + "up": (l.ff, D), f + "down": (D, l.ff)})
        elif l.ff_kind == "moe":
            s[f + "router"] = (l.experts, D)
            for e in range(l.experts):
                s.update({f + f"e{e}.gate": (l.expert_ff, D), f + f"e{e}.up": (l.expert_ff, D),
                          f + f"e{e}.down": (D, l.expert_ff)})
    return s


def tiny_config(**kw) -> NobonexConfig:
    """one small layer of every kind, unequal sizes, a layer that reads another one's keys and values (tests, smoke runs)"""
    moe = dict(ff_kind="moe", experts=7, top=2, expert_ff=40, limit=1.5)
    att = NobonexLayer(type="attention", heads=6, kv_heads=2, dim=24, vdim=24, scale=0.2, rot_dims=12, rot_base=5000.0, conv=3,
                       ff_kind="dense", ff=72)
    ssd = NobonexLayer(type="mamba2", heads=4, vdim=24, state=20, groups=2, norm_groups=3, conv=3, **moe)
    chk = NobonexLayer(type="attention_2", heads=4, kv_heads=2, dim=32, vdim=24, scale=0.2, rot_dims=16, rot_base=9000.0,
                       yarn=(4.0, 256.0, 16.0, 2.0), chunk=24, softcap=20.0, **moe)
    shr = NobonexLayer(type="attention_2", heads=8, kv_heads=2, dim=32, vdim=24, scale=0.15, rot_dims=16, rot_base=9000.0,
                       yarn=(4.0, 256.0, 16.0, 2.0), chunk=24, softcap=20.0, kv_from=2)
    base = dict(width=104, vocab_size=120, layers=[att, ssd, chk, shr], eps=1e-5, embed_scale=1.5, residual_mult=0.5,
                name="tiny")
    base.update(kw)
    return NobonexConfig(**base)


def sized_config(width: int, n_layers: int, heads: int, vocab: int = 32768, dim: int = 128, chunk: int = 1024,
                 ff: Optional[int] = None, experts: int = 0, top: int = 2, name: str = "nobonex-sized") -> NobonexConfig:
    """layers of a realistic size for throughput measurements (random weights), six in turn: state space (2 x width inner
    values in heads of 64, state 128) twice, convolved attention, state space, chunked attention, chunked attention with the
    keys and values of the one before.  Dense feed-forwards of width ff (3 x width by default), or `experts` experts of
    ff / (top + 1)"""
    ff = ff if ff is not None else 3 * width
    f = dict(ff_kind="moe", experts=experts, top=top, expert_ff=max(64, ff // (top + 1)), limit=7.0) if experts else \
        dict(ff_kind="dense", ff=ff)
    kv = max(1, heads // 4)
    rot = dict(rot_dims=dim // 2, rot_base=500000.0)
    ssd = NobonexLayer(type="mamba2", heads=2 * width // 64, vdim=64, state=128, groups=1, norm_groups=1, conv=4, **f)
    att = NobonexLayer(type="attention", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, conv=4, **rot, **f)
    chk = NobonexLayer(type="attention_2", heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                       yarn=(4.0, 4096.0, 32.0, 1.0), chunk=chunk, softcap=50.0, **rot, **f)
    cycle = (ssd, ssd, att, ssd, chk, chk)
    layers = [replace(cycle[i % 6], kv_from=i - 1) if i % 6 == 5 else cycle[i % 6] for i in range(n_layers)]
    return NobonexConfig(width=width, vocab_size=vocab, layers=layers, embed_scale=1.0, residual_mult=0.5, name=name)


def random_weights(cfg: NobonexConfig, seed: int, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Named state dict with variance-preserving random matrices, norm weights near one, decays that keep a state alive
    for tens of tokens (throughput runs and smoke tests; nothing trained)."""
    g = torch.Generator(device=device).manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        rnd = lambda: torch.randn(shape, generator=g, device=device)
        if leaf == "alpha":
            t = 0.6 + 0.1 * rnd()
        elif leaf.startswith("norm"):
            t = 1.0 + 0.1 * rnd()
        elif leaf == "conv":
            t = 0.4 * rnd()
        elif leaf == "b":
            t = 0.1 * rnd()
        elif leaf == "A_log":
            t = 0.3 * rnd()
        elif leaf == "dt_bias":
            t = -2.5 + rnd()
        elif leaf == "D":
            t = 1.0 + 0.1 * rnd()
        elif leaf == "embed":
            t = rnd()
        else:
            t = rnd() / math.sqrt(shape[-1])
        w[name] = t.to(dtype)
    return w


def pack(w: Dict[str, torch.Tensor], cfg: NobonexConfig, device, dtype) -> Dict[Tuple[int, str], torch.Tensor]:
    """checkpoint names -> engine buffers keyed (layer or -1, engine tensor name).  Matrices that read the same input
    are stacked into one; an expert's gate and up matrices are stacked and the experts laid out back to back.  Matrices
    take the engine's element type, everything that enters 32-bit arithmetic directly (norm weights and slopes, biases,
    convolution taps, decay parameters, router) stays fp32."""
    want = tensor_shapes(cfg)
    for k, shape in want.items():
        if k not in w:
            raise KeyError(f"checkpoint lacks tensor {k}")
        if tuple(w[k].shape) != tuple(shape):
            raise ValueError(f"tensor {k} has shape {tuple(w[k].shape)}, the configuration says {tuple(shape)}")
    mat = lambda t: t.to(device=device, dtype=dtype).contiguous()
    vec = lambda t: t.to(device=device, dtype=torch.float32).reshape(-1 if t.dim() == 0 else t.shape).contiguous()
    cat = lambda names: torch.cat([w[n] for n in names], 0)
    out = {(-1, "embed"): mat(w["embed"]), (-1, "head"): mat(w["head"])}

    def norm(layer, to, name):
        out[(layer, to)], out[(layer, to + "_b")] = vec(w[name]), vec(w[name + ".b"])
        out[(layer, to + "_alpha")] = vec(w[name + ".alpha"])
    norm(-1, "final_norm", "final.norm")
    for i, l in enumerate(cfg.layers):
        for n in norm_names(l):
            norm(i, n, f"l{i}.{n}")
        m, f = f"l{i}.mix.", f"l{i}.mlp."
        out[(i, "w_o")] = mat(w[m + "o"])
        if l.type == "mamba2":
            out[(i, "w_in")] = mat(w[m + "in"])
            out[(i, "conv_w")], out[(i, "conv_b")] = vec(w[m + "conv"]), vec(w[m + "conv.b"])
            out[(i, "a_log")], out[(i, "dt_bias")] = vec(w[m + "A_log"]), vec(w[m + "dt_bias"])
            out[(i, "skip")], out[(i, "out_norm")] = vec(w[m + "D"]), vec(w[m + "norm"])
        else:
            out[(i, "q_norm")] = vec(w[m + "q.norm"])
            if l.kv_from < 0:
                out[(i, "k_norm")] = vec(w[m + "k.norm"])
            if l.type == "attention":
                out[(i, "w_in")] = mat(cat([m + "q", m + "k"]))
                out[(i, "conv_w")] = vec(cat([m + "q.conv", m + "k.conv"]))
            else:
                own = ("q", "k", "v") if l.kv_from < 0 else ("q",)
                out[(i, "w_in")] = mat(cat([m + x for x in own] + [m + "g"]))
                out[(i, "in_bias")] = vec(cat([m + x + ".b" for x in own]))
        if l.ff_kind == "dense":
            out[(i, "w_gu")], out[(i, "w_down")] = mat(cat([f + "gate", f + "up"])), mat(w[f + "down"])
        elif l.ff_kind == "moe":
            out[(i, "router")] = vec(w[f + "router"])
            out[(i, "w_egu")] = mat(torch.stack([cat([f + f"e{e}.gate", f + f"e{e}.up"]) for e in range(l.experts)]))
            out[(i, "w_edown")] = mat(torch.stack([w[f + f"e{e}.down"] for e in range(l.experts)]))
    return out


def load_config_dir(path: str) -> NobonexConfig:
    with open(os.path.join(path, "config.json")) as f:
        return NobonexConfig.from_dict(json.load(f), name=os.path.basename(os.path.normpath(path)) or "nobonex")
