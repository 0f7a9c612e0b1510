"""Plain, slow restatement of the Dikopel decoder in PyTorch on the CPU: one function per mechanism, whole sequences
at a time, explicit loops over positions where a mechanism is a recurrence, no cache, no batching.
Test infrastructure only: the product package never imports it and it imports nothing of the product.

Notation: T tokens, D model width, H heads, G key/value heads, dk query/key size per head, dv value size, F
feed-forward width, E experts.  ``w`` maps tensor names to [out, in] matrices (or vectors); ``cfg`` is the dictionary
form of a checkpoint's ``config.json``."""
from __future__ import annotations

import math
from typing import Dict, List

import torch
import torch.nn.functional as F


# ------------------------------------------------------------------------------------------------ norms, activations
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps: float):
    """the row minus its mean, over the root of its mean squared deviation plus eps; then weight and bias"""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z * torch.sigmoid(z)


def unit_vector(x, tiny: float = 1e-6):
    """x / sqrt(sum(x^2) + tiny) over the last axis"""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + tiny)


# ------------------------------------------------------------------------------------------------ input
def sinusoids(positions, width: int, dtype):
    """[T, width]: sin(p base^(-2i/width)) at 2i and cos of the same angle at 2i + 1, base 10000"""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    p = positions.to(torch.float64)
    for c in range(width):
        ang = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(ang) if c % 2 == 0 else torch.cos(ang)
    return out.to(dtype)


def embedding(tokens, positions, table, scale: float):
    return table[tokens] * scale + sinusoids(positions, table.shape[1], table.dtype)


# ------------------------------------------------------------------------------------------------ short convolution
def causal_conv(x, taps):
    """x [T, C], taps [C, n] (last column weighs the current position, zeros before the start) -> [T, C]"""
    T, C = x.shape
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += taps[:, j] * x[:T - back]
    return out


def input_conv(h, taps):
    """what a mixer reads: the normed row plus its causal convolution over time"""
    return h + causal_conv(h, taps)


# ------------------------------------------------------------------------------------------------ mixers
def mlstm_core(q, k, v, i, f):
    """Matrix memory with exponential gates.  q, k [T, H, dk], v [T, H, dv], i and f [T, H] (logarithms of the input and
    forget gates) -> [T, H, dv].  The running maximum M keeps every exponential at most 1."""
    T, H, dk = q.shape
    dv = v.shape[2]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(dk, dv, dtype=q.dtype)
        n = torch.zeros(dk, dtype=q.dtype)
        M = torch.zeros((), dtype=q.dtype)
        for t in range(T):
            Mn = torch.maximum(f[t, h] + M, i[t, h])
            keep, put = torch.exp(f[t, h] + M - Mn), torch.exp(i[t, h] - Mn)
            S = keep * S + put * torch.outer(k[t, h], v[t, h])
            n = keep * n + put * k[t, h]
            M = Mn
            out[t, h] = (S.T @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-M)) + 1e-6)
    return out


def mlstm_mixer(h, w: Dict[str, torch.Tensor], m: dict, eps: float):
    T = h.shape[0]
    H, dk, cap = m["heads"], m["dim"], m["gate_cap"]
    dv = m.get("vdim", dk)
    q = (h @ w["q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dk)
    v = (h @ w["v"].T).reshape(T, H, dv)
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = F.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o = unit_rms(mlstm_core(q, k, v, i, f), eps).reshape(T, H * dv)
    return (o * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def sigmoid_attention(h, w, m: dict):
    """Causal attention whose weights are sigmoids of the scores plus a bias per head, not normalised over the keys"""
    T = h.shape[0]
    H, dk = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", dk)
    q = (h @ w["q"].T).reshape(T, H, dk)
    k = (h @ w["k"].T).reshape(T, G, dk)
    v = (h @ w["v"].T).reshape(T, G, dv)
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        p = torch.sigmoid((q[:, hd] @ k[:, g].T) * m["scale"] + w["pb"][hd])
        out[:, hd] = torch.where(seen, p, torch.zeros((), dtype=h.dtype)) @ v[:, g]
    return out.reshape(T, H * dv) @ w["o"].T


def gated_delta_core(q, k, v, beta, decay):
    """q, k [T, G, dk], v [T, H, dv], beta and decay [T, H] -> [T, H, dv]; the read-out sees the position's own write"""
    T, G, dk = q.shape
    H, dv = v.shape[1:]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for hd in range(H):
        g = hd // (H // G)
        S = torch.zeros(dk, dv, dtype=q.dtype)
        for t in range(T):
            S = decay[t, hd] * S
            u = beta[t, hd] * (v[t, hd] - S.T @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            out[t, hd] = S.T @ q[t, g]
    return out


def gated_delta_mixer(h, w, m: dict, eps: float):
    T = h.shape[0]
    H, dk = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", dk)
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).reshape(T, G, dk)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).reshape(T, G, dk)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).reshape(T, H, dv)
    beta = torch.sigmoid(h @ w["b"].T)
    decay = torch.exp(-torch.exp(w["A_log"]) * F.softplus(h @ w["a"].T + w["dt_bias"]))
    o = gated_delta_core(unit_vector(q) * dk ** -0.5, unit_vector(k), v, beta, decay)
    o = unit_rms(o, eps) * w["norm"] * silu(h @ w["g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w["o"].T


def sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def parallel_mixer(h, w, m: dict, eps: float):
    a = sigmoid_attention(h, sub(w, "left."), m["left"])
    b = gated_delta_mixer(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (unit_rms(a, eps) * w["left.out"] + unit_rms(b, eps) * w["right.out"])


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def choose_experts(z, correction, router: dict):
    """one token's router logits -> (expert indices, weights)"""
    E, top = router["experts"], router["top"]
    s = torch.sigmoid(z)
    c = s + correction
    grp = router.get("groups")
    if grp and grp["count"] > 1:
        n = E // grp["count"]
        score = torch.stack([c[g * n:(g + 1) * n].topk(min(2, n)).values.sum() for g in range(grp["count"])])
        kept = set(score.topk(grp["keep"]).indices.tolist())
        c = torch.stack([c[e] if e // n in kept else torch.tensor(-math.inf, dtype=c.dtype) for e in range(E)])
    idx = c.topk(top).indices
    g = s[idx]
    return idx, g / (g.sum() + 1e-20) * router.get("scale", 1.0)


def feed_forward(h, w, f: dict):
    if f.get("kind", "dense") == "dense":
        return gated_ff(h, w)
    z = h @ w["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        idx, g = choose_experts(z[t], w["correction"], f["router"])
        for e, ge in zip(idx.tolist(), g):
            out[t] += ge * gated_ff(h[t:t + 1], sub(w, f"e{e}."))[0]
    if f.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * gated_ff(h, sub(w, "shared."))
    return out


# ------------------------------------------------------------------------------------------------ the model
def owner(cfg: dict, i: int) -> int:
    """the layer whose tensors layer i uses"""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: list = None):
    """logits [T, vocab] of one sequence from position 0; every tensor is taken to ``dtype`` first"""
    w = {k: (t.to(dtype) if t.is_floating_point() else t) for k, t in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = embedding(tokens, torch.arange(len(tokens)), w["embed"], cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        lw = sub(w, f"l{owner(cfg, i)}.")
        h = layer_norm(x, lw["norm1"], lw["norm1.b"], eps)
        hm = input_conv(h, lw["canon1"])
        if L["type"] == "mlstm":
            y = mlstm_mixer(hm, sub(lw, "mix."), L["mixer"], eps)
        elif L["type"] == "parallel":
            y = parallel_mixer(hm, sub(lw, "mix."), L["mixer"], eps)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + feed_forward(h, sub(lw, "mlp."), L["mlp"])
        x = x + mult * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


# ------------------------------------------------------------------------------------------------ random models
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """every tensor of a checkpoint of this configuration, by name"""
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "final.norm": (D,), "final.norm.b": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        s.update({p + "norm1": (D,), p + "norm1.b": (D,), p + "canon1": (D, cfg["canon"]["taps"])})
        x = p + "mix."
        if L["type"] == "mlstm":
            H, dk, dv = m["heads"], m["dim"], m.get("vdim", m["dim"])
            s.update({x + "q": (H * dk, D), x + "k": (H * dk, D), x + "v": (H * dv, D), x + "g": (H * dv, D),
                      x + "o": (D, H * dv), x + "norm": (H * dv,), x + "i": (H, D), x + "i.b": (H,), x + "f": (H, D),
                      x + "f.b": (H,)})
        else:
            a, r = m["left"], m["right"]
            H, G, dk, dv = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a.get("vdim", a["dim"])
            y = x + "left."
            s.update({y + "q": (H * dk, D), y + "k": (G * dk, D), y + "v": (G * dv, D), y + "pb": (H,), y + "o": (D, H * dv),
                      y + "out": (D,)})
            H, G, dk, dv, n = r["heads"], r.get("kv_heads", r["heads"]), r["dim"], r.get("vdim", r["dim"]), r["conv"]
            y = x + "right."
            s.update({y + "q": (G * dk, D), y + "q.conv": (G * dk, n), y + "k": (G * dk, D), y + "k.conv": (G * dk, n),
                      y + "v": (H * dv, D), y + "v.conv": (H * dv, n), y + "b": (H, D), y + "A_log": (H,), y + "norm": (dv,),
                      y + "a": (H, D), y + "dt_bias": (H,), y + "g": (H * dv, D), y + "o": (D, H * dv), y + "out": (D,)})
        f = L.get("mlp")
        if f:
            x = p + "mlp."
            if f.get("kind", "dense") == "dense":
                s.update({x + "gate": (f["ff"], D), x + "up": (f["ff"], D), x + "down": (D, f["ff"])})
            else:
                E, Fe = f["router"]["experts"], f["expert"]["ff"]
                s.update({x + "router": (E, D), x + "correction": (E,)})
                for e in range(E):
                    s.update({x + f"e{e}.gate": (Fe, D), x + f"e{e}.up": (Fe, D), x + f"e{e}.down": (D, Fe)})
                if f.get("shared"):
                    Fs = f["shared"]["ff"]
                    s.update({x + "shared.gate": (Fs, D), x + "shared.up": (Fs, D), x + "shared.down": (D, Fs),
                              x + "shared.sg": (1, D)})
    return s


def random_model(cfg: dict, seed: int, scale: float = 1.0) -> Dict[str, torch.Tensor]:
    """weights whose every mechanism matters in the logits: matrices of unit-variance outputs, norm weights around
    one, biases, gate and decay parameters of order one; forget gates that let a state live for tens of tokens"""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        rnd = lambda: torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm", "out"):
            t = 1.0 + 0.3 * rnd()
        elif leaf in ("conv", "canon1"):
            t = 0.5 * rnd()
        elif name.endswith("f.b"):
            t = 2.0 + rnd()
        elif name.endswith("i.b"):
            t = rnd()
        elif leaf == "pb":
            t = rnd() - 2.0
        elif leaf == "A_log":
            t = rnd()
        elif leaf == "dt_bias":
            t = rnd() - 1.5
        elif leaf == "correction":
            t = 0.3 * rnd()
        elif leaf == "b" and len(shape) == 1:
            t = 0.3 * rnd()
        elif leaf == "embed":
            t = rnd() / math.sqrt(shape[-1])
        else:
            t = rnd() * (scale / math.sqrt(shape[-1]))
        w[name] = t.to(torch.bfloat16)          # what a checkpoint stores
    return w
