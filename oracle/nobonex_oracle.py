"""Plain, slow restatement of the Nobonex decoder in PyTorch on the CPU: one function per mechanism, whole sequences
at a time, explicit loops over positions where a mechanism is a recurrence, no cache, no batching.
Test infrastructure only: the product package never imports it and it imports nothing of the product.

Notation: T tokens, D model width, H heads, G key/value heads (mamba2: groups), dk query/key size per head, dv value size,
N state size, E experts.  ``w`` maps tensor names to [out, in] matrices (or vectors); ``cfg`` is the dictionary form of a
checkpoint's ``config.json``."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F


def sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


# ------------------------------------------------------------------------------------------------ norms, activations
def dynamic_tanh(x, w: Dict[str, torch.Tensor], name: str):
    """a norm without statistics: weight * tanh(alpha x) + bias"""
    return w[name] * torch.tanh(w[name + ".alpha"] * x) + w[name + ".b"]


def unit_rms(x, eps: float):
    """x / sqrt(mean(x^2) + eps) over the last axis"""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------ short convolution
def causal_conv(x, taps, bias=None):
    """x [T, C], taps [C, n] (last column weighs the current position, zeros before the start) -> [T, C]"""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += taps[:, j] * x[:T - back]
    return out if bias is None else out + bias


# ------------------------------------------------------------------------------------------------ rotation
def yarn(freq: List[float], base: float, dims: int, s: dict):
    """(frequencies, factor of cos and sin): fast-turning pairs keep their frequency, slow ones are divided by the factor,
    a linear ramp over the pair index in between"""
    def pair_of(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot: Optional[dict], interleaved: bool):
    """x [T, heads, d]: the first rot.dims coordinates turn by position-dependent angles, in pairs (2i, 2i+1) or
    (i, i + dims/2)"""
    if not rot or not rot["dims"]:
        return x
    n = rot["dims"]
    freq, mag = [rot["base"] ** (-2 * i / n) for i in range(n // 2)], 1.0
    if rot.get("scaling"):
        freq, mag = yarn(freq, rot["base"], n, rot["scaling"])
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freq):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n // 2)
        cs = (mag * torch.cos(pos * f)).to(x.dtype)[:, None]
        sn = (mag * torch.sin(pos * f)).to(x.dtype)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a] = u * cs - v * sn
        out[..., b] = v * cs + u * sn
    return out


# ------------------------------------------------------------------------------------------------ attention
def visible(T: int, chunk: int):
    """[T, T] bool: i sees j <= i, and with a chunk size only inside i's chunk (counted from position 0)"""
    i = torch.arange(T)
    m = i[None, :] <= i[:, None]
    return m & (i[None, :] // chunk == i[:, None] // chunk) if chunk else m


def softmax_attention(q, k, v, scale: float, seen, cap: float = 0.0):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H * dv]"""
    T, H, _ = q.shape
    G, dv = v.shape[1:]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = torch.where(seen, s, torch.tensor(-math.inf, dtype=s.dtype))
        out[:, hd] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(T, H * dv)


def conv_attention(h, w, m: dict, eps: float):
    """queries and keys: convolution over time, RMS norm over the whole projection, rotation; values: the convolved keys"""
    T, H, G, dk = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(h @ w["q"].T, w["q.conv"])
    k = causal_conv(h @ w["k"].T, w["k.conv"])
    v = k.reshape(T, G, dk)
    q = rotate((unit_rms(q, eps) * w["q.norm"]).reshape(T, H, dk), m.get("rot"), True)
    k = rotate((unit_rms(k, eps) * w["k.norm"]).reshape(T, G, dk), m.get("rot"), True)
    return softmax_attention(q, k, v, m["scale"], visible(T, 0)) @ w["o"].T


def chunk_attention(h, w, m: dict, eps: float, shared=None):
    """biased projections, an RMS norm per head, rotation, capped scores inside a chunk, an output gate.  ``shared``: another
    layer's (keys, values) to be used instead of own ones.  Returns (result, (keys, values))."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, dk)
    q = rotate(unit_rms(q, eps) * w["q.norm"], m.get("rot"), False)
    if shared is None:
        k = (h @ w["k"].T + w["k.b"]).reshape(T, G, dk)
        k = rotate(unit_rms(k, eps) * w["k.norm"], m.get("rot"), False)
        v = (h @ w["v"].T + w["v.b"]).reshape(T, G, dv)
    else:
        k, v = shared
    o = softmax_attention(q, k, v, m["scale"], visible(T, m["mask"]["size"]), m["softcap"])
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, (k, v)


# ------------------------------------------------------------------------------------------------ mamba2
def ssd_core(x, B, C, dt, a_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] -> [T, H, P]; one position after the other"""
    T, H, P = x.shape
    G, N = B.shape[1:]
    out = torch.zeros_like(x)
    for hd in range(H):
        g = hd // (H // G)
        S = torch.zeros(N, P, dtype=x.dtype)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[hd]) * dt[t, hd]) * S + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            out[t, hd] = S.T @ C[t, g] + D[hd] * x[t, hd]
    return out


def mamba2_mixer(h, w, m: dict, eps: float):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner, bc = H * P, G * N
    p = h @ w["in"].T
    z, dt = p[:, :inner], p[:, 2 * inner + 2 * bc:]
    xbc = silu(causal_conv(p[:, inner:2 * inner + 2 * bc], w["conv"], w["conv.b"]))
    y = ssd_core(xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + bc].reshape(T, G, N),
                 xbc[:, inner + bc:].reshape(T, G, N), F.softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    y = (y.reshape(T, inner) * silu(z)).reshape(T, m["norm_groups"], -1)
    return (unit_rms(y, eps).reshape(T, inner) * w["norm"]) @ w["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def expert(h, w, limit: float):
    g = torch.clamp(h @ w["gate"].T, max=limit)
    u = torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def feed_forward(h, w, f: dict):
    if f.get("kind", "dense") == "dense":
        return gated_ff(h, w)
    s = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in s[t].topk(f["router"]["top"]).indices.tolist():
            out[t] += expert(s[t, e] * h[t:t + 1], sub(w, f"e{e}."), f["expert"]["limit"])[0]
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: list = None):
    """logits [T, vocab] of one sequence from position 0; every tensor is taken to ``dtype`` first"""
    w = {k: (t.to(dtype) if t.is_floating_point() else t) for k, t in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    kv = {}
    for i, L in enumerate(cfg["layers"]):
        lw, m = sub(w, f"l{i}."), L["mixer"]
        mw = sub(lw, "mix.")
        h = dynamic_tanh(x, lw, "norm1")
        if L["type"] == "attention":
            y = conv_attention(h, mw, m, eps)
        elif L["type"] == "mamba2":
            y = mamba2_mixer(h, mw, m, eps)
        elif L["type"] == "attention_2":
            j = m.get("kv_from")
            y, kv[i] = chunk_attention(h, mw, m, eps, None if j is None else kv[j])
        else:
            raise ValueError(L["type"])
        x = x + mult * dynamic_tanh(y, lw, "norm1b")
        if L.get("mlp"):
            x = x + mult * dynamic_tanh(feed_forward(dynamic_tanh(x, lw, "norm2"), sub(lw, "mlp."), L["mlp"]), lw, "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return dynamic_tanh(x, w, "final.norm") @ w["head"].T


# ------------------------------------------------------------------------------------------------ random models
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """every tensor of a checkpoint of this configuration, by name"""
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "head": (V, D)}

    def norm(name):
        s.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        x = p + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            norm(p + n)
        if L["type"] == "mamba2":
            H, P, N, G, n = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            ch = H * P + 2 * G * N
            s.update({x + "in": (H * P + ch + H, D), x + "conv": (ch, n), x + "conv.b": (ch,), x + "dt_bias": (H,),
                      x + "A_log": (H,), x + "D": (H,), x + "norm": (H * P,), x + "o": (D, H * P)})
        else:
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            s.update({x + "q": (H * dk, D), x + "o": (D, H * dv)})
            if L["type"] == "attention":
                s.update({x + "k": (G * dk, D), x + "q.norm": (H * dk,), x + "k.norm": (G * dk,),
                          x + "q.conv": (H * dk, m["conv"]), x + "k.conv": (G * dk, m["conv"])})
            else:
                s.update({x + "q.b": (H * dk,), x + "q.norm": (dk,), x + "g": (H * dv, D)})
                if m.get("kv_from") is None:
                    s.update({x + "k": (G * dk, D), x + "k.b": (G * dk,), x + "k.norm": (dk,), x + "v": (G * dv, D),
                              x + "v.b": (G * dv,)})
        if f:
            x = p + "mlp."
            if f.get("kind", "dense") == "dense":
                s.update({x + "gate": (f["ff"], D), x + "up": (f["ff"], D), x + "down": (D, f["ff"])})
            else:
                E, Fe = f["router"]["experts"], f["expert"]["ff"]
                s[x + "router"] = (E, D)
                for e in range(E):
                    s.update({x + f"e{e}.gate": (Fe, D), x + f"e{e}.up": (Fe, D), x + f"e{e}.down": (D, Fe)})
    return s


def random_model(cfg: dict, seed: int, scale: float = 1.0) -> Dict[str, torch.Tensor]:
    """weights whose every mechanism matters in the logits: matrices of unit-variance outputs, norm weights around one,
    biases and norm slopes of order one, decays that let a state live for tens of tokens"""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        rnd = lambda: torch.randn(shape, generator=g)
        if leaf == "alpha":
            t = 0.7 + 0.2 * rnd()
        elif leaf.startswith("norm"):
            t = 1.0 + 0.3 * rnd()
        elif leaf == "conv":
            t = 0.5 * rnd()
        elif leaf == "b" and len(shape) == 1:
            t = 0.3 * rnd()
        elif leaf == "A_log":
            t = 0.7 * rnd() - 0.5
        elif leaf == "dt_bias":
            t = rnd() - 2.0
        elif leaf == "D":
            t = 0.5 + rnd()
        elif leaf == "embed":
            t = rnd()
        else:
            t = rnd() * (scale / math.sqrt(shape[-1]))
        w[name] = t.to(torch.bfloat16)          # what a checkpoint stores
    return w
