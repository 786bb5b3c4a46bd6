"""A plain, slow restatement of the Kilisun design in float64 on the CPU: one function per mechanism, no cache, no
batching.  The tests compare the engine with it; it shares nothing with the engine's code.

Notation.  x [T, W] is one request's residual stream, h a sublayer's input.  Linear weights are [out, in] and applied as
h @ W.T.  ``cfg`` is the config.json dictionary, ``w`` maps tensor names to float64 tensors.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------- small pieces
def unit_rms(x, eps):
    """x over the root of (its mean square + eps), along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_about_one(x, weight, eps):
    """The model's norm: the stored weight is what the factor differs from one by."""
    return unit_rms(x, eps) * (1.0 + weight)


def taps_over_time(u, taps):
    """u [T, C], taps [C, K]: each channel's last K inputs weighted, the newest by the last tap; zeros before the start."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    out = torch.zeros_like(u)
    for j in range(K):
        out = out + padded[j:j + T] * taps[:, j]
    return out


def query_temperature(positions, coef, every):
    """The factor on a query at each position: 1 until position ``every`` - 2, then growing with the logarithm."""
    steps = torch.div(positions + 1, every, rounding_mode="floor").to(F64)
    return 1.0 + coef * torch.log(steps + 1.0)


def turn_halves(x, positions, base, dims):
    """x [T, heads, d]: elements i and i + dims / 2 of the first ``dims`` turn together by position * base^(-2i / dims)."""
    n = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(n)], dtype=F64)
    ang = positions.to(F64)[:, None] * freq[None, :]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b, rest = x[..., :n], x[..., n:dims], x[..., dims:]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, rest], -1)


def in_window(T, size):
    """[T, T]: which keys (columns) a query (row) sees; ``size`` None: all up to itself, else the last ``size``."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def soft_capped(scores, cap):
    return scores if cap is None else cap * torch.tanh(scores / cap)


def softmax_rows(scores, visible):
    return torch.softmax(scores.masked_fill(~visible, -math.inf), -1)


# ---------------------------------------------------------------- mixers
def window_size(m):
    return None if m.get("mask") is None else m["mask"]["size"]


def attention(h, m, w, p, eps):
    """Grouped-query attention over all keys, without positions but for the queries' temperature: a short filter over time
    on q and k, values that are the filtered keys, then a norm per head, a gate per head on the output."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    if m.get("conv"):
        q, k = taps_over_time(q, w[p + "q.conv"]), taps_over_time(k, w[p + "k.conv"])
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    v = k
    q, k = unit_rms(q, eps) * w[p + "q.norm"], unit_rms(k, eps) * w[p + "k.norm"]
    if m.get("q_temp") is not None:
        q = q * query_temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    seen = in_window(T, None)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    heads = []
    for a in range(H):
        b = a // (H // G)
        heads.append(softmax_rows((q[:, a] @ k[:, b].T) * m["scale"], seen) @ v[:, b] * gate[:, a:a + 1])
    return torch.cat(heads, -1) @ w[p + "o"].T


def map_keys_values(h, m, w, p, eps):
    """The keys [T, G, 2, d] (normed, turned) and values [T, G, dv] of a differential attention layer."""
    T, G, d = h.shape[0], m["kv_heads"], m["dim"]
    k = unit_rms((h @ w[p + "k"].T).reshape(T, G * 2, d), eps) * w[p + "k.norm"]
    k = turn_halves(k, torch.arange(T), m["rot"]["base"], m["rot"]["dims"]).reshape(T, G, 2, d)
    return k, (h @ w[p + "v"].T).reshape(T, G, m["vdim"])


def map_share(m, w, p):
    """How much of the second map is taken off the first."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + m["diff"]


def maps_combined(a1, a2, share, diff, eps):
    return unit_rms(a1 - share * a2, eps) * (1.0 - diff)


def differential_attention(h, m, w, p, eps, kv):
    """Two softmax maps per head over the same values, the second taken off the first; capped scores; a window.  ``kv``:
    the keys and values, this layer's own or another layer's."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    k, v = kv
    q = unit_rms((h @ w[p + "q"].T).reshape(T, H * 2, d), eps) * w[p + "q.norm"]
    q = turn_halves(q, torch.arange(T), m["rot"]["base"], m["rot"]["dims"]).reshape(T, H, 2, d)
    seen = in_window(T, window_size(m))
    share = map_share(m, w, p)
    heads = []
    for a in range(H):
        b = a // (H // G)
        out = []
        for i in range(2):
            s = soft_capped((q[:, a, i] @ k[:, b, i].T) * m["scale"], m.get("softcap"))
            out.append(softmax_rows(s, seen) @ v[:, b])
        heads.append(maps_combined(out[0], out[1], share, m["diff"], eps))
    return torch.cat(heads, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forwards
def clamped_unit(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, correction, r):
    """(ids [T, top], weights [T, top]): sigmoid scores; the choice by score + correction among the groups whose two
    largest choice scores sum highest; the weights are the scores times a factor."""
    s = torch.sigmoid(h @ router.T)
    c = s + correction
    T, E = c.shape
    groups = r.get("groups") or dict(count=1, keep=1)
    per = c.reshape(T, groups["count"], E // groups["count"])
    worth = torch.topk(per, min(2, per.shape[-1]), dim=-1).values.sum(-1)
    best = torch.topk(worth, groups["keep"], dim=-1).indices
    open_ = torch.zeros(T, groups["count"], dtype=torch.bool).scatter_(1, best, True)
    c = per.masked_fill(~open_[..., None], -math.inf).reshape(T, E)
    ids = torch.topk(c, r["top"], dim=-1).indices
    return ids, torch.gather(s, 1, ids) * r.get("scale", 1.0)


def mixture(h, mlp, w, p):
    r = mlp["router"]
    ids, weights = route(h, w[p + "router"], w[p + "correction"], r)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        share = (weights * (ids == e)).sum(-1, keepdim=True)
        out = out + share * clamped_unit(h, w, f"{p}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * clamped_unit(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


# ---------------------------------------------------------------- the model
def layer_states(cfg, w, tokens):
    """The residual stream after every layer, [layers, T, W]."""
    eps = cfg["norm"]["eps"]
    x = norm_about_one(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    kept, states = {}, []
    for i, layer in enumerate(cfg["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        h = norm_about_one(x, w[l + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention(h, m, w, l + "mix.", eps)
        elif layer["type"] == "attention_2":
            src = m.get("kv_from")
            kept[i] = map_keys_values(h, m, w, l + "mix.", eps) if src is None else kept[src]
            y = differential_attention(h, m, w, l + "mix.", eps, kept[i])
        else:
            raise ValueError(layer["type"])
        x = x + norm_about_one(y, w[l + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm_about_one(x, w[l + "norm2"], eps)
            y = clamped_unit(h, w, l + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else mixture(h, mlp, w, l + "mlp.")
            x = x + norm_about_one(y, w[l + "norm2b"], eps)
        states.append(x)
    return torch.stack(states)


def forward(cfg, w, tokens):
    """Logits [T, vocab] of one request, every position."""
    x = layer_states(cfg, w, tokens)[-1]
    return norm_about_one(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


# ---------------------------------------------------------------- random weights for the tests
def tensor_shapes(cfg):
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "embed.norm": (W,), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        m, l = layer["mixer"], f"l{i}."
        p = l + "mix."
        for n in ("norm1", "norm1b") if layer.get("mlp") is None else ("norm1", "norm1b", "norm2", "norm2b"):
            shapes[l + n] = (W,)
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            shapes.update({p + "q": (H * d, W), p + "k": (G * d, W), p + "q.norm": (d,), p + "k.norm": (d,),
                           p + "g": (H, W), p + "o": (W, H * dv)})
            if m.get("conv"):
                shapes.update({p + "q.conv": (H * d, m["conv"]), p + "k.conv": (G * d, m["conv"])})
        else:
            shapes.update({p + "q": (H * 2 * d, W), p + "q.norm": (d,), p + "o": (W, H * dv)})
            shapes.update({p + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
            if m.get("kv_from") is None:
                shapes.update({p + "k": (G * 2 * d, W), p + "v": (G * dv, W), p + "k.norm": (d,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        p = l + "mlp."
        stacks = [(p, mlp["ff"])] if mlp["kind"] == "dense" else [(f"{p}e{e}.", mlp["expert"]["ff"])
                                                                 for e in range(mlp["router"]["experts"])]
        if mlp["kind"] == "moe":
            E = mlp["router"]["experts"]
            shapes.update({p + "router": (E, W), p + "correction": (E,)})
            if mlp.get("shared") is not None:
                stacks.append((p + "shared.", mlp["shared"]["ff"]))
                shapes[p + "shared.sg"] = (1, W)
        for s, ff in stacks:
            shapes.update({s + "gate": (ff, W), s + "up": (ff, W), s + "down": (W, ff)})
    return shapes


def random_weights(cfg, seed):
    """bfloat16 tensors under the checkpoint's names: matrices N(0, 1/in), norms that differ from channel to channel, the
    maps' vectors of a size that makes their share differ from its constant, corrections that change the choice."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=gen)
        if name.endswith((".q.norm", ".k.norm")):
            t = 1.0 + 0.2 * r
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 0.2 * r
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = 0.6 * r / shape[0] ** 0.25
        elif name.endswith(".correction"):
            t = 0.3 * r - 0.4
        elif name.endswith(".conv"):
            t = 0.6 * r
        elif name == "embed":
            t = r / math.sqrt(shape[-1]) * 2.0
        else:
            t = r / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
