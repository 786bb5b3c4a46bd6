"""A plain, slow restatement of the Vozorax design in float64 on the CPU: one function per mechanism, no cache, no
batching.  The tests compare the engine with it; it shares nothing with the engine's code.

Notation.  X [S, T, W] are the S copies of one request's residual stream, h a sublayer's input.  Linear weights are
[out, in] and applied as h @ W.T.  ``cfg`` is the config.json dictionary, ``w`` maps tensor names to float64 tensors.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------- small pieces
def unit_rms(x, eps):
    """x over the root of (its mean square + eps), along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def read_streams(X, read):
    """What a sublayer reads of the copies: their sum weighted by ``read`` [S]."""
    return torch.einsum("s,stw->tw", read, X)


def write_streams(X, mix, write, y):
    """The copies after a sublayer with output y: copy t becomes sum_s mix[s, t] X_s + write[t] y, every copy from
    the old ones."""
    return torch.einsum("sd,stw->dtw", mix, X) + write[:, None, None] * y[None]


def turn_neighbours(x, positions, base):
    """x [T, heads, n], n even: elements 2i and 2i + 1 of each head turn together by position * base^(-2i / n)."""
    n = x.shape[-1]
    freq = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * freq[None, :]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = x[..., 0::2], x[..., 1::2]
    return torch.stack([a * cos - b * sin, b * cos + a * sin], -1).flatten(-2)


def in_window(T, size):
    """[T, T]: which keys (columns) a query (row) sees; ``size`` None: all up to itself, else the last ``size``."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def softmax_rows(scores, visible, sink=None):
    """scores [T, T] for one head; ``sink``: a number whose exponential joins the denominator without a key."""
    s = scores.masked_fill(~visible, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, torch.full_like(top, float(sink)))
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return e / den


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------- mixers
def window_size(m):
    return None if m.get("mask") is None else m["mask"]["size"]


def latent_attention(h, m, w, p, eps):
    """Attention whose queries pass a normed latent and whose keys and values are expanded from one normed latent per
    token; one rotated key part for all heads; a sliding window; ordinary softmax."""
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = unit_rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, dn + dr)
    q_plain, q_rot = q[..., :dn], turn_neighbours(q[..., dn:], pos, m["rot"]["base"])
    kv = h @ w[p + "dkv"].T
    c = unit_rms(kv[:, :rank], eps) * w[p + "dkv.norm"]
    k_rot = turn_neighbours(kv[:, None, rank:], pos, m["rot"]["base"])[:, 0]
    k_plain = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    seen = in_window(T, window_size(m))
    heads = []
    for a in range(H):
        s = (q_plain[:, a] @ k_plain[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        heads.append(softmax_rows(s, seen) @ v[:, a])
    return torch.cat(heads, -1) @ w[p + "o"].T


def mixed_values(v, v_first, share):
    """(1 - share) v + share v_first."""
    return (1.0 - share) * v + share * v_first


def attention(h, m, w, p, eps, v_first=None):
    """Grouped-query attention without positions: q and k normed over all heads together, a sliding window, a sink per
    head; ``v_first`` [T, G dv]: the first value-mixing layer's values, mixed into this layer's.  Returns (output,
    this layer's own values before any mixing)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(T, G, d)
    own = h @ w[p + "v"].T
    v = own if v_first is None else mixed_values(own, v_first, w[p + "vmix"])
    v = v.reshape(T, G, dv)
    seen = in_window(T, window_size(m))
    heads = []
    for a in range(H):
        b = a // (H // G)
        s = (q[:, a] @ k[:, b].T) * m["scale"]
        heads.append(softmax_rows(s, seen, w[p + "sink"][a]) @ v[:, b])
    return torch.cat(heads, -1) @ w[p + "o"].T, own


# ---------------------------------------------------------------- feed-forwards
def gated_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def relu_squared_mlp(h, w, p):
    return (torch.relu(h @ w[p + "up"].T) ** 2) @ w[p + "down"].T


def route(h, router, bias, top):
    """The ``top`` largest logits per token and the softmax over these alone: (ids [T, top], weights [T, top])."""
    z = h @ router.T + bias
    vals, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(vals, -1)


def mixture(h, mlp, w, p):
    """Routed experts (up, squared relu, down), their outputs weighted, beside a shared expert with a gate per token."""
    ids, weights = route(h, w[p + "router"], w[p + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        share = (weights * (ids == e)).sum(-1, keepdim=True)
        out = out + share * relu_squared_mlp(h, w, f"{p}e{e}.")
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * relu_squared_mlp(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------- the model
def layer_states(cfg, w, tokens):
    """The sum of the streams after every layer, [layers, T, W]."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = x[None].repeat(cfg["streams"], 1, 1)
    v_first = None
    states = []
    for i, layer in enumerate(cfg["layers"]):
        l, m = f"l{i}.", layer["mixer"]
        h = unit_rms(read_streams(X, w[l + "hc1.in"]), eps) * w[l + "norm1"]
        if layer["type"] == "latent_attention":
            y = latent_attention(h, m, w, l + "mix.", eps)
        elif layer["type"] == "attention":
            y, own = attention(h, m, w, l + "mix.", eps, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = own
        else:
            raise ValueError(layer["type"])
        X = write_streams(X, w[l + "hc1.mix"], w[l + "hc1.out"], y)
        if layer.get("mlp") is not None:
            h = unit_rms(read_streams(X, w[l + "hc2.in"]), eps) * w[l + "norm2"]
            y = (gated_mlp(h, w, l + "mlp.") if layer["mlp"]["kind"] == "dense" else mixture(h, layer["mlp"], w, l + "mlp."))
            X = write_streams(X, w[l + "hc2.mix"], w[l + "hc2.out"], y)
        states.append(X.sum(0))
    return torch.stack(states)


def forward(cfg, w, tokens):
    """Logits [T, vocab] of one request, every position."""
    x = layer_states(cfg, w, tokens)[-1]
    return (unit_rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T


# ---------------------------------------------------------------- random weights for the tests
def tensor_shapes(cfg):
    W, S = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        m, l = layer["mixer"], f"l{i}."
        p = l + "mix."
        subs = (1,) if layer.get("mlp") is None else (1, 2)
        for n in subs:
            shapes.update({f"{l}norm{n}": (W,), f"{l}hc{n}.in": (S,), f"{l}hc{n}.out": (S,), f"{l}hc{n}.mix": (S, S)})
        if layer["type"] == "latent_attention":
            H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
            shapes.update({p + "dq": (m["q_rank"], W), p + "dq.norm": (m["q_rank"],), p + "uq": (H * (dn + dr), m["q_rank"]),
                           p + "dkv": (m["kv_rank"] + dr, W), p + "dkv.norm": (m["kv_rank"],),
                           p + "uk": (H * dn, m["kv_rank"]), p + "uv": (H * dv, m["kv_rank"]), p + "o": (W, H * dv)})
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            shapes.update({p + "q": (H * d, W), p + "k": (G * d, W), p + "v": (G * dv, W), p + "q.norm": (H * d,),
                           p + "k.norm": (G * d,), p + "sink": (H,), p + "o": (W, H * dv)})
            if m.get("v_mix"):
                shapes[p + "vmix"] = ()
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        p = l + "mlp."
        if mlp["kind"] == "dense":
            shapes.update({p + "gate": (mlp["ff"], W), p + "up": (mlp["ff"], W), p + "down": (W, mlp["ff"])})
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        shapes.update({p + "router": (E, W), p + "router.b": (E,)})
        for e in range(E):
            shapes.update({f"{p}e{e}.up": (ff, W), f"{p}e{e}.down": (W, ff)})
        if mlp.get("shared") is not None:
            sf = mlp["shared"]["ff"]
            shapes.update({p + "shared.up": (sf, W), p + "shared.down": (W, sf), p + "shared.sg": (1, W)})
    return shapes


def random_weights(cfg, seed):
    """bfloat16 tensors under the checkpoint's names: matrices N(0, 1/in), norms near 1, the streams' matrices near a
    mixing that keeps sizes, sinks, biases and the value share of a size that shows in the logits."""
    gen = torch.Generator().manual_seed(seed)
    S = cfg["streams"]
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=gen)
        if name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.2 * r
        elif name.endswith(".mix") and ".hc" in name:
            t = torch.eye(S) * 0.8 + 0.2 * r
        elif name.endswith((".in", ".out")) and ".hc" in name:
            t = 0.6 + 0.4 * r
        elif name.endswith(".vmix"):
            t = torch.tensor(0.35) + 0.1 * r
        elif name.endswith((".sink", ".router.b")) or name == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
