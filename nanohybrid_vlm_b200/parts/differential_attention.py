"""Differential attention: two softmax maps per head over the same values, the second taken off the first.

Parameters: ``num_heads`` (H), ``num_kv_heads`` (G), ``head_dim`` (d, of one map's queries and keys), ``v_head_dim``, ``scale``
(on q . k), ``position`` (a PartSpec of a position encoding with a rotary table, or None; it turns every map's first
elements by halves), ``eps`` (of the norms below), ``softcap`` (None, or c: scores become c tanh(score / c)), ``window`` (None:
all keys; n: the last n), ``keep_window`` (how many keys the pages keep, where another layer with a wider window reads them;
None: all), ``diff`` (the constant part of the second map's share), ``own_kv`` (False: the layer has no key / value
projections and norms and reads the keys and values that another run stored, ``LayerRun.cache_from``).

q has H and k has G heads of two maps of d elements each, [map 1, map 2]; every map is divided by its root mean square, times
a weight [d] of its kind, then rotated.  With a1 and a2 the two maps' outputs of a head, share = exp(lq1 . lk1) - exp(lq2 . lk2) +
diff, one number per layer:  o = a1 - share * a2, then o / rms(o) * (1 - diff) over the head's values, no weight.

Tensors: ``qkv`` [2 H d (+ 2 G d + G dv), width] from ``q``, ``k``, ``v``; ``q.norm``, ``k.norm`` [d]; ``lq1``, ``lk1``, ``lq2``, ``lk2`` [d]
(float32); ``o`` [width, H dv].

A page row holds a KV head's two key maps side by side, and a query of map m is padded with zeros to the whole row, so that its
product with a row is its own map's score: the 2 H / G queries of a KV head are one group of an ordinary grouped-query kernel,
which reads every key and value once for both maps.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, Mixer, PagedKVNeed
from .spec import ParamDecl, Source

MAPS = 2
SHARE_VECTORS = ("lq1", "lk1", "lq2", "lk2")


class DifferentialAttention(Mixer):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.nq = int(spec["num_heads"])
        self.nkv = int(spec["num_kv_heads"])
        self.d = int(spec["head_dim"])
        self.dv = int(spec["v_head_dim"])
        if self.nq % self.nkv:
            raise ValueError(f"{self.nq} query heads do not divide into {self.nkv} KV heads")
        self.scale = float(spec["scale"])
        self.eps = float(spec["eps"])
        self.diff = float(spec["diff"])
        cap = spec.get("softcap")
        self.softcap = None if cap is None else float(cap)
        if self.softcap is not None and self.softcap <= 0:
            raise ValueError("a cap on the scores must be positive")
        self.position = env.position(spec.get("position"))
        self.window = spec.get("window")
        self.keep_window = spec.get("keep_window", self.window)
        if self.keep_window is not None and (self.window is None or self.keep_window < self.window):
            raise ValueError("the pages must keep at least the keys that the layer's window shows")
        self.own_kv = bool(spec.get("own_kv", True))
        # what a page row and a padded query hold: on the tensor cores keys and values share one size in steps of 16
        self.D = MAPS * self.d
        if env.dtype == torch.bfloat16:
            self.D = -(-max(self.D, self.dv) // 16) * 16
        self.q_size = self.nq * MAPS * self.d
        self.k_size = self.nkv * MAPS * self.d if self.own_kv else 0
        self.v_size = self.nkv * self.dv if self.own_kv else 0

    def params(self):
        H = self.env.hidden_size
        sources = [Source("q", 0, self.q_size)]
        if self.own_kv:
            sources += [Source("k", self.q_size, self.k_size), Source("v", self.q_size + self.k_size, self.v_size)]
        decls = [ParamDecl("qkv", (self.q_size + self.k_size + self.v_size, H), sources=tuple(sources)),
                 ParamDecl("o", (H, self.nq * self.dv)), ParamDecl("q.norm", (self.d,), init="norm")]
        if self.own_kv:
            decls.append(ParamDecl("k.norm", (self.d,), init="norm"))
        return decls + [ParamDecl(name, (self.d,), init="map_share", storage="float32") for name in SHARE_VECTORS]

    def bind(self, tensors):
        super().bind(tensors)
        a, b, c, d = (tensors[name].double() for name in SHARE_VECTORS)
        self.share = (torch.exp((a * b).sum()) - torch.exp((c * d).sum()) + self.diff).reshape(1).float()

    def cache_need(self):
        return PagedKVNeed(self.nkv, self.D, self.keep_window, v_head_dim=self.dv)

    def streamed_weights(self):
        return [(self.w_qkv, 0), (self.w_o, 0)]

    def forward(self, x, batch, cache):
        T = x.shape[0]
        if cache.writes != self.own_kv:
            raise ValueError("a layer with keys of its own writes its pages; one without reads another run's (cache_from)")
        qkv = self.new(T, self.q_size + self.k_size + self.v_size)
        ops.linear(qkv, x, self.w_qkv)
        rot = self.position.rotary() if self.position is not None else None
        table, rotary_dim = rot if rot is not None else (None, 0)
        q = self.new(T, self.nq * MAPS * self.D)
        ops.heads_store(qkv, q, self.D, cache.pages if self.own_kv else None, cache.tables.slot_mapping, batch, table, rotary_dim,
                        self.nq, self.nkv, self.d, self.dv, self.eps, self.w_q_norm, self.w_k_norm if self.own_kv else None,
                        maps=MAPS)
        a = self.new(T, self.nq * MAPS * self.dv)
        ops.attention_sink(a, q, cache.pages, cache.tables, batch, self.nq * MAPS, self.nkv, self.D, self.dv, self.scale,
                           window=self.window or 0, softcap=self.softcap)
        o = self.new(T, self.nq * self.dv)
        ops.map_difference(o, a, self.share, 1.0 - self.diff, self.eps, self.nq, self.dv)
        y = self.new(T, self.env.hidden_size)
        ops.linear(y, o, self.w_o)
        return y


MIXERS.register("differential_attention", DifferentialAttention)
