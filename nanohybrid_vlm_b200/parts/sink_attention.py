"""Grouped-query attention with options that several designs combine differently: a learned sink per head, rotation
before a weightless q/k norm, value heads whose size may differ from the key heads', values that are the keys
themselves, a window or chunks, projection biases, and a sigmoid gate on the output.

Parameters: ``num_heads``, ``num_kv_heads``, ``head_dim`` (queries and keys), ``v_head_dim`` (values; default
``head_dim``), ``scale`` (on q . k; None: head_dim ** -0.5), ``position`` (a PartSpec of a position encoding with a
rotary table, or None), ``unit_norm_eps`` (after the rotation each q and k head is divided by its root mean square
with this eps inside the root; None: no norm), ``sink`` (True: the softmax denominator of head h also holds
exp(sink_h), a learned number with no key and no value, unscaled, counted once), ``window`` (None: all keys; n: the
last n), ``chunk`` (None, or n: a query sees only the keys of its own chunk of n positions, chunks counted from
position 0 of the request), ``values`` ("projected": a projection of their own; "keys": the values are the key heads as
projected, bias included, before the rotation, and there is no value projection), ``bias`` (True: q, k and the output
projection have biases ``q.b``, ``k.b``, ``o.b``), ``output_gate`` (None, or "sigmoid": the concatenated heads are
multiplied by sigmoid(g(x)) before the output projection, g a projection of the mixer's input; "sigmoid_head": g has one
output per head and head h is multiplied by sigmoid(g(x))_h), ``qk_norm_weight`` (True: after the unit norm each
q and k head is multiplied by a learned weight [head_dim], ``q.norm`` / ``k.norm``, shared by the heads),
``distance_slope_base`` (None, or b: the score of head h at distance n behind the query loses 2^(-b (h + 1) / H) * n),
``own_kv`` (False: the layer has no key / value projections, norms or pages of its own and reads the keys and values
that another run stored, ``LayerRun.cache_from``), ``keep_window`` (how many keys the pages keep, where that is more
than this layer's own ``window`` shows: a layer whose pages another layer with a wider window reads; None: all),
``keep_first`` (n, with a window: the keys at positions below n stay visible to every later query, at their true
positions, and their pages are kept), ``sink_constant`` (a number: the denominator of every head holds exp of it, as a
learned sink would, but no tensor is read; 0.0 adds one), ``qk_norm_order`` ("after_rotation", the default, or
"before_rotation": the unit norm and its weight come before the rotation), ``rope_layout`` ("half": element i turns
with element i + dims / 2, the default; "interleaved": element 2i with element 2i + 1), ``bias`` may also be "qk":
biases on q and k only, ``qk_norm_scope`` ("head", the default, or "projection": all query heads are divided by ONE root
mean square over the whole query projection, the key heads likewise, and the weights ``q.norm`` / ``k.norm`` have that
size; before the rotation, with a weight), ``value_mix`` (None; "source": the layer leaves its values to the later layers
of the step; "mixed": the values become (1 - lambda) v + lambda v_source of the same token, lambda a learned number
``vmix``, and the mixed values are what the pages keep; with ``qk_norm_scope`` "projection" only), ``conv_taps`` (K: q and k
pass a causal filter of K taps over time per channel, ``q.conv`` / ``k.conv`` [channels, K], directly after the projection; values
that are the keys are the filtered ones; the last K - 1 projected q and k of each request are kept beside the pages),
``query_temperature`` (None, or (coef, every): the queries are multiplied by 1 + coef ln(floor((position + 1) / every) + 1)
after norm and rotation).

Tensors: ``qkv`` [(nq + nkv) d (+ nkv dv) (+ nq dv), width], rows q then k then v then g, packed from the
checkpoint's ``q``, ``k``, ``v``, ``g`` (those that exist); ``qk_bias`` [(nq + nkv) d] from ``q.b``, ``k.b``; ``sink``
[nq] (float32); ``o`` [width, nq dv]; ``o.b`` [width].  Scores, softmax, rotation, bias and norm are computed in 32-bit.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import MIXERS, CompositeNeed, FixedStateNeed, Mixer, PagedKVNeed
from .spec import ParamDecl, Source


class SinkAttention(Mixer):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.nq = int(spec["num_heads"])
        self.nkv = int(spec["num_kv_heads"])
        self.d = int(spec["head_dim"])
        self.dv = int(spec.get("v_head_dim") or self.d)
        if self.nq % self.nkv:
            raise ValueError(f"{self.nq} query heads do not divide into {self.nkv} KV heads")
        scale = spec.get("scale")
        self.scale = float(scale) if scale is not None else self.d ** -0.5
        eps = spec.get("unit_norm_eps")
        self.eps = None if eps is None else float(eps)
        self.has_sink = bool(spec.get("sink", True))
        self.sink_constant = spec.get("sink_constant")
        if self.sink_constant is not None:
            if spec.get("sink", False):
                raise ValueError("a sink is learned (sink=True) or a constant (sink_constant), not both")
            self.has_sink = False
            self.fixed_sinks = torch.full((self.nq,), float(self.sink_constant), dtype=torch.float32, device=env.device)
        self.keep_first = int(spec.get("keep_first", 0) or 0)
        self.norm_scope = spec.get("qk_norm_scope", "head")
        self.value_mix = spec.get("value_mix")
        if self.norm_scope not in ("head", "projection") or self.value_mix not in (None, "source", "mixed"):
            raise ValueError(f"unknown qk_norm_scope {self.norm_scope!r} or value_mix {self.value_mix!r}")
        self.norm_order = spec.get("qk_norm_order", "before_rotation" if self.norm_scope == "projection" else "after_rotation")
        self.rope_layout = spec.get("rope_layout", "half")
        if self.norm_order not in ("after_rotation", "before_rotation") or self.rope_layout not in ("half", "interleaved"):
            raise ValueError(f"unknown qk_norm_order {self.norm_order!r} or rope_layout {self.rope_layout!r}")
        self.window = spec.get("window")
        self.keep_window = spec.get("keep_window", self.window)
        if self.keep_window is not None and (self.window is None or self.keep_window < self.window):
            raise ValueError("the pages must keep at least the keys that the layer's window shows")
        self.chunk = spec.get("chunk")
        if self.keep_first and (self.window is None or self.keep_window != self.window):
            raise ValueError("kept first keys go with a window of the layer's own")
        self.values = spec.get("values", "projected")
        if self.values not in ("projected", "keys"):
            raise ValueError(f"values are 'projected' or 'keys', not {self.values!r}")
        if self.values == "keys" and self.dv != self.d:
            raise ValueError(f"values that are the keys have the keys' size {self.d}, not {self.dv}")
        self.bias = bool(spec.get("bias", False))
        self.out_bias = self.bias and spec.get("bias") != "qk"
        self.gate = spec.get("output_gate")
        if self.gate not in (None, "sigmoid", "sigmoid_head"):
            raise ValueError(f"an output gate is None, 'sigmoid' or 'sigmoid_head', not {self.gate!r}")
        self.position = env.position(spec.get("position"))
        self.own_kv = bool(spec.get("own_kv", True))
        self.norm_weight = bool(spec.get("qk_norm_weight", False))
        if self.norm_weight and self.eps is None:
            raise ValueError("a weight on the q/k norm needs the norm (unit_norm_eps)")
        base = spec.get("distance_slope_base")
        self.slopes = None
        if base is not None:
            self.slopes = torch.tensor([2.0 ** (-float(base) * (h + 1) / self.nq) for h in range(self.nq)],
                                       dtype=torch.float32, device=env.device)
        self.rows = self.norm_scope == "projection"         # q and k pass the kernel that works on a token's whole rows
        if self.rows and (not self.norm_weight or self.norm_order != "before_rotation" or self.bias or not self.own_kv
                          or self.values != "projected"):
            raise ValueError("a norm over the whole projection has a weight, comes before the rotation and goes with keys "
                             "and values of the layer's own, without biases")
        if self.value_mix and not self.rows:
            raise ValueError("mixed values are offered with a norm over the whole projection")
        self.taps = int(spec.get("conv_taps") or 0)
        self.temperature = spec.get("query_temperature")
        if self.temperature is not None:
            coef, every = self.temperature
            self.temperature = (float(coef), int(every))
            if self.temperature[1] < 1:
                raise ValueError("a query temperature changes every so many positions, at least one")
        if self.taps < 0:
            raise ValueError("a filter over time has at least one tap")
        # heads that pass a filter or a temperature go through a kernel of their own
        self.prepared = self.taps > 0 or self.temperature is not None
        if self.prepared and (self.rows or self.bias or not self.own_kv or self.rope_layout != "half"
                              or (self.position is not None and self.eps is not None and self.norm_order != "before_rotation")):
            raise ValueError("a filter over time or a query temperature goes with keys of the layer's own, without biases, normed "
                             "per head before a rotation by halves")
        # what a page row and a query head hold: on the tensor cores keys and values of unequal size are padded to one
        self.D = self.d
        if self.rows and env.dtype == torch.bfloat16 and (self.dv > self.d or self.d % 16):
            self.D = -(-max(self.d, self.dv) // 16) * 16
        self.q_size = self.nq * self.d
        self.k_size = self.nkv * self.d if self.own_kv else 0
        self.v_size = self.nkv * self.dv if self.values == "projected" and self.own_kv else 0
        self.g_size = (self.nq if self.gate == "sigmoid_head" else self.nq * self.dv) if self.gate else 0

    def params(self):
        H = self.env.hidden_size
        sources = [Source("q", 0, self.q_size)]
        if self.k_size:
            sources.append(Source("k", self.q_size, self.k_size))
        if self.v_size:
            sources.append(Source("v", self.q_size + self.k_size, self.v_size))
        if self.g_size:
            sources.append(Source("g", self.q_size + self.k_size + self.v_size, self.g_size))
        decls = [
            ParamDecl("qkv", (self.q_size + self.k_size + self.v_size + self.g_size, H), sources=tuple(sources)),
            ParamDecl("o", (H, self.nq * self.dv)),
        ]
        if self.has_sink:
            decls.append(ParamDecl("sink", (self.nq,), storage="float32"))
        if self.norm_weight:
            decls.append(ParamDecl("q.norm", (self.q_size if self.rows else self.d,), init="norm"))
            if self.own_kv:
                decls.append(ParamDecl("k.norm", (self.k_size if self.rows else self.d,), init="norm"))
        if self.taps:
            decls.append(ParamDecl("qk_conv", (self.q_size + self.k_size, self.taps), init="filter_taps",
                                   sources=(Source("q.conv", 0, self.q_size), Source("k.conv", self.q_size, self.k_size))))
        if self.value_mix == "mixed":
            decls.append(ParamDecl("vmix", (1,), init="mix_share", storage="float32", sources=(Source("vmix", 0, 1, squeeze=True),)))
        if self.bias:
            if not self.own_kv:
                raise ValueError("projection biases are not offered for a layer without keys of its own")
            decls.append(ParamDecl("qk_bias", (self.q_size + self.k_size,), init="zeros_noise",
                                   sources=(Source("q.b", 0, self.q_size), Source("k.b", self.q_size, self.k_size))))
            if self.out_bias:
                decls.append(ParamDecl("o.b", (H,), init="zeros_noise"))
        return decls

    def bind(self, tensors):
        super().bind(tensors)
        if self.taps:
            self.w_taps = self.w_qk_conv.t().contiguous()       # one row per tap: what the kernel reads side by side

    def cache_need(self):
        pages = PagedKVNeed(self.nkv, self.D, self.keep_window, v_head_dim=self.dv, chunk=self.chunk,
                            keep_first=self.keep_first)
        if self.taps < 2:
            return pages
        return CompositeNeed((pages, FixedStateNeed(((self.taps - 1) * (self.q_size + self.k_size),))))

    def streamed_weights(self):
        return [(self.w_qkv, 0), (self.w_o, 0)]

    def forward(self, x, batch, cache):
        T = x.shape[0]
        state = None
        if self.taps > 1:
            cache, kept = cache.children
            state = kept.state
        qkv = self.new(T, self.q_size + self.k_size + self.v_size + self.g_size)
        ops.linear(qkv, x, self.w_qkv)
        rot = self.position.rotary() if self.position is not None else None
        table, rotary_dim = rot if rot is not None else (None, 0)
        q = self.new(T, self.nq * self.D)
        if cache.writes != self.own_kv:
            raise ValueError("a layer with keys of its own writes its pages; one without reads another run's (cache_from)")
        if self.prepared:
            ops.heads_store(qkv, q, self.D, cache.pages, cache.tables.slot_mapping, batch, table, rotary_dim, self.nq, self.nkv,
                            self.d, self.dv, self.eps, self.w_q_norm if self.norm_weight else None,
                            self.w_k_norm if self.norm_weight else None, values_from_keys=self.values == "keys",
                            taps=self.w_taps if self.taps else None, state=state, temperature=self.temperature)
        elif self.rows:
            self._store_rows(qkv, q, batch, cache, table, rotary_dim)
        else:
            ops.rope_norm_store(qkv, q, cache.pages if cache.writes else None, cache.tables.slot_mapping, batch.positions,
                                table, rotary_dim, self.nq, self.nkv, self.d, self.dv, self.eps,
                                bias=self.w_qk_bias if self.bias else None, values_from_keys=self.values == "keys",
                                q_weight=self.w_q_norm if self.norm_weight else None,
                                k_weight=self.w_k_norm if self.norm_weight and self.own_kv else None,
                                norm_first=self.norm_order == "before_rotation",
                                interleaved=self.rope_layout == "interleaved")
        o = self.new(T, self.nq * self.dv)
        ops.attention_sink(o, q, cache.pages, cache.tables, batch, self.nq, self.nkv, self.D, self.dv, self.scale,
                           self.w_sink if self.has_sink else getattr(self, "fixed_sinks", None), self.window or 0,
                           self.chunk or 0, self.slopes, self.keep_first)
        if self.gate == "sigmoid_head":
            ops.sigmoid_mul_heads(o, o, qkv[:, self.q_size + self.k_size + self.v_size:], self.dv)
        elif self.gate:
            ops.sigmoid_mul(o, o, qkv[:, self.q_size + self.k_size + self.v_size:])
        y = self.new(T, self.env.hidden_size)
        ops.linear(y, o, self.w_o)
        if self.out_bias:
            ops.add_row_bias(y, self.w_o_b)
        return y

    VALUE_SOURCE = "value_source"       # the key under which a step carries the values that later layers mix in

    def _store_rows(self, qkv, q, batch, cache, table, rotary_dim):
        v_first = share = None
        v = qkv[:, self.q_size + self.k_size:self.q_size + self.k_size + self.v_size]
        if self.value_mix == "source":
            batch.carried[self.VALUE_SOURCE] = v
        elif self.value_mix == "mixed":
            v_first, share = batch.carried.get(self.VALUE_SOURCE), self.w_vmix
            if v_first is None or v_first.shape != v.shape:
                raise ValueError("a layer that mixes values needs an earlier layer of the step that leaves values of its size")
        ops.row_norm_store(qkv, q, self.D, cache.pages, cache.tables.slot_mapping, batch.positions, table, rotary_dim,
                           self.nq, self.nkv, self.d, self.dv, self.eps, self.w_q_norm, self.w_k_norm,
                           interleaved=self.rope_layout == "interleaved", v_first=v_first, v_share=share)


MIXERS.register("sink_attention", SinkAttention)
