"""Kilisun: a decoder-only model whose layers are listed one by one in config.json.

config.json: ``architecture`` "Kilisun"; ``vocab``, ``width``; ``norm.eps``; ``layers``: a list of {``type``, ``mixer``, ``mlp``}.
Every sub-block has a norm before and after it: x <- x + norm1b(mixer(norm1(x))), then, if the layer has a feed-forward, x <- x +
norm2b(mlp(norm2(x))); the stream x is float32 and starts as the normed embedding; the norms are RMS norms whose stored weight
is the difference from one.  Layer types:

* ``attention`` (``mixer``: heads, kv_heads, dim, vdim, scale, conv, q_temp {coef, every}): grouped-query attention over all keys
  without rotation: q and k pass a causal filter of ``conv`` taps over time, the values are the filtered keys, q and k are normed
  per head, the queries are multiplied by a temperature that grows with the logarithm of the position, the output has a sigmoid
  gate per head;
* ``attention_2`` (``mixer``: heads, kv_heads, dim, vdim, scale, diff, rot {base, dims}, mask {size}, softcap, kv_from): differential
  attention: two maps per head over the same values, normed per head and map before a rotation by halves, capped scores, a
  sliding window; the second map times a share is taken off the first.  ``kv_from``: j: the layer has no keys and values of
  its own and reads those of layer j.

``mlp`` is null, {``kind``: "dense", ``ff``, ``limit``}: a clamped gated unit, or {``kind``: "moe", ``router`` {experts, top, groups
{count, keep}, scale}, ``expert`` {ff, limit}, ``shared`` {ff, limit} or null}: sigmoid scores, choice by score + ``correction``
among the groups whose two best choice scores sum highest, weights score * scale, experts and a gated shared expert of the same
form.

The logits are the last norm (``final.norm``) times the embedding table.  Tensors: ``embed``, ``embed.norm``, ``final.norm``, and
per layer i ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass

from ..config.model_config import ConfigError, ModelConfig, parse_dtype, take
from ..config.registry import register_architecture
from ..parts.spec import LayerRun, LayerSpec, ModelSpec, PartUse, part

ARCHITECTURE = "Kilisun"
NO_POSITION_LIMIT = 1 << 20     # the design names no longest sequence; the engine's max_model_len is the limit in use
LAYER_TYPES = ("attention", "attention_2")
NORM_OFFSET = 1.0               # norms store the difference from one: fixed by the design
UNIT_ALPHA = 1.702              # of the gated unit, g sigmoid(alpha g) (u + 1): fixed by the design


def _sub(raw: dict, key: str, where: str) -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: key {key!r} must be an object")
    return v


def _positive(m: dict, keys, where: str) -> list[int]:
    vals = [take(m, k, int, where=where) for k in keys]
    if min(vals) <= 0:
        raise ConfigError(f"{where}: {', '.join(keys)} must be positive")
    return vals


def _check_heads(m: dict, where: str) -> tuple[int, int]:
    heads, kv, dim, vdim = _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if heads % kv:
        raise ConfigError(f"{where}: heads {heads} must be a multiple of kv_heads {kv}")
    take(m, "scale", float, where=where)
    return dim, vdim


def _check_attention(m: dict, where: str) -> None:
    dim, vdim = _check_heads(m, where)
    if vdim != dim:
        raise ConfigError(f"{where}: the values are the keys, so vdim {vdim} must equal dim {dim}")
    if take(m, "conv", int, 0, where=where) < 0:
        raise ConfigError(f"{where}: conv must not be negative")
    if m.get("q_temp") is not None:
        qt = _sub(m, "q_temp", where)
        take(qt, "coef", float, where=where + ".q_temp")
        if take(qt, "every", int, where=where + ".q_temp") <= 0:
            raise ConfigError(f"{where}.q_temp: every must be positive")


def _check_differential(m: dict, where: str, index: int, layers: list) -> None:
    dim, _ = _check_heads(m, where)
    take(m, "diff", float, where=where)
    rot = _sub(m, "rot", where)
    dims = take(rot, "dims", int, where=where + ".rot")
    if take(rot, "base", float, where=where + ".rot") <= 0:
        raise ConfigError(f"{where}.rot: base must be positive")
    if dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{where}.rot: dims {dims} must be even and at most dim {dim}")
    if m.get("mask") is not None and take(_sub(m, "mask", where), "size", int, where=where + ".mask") <= 0:
        raise ConfigError(f"{where}.mask: size must be positive")
    cap = take(m, "softcap", float, None, where=where)
    if cap is not None and cap <= 0:
        raise ConfigError(f"{where}: softcap must be positive")
    src = take(m, "kv_from", int, None, where=where)
    if src is None:
        return
    if not 0 <= src < index or layers[src].get("type") != "attention_2":
        raise ConfigError(f"{where}: kv_from {src} must name an earlier layer of type 'attention_2'")
    theirs = layers[src]["mixer"]
    if theirs.get("kv_from") is not None:
        raise ConfigError(f"{where}: kv_from {src} must name a layer with keys and values of its own")
    if any(theirs.get(k) != m.get(k) for k in ("kv_heads", "dim", "vdim", "rot")):
        raise ConfigError(f"{where}: kv_heads, dim, vdim and rot must equal those of layer {src}, whose keys it reads")


def _check_unit(m: dict, where: str) -> None:
    _positive(m, ("ff",), where)
    if take(m, "limit", float, where=where) <= 0:
        raise ConfigError(f"{where}: limit must be positive")


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    kind = take(mlp, "kind", str, where=where)
    if kind == "dense":
        _check_unit(mlp, where)
    elif kind == "moe":
        r = _sub(mlp, "router", where)
        experts, top = _positive(r, ("experts", "top"), where + ".router")
        take(r, "scale", float, 1.0, where=where + ".router")
        count = keep = 1
        if r.get("groups") is not None:
            count, keep = _positive(_sub(r, "groups", where + ".router"), ("count", "keep"), where + ".router.groups")
        if experts % count or keep > count or top > keep * (experts // count):
            raise ConfigError(f"{where}.router: {experts} experts, top {top}, groups {count} of which {keep} are kept")
        for key in ("expert",) + (("shared",) if mlp.get("shared") is not None else ()):
            _check_unit(_sub(mlp, key, where), f"{where}.{key}")
    else:
        raise ConfigError(f"{where}: unknown kind {kind!r} (known: 'dense', 'moe', or null)")


@dataclass(frozen=True)
class KilisunConfig(ModelConfig):
    layers_json: str = "[]"         # the ``layers`` list as canonical JSON (the dataclass stays hashable)
    norm_eps: float = 1e-6

    @property
    def layers(self) -> list:
        return json.loads(self.layers_json)

    @classmethod
    def from_json_dict(cls, raw: dict) -> "KilisunConfig":
        vocab, width = _positive(raw, ("vocab", "width"), "config.json")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        for i, layer in enumerate(layers):
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, dict):
                raise ConfigError(f"{where} must be an object")
            kind = take(layer, "type", str, where=where)
            mixer = _sub(layer, "mixer", where)
            if kind == "attention":
                _check_attention(mixer, where + ".mixer")
            elif kind == "attention_2":
                _check_differential(mixer, where + ".mixer", i, layers)
            else:
                raise ConfigError(f"{where}: unknown layer type {kind!r} (known: {LAYER_TYPES})")
            _check_mlp(layer.get("mlp"), where + ".mlp")
        eos = raw.get("eos_token_id")
        return cls(
            architecture=ARCHITECTURE, model_type=take(raw, "model_type", str, "kilisun"), vocab_size=vocab,
            hidden_size=width, max_position_embeddings=take(raw, "max_position_embeddings", int, NO_POSITION_LIMIT),
            dtype=parse_dtype(raw.get("dtype", raw.get("torch_dtype", "bfloat16"))),
            eos_token_id=eos if isinstance(eos, int) and not isinstance(eos, bool) else None,
            layers_json=json.dumps(layers, sort_keys=True),
            norm_eps=take(_sub(raw, "norm", "config.json"), "eps", float, where="config.json: norm"))

    def to_json_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "layers": self.layers, "dtype": str(self.dtype).replace("torch.", ""),
                **({"eos_token_id": self.eos_token_id} if self.eos_token_id is not None else {})}


def _window(m: dict):
    return None if m.get("mask") is None else int(m["mask"]["size"])


def _kept_window(layers: list, index: int):
    """How many keys the pages of differential layer ``index`` must keep: the widest window among the layer itself and the
    layers that read its keys (None: all, when one of them has no window)."""
    sizes = [_window(layer["mixer"]) for i, layer in enumerate(layers)
             if layer["type"] == "attention_2" and (i == index or layer["mixer"].get("kv_from") == index)]
    return None if None in sizes else max(sizes)


def _mixer(layers: list, index: int, eps: float):
    m = layers[index]["mixer"]
    if layers[index]["type"] == "attention":
        qt = m.get("q_temp")
        return part("sink_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                    scale=float(m["scale"]), position=None, unit_norm_eps=eps, qk_norm_weight=True,
                    qk_norm_order="before_rotation", sink=False, values="keys", output_gate="sigmoid_head",
                    conv_taps=int(m.get("conv") or 0),
                    query_temperature=None if qt is None else (float(qt["coef"]), int(qt["every"])))
    src = m.get("kv_from")
    rope = None
    if m["rot"]["dims"]:
        rope = part("rope_banded", theta=float(m["rot"]["base"]), rotary_dim=int(m["rot"]["dims"]))
    return part("differential_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                v_head_dim=m["vdim"], scale=float(m["scale"]), position=rope, eps=eps, diff=float(m["diff"]),
                softcap=None if m.get("softcap") is None else float(m["softcap"]), window=_window(m),
                keep_window=_kept_window(layers, index if src is None else src), own_kv=src is None)


def _unit(m: dict):
    return part("clamped_glu", intermediate_size=int(m["ff"]), limit=float(m["limit"]), alpha=UNIT_ALPHA)


def _feed_forward(mlp: dict):
    if mlp["kind"] == "dense":
        return _unit(mlp)
    r, e, s = mlp["router"], mlp["expert"], mlp.get("shared")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return part("routed_moe", experts=int(r["experts"]), top=int(r["top"]), groups=int(groups["count"]),
                keep=int(groups["keep"]), group_best=2, scores="sigmoid", renorm=False, weight_factor=float(r.get("scale", 1.0)),
                correction=True, intermediate_size=int(e["ff"]), limit=float(e["limit"]), alpha=UNIT_ALPHA,
                shared=None if s is None else _unit(s), shared_gate=s is not None)


def build_spec(cfg: KilisunConfig) -> ModelSpec:
    """Kilisun as data: per layer a block with a norm before and after each sub-block over a float32 stream; a layer with
    ``kv_from`` runs on the pages of the layer it names."""
    def norm(name: str, prefix: str):
        return PartUse(part("rmsnorm", width=cfg.hidden_size, eps=cfg.norm_eps, weight_offset=NORM_OFFSET, source=name,
                            own_name=True), prefix)

    block = part("sandwich_residual")
    raw_layers = cfg.layers
    layers, order, unused = [], [], []
    for i, layer in enumerate(raw_layers):
        p = f"l{i}."
        uses = dict(mixer=PartUse(_mixer(raw_layers, i, cfg.norm_eps), p + "mix."), mixer_norm=norm("norm1", p),
                    mixer_post_norm=norm("norm1b", p))
        if layer.get("mlp") is not None:
            uses.update(ffn=PartUse(_feed_forward(layer["mlp"]), p + "mlp."), ffn_norm=norm("norm2", p),
                        ffn_post_norm=norm("norm2b", p))
        else:
            unused += [p + "norm2", p + "norm2b"]   # a checkpoint may carry them for a layer that has no use for them
        layers.append(LayerSpec(block, **uses))
        order.append(LayerRun(i, cache_from=layer["mixer"].get("kv_from") if layer["type"] == "attention_2" else None))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size,
        max_position=cfg.max_position_embeddings,
        embedding=PartUse(part("token_embedding", vocab_size=cfg.vocab_size, stream="float32", source="embed",
                               norm=norm("embed.norm", "").spec), ""),
        layers=tuple(layers), order=tuple(order), final_norm=norm("norm", "final."),
        head=PartUse(part("lm_head", vocab_size=cfg.vocab_size, tied=True, exact=True), "head."),
        ignored_checkpoint_tensors=tuple(unused))


register_architecture(ARCHITECTURE, model_types=("kilisun",), parse_config=KilisunConfig.from_json_dict, build_spec=build_spec)
