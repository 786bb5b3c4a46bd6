"""Vozorax: a decoder-only model whose layers are listed one by one in config.json.

config.json: ``architecture`` "Vozorax"; ``vocab``, ``width``; ``streams``; ``norm.eps``; ``layers``: a list of
{``type``, ``mixer``, ``mlp``}.  The residual stream is ``streams`` copies per token (hyper-connections), float32: a
sub-block reads an RMS norm of a weighted sum of the copies, and its output makes new copies from all of them.  Layer
types:

* ``latent_attention`` (``mixer``: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims}, mask {size}):
  queries through a normed latent, keys and values expanded from one normed latent per token, one key part for all
  heads with neighbouring elements rotated together, a sliding window, ordinary softmax;
* ``attention`` (``mixer``: heads, kv_heads, dim, vdim, scale, mask {size}, v_mix): grouped-query attention in a sliding
  window without positions, q and k each normed over the whole projection, a sink per head; with ``v_mix`` the values
  are mixed with those of the first such layer (which itself keeps its own).

``mlp`` is null, {``kind``: "dense", ``ff``}: down(gelu_tanh(gate h) * (up h)), or {``kind``: "moe", ``router`` {experts,
top}, ``expert`` {ff}, ``shared`` {ff} or null}: the ``top`` largest logits (with a bias) chosen, weighted by the softmax
over these alone, experts down(relu(up h)^2), a shared expert of the same form with a sigmoid gate per token.

The logits are the last norm (``final.norm``) of the sum of the copies, times ``head``.  Tensors: ``embed``, ``head``,
``final.norm``, and per layer i ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.{in,out,mix}``,
``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass

from ..config.model_config import ConfigError, ModelConfig, parse_dtype, take
from ..config.registry import register_architecture
from ..parts.spec import LayerRun, LayerSpec, ModelSpec, PartUse, part

ARCHITECTURE = "Vozorax"
NO_POSITION_LIMIT = 1 << 20     # the design names no longest sequence; the engine's max_model_len is the limit in use
LAYER_TYPES = ("latent_attention", "attention")
MAX_STREAMS = 16                # what the streams' kernel takes


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


def _check_mask(m: dict, where: str) -> None:
    if m.get("mask") is not None and take(_sub(m, "mask", where), "size", int, where=where + ".mask") <= 0:
        raise ConfigError(f"{where}.mask: size must be positive")


def _check_latent(m: dict, where: str) -> None:
    _positive(m, ("heads", "vdim", "q_rank", "kv_rank"), where)
    dim, rot_dim = take(m, "dim", int, where=where), take(m, "rot_dim", int, where=where)
    if dim < 0 or rot_dim < 0 or dim + rot_dim <= 0:
        raise ConfigError(f"{where}: dim {dim} and rot_dim {rot_dim} must not be negative, nor both zero")
    take(m, "scale", float, where=where)
    if rot_dim:
        rot = _sub(m, "rot", where)
        take(rot, "base", float, where=where + ".rot")
        dims = take(rot, "dims", int, where=where + ".rot")
        if dims <= 0 or dims % 2 or dims > rot_dim:
            raise ConfigError(f"{where}.rot: dims {dims} must be even and at most rot_dim {rot_dim}")
    _check_mask(m, where)


def _check_attention(m: dict, where: str) -> None:
    heads, kv, _, _ = _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if heads % kv:
        raise ConfigError(f"{where}: heads {heads} must be a multiple of kv_heads {kv}")
    take(m, "scale", float, where=where)
    take(m, "v_mix", bool, False, where=where)
    _check_mask(m, where)


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where} must be an object or null")
    kind = take(mlp, "kind", str, where=where)
    if kind == "dense":
        _positive(mlp, ("ff",), where)
    elif kind == "moe":
        experts, top = _positive(_sub(mlp, "router", where), ("experts", "top"), where + ".router")
        if top > experts:
            raise ConfigError(f"{where}.router: {experts} experts, top {top}")
        for key in ("expert",) + (("shared",) if mlp.get("shared") is not None else ()):
            _positive(_sub(mlp, key, where), ("ff",), f"{where}.{key}")
    else:
        raise ConfigError(f"{where}: unknown kind {kind!r} (known: 'dense', 'moe', or null)")


def _value_layers(layers: list) -> list[int]:
    """The attention layers that mix values; the first of them is where the values come from."""
    return [i for i, layer in enumerate(layers) if layer["type"] == "attention" and layer["mixer"].get("v_mix")]


@dataclass(frozen=True)
class VozoraxConfig(ModelConfig):
    layers_json: str = "[]"         # the ``layers`` list as canonical JSON (the dataclass stays hashable)
    norm_eps: float = 1e-6
    streams: int = 1

    @property
    def layers(self) -> list:
        return json.loads(self.layers_json)

    @classmethod
    def from_json_dict(cls, raw: dict) -> "VozoraxConfig":
        vocab, width, streams = _positive(raw, ("vocab", "width", "streams"), "config.json")
        if streams > MAX_STREAMS:
            raise ConfigError(f"config.json: {streams} streams are beyond the supported {MAX_STREAMS}")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        for i, layer in enumerate(layers):
            where = f"config.json: layers[{i}]"
            if not isinstance(layer, dict):
                raise ConfigError(f"{where} must be an object")
            kind = take(layer, "type", str, where=where)
            mixer = _sub(layer, "mixer", where)
            if kind == "latent_attention":
                _check_latent(mixer, where + ".mixer")
            elif kind == "attention":
                _check_attention(mixer, where + ".mixer")
            else:
                raise ConfigError(f"{where}: unknown layer type {kind!r} (known: {LAYER_TYPES})")
            _check_mlp(layer.get("mlp"), where + ".mlp")
        sizes = {i: layers[i]["mixer"]["kv_heads"] * layers[i]["mixer"]["vdim"] for i in _value_layers(layers)}
        if len(set(sizes.values())) > 1:
            raise ConfigError(f"config.json: layers that mix values have values of one size, not {sizes}")
        eos = raw.get("eos_token_id")
        return cls(
            architecture=ARCHITECTURE, model_type=take(raw, "model_type", str, "vozorax"), vocab_size=vocab,
            hidden_size=width, max_position_embeddings=take(raw, "max_position_embeddings", int, NO_POSITION_LIMIT),
            dtype=parse_dtype(raw.get("dtype", raw.get("torch_dtype", "bfloat16"))),
            eos_token_id=eos if isinstance(eos, int) and not isinstance(eos, bool) else None,
            layers_json=json.dumps(layers, sort_keys=True), streams=streams,
            norm_eps=take(_sub(raw, "norm", "config.json"), "eps", float, where="config.json: norm"))

    def to_json_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                "norm": {"eps": self.norm_eps}, "layers": self.layers, "dtype": str(self.dtype).replace("torch.", ""),
                **({"eos_token_id": self.eos_token_id} if self.eos_token_id is not None else {})}


def _mixer(kind: str, m: dict, eps: float, value_mix):
    window = None if m.get("mask") is None else int(m["mask"]["size"])
    if kind == "latent_attention":
        rope = None
        if m["rot_dim"]:
            rope = part("rope_banded", theta=float(m["rot"]["base"]), rotary_dim=int(m["rot"]["dims"]))
        return part("latent_attention", num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"],
                    v_head_dim=m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=float(m["scale"]),
                    position=rope, rope_layout="interleaved", eps=eps, sink=False, window=window)
    return part("sink_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                v_head_dim=m["vdim"], scale=float(m["scale"]), position=None, unit_norm_eps=eps, qk_norm_weight=True,
                qk_norm_scope="projection", sink=True, window=window, value_mix=value_mix)


def _feed_forward(mlp: dict):
    if mlp["kind"] == "dense":
        return part("gated_mlp", intermediate_size=int(mlp["ff"]), activation="gelu_tanh")
    r, s = mlp["router"], mlp.get("shared")
    shared = None if s is None else part("dense_mlp", intermediate_size=int(s["ff"]), activation="relu2")
    return part("routed_moe", experts=int(r["experts"]), top=int(r["top"]), unit="relu2", scores="chosen_softmax",
                correction=True, correction_source="router.b", intermediate_size=int(mlp["expert"]["ff"]), limit=None,
                shared=shared, shared_gate=shared is not None)


def build_spec(cfg: VozoraxConfig) -> ModelSpec:
    """Vozorax as data: per layer a block whose sub-blocks read and write several copies of a float32 stream."""
    block = part("hyper_connections")
    raw_layers = cfg.layers
    mixing = _value_layers(raw_layers)
    layers, unused = [], []
    for i, layer in enumerate(raw_layers):
        p = f"l{i}."

        def norm(name: str):
            return PartUse(part("rmsnorm", width=cfg.hidden_size, eps=cfg.norm_eps, source=name, own_name=True), p)

        def connection(name: str):
            return PartUse(part("hyper_connection", streams=cfg.streams, source=name), p)

        value_mix = None if i not in mixing else ("source" if i == mixing[0] else "mixed")
        uses = dict(mixer=PartUse(_mixer(layer["type"], layer["mixer"], cfg.norm_eps, value_mix), p + "mix."),
                    mixer_norm=norm("norm1"), mixer_connection=connection("hc1"))
        if layer.get("mlp") is not None:
            uses.update(ffn=PartUse(_feed_forward(layer["mlp"]), p + "mlp."), ffn_norm=norm("norm2"),
                        ffn_connection=connection("hc2"))
        else:       # a checkpoint may carry them for a layer that has no use for them
            unused += [p + "norm2", p + "hc2.in", p + "hc2.out", p + "hc2.mix"]
        if value_mix != "mixed":
            unused.append(p + "mix.vmix")
        layers.append(LayerSpec(block, **uses))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=cfg.hidden_size, vocab_size=cfg.vocab_size,
        max_position=cfg.max_position_embeddings,
        embedding=PartUse(part("token_embedding", vocab_size=cfg.vocab_size, stream="float32", source="embed"), ""),
        layers=tuple(layers), order=tuple(LayerRun(i) for i in range(len(layers))),
        final_norm=PartUse(part("rmsnorm", width=cfg.hidden_size, eps=cfg.norm_eps, source="norm"), "final."),
        head=PartUse(part("lm_head", vocab_size=cfg.vocab_size, tied=False, exact=True, source="head"), ""),
        ignored_checkpoint_tensors=tuple(unused))


register_architecture(ARCHITECTURE, model_types=("vozorax",), parse_config=VozoraxConfig.from_json_dict,
                      build_spec=build_spec)
