"""Vozorax on the CPU: its config.json keys and their checks, the tensor table against the design's tensor names, what
each layer keeps between steps, which layer leaves its values to the others, and which tiles of latents a step with a
window expands."""
import copy

import pytest
import torch

import plain_vozorax as pv
from nanohybrid_vlm_b200.config.model_config import ConfigError
from nanohybrid_vlm_b200.config.registry import ARCHITECTURES
from nanohybrid_vlm_b200.engine.model import CausalLM
from nanohybrid_vlm_b200.parts.base import PagedKVNeed

LATENT = dict(heads=3, dim=12, rot_dim=6, vdim=10, q_rank=14, kv_rank=18, scale=0.2, rot=dict(base=5000.0, dims=6),
              mask=dict(size=21))
ATTN = dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.3, mask=dict(size=9), v_mix=True)
MOE = dict(kind="moe", router=dict(experts=4, top=2), expert=dict(ff=12), shared=dict(ff=16))
CFG = dict(architecture="Vozorax", vocab=120, width=48, streams=2, norm=dict(eps=1e-5), layers=[
    dict(type="latent_attention", mixer=LATENT, mlp=dict(kind="dense", ff=40)),
    dict(type="attention", mixer=ATTN, mlp=MOE),
    dict(type="attention", mixer=dict(ATTN, heads=2, mask=dict(size=30)), mlp=None),
    dict(type="attention", mixer=dict(ATTN, dim=16, v_mix=False), mlp=dict(MOE, shared=None)),
])


def build(cfg):
    import nanohybrid_vlm_b200.models  # noqa: F401
    entry = ARCHITECTURES.resolve(cfg)
    parsed = entry.parse_config(cfg)
    return parsed, entry.build_spec(parsed)


def checkpoint_table(model):
    return {s.name: tuple(s.checkpoint_shape(bp.decl.shape)) for bp in model.param_table() for s in bp.decl.sources}


def test_tensor_table_names_and_shapes_are_the_designs():
    parsed, spec = build(CFG)
    got = checkpoint_table(CausalLM(spec, torch.bfloat16, "cpu"))
    want = {k: tuple(v.shape) for k, v in pv.random_weights(CFG, 1).items()}
    # the first layer that mixes values has a share it does not use; a layer without a feed-forward, no second norm
    assert got == {k: v for k, v in want.items() if k != "l1.mix.vmix"}
    assert set(spec.ignored_checkpoint_tensors) == {"l0.mix.vmix", "l1.mix.vmix", "l3.mix.vmix", "l2.norm2", "l2.hc2.in",
                                                    "l2.hc2.out", "l2.hc2.mix"}
    assert parsed.to_json_dict()["layers"] == CFG["layers"] and parsed.streams == 2


def test_constants_of_the_stream_and_the_router_stay_in_32_bit():
    _, spec = build(CFG)
    kinds = {bp.name: bp.decl.storage for bp in CausalLM(spec, torch.bfloat16, "cpu").param_table()}
    for name in ("l0.hc1.in", "l0.hc2.mix", "l1.hc1.out", "l1.mlp.correction", "l1.mix.sink", "l2.mix.vmix"):
        assert kinds[name] == "float32", name
    assert kinds["l1.mlp.router"] == "model"


def test_cache_needs_follow_the_layers():
    _, spec = build(CFG)
    needs = CausalLM(spec, torch.float32, "cpu").cache_needs()
    assert needs == [PagedKVNeed(1, 24, 21, v_head_dim=18, planes=1), PagedKVNeed(2, 8, 9, v_head_dim=6),
                     PagedKVNeed(2, 8, 30, v_head_dim=6), PagedKVNeed(2, 16, 9, v_head_dim=6)]
    # in bfloat16 a row is padded to what the tensor-core kernels take, where the values are wider than the keys too
    cfg = copy.deepcopy(CFG)
    cfg["layers"][1]["mixer"].update(dim=8, vdim=20)
    cfg["layers"][2]["mixer"].update(dim=32, vdim=20)
    rows = [n.row_dim for n in CausalLM(build(cfg)[1], torch.bfloat16, "cpu").cache_needs()]
    assert rows == [24, 32, 32, 16]


def test_the_first_layer_that_mixes_values_is_their_source():
    _, spec = build(CFG)
    assert [lay.mixer.spec.get("value_mix") for lay in spec.layers] == [None, "source", "mixed", None]
    assert all(lay.mixer.spec.get("sink") is (lay.mixer.spec.kind == "sink_attention") for lay in spec.layers)


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "mixer", "mask", "size"), 0, "size"),
    (("layers", 0, "mixer", "rot", "dims"), 5, "dims"),
    (("layers", 0, "mixer", "rot", "dims"), 8, "dims"),
    (("layers", 0, "mixer", "kv_rank"), 0, "positive"),
    (("layers", 0, "mixer", "rot_dim"), -2, "rot_dim"),
    (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "v_mix"), 1, "bool"),
    (("layers", 2, "mixer", "vdim"), 7, "one size"),
    (("layers", 1, "mlp", "router", "top"), 5, "top"),
    (("layers", 1, "mlp", "expert", "ff"), 0, "positive"),
    (("layers", 1, "mlp", "shared", "ff"), 0, "positive"),
    (("layers", 1, "mlp", "kind"), "glu", "unknown kind"),
    (("layers", 2, "type"), "conv", "unknown layer type"),
    (("streams",), 0, "positive"),
    (("streams",), 17, "streams"),
    (("norm",), None, "norm"),
])
def test_bad_values_are_refused(path, value, words):
    cfg = copy.deepcopy(CFG)
    at = cfg
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=words):
        build(cfg)


def test_optional_keys():
    cfg = copy.deepcopy(CFG)
    del cfg["layers"][0]["mixer"]["mask"]               # no window: every key is kept
    cfg["layers"][3]["mixer"]["mask"] = None
    del cfg["layers"][3]["mixer"]["v_mix"]
    cfg["layers"][0]["mixer"]["rot_dim"] = 0            # nothing is rotated
    del cfg["layers"][0]["mixer"]["rot"]
    _, spec = build(cfg)
    needs = CausalLM(spec, torch.float32, "cpu").cache_needs()
    assert needs[0] == PagedKVNeed(1, 18, None, v_head_dim=18, planes=1) and needs[3].window is None


def test_tiles_of_latents_that_a_step_expands():
    """Portions of 5 and 1 tokens behind 200 and 300: without a window all tiles up to the last token; with one, from
    the tile of the first key that the portion's first token sees."""
    from nanohybrid_vlm_b200.kernels.ops import latent_tiles
    cu, kv = [0, 5, 6, 70], [205, 301, 64]
    assert latent_tiles(cu, kv, 0) == [(0, 4), (0, 5), (0, 1)]
    # window 73: the portion that starts at 200 sees keys from 128 = 2 * 64 on; window 74 reaches one key further back
    assert latent_tiles(cu, kv, 73) == [(2, 4), (3, 5), (0, 1)]
    assert latent_tiles(cu, kv, 74) == [(1, 4), (3, 5), (0, 1)]
    assert latent_tiles(cu, kv, 1) == [(3, 4), (4, 5), (0, 1)]
    assert latent_tiles(cu, kv, 1000) == latent_tiles(cu, kv, 0)
