"""Kilisun on the CPU: its config.json keys and their checks, the tensor table against the design's tensor names, what
each layer keeps between steps, which layers read another's pages, and the plain functions' own edges."""
import json

import pytest
import torch

import plain_kilisun as pk
from nanohybrid_vlm_b200.config.model_config import ConfigError
from nanohybrid_vlm_b200.config.registry import ARCHITECTURES
from nanohybrid_vlm_b200.engine.model import CausalLM
from nanohybrid_vlm_b200.parts.base import CompositeNeed, FixedStateNeed, PagedKVNeed, SharedPagesNeed

FULL = dict(heads=6, kv_heads=3, dim=10, vdim=10, scale=0.3, conv=4, q_temp=dict(coef=0.2, every=7))
MAPS = dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.25, diff=0.4, softcap=9.0, rot=dict(base=500.0, dims=8),
            mask=dict(size=21))
MOE = dict(kind="moe", router=dict(experts=8, top=3, groups=dict(count=4, keep=2), scale=1.5), expert=dict(ff=12, limit=0.5),
           shared=dict(ff=16, limit=3.0))
CFG = dict(architecture="Kilisun", vocab=120, width=48, norm=dict(eps=1e-5), layers=[
    dict(type="attention", mixer=FULL, mlp=MOE),
    dict(type="attention_2", mixer=MAPS, mlp=dict(kind="dense", ff=40, limit=1.5)),
    dict(type="attention_2", mixer=dict(MAPS, heads=2, mask=dict(size=30), kv_from=1), mlp=dict(MOE, shared=None)),
    dict(type="attention_2", mixer=MAPS, mlp=None),
    dict(type="attention", mixer=dict(FULL, conv=1), mlp=None),
])


def build(cfg):
    import nanohybrid_vlm_b200.models  # noqa: F401
    entry = ARCHITECTURES.resolve(cfg)
    parsed = entry.parse_config(cfg)
    return parsed, entry.build_spec(parsed)


def test_tensor_table_names_and_shapes_are_the_designs():
    parsed, spec = build(CFG)
    got = {s.name: tuple(s.checkpoint_shape(bp.decl.shape)) for bp in CausalLM(spec, torch.bfloat16, "cpu").param_table()
           for s in bp.decl.sources}
    assert got == {k: tuple(v) for k, v in pk.tensor_shapes(CFG).items()}
    assert "l2.mix.k" not in got and "l2.mix.k.norm" not in got and "l2.mix.q.norm" in got and "head" not in got
    assert set(spec.ignored_checkpoint_tensors) == {"l3.norm2", "l3.norm2b", "l4.norm2", "l4.norm2b"}
    assert parsed.to_json_dict()["layers"] == CFG["layers"] and parsed.norm_eps == 1e-5


def test_what_enters_a_decision_or_a_share_stays_in_32_bit():
    _, spec = build(CFG)
    kinds = {bp.name: bp.decl.storage for bp in CausalLM(spec, torch.bfloat16, "cpu").param_table()}
    for name in ("l0.mlp.correction", "l1.mix.lq1", "l2.mix.lk2"):
        assert kinds[name] == "float32", name
    assert kinds["l0.mlp.router"] == kinds["l0.mix.qk_conv"] == "model"


def test_cache_needs_follow_the_layers():
    _, spec = build(CFG)
    needs = CausalLM(spec, torch.float32, "cpu").cache_needs()
    full = PagedKVNeed(3, 10, None, v_head_dim=10)
    # both maps of a key head in one row; the pages of layer 1 keep what layer 2's wider window shows
    assert needs == [CompositeNeed((full, FixedStateNeed((3 * 90,)))), PagedKVNeed(2, 24, 30, v_head_dim=20), SharedPagesNeed(),
                     PagedKVNeed(2, 24, 21, v_head_dim=20), full]
    # in bfloat16 a row is padded to what the tensor-core kernels take, where the values are wider than both maps too
    assert [n.row_dim for n in CausalLM(spec, torch.bfloat16, "cpu").cache_needs() if isinstance(n, PagedKVNeed)] == [32, 32, 10]
    cfg = json.loads(json.dumps(CFG))
    cfg["layers"][3]["mixer"]["vdim"] = 40
    assert CausalLM(build(cfg)[1], torch.bfloat16, "cpu").cache_needs()[3].row_dim == 48
    cfg["layers"][2]["mixer"]["mask"] = None              # a reader without a window: the pages keep every key
    assert CausalLM(build(cfg)[1], torch.float32, "cpu").cache_needs()[1].window is None


def test_a_layer_reads_the_pages_of_the_layer_it_names():
    _, spec = build(CFG)
    assert [run.cache_from for run in spec.order] == [None, None, 1, None, None]
    assert [lay.mixer.spec.get("own_kv", True) for lay in spec.layers] == [True, True, False, True, True]


def test_the_share_of_the_second_map_is_computed_once_in_32_bit():
    _, spec = build(CFG)
    model = CausalLM(spec, torch.bfloat16, "cpu")
    w = {k: v.double() for k, v in pk.random_weights(CFG, 3).items()}
    tensors = {}
    for bp in model.param_table():
        t = torch.zeros(bp.decl.shape, dtype=torch.float32 if bp.decl.storage == "float32" else torch.bfloat16)
        for s in bp.decl.sources:
            t.narrow(s.dim, s.row, s.rows).copy_(s.to_slice(w[s.name].to(t.dtype), bp.decl.shape))
        tensors[bp.name] = t
    model.bind(tensors)
    for i in (1, 2, 3):
        m = CFG["layers"][i]["mixer"]
        share = model.blocks[i].mixer.share
        want = pk.map_share(m, w, f"l{i}.mix.").item()
        assert share.dtype == torch.float32 and abs(share.item() - want) < 1e-6 and abs(want - m["diff"]) > 0.02


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "vdim"), 12, "values are the keys"),
    (("layers", 0, "mixer", "conv"), -1, "conv"),
    (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
    (("layers", 0, "mixer", "scale"), "big", "scale"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"),
    (("layers", 1, "mixer", "rot", "dims"), 5, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 14, "dims"),
    (("layers", 1, "mixer", "softcap"), 0.0, "softcap"),
    (("layers", 1, "mixer", "diff"), None, "diff"),
    (("layers", 2, "mixer", "kv_from"), 2, "kv_from"),
    (("layers", 2, "mixer", "kv_from"), 0, "kv_from"),
    (("layers", 2, "mixer", "vdim"), 24, "must equal"),
    (("layers", 3, "mixer", "kv_from"), 2, "of its own"),
    (("layers", 0, "mlp", "router", "top"), 5, "top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 3, "groups"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5, "groups"),
    (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 0, "mlp", "shared", "ff"), 0, "positive"),
    (("layers", 1, "mlp", "kind"), "glu", "unknown kind"),
    (("layers", 2, "type"), "conv", "unknown layer type"),
    (("width",), 0, "positive"),
    (("norm",), None, "norm"),
])
def test_bad_values_are_refused(path, value, words):
    cfg = json.loads(json.dumps(CFG))
    at = cfg
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=words):
        build(cfg)


def test_optional_keys():
    cfg = json.loads(json.dumps(CFG))
    full, maps = cfg["layers"][0]["mixer"], cfg["layers"][3]["mixer"]
    del full["conv"], full["q_temp"], maps["softcap"], cfg["layers"][0]["mlp"]["router"]["groups"]
    maps.update(mask=None, rot=dict(base=500.0, dims=0))
    _, spec = build(cfg)
    model = CausalLM(spec, torch.float32, "cpu")
    assert model.cache_needs()[0] == PagedKVNeed(3, 10, None, v_head_dim=10) and model.cache_needs()[3].window is None
    assert model.blocks[3].mixer.position is None and model.blocks[3].mixer.softcap is None
    assert model.blocks[0].ffn.groups == 1 and not any(bp.name == "l0.mix.qk_conv" for bp in model.param_table())


def test_plain_functions_at_their_edges():
    # the temperature's first step is at position every - 1
    t = pk.query_temperature(torch.tensor([0, 5, 6, 13, 20]), 0.5, 7)
    assert torch.allclose(t, 1 + 0.5 * torch.tensor([1.0, 1.0, 2.0, 3.0, 4.0], dtype=torch.float64).log())
    # the newest input meets the last tap
    y = pk.taps_over_time(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[3.0, 2.0]]))
    assert y[:, 0].tolist() == [2.0, 23.0, 230.0]
    # two good experts beat one excellent one; negative choice scores stay above the closed groups
    z = torch.logit(torch.tensor([[0.9, 0.1, 0.6, 0.55]], dtype=torch.float64))
    r = dict(experts=4, top=1, groups=dict(count=2, keep=1), scale=3.0)
    ids, weights = pk.route(z, torch.eye(4, dtype=torch.float64), torch.zeros(4), r)
    assert ids.tolist() == [[2]] and abs(weights.item() - 1.8) < 1e-9
    ids, _ = pk.route(z, torch.eye(4, dtype=torch.float64), torch.full((4,), -5.0), dict(r, top=2))
    assert sorted(ids[0].tolist()) == [2, 3]
