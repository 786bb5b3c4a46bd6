"""Kilisun through the engine against the plain model (float64): the same requests whole, with their last tokens decoded
one by one, in portions down to two tokens, and mixed with other requests in a pool so small that pages and state slots are
used again; long decoding from a single token; greedy generation through ``LLM.generate`` and the scheduler, and through the
command line.  Small configurations that differ in every size, in the order of their layers and in what the design leaves
open: windows of one key, smaller and larger than a page and none at all, layers that read another's keys under a narrower
or wider window, value heads smaller and larger than both maps, filters of one to six taps and none, groups of experts of
which one, some or all are kept, a mixture without a shared expert, layers without a feed-forward, sizes that are no multiple
of 8."""
import json
import os

import numpy as np
import pytest
import torch

import plain_kilisun as pk
import trace_tools as tt

pytestmark = pytest.mark.gpu


def full(heads, kv, dim, scale, conv, coef=0.3, every=16):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale, conv=conv,
                                             q_temp=dict(coef=coef, every=every)))


def maps(heads, kv, dim, vdim, scale, diff, cap, base, dims, size, kv_from=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, diff=diff, softcap=cap, rot=dict(base=base, dims=dims))
    if size is not None:
        m["mask"] = dict(size=size)
    return dict(type="attention_2", mixer=m if kv_from is None else dict(m, kv_from=kv_from))


def dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts, top, count, keep, ff, limit, scale, shared=None, shared_limit=1.0):
    m = dict(kind="moe", router=dict(experts=experts, top=top, groups=dict(count=count, keep=keep), scale=scale),
             expert=dict(ff=ff, limit=limit))
    return m if shared is None else dict(m, shared=dict(ff=shared, limit=shared_limit))


KIL_A = dict(architecture="Kilisun", vocab=300, width=96, norm=dict(eps=1e-6), layers=[
    dict(full(6, 3, 16, 0.3, 3), mlp=moe(6, 2, 3, 2, 24, 0.8, 1.5, 32, 2.0)),
    dict(maps(4, 2, 16, 32, 0.25, 0.5, 12.0, 10000.0, 16, 33), mlp=dense(80, 1.5)),
    dict(maps(2, 2, 16, 32, 0.25, 0.2, 3.0, 10000.0, 16, 50, 1), mlp=moe(4, 1, 2, 1, 16, 1.0, 2.0)),
    dict(full(2, 1, 64, 0.15, 4, 0.8, 40), mlp=None),
    dict(maps(3, 1, 32, 64, 0.2, 0.7, 30.0, 500.0, 8, 12), mlp=moe(8, 3, 4, 2, 8, 0.5, 1.0, 16, 0.7)),
])
KIL_B = dict(architecture="Kilisun", vocab=211, width=64, norm=dict(eps=1e-5), layers=[
    dict(maps(2, 1, 32, 48, 0.2, 0.8, 20.0, 300.0, 32, 70), mlp=moe(6, 4, 1, 1, 8, 2.0, 0.5, 16, 1.0)),
    dict(maps(4, 1, 32, 48, 0.2, 0.3, 5.0, 300.0, 32, 9, 0), mlp=None),
    dict(full(4, 4, 8, 0.4, 6, 0.5, 5), mlp=dense(40, 0.9)),
    dict(maps(2, 2, 8, 8, 0.4, 0.1, 2.0, 40.0, 4, 1), mlp=moe(4, 2, 2, 2, 12, 1.2, 1.0)),
    dict(maps(4, 2, 16, 40, 0.3, 0.4, 9.0, 100.0, 16, None), mlp=dense(32, 3.0)),
    dict(full(8, 2, 16, 0.3, 1, 0.2, 1), mlp=None),
])
# sizes that are no multiple of 8 anywhere: every product and the attention take their general paths
KIL_C = dict(architecture="Kilisun", vocab=97, width=100, norm=dict(eps=1e-5), layers=[
    dict(full(3, 1, 20, 0.25, 5, 0.4, 11), mlp=moe(5, 3, 1, 1, 18, 1.0, 1.3, 14, 0.6)),
    dict(maps(3, 1, 14, 22, 0.25, 0.6, 7.0, 7000.0, 10, 50), mlp=moe(9, 2, 3, 1, 10, 0.7, 2.2)),
    dict(maps(2, 1, 14, 22, 0.25, 0.6, 7.0, 7000.0, 10, 19, 1), mlp=dense(36, 1.0)),
    dict(full(2, 2, 34, 0.2, 2, 0.1, 30), mlp=dense(22, 0.5)),
])
# neither a filter, a temperature, a cap, a rotation nor groups: what the design's keys may leave out
KIL_D = dict(architecture="Kilisun", vocab=64, width=48, norm=dict(eps=1e-4), layers=[
    dict(type="attention", mixer=dict(heads=3, kv_heads=3, dim=16, vdim=16, scale=0.3),
         mlp=dict(kind="moe", router=dict(experts=2, top=1), expert=dict(ff=8, limit=1.0))),
    dict(type="attention_2", mixer=dict(heads=2, kv_heads=2, dim=16, vdim=16, scale=0.3, diff=0.5, rot=dict(base=10.0, dims=0),
                                        mask=dict(size=20)), mlp=dense(64, 1.0)),
])
MODELS = {"A": (KIL_A, 61), "B": (KIL_B, 62), "C": (KIL_C, 63), "D": (KIL_D, 64)}
LENGTHS = (70, 41, 97, 2, 33, 129, 1, 9, 55)
F32_TOL = 1e-4          # float32 sums in another order than float64
BF16_TOL = 0.05         # activations rounded to 8 bits of mantissa after every op


def write_model(folder, cfg, seed):
    from safetensors.torch import save_file
    w = pk.random_weights(cfg, seed)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    return {k: v.to(torch.float64) for k, v in w.items()}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, seed) in MODELS.items():
        d = str(tmp_path_factory.mktemp(f"kilisun_{name}"))
        out[name] = (d, cfg, write_model(d, cfg, seed))
    return out


def requests_for(name):
    cfg, seed = MODELS[name]
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(LENGTHS)}


@pytest.fixture(scope="module")
def references(models):
    return {name: {rid: pk.forward(cfg, w, t).numpy() for rid, t in requests_for(name).items()}
            for name, (_, cfg, w) in models.items()}


def check(got, ref, reqs, dtype):
    """float32: every position within the limit.  bfloat16: the rounding of a router's input can tip a choice between two
    experts whose logits are nearly equal, which changes that token (and, less, the later ones of its request) by more
    than rounding does elsewhere; so the typical position stays within the limit and few are far over it.  What is cut
    or placed wrongly shows in float32, where nothing is left to chance."""
    for rid, toks in reqs.items():
        assert sorted(got[rid]) == list(range(len(toks))), f"{rid}: positions missing"
        g = np.stack([got[rid][p] for p in range(len(toks))])
        assert np.isfinite(g).all(), f"{rid}: position {int((~np.isfinite(g)).any(axis=1).argmax())} is not finite"
        diff = g - ref[rid]
        err = (diff - diff.mean(axis=1, keepdims=True)).std(axis=1) / ref[rid].std()
        if dtype == "float32":
            assert err.max() <= F32_TOL, f"{rid}: first bad position {int((err > F32_TOL).argmax())}, worst {err.max():.2e}"
        else:
            over = err > 2 * BF16_TOL
            middle = np.sort(err)[(len(toks) - 1) // 2]
            assert middle <= BF16_TOL and over.sum() <= max(2, len(toks) // 5), \
                f"{rid}: first bad position {int(over.argmax())}, {int(over.sum())} far over, median {middle:.2e}"


def pairs(requests, n=2):
    return tt.portions(requests, sizes=(n,))


MODES = {"whole": tt.whole, "decode_tail": tt.decode_tail, "portions": tt.portions, "pairs": pairs, "mixed": tt.mixed}


def one_after_another(reqs, modes):
    """The schedules of several modes as one trace (requests named mode/request; each mode ends all of its requests)."""
    steps = []
    for mode in modes:
        for st in MODES[mode]({f"{mode}/{rid}": toks for rid, toks in reqs.items()}):
            steps.append(dict(st, step=len(steps)))
    return steps


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_replay_matches_plain(name, dtype, models, references, tmp_path):
    """Whole, with a decoded tail, in portions, in pairs and mixed, one schedule after the other in one process."""
    folder, cfg, _ = models[name]
    reqs = requests_for(name)
    got = tt.run_trace(folder, dtype, one_after_another(reqs, MODES), str(tmp_path), vocab=cfg["vocab"],
                       page_size=16 if name == "A" else 5)
    for mode in MODES:
        mine = {rid: got[f"{mode}/{rid}"] for rid in reqs}
        try:
            check(mine, references[name], reqs, dtype)
        except AssertionError as e:
            raise AssertionError(f"{mode}: {e}") from e


@pytest.mark.parametrize("name", ["A", "B"])
def test_float32_logits_do_not_depend_on_the_cutting(name, models, tmp_path):
    """Every kernel fixes the order of its sums per output, so in float32 a position's logits agree to the last few
    bits however its tokens were cut and batched and wherever its pages lie."""
    folder, cfg, _ = models[name]
    reqs = requests_for(name)
    outs = []
    for i, mode in enumerate(("whole", "mixed", "pairs")):
        d = tmp_path / mode
        d.mkdir()
        outs.append(tt.run_trace(folder, "float32", MODES[mode](reqs), str(d), page_size=(8, 3, 64)[i]))
    for rid, toks in reqs.items():
        a = np.stack([outs[0][rid][p] for p in range(len(toks))])
        for other in outs[1:]:
            b = np.stack([other[rid][p] for p in range(len(toks))])
            worst = np.abs(a - b).max(axis=1)
            assert worst.max() <= 2e-5 * np.abs(a).max(), f"{rid} position {int(worst.argmax())} differs between cuttings"


def test_bfloat16_with_pages_of_64_agrees_with_float32(models, tmp_path):
    """Pages of 64 keys: the shapes at which bfloat16 steps take the engine's widest kernels.  The same trace in
    float32 is the comparison."""
    folder, cfg, _ = models["A"]
    reqs = {k: v for k, v in requests_for("A").items() if len(v) > 30}
    steps = tt.mixed(reqs, live=3, first=40)
    out = {}
    for dtype in ("float32", "bfloat16"):
        d = tmp_path / dtype
        d.mkdir()
        out[dtype] = tt.run_trace(folder, dtype, steps, str(d), vocab=cfg["vocab"], page_size=64)
    ref = {rid: np.stack([out["float32"][rid][p] for p in range(len(t))]) for rid, t in reqs.items()}
    check(out["bfloat16"], ref, reqs, "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_from_one_token(name, dtype, models, tmp_path):
    """One token of prompt, then 200 tokens one by one: the cache written by single-token steps only, with every window
    passing over decoded tokens and many page borders; pages behind the windows go back to the pool meanwhile."""
    folder, cfg, w = models[name]
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 201).tolist()
    reqs = {"long": toks}
    got = tt.run_trace(folder, dtype, tt.decode_tail(reqs, tail=200), str(tmp_path), vocab=cfg["vocab"], page_size=16)
    check(got, {"long": pk.forward(cfg, w, toks).numpy()}, reqs, dtype)


def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(pk.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("eager", [True, False])
def test_greedy_generation_through_the_engine(eager, name, models):
    """``LLM.generate`` with more prompts than places in a batch and a token budget that cuts prompts into portions: the
    scheduler admits, batches, frees and reuses pages; tokens equal the plain model's greedy choice, with
    and without captured decode steps."""
    from nanohybrid_vlm_b200 import LLM, SamplingParams
    folder, cfg, w = models[name]
    rng = np.random.default_rng(9)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (23, 5, 41, 1, 12)]
    llm = LLM(folder, dtype="float32", kvcache_block_size=8, num_kvcache_blocks=40, max_num_batched_tokens=16,
              max_num_seqs=3, max_model_len=64, enforce_eager=eager)
    out = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=7, ignore_eos=True), use_tqdm=False)
    for p, o in zip(prompts, out):
        assert o["token_ids"] == plain_greedy(cfg, w, p, 7)


def test_command_line_generates_the_plain_models_tokens(models):
    """``python -m nanohybrid_vlm_b200.cli generate`` on a Kilisun folder: the registry picks the model by config.json."""
    import subprocess
    import sys
    folder, cfg, w = models["C"]
    rng = np.random.default_rng(4)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (6, 19)]
    args = [sys.executable, "-m", "nanohybrid_vlm_b200.cli", "generate", "--model", folder, "--dtype", "float32",
            "--temperature", "0", "--max-tokens", "5", "--ignore-eos", "--kvcache-block-size", "16", "--num-kvcache-blocks",
            "16", "--max-num-seqs", "2", "--max-model-len", "64", "--max-num-batched-tokens", "32", "--quiet"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    env = dict(os.environ, PYTHONPATH=tt.ROOT + os.pathsep + os.environ.get("PYTHONPATH", ""))
    r = subprocess.run(args, capture_output=True, text=True, env=env, cwd=tt.ROOT)
    assert r.returncode == 0, r.stderr[-3000:]
    lines = [json.loads(l) for l in r.stdout.splitlines() if l.startswith("{")]
    assert [l["token_ids"] for l in lines] == [plain_greedy(cfg, w, p, 5) for p in prompts]


def test_random_weights_folder_round_trip(tmp_path):
    """The random-weights mode writes a Kilisun folder from its configuration that the engine loads and runs."""
    from nanohybrid_vlm_b200.weights import write_random_model
    folder = str(tmp_path / "m")
    write_random_model(folder, dict(KIL_B, dtype="bfloat16"), seed=5)
    reqs = {"a": list(range(40)), "b": [7, 3, 9]}
    out = tmp_path / "o"
    out.mkdir()
    got = tt.run_trace(folder, "bfloat16", tt.mixed(reqs, live=2, first=8), str(out), vocab=KIL_B["vocab"])
    assert all(np.isfinite(row).all() for rows in got.values() for row in rows.values())
