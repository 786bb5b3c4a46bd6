"""Vozorax through the engine against the plain model (float64): the same requests whole, with their last tokens
decoded one by one, in portions down to two tokens, and mixed with other requests in a pool so small that pages are used
again; long decoding from a single token; greedy generation through ``LLM.generate`` and the scheduler, and through the
command line.  Small configurations that differ in every size, in the order of their layers and in what the design leaves
open: one to five copies of the stream, windows of one key, smaller and larger than a page and none at all, value heads
smaller and larger than key heads, value mixing in all attention layers, in some and in none, one to four experts chosen,
a mixture without a shared expert, layers without a feed-forward, sizes that are no multiple of 8."""
import json
import os

import numpy as np
import pytest
import torch

import plain_vozorax as pv
import trace_tools as tt

pytestmark = pytest.mark.gpu


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, size, scale):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
             rot=dict(base=base, dims=rot_dim))
    return m if size is None else dict(m, mask=dict(size=size))


def attn(heads, kv, dim, vdim, size, scale, v_mix):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    return m if size is None else dict(m, mask=dict(size=size))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared):
    m = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
    return m if shared is None else dict(m, shared=dict(ff=shared))


VOZ_A = dict(architecture="Vozorax", vocab=300, width=96, streams=4, norm=dict(eps=1e-6), layers=[
    dict(type="latent_attention", mixer=latent(3, 16, 8, 24, 40, 48, 10000.0, 33, 0.2), mlp=moe(4, 2, 24, 32)),
    dict(type="attention", mixer=attn(6, 3, 32, 16, 12, 0.2, True), mlp=dense(80)),
    dict(type="latent_attention", mixer=latent(4, 32, 32, 16, 24, 64, 500.0, 70, 0.15), mlp=None),
    dict(type="attention", mixer=attn(4, 1, 16, 48, 40, 0.3, True), mlp=moe(3, 1, 16, None)),
])
VOZ_B = dict(architecture="Vozorax", vocab=211, width=64, streams=2, norm=dict(eps=1e-5), layers=[
    dict(type="attention", mixer=attn(2, 2, 64, 8, 5, 0.15, False), mlp=moe(6, 4, 8, 16)),
    dict(type="attention", mixer=attn(4, 2, 16, 16, 25, 0.3, True), mlp=dense(40)),
    dict(type="latent_attention", mixer=latent(2, 8, 4, 8, 16, 24, 300.0, 1, 0.4), mlp=dense(32)),
    dict(type="attention", mixer=attn(8, 4, 8, 8, 64, 0.4, True), mlp=None),
    dict(type="latent_attention", mixer=latent(1, 40, 24, 48, 8, 32, 100.0, None, 0.12), mlp=moe(2, 2, 12, 20)),
    dict(type="attention", mixer=attn(2, 2, 32, 16, None, 0.2, True), mlp=None),
])
# sizes that are no multiple of 8 anywhere: every product and the attention take their general paths
VOZ_C = dict(architecture="Vozorax", vocab=97, width=100, streams=5, norm=dict(eps=1e-5), layers=[
    dict(type="attention", mixer=attn(3, 1, 20, 14, 19, 0.25, True), mlp=moe(5, 3, 18, 14)),
    dict(type="latent_attention", mixer=latent(3, 14, 6, 10, 22, 30, 7000.0, 50, 0.25), mlp=moe(7, 1, 10, None)),
    dict(type="attention", mixer=attn(2, 1, 34, 14, 33, 0.2, True), mlp=dense(36)),
    dict(type="latent_attention", mixer=latent(5, 6, 2, 18, 9, 13, 20.0, 9, 0.4), mlp=dense(22)),
])
# one copy of the stream, which its connection still scales
VOZ_D = dict(architecture="Vozorax", vocab=64, width=48, streams=1, norm=dict(eps=1e-4), layers=[
    dict(type="latent_attention", mixer=latent(2, 16, 16, 16, 16, 16, 1000.0, 20, 0.2), mlp=dense(64)),
    dict(type="attention", mixer=attn(3, 3, 16, 16, 16, 0.3, False), mlp=moe(2, 1, 8, 8)),
])
MODELS = {"A": (VOZ_A, 51), "B": (VOZ_B, 52), "C": (VOZ_C, 75), "D": (VOZ_D, 54)}
LENGTHS = (70, 41, 97, 2, 33, 129, 1, 9, 55)
F32_TOL = 1e-4          # float32 sums in another order than float64
BF16_TOL = 0.05         # activations rounded to 8 bits of mantissa after every op


def write_model(folder, cfg, seed):
    from safetensors.torch import save_file
    w = pv.random_weights(cfg, seed)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    return {k: v.to(torch.float64) for k, v in w.items()}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, seed) in MODELS.items():
        d = str(tmp_path_factory.mktemp(f"vozorax_{name}"))
        out[name] = (d, cfg, write_model(d, cfg, seed))
    return out


def requests_for(name):
    cfg, seed = MODELS[name]
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(LENGTHS)}


@pytest.fixture(scope="module")
def references(models):
    return {name: {rid: pv.forward(cfg, w, t).numpy() for rid, t in requests_for(name).items()}
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
    check(got, {"long": pv.forward(cfg, w, toks).numpy()}, reqs, dtype)


def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(pv.forward(cfg, w, toks)[-1].argmax()))
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
    """``python -m nanohybrid_vlm_b200.cli generate`` on a Vozorax folder: the registry picks the model by config.json."""
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
    """The random-weights mode writes a Vozorax folder from its configuration that the engine loads and runs."""
    from nanohybrid_vlm_b200.weights import write_random_model
    folder = str(tmp_path / "m")
    write_random_model(folder, dict(VOZ_B, dtype="bfloat16"), seed=5)
    reqs = {"a": list(range(40)), "b": [7, 3, 9]}
    out = tmp_path / "o"
    out.mkdir()
    got = tt.run_trace(folder, "bfloat16", tt.mixed(reqs, live=2, first=8), str(out), vocab=VOZ_B["vocab"])
    assert all(np.isfinite(row).all() for rows in got.values() for row in rows.values())
