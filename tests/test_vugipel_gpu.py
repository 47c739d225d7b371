"""Vugipel through the engine: the step function, the cache manager and the runtime against the plain
implementation (``plain_vugipel``), on five tiny configurations that differ in every size, in both
dtypes: whole prompts, token-by-token decoding, portions down to two tokens, batches of unequal
requests over pools whose pages and slots are used again, long decoding over page and window borders,
the stream after every layer, and greedy generation through the entry point and its scheduler."""
import numpy as np
import pytest
import torch

import plain_vugipel as P
from gpu_util import (DTYPES, TOL_ORACLE, assert_close, mixed_trace, model_dir, new_runner, oracle_rows,
                      plain_logits, plain_model, random_tokens, replay_in_process, run_portions, run_whole)
from tiny_configs import TINY, vocab_of

pytestmark = pytest.mark.gpu
NAMES = ("VA", "VB", "VC")
ALL = NAMES + ("VD", "VE")


@pytest.mark.parametrize("name", ALL)
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts(name, dtype):
    runner = new_runner(name, dtype)
    for n in (1, 2, 3, 37, 38, 64, 65, 71, 131, 200):
        tokens = random_tokens(name, n, seed=n)
        assert_close(run_whole(runner, f"w{n}", tokens), plain_logits(name, dtype, tokens),
                     oracle_rows(name, dtype, tokens), f"{name} {dtype} whole prompt of {n}")
    runner.check_health()


@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_prefill_against_token_by_token_decoding(name, dtype):
    runner = new_runner(name, dtype)
    tokens = random_tokens(name, 140, seed=5)
    whole = run_whole(runner, "whole", tokens)
    single = run_portions(runner, "single", tokens, [1])
    want = plain_logits(name, dtype, tokens)
    bound = oracle_rows(name, dtype, tokens)
    assert_close(single, want, bound, "token by token")
    assert_close(single, whole, 2e-5 if dtype == "float32" else 2.0 * bound, "token by token against the whole prompt")
    late = run_portions(runner, "late", tokens, [100] + [1] * 40)
    assert_close(late, want, bound, "a prompt, then decoding")


@pytest.mark.parametrize("name", ALL)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2,), (3, 2, 7, 1, 64, 2, 33), (63, 2, 64, 1, 1, 65), (128, 2), (36, 1, 1, 2)])
def test_portions_of_any_size(name, dtype, sizes):
    runner = new_runner(name, dtype)
    tokens = random_tokens(name, 197, seed=11)
    want = plain_logits(name, dtype, tokens)
    assert_close(run_portions(runner, "p", tokens, list(sizes)), want, oracle_rows(name, dtype, tokens),
                 f"portions {sizes}")


@pytest.mark.parametrize("name", ALL)
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_over_a_small_pool(name, dtype):
    """Up to four live requests, portions beside single tokens, requests left out of steps; the pool
    has fewer pages than the requests need together, so pages and state slots are used again, and a
    stale recurrent state or a cache row of an earlier owner would show."""
    lengths = [150, 40, 97, 1, 130, 64, 2, 70, 129]
    steps, tokens = mixed_trace(lengths, vocab_of(TINY[name]), num_pages=7, max_live=4, seed=4, tail=20)
    runner = new_runner(name, dtype, num_pages=7, num_slots=4, max_model_len=256)
    got = replay_in_process(runner, steps)
    for rid, ids in tokens.items():
        assert_close(got[rid], plain_logits(name, dtype, ids), oracle_rows(name, dtype, ids),
                     f"{name} {dtype} request {rid}")
    assert all(group.pool.n_used == 0 for group in runner.cache.groups)
    runner.check_health()


@pytest.mark.parametrize("name", ("VA", "VB", "VE"))
def test_a_slot_and_pages_used_again_hold_nothing_of_their_last_owner(name):
    dtype = "float32"
    runner = new_runner(name, dtype, num_pages=3, num_slots=1, max_model_len=192)
    first = random_tokens(name, 180, seed=1)
    second = random_tokens(name, 150, seed=2)
    run_whole(runner, "first", first)
    got = run_portions(runner, "second", second, [70, 1, 1, 50, 28])
    assert_close(got, plain_logits(name, dtype, second), TOL_ORACLE[dtype], "second owner")


@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_page_and_window_borders(name, dtype):
    """Three requests decode together for 200 steps from prompts of different lengths: every page border
    is crossed by a decoded token, windows leave pages behind and kept first tokens stay, in a replayed graph once the
    shape has settled."""
    prompts = [random_tokens(name, n, seed=30 + n) for n in (1, 60, 127)]
    cont = [random_tokens(name, 200, seed=40 + i) for i in range(3)]
    runner = new_runner(name, dtype, num_pages=16, num_slots=4, max_model_len=512)
    rows = [[runner.step([(f"d{i}", p, list(range(len(p))))]).cpu().numpy()] for i, p in enumerate(prompts)]
    for step in range(200):
        out = runner.step([(f"d{i}", [cont[i][step]], [0]) for i in range(3)]).cpu().numpy()
        for i in range(3):
            rows[i].append(out[i:i + 1])
    assert runner.graph_replays > 0
    for i in range(3):
        assert_close(np.concatenate(rows[i]), plain_logits(name, dtype, prompts[i] + cont[i]),
                     oracle_rows(name, dtype, prompts[i] + cont[i]), f"{name} {dtype} request {i}")
    runner.check_health()


@pytest.mark.parametrize("name", ("VA", "VB", "VC"))
def test_the_stream_after_every_layer(name):
    """float32, layer by layer: the engine's residual stream behind each layer against the plain one, so a
    fault shows in the first layer that has it and not only in the logits."""
    dtype = "float32"
    tokens = random_tokens(name, 90, seed=8)
    cfg, w = plain_model(name, dtype)
    want = []
    P.forward(cfg, w, tokens, layers_out=want)
    runner = new_runner(name, dtype)
    model = runner.model
    seen = []
    hooks = []
    for layer in model.layers:
        original = layer.forward

        def wrapped(ctx, x, pending, cache, _f=original):
            out, pending = _f(ctx, x, pending, cache)
            seen.append((out if pending is None else out + pending).detach().to(torch.float64).cpu().clone())
            return out, pending
        layer.forward = wrapped
        hooks.append((layer, original))
    try:
        run_whole(runner, "layers", tokens)
    finally:
        for layer, original in hooks:
            layer.forward = original
    assert len(seen) == len(want) == len(cfg["layers"])
    for index, (got, plain) in enumerate(zip(seen, want)):
        assert_close(got.numpy(), plain.numpy(), 2e-5, f"{name} stream behind layer {index}")


@pytest.mark.parametrize("name", NAMES + ("VD",))
def test_greedy_generation_through_the_runtime(name):
    from flyweight_b200 import Model
    cfg, w = plain_model(name, "float32")
    prompts = [random_tokens(name, n, seed=50 + n) for n in (1, 9, 70)]
    with Model(model_dir(name, "float32"), dtype="float32").native_runtime(
            context_limit=192, parallel_sequences=3) as runtime:
        alone = runtime.generate(prompts[1], 24)
        assert alone == P.greedy_generate(cfg, w, prompts[1], 24)
        for prompt, result in zip(prompts, runtime.generate_batch(prompts, 24)):
            assert list(result.generated_ids) == P.greedy_generate(cfg, w, prompt, 24)
        assert all(group["pages_in_use"] == 0 for group in runtime.info["cache"]["groups"])


def test_bfloat16_generation_with_more_requests_than_slots():
    """Requests queue for slots and pages, are admitted as others end, and every generated token is
    (within the bfloat16 bound) the best of the plain implementation's logits at its place."""
    from flyweight_b200 import Model
    name, dtype = "VC", "bfloat16"
    prompts = [random_tokens(name, n, seed=70 + n) for n in (3, 40, 66, 12, 90, 5)]
    with Model(model_dir(name, dtype), dtype=dtype).native_runtime(
            context_limit=128, parallel_sequences=2) as runtime:
        results = runtime.generate_batch(prompts, 20)
    for prompt, result in zip(prompts, results):
        made = list(result.generated_ids)
        assert len(made) == 20
        logits = plain_logits(name, dtype, prompt + made)
        scale = max(1.0, np.abs(logits).max())
        bound = oracle_rows(name, dtype, prompt + made)
        for i, token in enumerate(made):
            row = logits[len(prompt) - 1 + i]
            assert row.max() - row[token] <= 2 * bound[len(prompt) - 1 + i, 0] * scale


def test_the_model_folder_round_trip_the_command_line_and_the_trace_runner(tmp_path):
    """`make-random` writes a Vugipel folder from a configuration file, `inspect` and `generate` read it,
    and the trace runner replays steps over it."""
    import json
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    config = tmp_path / "config.json"
    config.write_text(json.dumps(TINY["VA"]))
    folder = tmp_path / "model"
    run = lambda *args: subprocess.run([sys.executable, "-m", "flyweight_b200", *args], cwd=root,
                                       capture_output=True, text=True, timeout=600)
    made = run("make-random", str(config), "--out", str(folder), "--seed", "5", "--preset", "unit",
               "--dtype", "float32")
    assert made.returncode == 0, made.stderr
    seen = run("inspect", str(folder))
    assert seen.returncode == 0 and "Vugipel" in seen.stdout, seen.stderr
    prompt = random_tokens("VA", 6, seed=1)
    out = run("generate", str(folder), "--dtype", "float32", "--prompt", ",".join(map(str, prompt)),
              "--max-tokens", "8", "--temperature", "0")
    assert out.returncode == 0, out.stderr[-2000:]
    cfg, w = P.load_model_dir(folder)
    assert [int(t) for t in out.stdout.split()] == P.greedy_generate(cfg, w, prompt, 8)
    tokens = random_tokens("VA", 75, seed=2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[70:72], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[72:], "want": [2]}], "end": ["a"]}]
    replay = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
                             str(tmp_path / "out"), "--max-tokens", "128"], cwd=root, capture_output=True, text=True,
                            timeout=600, input="".join(json.dumps(line) + "\n" for line in lines))
    assert replay.returncode == 0, replay.stderr[-2000:]
    assert [l for l in replay.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = np.asarray(P.forward(cfg, w, tokens))
    got = np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").reshape(2, -1)
    assert_close(got, want[[0, 69]], TOL_ORACLE["float32"], "step 0")
    assert not (tmp_path / "out" / "1.f32").exists()
    got = np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(1, -1)
    assert_close(got, want[[74]], TOL_ORACLE["float32"], "step 2")


# ------------------------------------------------------------------ wider layers, longer prompts
def _wider_config(v):
    mlp = {"kind": "moe", "expert": {"ff": 96}, "router": {"experts": 5, "top": 2}}
    if v == 0:
        left = {"heads": 4, "kv_heads": 4, "dim": 64, "vdim": 128, "scale": 0.2, "softcap": 5.0,
                "mask": {"size": 100, "keep_first": 9}, "rot": {"base": 10000.0, "dims": 32}}
        wide = {"heads": 6, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.3, "softcap": 30.0,
                "mask": {"size": 300, "keep_first": 130}, "rot": {"base": 500.0, "dims": 32}}
        right = {"heads": 4, "dim": 64, "vdim": 32, "decay": [0.9, 0.97, 0.99, 0.999]}
        layers = [{"type": "mingru", "mixer": {"width": 256}, "mlp": mlp},
                  {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.9}, "mlp": None},
                  {"type": "parallel", "mixer": {"left": wide, "right": right, "left_scale": 1.1, "right_scale": 0.4}, "mlp": mlp},
                  {"type": "mingru", "mixer": {"width": 384}, "mlp": mlp}]
        return {"architecture": "Vugipel", "vocab": 1000, "width": 256, "norm": {"eps": 1e-6}, "layers": layers}
    left = {"heads": 12, "kv_heads": 3, "dim": 128, "vdim": 64, "scale": 0.15, "mask": {"size": 257, "keep_first": 64},
            "rot": {"base": 500000.0, "dims": 80}}
    right = {"heads": 2, "dim": 96, "vdim": 160, "decay": [0.95, 0.9995]}
    layers = [{"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}, "mlp": mlp},
              {"type": "mingru", "mixer": {"width": 200}, "mlp": {"kind": "moe", "expert": {"ff": 200}, "router": {"experts": 9, "top": 4}}},
              {"type": "mingru", "mixer": {"width": 1000}, "mlp": None},
              {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.9, "right_scale": 0.3}, "mlp": mlp}]
    return {"architecture": "Vugipel", "vocab": 777, "width": 320, "norm": {"eps": 1e-5}, "layers": layers}


@pytest.mark.parametrize("variant", (0, 1))
@pytest.mark.parametrize("dtype", DTYPES)
def test_wider_layers_and_longer_prompts(variant, dtype, tmp_path):
    """Two configurations with heads of 32 to 128 channels (values wider than keys and narrower), windows of 100 to
    300 keys with 9 to 130 kept ones, states of 64 x 32 and 96 x 160, minGRU layers wider and narrower than the
    model: 1,300 tokens whole (more than one round of the recurrence's cluster), in portions that end on and off
    the borders of pages and windows, and as a prompt of 1,200 followed by 100 single tokens."""
    from gpu_util import _class_routers
    from tiny_configs import make_model_dir
    from flyweight_b200.engine import ModelRunner, load_model
    config = _wider_config(variant)
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    edit = None if dtype == "float32" else (lambda tensors: _class_routers(tensors, config))
    folder = make_model_dir(str(tmp_path / "model"), config, seed=7 + variant, dtype=stored, edit=edit)
    cfg, w = P.load_model_dir(folder)
    rng = np.random.default_rng(variant)
    tokens = [int(t) for t in rng.integers(0, config["vocab"], size=1300)]
    want = np.asarray(P.forward(cfg, w, tokens))
    bound = 2e-4
    if dtype == "bfloat16":
        rows = np.max([np.abs(np.asarray(P.forward(cfg, w, tokens, rnd=rnd)) - want).max(axis=1)
                       for rnd in (P.bf16, P.dither(0), P.dither(1))], axis=0)
        bound = np.maximum(TOL_ORACLE[dtype], 3.0 * rows / max(1.0, float(np.abs(want).max())))[:, None]
    runner = ModelRunner(load_model(folder, dtype), num_pages=24, num_slots=4, max_model_len=1536,
                         max_batched_tokens=4096)
    for what, sizes in (("whole", [1300]), ("portions", [300, 2, 1, 257, 64, 1, 1, 674]), ("decoding", [1200] + [1] * 100)):
        assert_close(run_portions(runner, what, tokens, sizes), want, bound, f"variant {variant} {dtype} {what}")
    runner.check_health()


def test_pages_a_window_has_passed_go_back_and_kept_ones_stay():
    """One request far longer than the pool's pages could hold if every page stayed: the window's old pages are
    given back, the page of the kept first tokens is not, and the logits stay right to the end."""
    name, dtype = "VA", "float32"
    config = {**TINY[name], "layers": [TINY[name]["layers"][0], TINY[name]["layers"][1]]}
    from tiny_configs import make_model_dir
    import tempfile
    from flyweight_b200.engine import ModelRunner, load_model
    with tempfile.TemporaryDirectory() as folder:
        make_model_dir(folder, config, seed=12, dtype=torch.float32)
        cfg, w = P.load_model_dir(folder)
        runner = ModelRunner(load_model(folder, dtype), num_pages=4, num_slots=2, max_model_len=640, max_batched_tokens=512)
    tokens = random_tokens(name, 600, seed=3)
    sizes = [60, 64, 30, 1, 1, 64, 64, 64] + [1] * 12 + [40] * 6
    got = run_portions(runner, "long", tokens, sizes, finish=False)
    group = runner.cache.groups[0]
    table = group.tables["long"]
    assert len(table) == -(-600 // 64) and table[0] >= 0 and all(page < 0 for page in table[1:8])
    assert group.pool.high_water <= 4 and (group.window, group.keep_first) == (37, 5)
    runner.finish("long")
    assert group.pool.n_used == 0
    assert_close(got, np.asarray(P.forward(cfg, w, tokens)), TOL_ORACLE[dtype], "a long request over four pages")
