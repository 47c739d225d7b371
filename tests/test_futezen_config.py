"""Futezen without a GPU: the typed configuration (keys, checks, the model in parts, the schedule of repeated layers,
the tensors it declares), the registry, random model folders, and properties of the plain implementation that the
GPU tests lean on."""
import copy

import pytest
import torch

import plain_futezen as P
from tiny_configs import TINY, make_model_dir

F64 = torch.float64
NAMES = ("ZA", "ZB", "ZC", "ZD", "ZE")


def typed(raw):
    from flyweight_b200.config.futezen import FutezenConfig
    return FutezenConfig.from_dict(raw)


def model_of(raw):
    from flyweight_b200.models import FutezenForCausalLM
    from flyweight_b200.parts import Precision
    return FutezenForCausalLM(typed(raw), Precision("float32"), torch.device("cpu"))


def test_the_registry_finds_the_architecture_by_either_key():
    import flyweight_b200.models  # noqa: F401
    from flyweight_b200.config import architecture_name, lookup
    raw = TINY["ZA"]
    assert architecture_name(raw) == "Futezen"
    assert architecture_name({"architectures": ["Futezen"]}) == "Futezen"
    assert lookup("Futezen").config_class.from_dict(raw).to_dict() == typed(raw).to_dict()


@pytest.mark.parametrize("name", NAMES)
def test_the_model_in_parts_follows_the_configuration(name):
    raw = TINY[name]
    config = typed(raw)
    back = config.to_dict()
    assert back["layers"] == raw["layers"] and back["vocab"] == raw["vocab"] and back["width"] == raw["width"]
    assert back.get("loop") == raw.get("loop") and typed(back) == config
    spec = config.model_spec()
    eps = raw["norm"]["eps"]
    assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"] and spec.head_tensor is None
    assert spec.final_norm.params == {"size": raw["width"], "eps": eps, "offset": 1.0}
    for layer, given in zip(spec.layers, raw["layers"]):
        assert layer.arrangement == "sandwich_residual"
        has_ff = given["mlp"] is not None
        assert ("feed_forward" in layer.parts) == has_ff == ("ffn_norm" in layer.parts) == ("ffn_out_norm" in layer.parts)
        for role in ("mixer_norm", "mixer_out_norm") + (("ffn_norm", "ffn_out_norm") if has_ff else ()):
            assert layer.parts[role].params == {"size": raw["width"], "eps": eps, "offset": 1.0}
        mixer, m = layer.parts["mixer"], given["mixer"]
        p = mixer.params
        if given["type"] == "mamba2":
            assert mixer.kind == "state_space"
            assert (p["num_heads"], p["vdim"], p["state"], p["groups"], p["taps"], p["norm_groups"], p["eps"]) == \
                (m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"], eps)
        else:
            if given["type"] == "attention":
                assert mixer.kind == "gqa_attention" and p["qk_norm_eps"] is None
                assert (p["num_heads"], p["num_kv_heads"], p["head_dim"], p["value_dim"], p["scale"]) == \
                    (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"])
                dims, pairing = m["rot"]["dims"], "half_split"
            else:
                assert mixer.kind == "latent_attention" and p["sink"] is False and p["eps"] == eps
                assert (p["num_heads"], p["dim"], p["rot_dim"], p["vdim"], p["q_rank"], p["kv_rank"], p["scale"]) == \
                    (m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"])
                dims, pairing = m["rot_dim"], "interleaved"
            assert p["position"].params == {"theta": m["rot"]["base"], "rotary_dim": dims, "pairing": pairing}
        if not has_ff:
            continue
        ff, g = layer.parts["feed_forward"], given["mlp"]
        if g["kind"] == "dense":
            assert ff.kind == "swiglu" and ff.params["activation"] == "relu" and ff.params["ffn_dim"] == g["ff"]
        else:
            assert ff.kind == "routed_experts" and ff.params["scores"] == "softmax_chosen" and not ff.params["gated"]
            assert (ff.params["ffn_dim"], ff.params["experts"], ff.params["top"], ff.params["activation"]) == \
                (g["expert"]["ff"], g["router"]["experts"], g["router"]["top"], "relu_squared")
            assert ff.params.get("shared_ffn_dim") == (g.get("shared") or {}).get("ff")
            assert ("shared_scale" in ff.tensors) == ("shared" in g)


@pytest.mark.parametrize("name", NAMES)
def test_the_schedule_repeats_the_looped_layers_with_caches_of_their_own(name):
    raw = TINY[name]
    n, loop = len(raw["layers"]), raw.get("loop")
    want = list(range(n)) if loop is None else (list(range(loop["start"]))
                                                + list(range(loop["start"], loop["stop"])) * loop["times"]
                                                + list(range(loop["stop"], n)))
    model = model_of(raw)
    assert [entry.layer for entry in model.spec.schedule] == want == P.layer_runs(raw)
    assert all(entry.cache_of is None and not entry.add_embedding for entry in model.spec.schedule)
    from flyweight_b200.cache.manager import CacheManager
    manager = CacheManager(model.state_specs(), num_pages=4, num_slots=2, device=None)
    assert len(manager.layer_caches) == len(want)
    paged = sum(raw["layers"][i]["type"] != "mamba2" for i in want)
    assert sum(len(group.members) for group in manager.groups) == paged


def test_declared_tensors_and_what_a_request_keeps():
    from flyweight_b200.parts.base import FixedState, PagedKV
    raw = TINY["ZA"]
    model = model_of(raw)
    declared = {name: tuple(decl.shape) for name, decl in model.declare().items()}
    W = raw["width"]
    assert declared["embed"] == (raw["vocab"], W) and "head" not in declared and declared["final.norm"] == (W,)
    for i, given in enumerate(raw["layers"]):
        assert declared[f"l{i}.norm1"] == declared[f"l{i}.norm1b"] == (W,)
        assert (f"l{i}.norm2" in declared) == (f"l{i}.norm2b" in declared) == (given["mlp"] is not None)
    a = raw["layers"][0]["mixer"]
    inner, bc = a["heads"] * a["vdim"], 2 * a["groups"] * a["state"]
    assert declared["l0.mix.in"] == (2 * inner + bc + a["heads"], W) and declared["l0.mix.o"] == (W, inner)
    assert declared["l0.mix.conv"] == (inner + bc, a["conv"]) and declared["l0.mix.conv.b"] == (inner + bc,)
    assert all(declared[f"l0.mix.{name}"] == (a["heads"],) for name in ("dt_bias", "A_log", "D"))
    assert declared["l0.mix.norm"] == (inner,)
    g = raw["layers"][0]["mlp"]
    E = g["router"]["experts"]
    assert declared["l0.mlp.router"] == (E, W) and declared["l0.mlp.router.b"] == (E,)
    assert all(declared[f"l0.mlp.e{j}.up"] == (g["expert"]["ff"], W) for j in range(E)) and f"l0.mlp.e{E}.up" not in declared
    assert declared["l0.mlp.e0.down"] == (W, g["expert"]["ff"]) and "l0.mlp.e0.gate" not in declared
    assert declared["l0.mlp.shared.up"] == (g["shared"]["ff"], W) and declared["l0.mlp.shared.sg"] == (1, W)
    b = raw["layers"][1]["mixer"]
    assert declared["l1.mix.dq"] == (b["q_rank"], W) and declared["l1.mix.dq.norm"] == (b["q_rank"],)
    assert declared["l1.mix.uq"] == (b["heads"] * (b["dim"] + b["rot_dim"]), b["q_rank"]) and "l1.mix.q" not in declared
    assert declared["l1.mix.dkv"] == (b["kv_rank"] + b["rot_dim"], W) and declared["l1.mix.dkv.norm"] == (b["kv_rank"],)
    assert declared["l1.mlp.gate"] == declared["l1.mlp.up"] == (raw["layers"][1]["mlp"]["ff"], W)
    c = raw["layers"][2]["mixer"]
    assert declared["l2.mix.v"] == (c["kv_heads"] * c["vdim"], W) and declared["l2.mix.o"] == (W, c["heads"] * c["vdim"])
    state, rows, pages = (layer.state_spec() for layer in model.layers)
    # the matrices, and the convolution's last inputs behind them
    assert isinstance(state, FixedState)
    assert state.shape[0] >= a["heads"] * a["state"] * a["vdim"] + (a["conv"] - 1) * (inner + bc) and state.shape[0] % 4 == 0
    assert isinstance(rows, PagedKV) and rows.values is False and rows.head_dim >= b["kv_rank"] + b["rot_dim"]
    assert isinstance(pages, PagedKV) and pages.n_kv_heads == c["kv_heads"] and pages.window == 0


def test_a_random_model_folder_loads_back(tmp_path):
    folder = make_model_dir(tmp_path / "m", TINY["ZA"], seed=11, dtype=torch.bfloat16)
    cfg, w = P.load_model_dir(folder)
    assert cfg["architecture"] == "Futezen" and cfg["loop"] == TINY["ZA"]["loop"]
    assert abs(float(w["l0.norm1"].mean())) < 0.2                 # (norm weights are stored around zero)
    assert abs(float(w["l0.mix.norm"].mean()) - 1.0) < 0.2        # (a mixer's own norm is not)
    from flyweight_b200.models import FutezenForCausalLM
    from flyweight_b200.parts import Precision
    from flyweight_b200.weights import load_checkpoint
    model = FutezenForCausalLM(typed(cfg), Precision("bfloat16"), torch.device("cpu"))
    model.load(load_checkpoint(folder, model.declare(), model.spec.unused_tensors))
    assert model.head is model.embedding and model.graph_safe
    assert torch.equal(model.layers[0].mixer_norm.weight, w["l0.norm1"].float() + 1.0)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "multiple of groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "multiple of norm_groups"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "missing state"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top exceeds"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "missing ff"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "missing q_rank"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=3), "rot_dim must be even"),
    (lambda c: c["layers"][1]["mlp"].update(kind="table"), "unknown feed-forward"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["loop"].update(stop=9), "'loop'"),
    (lambda c: c["loop"].update(times=0), "'loop'"),
    (lambda c: c.pop("norm"), "missing norm"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_its_reason(change, message):
    from flyweight_b200.config.lfm2 import ConfigError
    raw = copy.deepcopy(TINY["ZA"])
    change(raw)
    with pytest.raises(ConfigError, match=message):
        typed(raw)


def test_visible_pages_of_a_step_are_listed_once():
    from flyweight_b200.engine import Segment, StepBatch
    batch = StepBatch([Segment("a", 0, 10, [1], []), Segment("b", 1, 100, [1] * 60, []), Segment("c", 2, 0, [1] * 64, [])],
                      [[[0, -1, -1], [1, 2, 3], [4, -1, -1]]], None)
    seg, page, table, n = batch.visible_pages(64, 1)
    assert n == 4 and seg.tolist() == [1, 1, 1, 2] and page.tolist() == [0, 1, 2, 0]
    assert table.shape == (3, 3) and table[1].tolist() == [0, 1, 2] and table[2, 0] == 3
    assert batch.visible_pages(64, 1)[0] is seg


def test_pieces_of_the_recurrence_and_slices_of_the_context():
    from flyweight_b200.kernels import latent, state_space
    assert state_space.piece_tokens(64, 2) == 128 and state_space.piece_tokens(8192, 64) == 1024
    for longest in (100, 2048, 4096):
        piece = state_space.piece_tokens(longest, 64)
        assert piece % 64 == 0 and (piece == 128 or -(-longest // piece) * 64 >= 2 * state_space.SM_COUNT)
    for items in (1, 8, 64, 500):
        for tiles in (1, 3, 64, 2000):
            splits, per = latent.rows_splits(items, tiles, 288)
            assert splits * per >= tiles and (splits - 1) * per < tiles and per <= 128
    assert latent.expanded_head(64, 32, 64) == 128 and latent.expanded_head(32, 32, 64) == 64
    assert latent.expanded_head(128, 64, 128) == 0


# ------------------------------------------------------------------ the plain implementation itself
def test_plain_recurrence_against_its_closed_form_and_its_state():
    g = torch.Generator().manual_seed(0)
    T, H, G, n, e = 12, 4, 2, 3, 5
    x, dt = torch.randn(T, H, e, generator=g, dtype=F64), torch.rand(T, H, generator=g, dtype=F64)
    b, c = torch.randn(T, G, n, generator=g, dtype=F64), torch.randn(T, G, n, generator=g, dtype=F64)
    a, skip = torch.rand(H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64)
    y, S = P.scalar_decay_scan(x, b, c, dt, a, skip)
    for t in (0, 5, 11):
        for h in range(H):
            want = skip[h] * x[t, h]
            for j in range(t + 1):
                want = want + torch.exp(-a[h] * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (c[t, h // 2] @ b[j, h // 2]) * x[j, h]
            assert torch.allclose(y[t, h], want)
    first, mid = P.scalar_decay_scan(x[:7], b[:7], c[:7], dt[:7], a, skip)
    rest, end = P.scalar_decay_scan(x[7:], b[7:], c[7:], dt[7:], a, skip, mid)
    assert torch.allclose(torch.cat([first, rest]), y) and torch.allclose(end, S)
    z = torch.tensor([-800.0, -1.0, 0.0, 2.0, 800.0], dtype=F64)
    assert torch.allclose(P.softplus(z), torch.nn.functional.softplus(z))


def test_plain_router_norm_and_feed_forward():
    logits = torch.tensor([[1.0, 3.0, 2.0, -5.0]], dtype=F64)
    ids, weights = P.chosen_experts(logits, 2)
    assert ids.tolist() == [[1, 2]] and torch.allclose(weights, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=F64), dim=1))
    h = torch.tensor([[1.0, -2.0]], dtype=F64)
    assert P.squared_relu(h, torch.tensor([[3.0, 0.0], [0.0, 1.0]], dtype=F64), torch.eye(2, dtype=F64)).tolist() == [[9.0, 0.0]]
    gate, up = torch.tensor([[-1.0, 0.0], [2.0, 0.0]], dtype=F64), torch.tensor([[1.0, 1.0], [0.0, 1.0]], dtype=F64)
    assert P.gated_relu(h, gate, up, torch.eye(2, dtype=F64)).tolist() == [[0.0, -4.0]]
    y, z = torch.tensor([[1.0, 1.0, 4.0, 4.0]], dtype=F64), torch.full((1, 4), 50.0, dtype=F64)
    out = P.gated_group_norm(y, z, torch.ones(4, dtype=F64), 2, 0.0)
    assert torch.allclose(out, torch.ones(1, 4, dtype=F64))


@pytest.mark.parametrize("name", ("ZA", "ZB"))
def test_plain_logits_are_causal_and_the_loop_counts(name, tmp_path):
    folder = make_model_dir(tmp_path / "m", TINY[name], seed=5, dtype=torch.float32)
    cfg, w = P.load_model_dir(folder)
    tokens = [int(t) for t in torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1))]
    runs = []
    full = P.forward(cfg, w, tokens, layers_out=runs)
    assert len(runs) == len(P.layer_runs(cfg))
    changed = list(tokens)
    changed[20] = (changed[20] + 1) % cfg["vocab"]
    other = P.forward(cfg, w, changed)
    assert torch.equal(other[:20], full[:20]) and not torch.allclose(other[20:], full[20:])
    once = copy.deepcopy(cfg)
    once["loop"]["times"] = 1
    assert not torch.allclose(P.forward(once, w, tokens), full)
