"""Vugipel without a GPU: the typed configuration (keys, checks, the model in parts, the tensors it declares), the
registry, random model folders, what the cache manager keeps for a window with kept first tokens, and properties
of the plain implementation that the GPU tests lean on."""
import copy
import math
import random

import pytest
import torch

import plain_vugipel as P
from tiny_configs import TINY, make_model_dir

F64 = torch.float64
NAMES = ("VA", "VB", "VC", "VD", "VE")


def typed(raw):
    from flyweight_b200.config.vugipel import VugipelConfig
    return VugipelConfig.from_dict(raw)


def built(raw, precision="float32"):
    from flyweight_b200.models import VugipelForCausalLM
    from flyweight_b200.parts import Precision
    return VugipelForCausalLM(typed(raw), Precision(precision), torch.device("cpu"))


def test_the_registry_finds_the_architecture_by_either_key():
    import flyweight_b200.models  # noqa: F401
    from flyweight_b200.config import architecture_name, lookup
    raw = TINY["VA"]
    assert architecture_name(raw) == "Vugipel"
    assert architecture_name({"architectures": ["Vugipel"]}) == "Vugipel"
    assert lookup("Vugipel").config_class.from_dict(raw).to_dict() == typed(raw).to_dict() == raw


@pytest.mark.parametrize("name", NAMES)
def test_the_model_in_parts_follows_the_configuration(name):
    raw = TINY[name]
    config = typed(raw)
    assert config.to_dict() == raw
    spec = config.model_spec()
    eps = raw["norm"]["eps"]
    assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"] and spec.head_tensor == "head"
    assert [entry.layer for entry in spec.schedule] == list(range(len(raw["layers"])))
    for index, (layer, given) in enumerate(zip(spec.layers, raw["layers"])):
        assert layer.arrangement == "prenorm_residual"
        has_ff = given["mlp"] is not None
        assert ("feed_forward" in layer.parts) == has_ff == ("ffn_norm" in layer.parts)
        assert (f"l{index}.norm2" in spec.unused_tensors) == (not has_ff)
        assert layer.parts["mixer_norm"].params == {"size": raw["width"], "eps": eps, "offset": 1.0}
        mixer, m = layer.parts["mixer"], given["mixer"]
        if given["type"] == "mingru":
            assert mixer.kind == "mingru" and mixer.params["width"] == m["width"]
        else:
            assert mixer.kind == "mixer_pair" and mixer.params["combine"] == "scaled"
            assert (mixer.params["left_scale"], mixer.params["right_scale"]) == (m["left_scale"], m["right_scale"])
            p, a = mixer.params["left"].params, m["left"]
            assert mixer.params["left"].kind == "gqa_attention"
            assert (p["num_heads"], p["num_kv_heads"], p["head_dim"], p["value_dim"], p["scale"], p["qk_norm_eps"]) == \
                (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], eps)
            mask = a.get("mask") or {}
            assert (p["window"], p["keep_first"]) == (mask.get("size", 0), mask.get("keep_first", 0))
            assert p["softcap"] == a.get("softcap", 0.0) and p["bias"] and p["temp"]
            assert p["turned_values"] == ("rot" in a)
            if "rot" in a:
                assert p["position"].params == {"theta": a["rot"]["base"], "rotary_dim": a["rot"]["dims"], "pairing": "interleaved"}
            else:
                assert p["position"].kind == "no_position"
            p, a = mixer.params["right"].params, m["right"]
            assert mixer.params["right"].kind == "decayed_linear_attention"
            assert (p["num_heads"], p["dim"], p["vdim"], list(p["decay"]), p["eps"]) == (a["heads"], a["dim"], a["vdim"], a["decay"], eps)
            assert (p["activation"], p["norm"], p["gate"]) == (None, "head", "silu") and p["k_scale"] == pytest.approx(a["dim"] ** -0.5)
        if has_ff:
            ff, g = layer.parts["feed_forward"].params, given["mlp"]
            assert (ff["ffn_dim"], ff["experts"], ff["top"]) == (g["expert"]["ff"], g["router"]["experts"], g["router"]["top"])
            assert (ff["scores"], ff["corrected"], ff["weights_on"], ff["activation"]) == ("sigmoid", False, "input", "silu")


def test_declared_tensors_their_shapes_and_what_a_request_keeps():
    from flyweight_b200.parts.base import FixedState, PagedKV
    raw = TINY["VA"]
    model = built(raw)
    declared = {name: tuple(decl.shape) for name, decl in model.declare().items()}
    W = raw["width"]
    assert declared["embed"] == declared["head"] == (raw["vocab"], W) and declared["final.norm"] == (W,)
    left, right = raw["layers"][0]["mixer"]["left"], raw["layers"][0]["mixer"]["right"]
    H, G, d, e = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
    p = "l0.mix.left."
    assert declared[p + "q"] == (H * d, W) and declared[p + "k"] == (G * d, W) and declared[p + "v"] == (G * e, W)
    assert declared[p + "q.b"] == (H * d,) and declared[p + "k.b"] == (G * d,) and declared[p + "v.b"] == (G * e,)
    assert declared[p + "q.norm"] == declared[p + "k.norm"] == (d,) and declared[p + "temp"] == (H,)
    assert declared[p + "o"] == (W, H * e) and declared[p + "o.b"] == (W,)
    h, rd, re = right["heads"], right["dim"], right["vdim"]
    p = "l0.mix.right."
    assert declared[p + "q"] == declared[p + "k"] == (h * rd, W) and declared[p + "v"] == declared[p + "g"] == (h * re, W)
    assert declared[p + "o"] == (W, h * re) and p + "norm" not in declared
    w = raw["layers"][1]["mixer"]["width"]
    assert declared["l1.mix.z"] == declared["l1.mix.x"] == declared["l1.mix.g"] == (w, W)
    assert declared["l1.mix.z.b"] == declared["l1.mix.x.b"] == (w,) and declared["l1.mix.o"] == (W, w)
    g = raw["layers"][0]["mlp"]
    assert declared["l0.mlp.router"] == (g["router"]["experts"], W) and "l0.mlp.correction" not in declared
    for j in range(g["router"]["experts"]):
        assert declared[f"l0.mlp.e{j}.gate"] == declared[f"l0.mlp.e{j}.up"] == (g["expert"]["ff"], W)
        assert declared[f"l0.mlp.e{j}.down"] == (W, g["expert"]["ff"])
    assert f"l0.mlp.e{g['router']['experts']}.gate" not in declared and "l2.norm2" not in declared
    pages, state = model.layers[0].state_spec()
    assert isinstance(pages, PagedKV) and (pages.n_kv_heads, pages.head_dim, pages.window, pages.keep_first) == (G, 32, 37, 5)
    assert isinstance(state, FixedState) and state.shape == (h * rd * re,) and state.dtype == torch.float32
    state = model.layers[1].state_spec()
    assert isinstance(state, FixedState) and state.shape == (w,) and state.dtype == torch.float32
    assert built(TINY["VB"]).layers[0].state_spec().shape == (36,)          # (33 channels, slots on 16-byte borders)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_a_random_model_folder_loads_back(tmp_path, dtype):
    folder = make_model_dir(tmp_path / "m", TINY["VB"], seed=11, dtype=dtype)
    cfg, w = P.load_model_dir(folder)
    assert cfg["architecture"] == "Vugipel"
    # weights stored around zero come out around zero, factors and plain norm weights around one
    assert abs(float(w["l0.norm1"].mean())) < 0.1 < abs(float(w["l1.mix.left.q.norm"].mean()))
    from flyweight_b200.weights import load_checkpoint
    model = built(cfg, "bfloat16" if dtype == torch.bfloat16 else "float32")
    model.load(load_checkpoint(folder, model.declare(), model.spec.unused_tensors))
    assert torch.equal(model.layers[0].mixer_norm.weight, 1.0 + w["l0.norm1"].to(torch.float32))
    pair = model.layers[1].mixer
    left, right = cfg["layers"][1]["mixer"]["left"], cfg["layers"][1]["mixer"]["right"]
    D = pair.left.head_dim
    assert pair.joined and pair.w_in.shape[0] == (left["heads"] + 2 * left["kv_heads"]) * D + right["heads"] * 2 * (right["dim"] + right["vdim"])
    # one output matrix: the left heads' columns, the bias twice, zeros, the right heads' columns, zeros
    used = left["heads"] * left["vdim"]
    bias = w["l1.mix.left.o.b"].to(pair.w_o.dtype)
    assert torch.equal(pair.w_o[:, :used], w["l1.mix.left.o"].to(pair.w_o.dtype))
    assert torch.equal(pair.w_o[:, used], bias) and torch.equal(pair.w_o[:, used + 1], bias)
    at = pair.left.out_width
    assert at % 8 == 0 and (pair.w_o[:, used + 2:at] == 0).all()
    assert torch.equal(pair.w_o[:, at:at + right["heads"] * right["vdim"]], w["l1.mix.right.o"].to(pair.w_o.dtype))
    assert pair.w_o.shape[1] % 8 == 0 and pair.weight_bytes() > 0 and pair.flops_per_token() > 0


def test_a_checkpoint_may_carry_the_norm_of_a_feed_forward_it_leaves_out(tmp_path):
    def edit(tensors):
        tensors["l2.norm2"] = torch.zeros(TINY["VA"]["width"])
    folder = make_model_dir(tmp_path / "m", TINY["VA"], seed=1, dtype=torch.float32, edit=edit)
    from flyweight_b200.weights import load_checkpoint
    model = built(TINY["VA"])
    model.load(load_checkpoint(folder, model.declare(), model.spec.unused_tensors))


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="attention"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].pop("base"), "missing base"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=25), "even vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size must be positive"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "missing left_scale"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(heads=2), "one decay per head"),
    (lambda c: c["layers"][1]["mixer"].pop("width"), "missing width"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top exceeds"),
    (lambda c: c.pop("norm"), "missing norm"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_its_reason(change, message):
    from flyweight_b200.config.lfm2 import ConfigError
    raw = copy.deepcopy(TINY["VA"])
    change(raw)
    with pytest.raises(ConfigError, match=message):
        typed(raw)


def test_options_that_do_not_combine_are_refused():
    from flyweight_b200.config.spec import PartSpec
    from flyweight_b200.parts import build_arrangement, build_mixer
    from flyweight_b200.config.spec import LayerSpec
    base = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "position": PartSpec("no_position")}
    for extra, message in (({"keep_first": 3}, "sliding window"), ({"bias": True, "gate": "head"}, "do not combine"),
                           ({"turned_values": True}, "rotary position part"),
                           ({"temp": True, "shares_cache": True}, "do not combine")):
        with pytest.raises(ValueError, match=message):
            build_mixer(PartSpec("gqa_attention", {**base, **extra}, {}))
    with pytest.raises(ValueError, match="has no form"):
        build_mixer(PartSpec("decayed_linear_attention", {"hidden_size": 8, "num_heads": 1, "dim": 4, "vdim": 4, "decay": (0.9,),
                                                          "eps": 1e-5, "norm": "head", "gate": "sigmoid"}, {}))
    norm = PartSpec("rmsnorm", {"size": 8, "eps": 1e-5}, {"weight": "n"})
    with pytest.raises(ValueError, match="go together"):
        build_arrangement(LayerSpec("prenorm_residual", parts={"mixer_norm": norm, "ffn_norm": norm,
                                                               "mixer": PartSpec("mingru", {"hidden_size": 8, "width": 8}, {})}))


# ------------------------------------------------------------------ what a window with kept first tokens keeps
@pytest.mark.parametrize("window,keep", [(37, 5), (64, 64), (1, 3), (10, 70), (130, 65), (200, 0)])
def test_the_cache_keeps_the_first_pages_and_gives_the_passed_ones_back(window, keep):
    from flyweight_b200.cache import PAGE_SIZE, CacheManager
    from flyweight_b200.parts import PagedKV
    manager = CacheManager([PagedKV(1, 16, window, keep), PagedKV(1, 16, window, keep), PagedKV(1, 16, window), PagedKV(1, 16, 0, keep),
                            PagedKV(2, 16)], num_pages=40, num_slots=3, device=None)
    # one group for each need: the first two share one; without a window kept positions mean nothing
    assert [len(g.members) for g in manager.groups] == ([2, 1, 2] if keep else [3, 2])
    group = manager.groups[0]
    assert (group.window, group.keep_first) == (window, keep)
    rnd = random.Random(window)
    manager.admit("a")
    length = 0
    while length < 1000:
        new = length + rnd.choice((1, 2, 5, 64, 63, 130))
        manager.release_passed("a")
        # every page that a query of this step may read is mapped, every other page is free again
        needed = set(range(-(-min(keep, length) // PAGE_SIZE)))
        needed |= {j // PAGE_SIZE for j in range(max(0, length - window + 1), length)}
        mapped = {i for i, page in enumerate(group.tables["a"]) if page >= 0}
        assert needed <= mapped
        spare = mapped - needed
        assert all(page in (length // PAGE_SIZE, (length - window + 1) // PAGE_SIZE) or page < -(-keep // PAGE_SIZE) for page in spare)
        manager.extend("a", new)
        manager.check()
        length = new
    assert group.pool.high_water <= -(-keep // PAGE_SIZE) + (window + 62) // PAGE_SIZE + 5
    manager.release("a")
    manager.check()
    assert all(g.pool.n_used == 0 for g in manager.groups)


def test_a_decoded_token_walks_the_windows_tiles_and_the_kept_ones():
    from flyweight_b200.kernels.attention import window_tiles
    for window in (1, 2, 63, 64, 65, 66, 129, 1024):
        for keep in (0, 1, 64, 65):
            bound = window_tiles(1000, window, keep)
            for pos in list(range(0, 400)) + [5000 + i for i in range(130)]:
                seen = {j // 64 for j in range(max(0, pos - window + 1), pos + 1)} | {j // 64 for j in range(min(keep, pos + 1))}
                assert len(seen) <= bound
    assert window_tiles(7, 0) == 7 and window_tiles(3, 1024, 5) == 3


# ------------------------------------------------------------------ the plain implementation itself
def test_plain_recurrences_by_hand():
    z = torch.tensor([[0.25, 1.0], [0.5, 0.0]], dtype=F64)
    c = torch.tensor([[2.0, 3.0], [4.0, 9.0]], dtype=F64)
    got = P.gated_average(z, c)
    assert torch.allclose(got, torch.tensor([[0.5, 3.0], [0.25 + 2.0, 3.0]], dtype=F64))
    assert torch.allclose(P.gated_average(z[1:], c[1:], got[0]), got[1:])
    u = torch.tensor([0.0, 2.0, -1.0], dtype=F64)
    assert torch.allclose(P.positive_part(u), torch.tensor([0.5, 2.5, 1.0 / (1.0 + math.e)], dtype=F64))
    q, k, v = (torch.randn(6, 2, 3, dtype=F64) for _ in range(3))
    decay = torch.tensor([0.5, 0.9], dtype=F64)
    o = P.decayed_sums(q, k, v, decay)
    for t in (0, 3, 5):
        for h in range(2):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)


def test_plain_window_and_rotation():
    pos = torch.arange(12)
    seen = P.visible(pos, pos, size=3, keep_first=2)
    assert seen[8].nonzero().flatten().tolist() == [0, 1, 6, 7, 8] and seen[1].nonzero().flatten().tolist() == [0, 1]
    x = torch.randn(12, 2, 6, dtype=F64)
    turned = P.turn_neighbours(x, pos, 50.0, 4)
    assert torch.equal(turned[..., 4:], x[..., 4:]) and torch.allclose(P.turn_neighbours(turned, pos, 50.0, 4, sign=-1.0), x)
    assert torch.allclose(turned[3, 0, 0], x[3, 0, 0] * math.cos(3.0) - x[3, 0, 1] * math.sin(3.0))
    f = 50.0 ** -0.5
    assert torch.allclose(turned[3, 0, 3], x[3, 0, 3] * math.cos(3.0 * f) + x[3, 0, 2] * math.sin(3.0 * f))
    # scores of turned heads depend on distances alone
    a, b = torch.randn(1, 1, 4, dtype=F64), torch.randn(1, 1, 4, dtype=F64)
    dot = lambda i, j: float((P.turn_neighbours(a, torch.tensor([i]), 9.0, 4) * P.turn_neighbours(b, torch.tensor([j]), 9.0, 4)).sum())
    assert dot(7, 3) == pytest.approx(dot(104, 100), rel=1e-12)


def test_plain_experts_weigh_their_inputs():
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0], [-1.0, 0.0]], dtype=F64)}
    for j in range(3):
        w[f"e{j}.gate"] = w[f"e{j}.up"] = torch.full((1, 2), float(j + 1), dtype=F64)
        w[f"e{j}.down"] = torch.tensor([[1.0], [0.5]], dtype=F64)
    h = torch.tensor([[0.3, 2.0]], dtype=F64)
    got = P.input_weighted_experts(h, w, "", {"router": {"top": 2}})
    want = torch.zeros(2, dtype=F64)
    for j, z in ((1, 2.0), (0, 0.3)):
        g = (j + 1) * 2.3 / (1.0 + math.exp(-z))
        want += g / (1.0 + math.exp(-g)) * g * torch.tensor([1.0, 0.5], dtype=F64)
    assert torch.allclose(got[0], want)


@pytest.mark.parametrize("name", ("VA", "VB"))
def test_plain_logits_are_causal(name, tmp_path):
    folder = make_model_dir(tmp_path / "m", TINY[name], seed=5, dtype=torch.float32)
    cfg, w = P.load_model_dir(folder)
    tokens = [int(t) for t in torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(1))]
    layers = []
    full = P.forward(cfg, w, tokens, layers_out=layers)
    assert len(layers) == len(cfg["layers"])
    changed = list(tokens)
    changed[20] = (changed[20] + 1) % cfg["vocab"]
    other = P.forward(cfg, w, changed)
    assert torch.equal(other[:20], full[:20]) and not torch.allclose(other[20:], full[20:])


def test_class_routers_leave_no_close_call(tmp_path):
    """The 16-bit model folders of the GPU tests: every token's chosen scores stand clear of the others in every layer."""
    from gpu_util import _class_routers
    raw = TINY["VA"]
    folder = make_model_dir(tmp_path / "m", raw, seed=5, dtype=torch.bfloat16, edit=lambda t: _class_routers(t, raw))
    cfg, w = P.load_model_dir(folder)
    gaps, chosen = [], set()
    original = P.sigmoid_choice

    def watched(h, router, top):
        z = (h @ router.T).sort(dim=1, descending=True).values
        if top < z.shape[1]:
            gaps.append(float((z[:, top - 1] - z[:, top]).min()))
        ids, scores = original(h, router, top)
        chosen.update(ids[:, 0].tolist())
        return ids, scores
    P.sigmoid_choice = watched
    try:
        P.forward(cfg, w, list(range(60)))
    finally:
        P.sigmoid_choice = original
    assert min(gaps) > 0.1 and len(chosen) > 2
