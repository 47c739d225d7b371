"""The mechanisms Vugipel brought to the engine, each alone: the kernel (or the part) against the function of
``plain_vugipel`` that states the same mechanism, on hand-made batches whose segments start at position 0, in
the middle of a sequence and on single tokens, over shuffled pages and slots.  Where random numbers would hide a
fault (a window's edge, the last kept token, one key far back) the inputs are made so that it shows."""
import math

import pytest
import torch

import plain_vugipel as P

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
F64 = torch.float64
EPS = 1e-5
TOL = {torch.float32: 2e-4, torch.bfloat16: 4e-2}
SHOWS = 20 * TOL[torch.float32]     # what a fault has to change in the plain result for the inputs to count as telling
DTYPES = [torch.float32, torch.bfloat16]


def dev(t, dtype=None):
    return t.to(device=DEV, dtype=dtype or t.dtype).contiguous()


def close(got, want, rel, what=""):
    got, want = got.detach().cpu().to(F64), want.detach().cpu().to(F64)
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite"
    scale = max(1.0, float(want.abs().max()))
    worst = float((got - want).abs().max())
    assert worst <= rel * scale, f"{what}: max|delta| {worst:.3e} > {rel:.1e} * {scale:.3g}"


def bf16_round(t):
    return t.to(torch.bfloat16).to(F64)


def rounding(dtype):
    return bf16_round if dtype == torch.bfloat16 else (lambda t: t.float().to(F64))


def batch_of(step, done, slot_of, pages=None):
    """A ``StepBatch`` of (sequence, tokens) pairs that continue where ``done`` says."""
    from flyweight_b200.engine import Segment, StepBatch
    segments = [Segment(f"s{s}", slot_of(s), done[s], [0] * m, []) for s, m in step]
    table = [[0]] * len(step)
    if pages is not None:
        width = max(len(pages[s]) for s, _ in step)
        table = [pages[s] + [-1] * (width - len(pages[s])) for s, _ in step]
    return StepBatch(segments, [table], DEV)


# ------------------------------------------------------------------ the gated average
# decoding requests first, portions of 1 to 1,100 tokens (below, at and above a warp's, a CTA's and a cluster's share)
AVERAGE_CUTS = [[(0, 9), (1, 1), (2, 128)], [(1, 1), (0, 2), (2, 129)], [(0, 1), (1, 1), (2, 1)],
                [(3, 1), (2, 1100), (0, 8), (1, 7)], [(3, 257), (0, 600)], [(1, 1), (3, 1), (0, 64), (2, 2)]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,out_width", [(33, 40), (64, 64), (50, 56), (7, 8), (192, 192), (320, 320), (1, 8)])
def test_gated_average_over_portions_single_tokens_and_shuffled_slots(dtype, width, out_width):
    """Four sequences in shuffled slots; gates from nearly shut (a state that lives for thousands of tokens) to
    wide open, so that a state lost at any border shows; a slot nobody owns must stay as it was."""
    from flyweight_b200.kernels import mixing
    g = torch.Generator().manual_seed(width)
    lengths = [sum(m for step in AVERAGE_CUTS for s, m in step if s == q) for q in range(4)]
    shift = torch.linspace(-7.0, 4.0, width, dtype=F64)              # (a channel's usual gate)
    z = [(torch.randn(n, width, generator=g, dtype=F64) + shift).float().to(F64) for n in lengths]
    x = [(1.5 * torch.randn(n, width, generator=g, dtype=F64)).float().to(F64) for n in lengths]
    o = [torch.randn(n, width, generator=g, dtype=F64).float().to(F64) for n in lengths]
    zb, xb = (torch.randn(width, generator=g, dtype=F64).float().to(F64) for _ in range(2))
    state = torch.full((6, width + 3), 7.0, device=DEV)
    slot_of = lambda s: 4 - s
    for s in range(4):
        state[slot_of(s)] = 0.0
    done, got = [0] * 4, [[] for _ in range(4)]
    for step in AVERAGE_CUTS:
        rows = torch.cat([torch.cat([o[s][done[s]:done[s] + m], z[s][done[s]:done[s] + m], torch.zeros(m, 2, dtype=F64),
                                     x[s][done[s]:done[s] + m]], dim=1) for s, m in step])
        batch = batch_of(step, done, slot_of)
        y = mixing.gated_average(dev(rows, torch.float32), width, 2 * width + 2, 0, dev(zb, torch.float32),
                                 dev(xb, torch.float32), state, batch, width, dtype, out_width)
        assert y.dtype == dtype and tuple(y.shape) == (rows.shape[0], out_width)
        assert (y[:, width:] == 0).all()
        at = 0
        for s, m in step:
            got[s].append(y[at:at + m, :width].cpu().to(F64))
            at += m
            done[s] += m
    for s in range(4):
        states = P.gated_average(torch.sigmoid(z[s] + zb), P.positive_part(x[s] + xb))
        close(torch.cat(got[s]), states * P.silu(o[s]), 2e-5 if dtype == torch.float32 else 8e-3, f"sequence {s}")
        close(state[slot_of(s), :width], states[-1], 1e-5, f"state {s}")
    assert (state[0] == 7.0).all() and (state[5] == 7.0).all() and (state[1:5, width:] == 0).all()


def test_gated_average_candidate_at_zero_and_extreme_gates():
    """The candidate's two branches meet at 1/2; gates at the ends of fp32's range neither overflow nor lose the state."""
    from flyweight_b200.kernels import mixing
    u = torch.tensor([0.0, -0.0, 1e-30, -1e-30, -100.0, 100.0, -5.0, 3.0])
    z = torch.tensor([100.0, 100.0, 100.0, 100.0, 100.0, 100.0, -100.0, -200.0])
    want = torch.tensor([0.5, 0.5, 0.5, 0.5, 0.0, 100.5, 9.0, 9.0], dtype=F64)
    for dtype in DTYPES:
        for m in (1, 5):
            state = torch.full((1, 8), 9.0, device=DEV)
            rows = torch.cat([z, u, torch.full((8,), 30.0)]).repeat(m, 1).to(DEV)
            y = mixing.gated_average(rows, 0, 8, 16, None, None, state, batch_of([(0, m)], [0], lambda s: 0), 8, dtype)
            close(state[0], want, 1e-6, "state")
            close(y[-1], want * 30.0, 1e-6 if dtype == torch.float32 else 4e-3, "output")


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_average_does_not_depend_on_the_cut(dtype):
    from flyweight_b200.kernels import mixing
    W, n = 96, 700
    rows = torch.randn(n, 3 * W, generator=torch.Generator().manual_seed(1)).to(DEV)
    rows[:, :W] -= 3.0
    results = []
    for cut in ([700], [1] * 40 + [660], [333, 2, 300, 65], [128] * 5 + [60]):
        state, done, parts = torch.zeros(1, W, device=DEV), [0], []
        for m in cut:
            batch = batch_of([(0, m)], done, lambda s: 0)
            parts.append(mixing.gated_average(rows[done[0]:done[0] + m].contiguous(), 0, W, 2 * W, None, None, state, batch,
                                              W, dtype).float())
            done[0] += m
        results.append(torch.cat(parts))
    for other in results[1:]:
        close(other, results[0], 3e-6 if dtype == torch.float32 else 8e-3)


# ------------------------------------------------------------------ the head kernel's additions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pairing", ["interleaved", "half_split"])
@pytest.mark.parametrize("heads,kv,D,dim,rot,vdim", [(4, 2, 64, 64, 32, 64), (3, 1, 32, 20, 20, 32), (4, 4, 128, 128, 128, 96),
                                                     (2, 2, 48, 40, 16, 42), (6, 2, 16, 16, 0, 16)])
@pytest.mark.parametrize("wide", [0, 24])
def test_bias_factor_and_turned_values_in_the_head_kernel(dtype, pairing, heads, kv, D, dim, rot, vdim, wide):
    """Rows of fp32 (as the products leave them), alone or as the first columns of a wider buffer; the 16-byte form
    and the general one."""
    from flyweight_b200.kernels import ops
    g = torch.Generator().manual_seed(D + rot)
    T, columns = 70, (heads + 2 * kv) * D
    pos = torch.randint(0, 500, (T,), generator=g)
    pos[:3] = torch.tensor([0, 63, 64])
    seg = torch.arange(T) % 2
    buf = torch.randn(T, columns + wide, generator=g).to(DEV)
    qkv = buf[:, :columns]
    live = torch.zeros(heads + 2 * kv, D)
    live[:heads + kv, :dim] = 1.0
    live[heads + kv:, :vdim] = 1.0
    buf[:, :columns] *= live.reshape(-1).to(DEV)
    bias = (torch.randn(columns, generator=g) * live.reshape(-1)).to(DEV)
    temp = (1.0 + 0.5 * torch.randn(heads, generator=g)).to(DEV)
    wq, wk = ((1.0 + 0.2 * torch.randn(D, generator=g)) for _ in range(2))
    wq[dim:], wk[dim:] = 0.0, 0.0
    angle = torch.arange(512, dtype=F64)[:, None] * (10000.0 ** (-2.0 * torch.arange(max(rot // 2, 1), dtype=F64) / max(rot, 1)))
    table = torch.stack([angle.cos(), angle.sin()], -1).float().to(DEV)
    v_angle = torch.arange(512, dtype=F64)[:, None] * (300.0 ** (-2.0 * torch.arange(vdim // 2, dtype=F64) / vdim))
    v_table = torch.stack([v_angle.cos(), v_angle.sin()], -1).float().to(DEV)
    pages = torch.arange(16, dtype=torch.int32).view(2, 8).to(DEV)
    pools = [torch.zeros(16, kv, 64, D, dtype=dtype, device=DEV) for _ in range(2)]
    q = ops.qk_norm_rope(qkv, dev(wq), dev(wk), table, dev(pos, torch.int32), dev(seg, torch.int32), pages, pools[0], pools[1],
                         heads, kv, D, rot, EPS, dtype, pairing=pairing, norm_dim=dim, bias=bias, temp=temp,
                         value_table=v_table, value_rotary=vdim)

    def turn(x, base_angle, n):
        c, s = base_angle[pos].cos()[:, None], base_angle[pos].sin()[:, None]
        out = x.clone()
        a, b = (x[..., 0:n:2], x[..., 1:n:2]) if pairing == "interleaved" else (x[..., :n // 2], x[..., n // 2:n])
        lo, hi = a * c - b * s, b * c + a * s
        if pairing == "interleaved":
            out[..., 0:n:2], out[..., 1:n:2] = lo, hi
        else:
            out[..., :n // 2], out[..., n // 2:n] = lo, hi
        return out

    rows = (qkv.cpu().to(F64) + bias.cpu().to(F64)).view(T, heads + 2 * kv, D)
    unit = lambda x: x / torch.sqrt((x[..., :dim] ** 2).mean(-1, keepdim=True) + EPS)
    want_q, want_k = unit(rows[:, :heads]) * wq.to(F64), unit(rows[:, heads:heads + kv]) * wk.to(F64)
    if rot:
        want_q, want_k = turn(want_q, angle, rot), turn(want_k, angle, rot)
    want_q = want_q * temp.cpu().to(F64)[None, :, None]
    want_v = turn(rows[:, heads + kv:], v_angle, vdim)
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    close(q.view(T, heads, D), want_q, tol, "queries")
    # (two tokens of one segment may share a position: the later row wins, so compare only the last of each)
    last = {(int(s), int(p)): t for t, (s, p) in enumerate(zip(seg, pos))}
    count = {}
    for s, p in zip(seg.tolist(), pos.tolist()):
        count[s, p] = count.get((s, p), 0) + 1
    for (s, p), t in last.items():
        if count[s, p] > 1:
            continue
        page = int(pages[s, p // 64])
        close(pools[0][page, :, p % 64], want_k[t], tol, f"key {t}")
        close(pools[1][page, :, p % 64], want_v[t], tol, f"value {t}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pairing", ["interleaved", "half_split"])
@pytest.mark.parametrize("heads,D,e,turned,col0,width,ld", [(4, 64, 64, True, 0, 264, 264), (3, 32, 24, True, 16, 80, 120),
                                                            (2, 128, 96, True, 8, 200, 208), (5, 16, 10, True, 3, 57, 61),
                                                            (4, 64, 64, False, 0, 256, 256), (3, 48, 42, False, 1, 130, 140)])
def test_heads_are_packed_turned_back_and_scaled(dtype, pairing, heads, D, e, turned, col0, width, ld):
    """Columns outside the mixer's own stay as they were; the constant behind the heads carries the scale to more
    digits than the row's type has."""
    from flyweight_b200.kernels import mixing
    g = torch.Generator().manual_seed(D + e)
    T, scale = 41, 0.7123456
    o = torch.randn(T, heads * D, generator=g).to(dtype).to(DEV)
    pos = torch.randint(0, 300, (T,), generator=g)
    angle = torch.arange(300, dtype=F64)[:, None] * (1000.0 ** (-2.0 * torch.arange(e // 2, dtype=F64) / e))
    table = torch.stack([angle.cos(), angle.sin()], -1).float().to(DEV) if turned else None
    out = torch.full((T, ld), 5.0, dtype=dtype, device=DEV)
    mixing.place_heads_(o, heads, D, e, out, col0, width, scale, dev(pos, torch.int32), table, pairing)
    x = o.cpu().to(F64).view(T, heads, D)[..., :e]
    if turned:
        c, s = angle[pos].cos()[:, None], angle[pos].sin()[:, None]
        if pairing == "interleaved":
            a, b = x[..., 0::2], x[..., 1::2]
            x = torch.stack([a * c + b * s, b * c - a * s], -1).reshape(T, heads, e)
        else:
            a, b = x[..., :e // 2], x[..., e // 2:]
            x = torch.cat([a * c + b * s, b * c - a * s], -1)
    close(out[:, col0:col0 + heads * e], (x * scale).reshape(T, -1), 1e-6 if dtype == torch.float32 else 6e-3)
    rest = out[:, col0 + heads * e:col0 + width].cpu().to(F64)
    if rest.shape[1] >= 2:
        assert (rest[:, 0] + rest[:, 1] - scale).abs().max() < (1e-7 if dtype == torch.float32 else 2e-5)
        assert (rest[:, 2:] == 0).all()
    assert (out[:, :col0] == 5.0).all() and (out[:, col0 + width:] == 5.0).all()


# ------------------------------------------------------------------ parts from a configuration
def tiny_config(**kw):
    left = {"heads": kw.get("heads", 4), "kv_heads": kw.get("kv", 2), "dim": kw.get("dim", 16), "vdim": kw.get("vdim", 24),
            "scale": kw.get("scale", 0.3)}
    if kw.get("window"):
        left["mask"] = {"size": kw["window"], "keep_first": kw.get("keep", 0)}
    if kw.get("softcap"):
        left["softcap"] = kw["softcap"]
    if kw.get("rot_dims") is not None:
        left["rot"] = {"base": kw.get("base", 10000.0), "dims": kw["rot_dims"]}
    r_heads, r_dim, r_vdim = kw.get("right", (3, 12, 20))
    right = {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": [1.0 - 0.4 / 4.0 ** h for h in range(r_heads)]}
    ff, experts, top = kw.get("mlp", (32, 4, 2))
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {"architecture": "Vugipel", "vocab": 61, "width": kw.get("width", 48), "norm": {"eps": EPS},
            "layers": [{"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": kw.get("left_scale", 0.8),
                                                      "right_scale": kw.get("right_scale", 1.3)}, "mlp": mlp},
                       {"type": "mingru", "mixer": {"width": kw.get("mingru", 36)}, "mlp": None}]}


def random_weights(raw, seed, dtype):
    from flyweight_b200.config.vugipel import VugipelConfig
    from flyweight_b200.parts import build_arrangement
    g = torch.Generator().manual_seed(seed)
    spec = VugipelConfig.from_dict(raw).model_spec()
    w = {}
    for layer in spec.layers:
        declared = {}
        for part in build_arrangement(layer).parts():
            declared.update(part.declare())
        for name, decl in declared.items():
            t = torch.randn(decl.shape, generator=g, dtype=F64)
            if len(decl.shape) == 2:
                t = t / math.sqrt(decl.shape[1])
            elif name.endswith((".q.norm", ".k.norm", ".temp")):
                t = 1.0 + 0.2 * t
            elif name.endswith(".b"):
                t = 0.5 * t
            else:
                t = 0.1 * t
            w[name] = rounding(dtype)(t)
    return spec, w


def run_part(part_spec, w, dtype, h_seqs, cuts, n_pages=24, seed=0):
    """A mixer over several sequences fed in the portions ``cuts``; pages in shuffled order, slot = 3 - s; pages
    that nobody wrote hold NaN.  Returns the outputs by sequence."""
    from flyweight_b200.engine import StepContext
    from flyweight_b200.parts import Precision, build_mixer
    from flyweight_b200.parts.base import FixedState, PagedKV
    precision = Precision("float32" if dtype == torch.float32 else "bfloat16")
    order = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
    part = build_mixer(part_spec)
    part.bind(lambda n: w[n].to(dtype), precision, DEV)
    part.prepare(1024, DEV)
    cache = type("Cache", (), {})()
    cache.k_pool = cache.v_pool = cache.state = None
    cache.group = 0
    specs = part.state_spec()
    for one in specs if isinstance(specs, tuple) else (specs,):
        if isinstance(one, PagedKV):
            shape = (n_pages, one.n_kv_heads, 64, one.head_dim)
            cache.k_pool = torch.full(shape, float("nan"), dtype=precision.cache_dtype, device=DEV)
            cache.v_pool = torch.full(shape, float("nan"), dtype=precision.cache_dtype, device=DEV)
        elif isinstance(one, FixedState):
            cache.state = torch.zeros((4,) + tuple(one.shape), dtype=one.dtype, device=DEV)
    pages = {s: [] for s in range(len(h_seqs))}
    done = {s: 0 for s in range(len(h_seqs))}
    outs = {s: [] for s in range(len(h_seqs))}
    for step in cuts:
        for s, m in step:
            while len(pages[s]) * 64 < done[s] + m:
                pages[s].append(order.pop())
        ctx = StepContext(batch_of(step, done, lambda s: 3 - s, pages), precision, DEV)
        h = dev(torch.cat([h_seqs[s][done[s]:done[s] + m] for s, m in step]).to(precision.act_dtype))
        out = part.forward(ctx, h, cache)
        at = 0
        for s, m in step:
            outs[s].append(out[at:at + m].float().cpu())
            at += m
            done[s] += m
    return {s: torch.cat(parts) for s, parts in outs.items() if parts}


def inputs_with_partners(lengths, width, pairs, seed, dtype, strength=6.0, query_sign=-1.0):
    """Random rows; for every (sequence, key position, query position) in ``pairs`` both rows get a large share of
    one direction (the query's with ``query_sign``), so that this query's score on this key stands far out."""
    g = torch.Generator().manual_seed(seed)
    seqs = [torch.randn(n, width, generator=g, dtype=F64) for n in lengths]
    for index, (s, j, i) in enumerate(pairs):
        u = torch.randn(width, generator=torch.Generator().manual_seed(1000 + index), dtype=F64)
        seqs[s][j] += strength * u
        seqs[s][i] += query_sign * strength * u
    return [rounding(dtype)(h) for h in seqs]


def tie_queries_to_keys(w, prefix, heads, kv, dim):
    """Makes every query head's projection minus its key head's, with the key head's norm weight and no biases: a
    row that is the opposite of an earlier one then scores high on it whatever the random weights are, and every
    row scores far below zero on itself."""
    rep = heads // kv
    w[prefix + "q"] = -w[prefix + "k"].view(kv, dim, -1).repeat_interleave(rep, dim=0).reshape(heads * dim, -1).clone()
    w[prefix + "q.norm"] = w[prefix + "k.norm"].clone()
    w[prefix + "temp"] = w[prefix + "temp"].abs()
    for name in ("q.b", "k.b"):
        w[prefix + name] = torch.zeros_like(w[prefix + name])


# sequence 0: 0-99, 100-101, 102, 103-139, 140, 141, 142-199 (102, 140 and 141 are decoded alone)
CUTS = [[(0, 100), (1, 3)], [(1, 1), (0, 2), (2, 64)], [(0, 1), (1, 1), (2, 1)], [(2, 63), (0, 37), (1, 60)],
        [(0, 1), (2, 2)], [(0, 1)], [(0, 58), (1, 70)]]
LENGTHS = [200, 135, 130]
SINGLE = {(0, 102), (0, 140), (0, 141), (1, 3), (1, 4), (2, 64)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep,heads,kv,dim,vdim,rot_dims,softcap", [
    (37, 5, 4, 2, 16, 24, None, 0.0), (40, 1, 4, 2, 16, 24, 0, 25.0), (64, 64, 2, 2, 32, 32, None, 0.0),
    (10, 70, 3, 1, 24, 16, 0, 0.0), (1, 3, 4, 1, 16, 16, None, 30.0), (50, 4, 8, 2, 64, 64, None, 0.0),
    (33, 66, 4, 1, 64, 128, 0, 40.0), (70, 2, 4, 1, 128, 128, None, 0.0), (90, 0, 6, 2, 32, 48, 0, 0.0)])
def test_a_window_with_kept_first_tokens_shows_its_edges(dtype, window, keep, heads, kv, dim, vdim, rot_dims, softcap):
    """The whole mixer pair over three sequences in portions and single tokens.  Keys stand out just inside and just
    outside the window and among the first tokens (the last kept one and the next); the plain result with the window
    or the kept run one longer or shorter must differ by far more than the tolerance wherever it changes what a
    query sees, in portions and for tokens decoded alone."""
    raw = tiny_config(window=window, keep=keep, heads=heads, kv=kv, dim=dim, vdim=vdim, rot_dims=rot_dims, softcap=softcap,
                      scale=10.0 / dim, width=48 if dim < 64 else 128)
    spec, w = random_weights(raw, 3, dtype)
    tie_queries_to_keys(w, "l0.mix.left.", heads, kv, dim)
    m = raw["layers"][0]["mixer"]["left"]
    pairs = []
    queries = [(0, 102), (0, 140), (0, 141), (0, 150), (0, 111), (0, 199), (2, 64), (2, 110), (2, 120)]
    offsets = [window - 1, window, None, None, window - 1, window, window, window - 1, None]
    firsts = [None, None, keep - 1, keep, None, None, None, None, keep - 1]
    taken = set()
    for (s, i), off, j in zip(queries, offsets, firsts):
        j = i - off if off is not None else j
        if 0 <= j < i and (s, j) not in taken and (s, i) not in taken:
            pairs.append((s, j, i))
            taken |= {(s, j), (s, i)}
    seqs = inputs_with_partners(LENGTHS, raw["width"], pairs, 7, dtype)
    rnd = rounding(dtype)
    got = run_part(spec.layers[0].parts["mixer"], w, dtype, seqs, CUTS)
    mixer = raw["layers"][0]["mixer"]
    changed, shown = set(), set()
    for s, h in enumerate(seqs):
        pos = torch.arange(h.shape[0])
        want = P.parallel_mixer(h, w, "l0.mix.", mixer, EPS, pos, rnd=rnd)
        close(got[s], want, TOL[dtype], f"sequence {s}")
        for key, delta in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1)):
            mask = dict(m["mask"])
            mask[key] += delta
            if mask["size"] < 1 or mask["keep_first"] < 0:
                continue
            off = P.parallel_mixer(h, w, "l0.mix.", {**mixer, "left": {**m, "mask": mask}}, EPS, pos, rnd=rnd)
            differs = P.visible(pos, pos, **m["mask"]) != P.visible(pos, pos, **mask)
            for q, j, i in pairs:
                if q == s and differs[i, j]:
                    changed.add((key, delta, s, i))
                    if (off[i] - want[i]).abs().max() > SHOWS * max(1.0, want.abs().max()):
                        shown.add((key, delta, s, i))
    assert changed and shown == changed, f"an edge that is one off must show wherever it changes what a query sees: {changed - shown}"
    assert {(s, i) in SINGLE for _, _, s, i in shown} == {True, False}     # decoded alone, and in a portion
    if keep > 0 and window + keep < 140:
        assert {key for key, _, _, _ in shown} == {"size", "keep_first"}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [
    dict(window=37, keep=5, rot_dims=8, softcap=2.0, scale=0.8), dict(rot_dims=16, scale=0.5), dict(window=20, keep=2, rot_dims=0),
    dict(heads=3, kv=3, dim=20, vdim=12, rot_dims=20, softcap=1.0, scale=0.6), dict(heads=8, kv=2, dim=64, vdim=64, rot_dims=32, window=130, keep=70, width=128),
    dict(heads=4, kv=1, dim=128, vdim=128, rot_dims=128, window=70, keep=3, width=128, softcap=3.0),
    dict(heads=2, kv=2, dim=40, vdim=88, rot_dims=30, window=100, keep=0), dict(heads=2, kv=1, dim=160, vdim=40, rot_dims=64, window=64, keep=8),
    dict(right=(5, 33, 17)), dict(right=(1, 64, 64), left_scale=-0.4, right_scale=0.0), dict(right=(2, 130, 40), left_scale=1.0, right_scale=1.0)])
def test_the_pair_of_attention_and_retention(dtype, kw):
    """Biases, norm per head, rotation of keys and of values (all, some and none of the key channels), the factor per
    head, the cap, and the retention's state over portions and single tokens; each of them is felt."""
    raw = tiny_config(**kw)
    spec, w = random_weights(raw, 5, dtype)
    mixer = raw["layers"][0]["mixer"]
    seqs = inputs_with_partners(LENGTHS, raw["width"], [], 9, dtype)
    rnd = rounding(dtype)
    got = run_part(spec.layers[0].parts["mixer"], w, dtype, seqs, CUTS, seed=2)
    for s, h in enumerate(seqs):
        pos = torch.arange(h.shape[0])
        want = P.parallel_mixer(h, w, "l0.mix.", mixer, EPS, pos, rnd=rnd)
        close(got[s], want, TOL[dtype], f"sequence {s}")
    h, pos = seqs[0], torch.arange(LENGTHS[0])
    base = P.parallel_mixer(h, w, "l0.mix.", mixer, EPS, pos, rnd=rnd)

    def felt(weights, m, what):
        other = P.parallel_mixer(h, weights, "l0.mix.", m, EPS, pos, rnd=rnd)
        assert (other - base).abs().max() > SHOWS * max(1.0, float(base.abs().max())), what

    for name in ("q.b", "k.b", "v.b", "o.b", "temp"):
        changed = dict(w)
        changed["l0.mix.left." + name] = torch.ones_like(w["l0.mix.left." + name]) if name == "temp" else 0.0 * w["l0.mix.left." + name]
        felt(changed, mixer, name)
    if kw.get("softcap"):
        felt(w, {**mixer, "left": {k: v for k, v in mixer["left"].items() if k != "softcap"}}, "softcap")
    if mixer["right_scale"]:
        felt(w, {**mixer, "right": {**mixer["right"], "decay": [0.5 * d for d in mixer["right"]["decay"]]}}, "decay")
    felt(w, {**mixer, "right_scale": mixer["right_scale"] + 0.5}, "right_scale")


def test_rotated_values_are_felt_and_turned_back():
    """With one visible key at the query's own position turning and turning back cancel; with a key far back they do
    not, and the engine follows (a value that was not turned, or not turned back, would show)."""
    raw = tiny_config(window=5, keep=1, rot_dims=0, scale=2.0, vdim=16, dim=16, base=3.0, right_scale=0.0)
    dtype = torch.float32
    spec, w = random_weights(raw, 8, dtype)
    tie_queries_to_keys(w, "l0.mix.left.", 4, 2, 16)
    seqs = inputs_with_partners(LENGTHS, raw["width"], [(0, 0, 150), (0, 101, 102)], 4, dtype)
    mixer = raw["layers"][0]["mixer"]
    got = run_part(spec.layers[0].parts["mixer"], w, dtype, seqs, CUTS)
    pos = torch.arange(LENGTHS[0])
    want = P.parallel_mixer(seqs[0], w, "l0.mix.", mixer, EPS, pos)
    close(got[0], want, TOL[dtype])
    still = P.parallel_mixer(seqs[0], w, "l0.mix.", {**mixer, "left": {k: v for k, v in mixer["left"].items() if k != "rot"}}, EPS, pos)
    for i in (102, 150):
        assert (still[i] - want[i]).abs().max() > SHOWS * float(want.abs().max())
    assert (still[0] - want[0]).abs().max() < 1e-9           # (position 0 sees itself only)


def test_a_pair_that_cannot_join_adds_its_scaled_halves():
    """The general form: an attention with an output gate beside a lightning attention, each part run alone."""
    from flyweight_b200.config.spec import PartSpec
    W = 32
    left = PartSpec("gqa_attention", {"hidden_size": W, "num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "qk_norm_eps": EPS,
                                      "position": PartSpec("rope", {"theta": 100.0, "rotary_dim": 8}), "gate": "head"},
                    {n: "a." + n for n in ("q", "k", "v", "o", "q_norm", "k_norm", "g")})
    right = PartSpec("decayed_linear_attention", {"hidden_size": W, "num_heads": 2, "dim": 8, "vdim": 8, "decay": (0.9, 0.99), "eps": EPS},
                     {n: "b." + n for n in ("q", "k", "v", "g", "norm", "o")})
    pair = PartSpec("mixer_pair", {"hidden_size": W, "combine": "scaled", "left_scale": 0.25, "right_scale": -1.5, "left": left,
                                   "right": right})
    g = torch.Generator().manual_seed(2)
    shapes = {"a.q": (32, W), "a.k": (16, W), "a.v": (16, W), "a.o": (W, 32), "a.q_norm": (16,), "a.k_norm": (16,), "a.g": (2, W),
              "b.q": (16, W), "b.k": (16, W), "b.v": (16, W), "b.g": (16, W), "b.norm": (16,), "b.o": (W, 16)}
    w = {n: (torch.randn(s, generator=g, dtype=F64) / math.sqrt(s[-1])).float().to(F64) for n, s in shapes.items()}
    seqs = inputs_with_partners(LENGTHS, W, [], 3, torch.float32)
    both, a, b = (run_part(spec, w, torch.float32, seqs, CUTS) for spec in (pair, left, right))
    for s in both:
        close(both[s], 0.25 * a[s].to(F64) - 1.5 * b[s].to(F64), 1e-5)


def test_an_attention_with_the_new_options_alone():
    """The same attention outside a pair: the bias rides on the output product, heads leave unscaled."""
    from flyweight_b200.config.vugipel import VugipelConfig
    for dtype in DTYPES:
        raw = tiny_config(window=37, keep=5, rot_dims=8, softcap=4.0)
        _, w = random_weights(raw, 6, dtype)
        spec = VugipelConfig.from_dict(raw).model_spec().layers[0].parts["mixer"].params["left"]
        seqs = inputs_with_partners(LENGTHS, raw["width"], [], 5, dtype)
        got = run_part(spec, w, dtype, seqs, CUTS)
        for s, h in enumerate(seqs):
            want = P.turned_attention(h, w, "l0.mix.left.", raw["layers"][0]["mixer"]["left"], EPS, torch.arange(h.shape[0]),
                                      rnd=rounding(dtype))
            close(got[s], want, TOL[dtype], f"sequence {s}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("right", [(3, 12, 20), (2, 64, 64), (5, 33, 17), (1, 256, 8), (2, 300, 12)])
def test_retention_alone(dtype, right):
    """The recurrence without an activation, keys scaled, a norm per head and a silu gate, over portions and single
    tokens (the token-by-token kernel, the tensor-core one, and states too tall for the latter); the norm's eps is
    large enough to be felt, so a key scale that is missing would show."""
    from flyweight_b200.config.spec import PartSpec
    H, d, e = right
    W, eps = 48, 0.05
    m = {"heads": H, "dim": d, "vdim": e, "decay": [0.7 + 0.29 * h / max(H - 1, 1) for h in range(H)]}
    spec = PartSpec("decayed_linear_attention", {"hidden_size": W, "num_heads": H, "dim": d, "vdim": e, "decay": m["decay"],
                                                 "eps": eps, "activation": None, "k_scale": d ** -0.5, "norm": "head", "gate": "silu"},
                    {n: "r." + n for n in ("q", "k", "v", "g", "o")})
    g = torch.Generator().manual_seed(d)
    shapes = {"q": (H * d, W), "k": (H * d, W), "v": (H * e, W), "g": (H * e, W), "o": (W, H * e)}
    w = {"r." + n: rounding(dtype)(torch.randn(s, generator=g, dtype=F64) / math.sqrt(s[-1])) for n, s in shapes.items()}
    seqs = inputs_with_partners(LENGTHS, W, [], 13, dtype)
    got = run_part(spec, w, dtype, seqs, CUTS)
    for s, h in enumerate(seqs):
        close(got[s], P.retention(h, w, "r.", m, eps, rnd=rounding(dtype)), TOL[dtype], f"sequence {s}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mingru,width", [(36, 48), (33, 40), (7, 24), (256, 64), (130, 100)])
def test_the_mingru_mixer(dtype, mingru, width):
    """Projections, biases, recurrence and output together (widths that the products' tiles take and that they do
    not), and the biases are felt."""
    raw = tiny_config(mingru=mingru, width=width)
    spec, w = random_weights(raw, 4, dtype)
    seqs = inputs_with_partners(LENGTHS, width, [], 6, dtype)
    got = run_part(spec.layers[1].parts["mixer"], w, dtype, seqs, CUTS)
    for s, h in enumerate(seqs):
        want = P.mingru_mixer(h, w, "l1.mix.", rnd=rounding(dtype))
        close(got[s], want, TOL[dtype], f"sequence {s}")
    for name in ("z.b", "x.b"):
        changed = dict(w)
        changed["l1.mix." + name] = 0.0 * w["l1.mix." + name]
        assert (P.mingru_mixer(seqs[0], changed, "l1.mix.") - P.mingru_mixer(seqs[0], w, "l1.mix.")).abs().max() > SHOWS


# ------------------------------------------------------------------ the router and the experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,N,top", [(1, 48, 4, 1), (65, 80, 7, 3), (8, 1024, 32, 8), (300, 512, 5, 5), (300, 2048, 64, 6), (9, 50, 3, 2),
                                       (1000, 768, 16, 4)])
def test_sigmoid_router(dtype, T, W, N, top):
    """Scores of each output on its own, no correction, the largest chosen, weights not renormalised; the softmax of
    the same rows gives other weights, and a correction still moves the choice but not the weights."""
    from flyweight_b200.kernels import experts
    g = torch.Generator().manual_seed(N + top)
    h = rounding(dtype)(torch.randn(T, W, generator=g, dtype=F64))
    router = (2.0 * torch.randn(N, W, generator=g, dtype=F64) / math.sqrt(W)).float().to(F64)
    ids, weights = experts.route(dev(h, dtype), dev(router, torch.float32), None, 1, 1, top, "sigmoid")
    scores = torch.sigmoid(h @ router.T)
    ranked = scores.sort(dim=1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == N else (ranked[:, top - 1] - ranked[:, top] > 1e-5)
    assert clear.float().mean() > 0.9
    want_ids, want = P.sigmoid_choice(h, router, top)
    got_ids = ids.cpu().long()
    assert (got_ids.sort(dim=1).values == want_ids.sort(dim=1).values)[clear].all()
    close(weights.cpu().to(F64), torch.gather(scores, 1, got_ids), 1e-5)
    close(weights.cpu()[clear], want[clear], 1e-5)
    soft = experts.route(dev(h, dtype), dev(router, torch.float32), torch.zeros(N, device=DEV), 1, 1, top)[1]
    close(soft, torch.gather(torch.softmax(h @ router.T, dim=1), 1, got_ids), 1e-5)
    correction = torch.linspace(9.0, 0.0, N)
    ids, weights = experts.route(dev(h, dtype), dev(router, torch.float32), dev(correction), 1, 1, top, "sigmoid")
    assert (ids.cpu().sort(dim=1).values == torch.arange(top)[None]).all() or N > 10
    close(weights, torch.gather(scores, 1, ids.cpu().long()), 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tensor_cores", [True, False])
@pytest.mark.parametrize("T,W,F,E,top", [(1, 48, 32, 4, 1), (90, 64, 64, 6, 2), (33, 40, 16, 3, 3), (300, 128, 96, 9, 4), (20, 36, 20, 5, 2),
                                         (700, 64, 40, 2, 1)])
def test_experts_whose_inputs_are_weighted(dtype, tensor_cores, T, W, F, E, top):
    """sum of expert(w h): not the same as the weighted sum of expert(h), which the other setting still gives."""
    from flyweight_b200.kernels import experts
    g = torch.Generator().manual_seed(T + E)
    rnd = rounding(dtype)
    h = rnd(2.0 * torch.randn(T, W, generator=g, dtype=F64))
    w = {}
    for j in range(E):
        w[f"e{j}.gate"], w[f"e{j}.up"] = (rnd(torch.randn(F, W, generator=g, dtype=F64) / math.sqrt(W)) for _ in range(2))
        w[f"e{j}.down"] = rnd(torch.randn(W, F, generator=g, dtype=F64) / math.sqrt(F))
    ids = torch.rand(T, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32)
    weights = torch.rand(T, top, generator=g, dtype=F64).float().to(F64)
    gate_up = torch.stack([torch.cat([w[f"e{j}.gate"], w[f"e{j}.up"]]) for j in range(E)])
    down = torch.stack([w[f"e{j}.down"] for j in range(E)])
    before = experts._use_tensor_cores
    experts.set_tensor_cores(tensor_cores)
    try:
        got = {on: experts.experts_forward(dev(h, dtype), dev(ids), dev(weights, torch.float32), dev(gate_up, dtype), dev(down, dtype),
                                           weights_on=on) for on in ("input", "output")}
    finally:
        experts.set_tensor_cores(before)
    want = {"input": torch.zeros(T, W, dtype=F64), "output": torch.zeros(T, W, dtype=F64)}
    for t in range(T):
        for slot in range(top):
            p, s = f"e{int(ids[t, slot])}.", float(weights[t, slot])
            for on, x, out in (("input", rnd(h[t] * s), 1.0), ("output", h[t], s)):
                want[on][t] += out * (w[p + "down"] @ rnd(P.silu(w[p + "gate"] @ x) * (w[p + "up"] @ x)))
    for on in want:
        close(got[on], want[on], 1e-5 if dtype == torch.float32 else 2e-2, on)
    assert (want["input"] - want["output"]).abs().max() > SHOWS * want["output"].abs().max()


@pytest.mark.parametrize("T,W,N,top,groups,keep", [(256, 512, 32, 8, 1, 1), (700, 1024, 12, 3, 4, 2), (2049, 256, 5, 5, 1, 1), (300, 2048, 100, 1, 1, 1)])
@pytest.mark.parametrize("scores", ["sigmoid", "softmax"])
def test_the_router_as_a_matrix_product_chooses_alike(T, W, N, top, groups, keep, scores):
    """bfloat16 rows of a prompt through the tensor-core product and the choosing kernel, against the kernel that does
    both in fp32; where a choice is no close call it must be the same."""
    from flyweight_b200.kernels import experts
    g = torch.Generator().manual_seed(N)
    h = torch.randn(T, W, generator=g).to(torch.bfloat16).to(DEV)
    router16 = (2.0 * torch.randn(N, W, generator=g) / math.sqrt(W)).to(torch.bfloat16).to(DEV)
    correction = (0.1 * torch.randn(N, generator=g)).to(DEV)
    one = experts.route(h, router16.float(), correction, groups, keep, top, scores)
    two = experts.route(h, router16.float(), correction, groups, keep, top, scores, router16=router16)
    same = (one[0] == two[0]).all(dim=1)
    assert same.float().mean() > 0.99
    close(two[1][same], one[1][same], 1e-5)


@pytest.mark.parametrize("A,top,E", [(1, 1, 1), (130, 2, 7), (1024, 4, 40), (1025, 5, 3), (17000, 4, 33), (40000, 8, 70)])
@pytest.mark.parametrize("tile_rows", [16, 64])
def test_pairs_are_sorted_by_expert(A, top, E, tile_rows):
    """Every pair of a real expert gets one row among its expert's, the tiles cover the rows once and never two experts;
    outputs from E on (identity experts) get no row."""
    from flyweight_b200.kernels import lib
    from flyweight_b200.kernels.lib import ptr, stream
    g = torch.Generator().manual_seed(A)
    ids = torch.randint(0, E + 1, (A,), generator=g).to(torch.int32)
    weights = torch.rand(A, generator=g)
    most = A // tile_rows + E + 1
    offsets, row_token, pair_row, tiles = (torch.full((n,), -7, dtype=torch.int32, device=DEV) for n in (E + 1, A, A, 1 + 2 * most))
    row_weight = torch.full((A,), -7.0, device=DEV)
    ids_d, weights_d = dev(ids), dev(weights)
    lib.call("fwb_moe_sort", ptr(ids_d), A, top, E, tile_rows, ptr(offsets), ptr(row_token), ptr(pair_row), ptr(tiles),
             ptr(weights_d), ptr(row_weight), stream())
    counts = torch.bincount(ids.long(), minlength=E + 1)[:E]
    starts = torch.cat([torch.zeros(1, dtype=torch.long), counts.cumsum(0)])
    assert offsets.cpu().long().tolist() == starts.tolist()
    rows, total = pair_row.cpu().long(), int(starts[-1])
    real = ids < E
    assert (rows[~real] == -1).all() and sorted(rows[real].tolist()) == list(range(total))
    expert_of_row = torch.repeat_interleave(torch.arange(E), counts)
    assert (expert_of_row[rows[real]] == ids[real].long()).all()
    pairs = torch.arange(A)[real]
    assert (row_token.cpu().long()[rows[real]] == pairs // top).all() and (row_weight.cpu()[rows[real]] == weights[real]).all()
    n = int(tiles[0])
    listed = tiles[1:1 + 2 * n].cpu().view(n, 2).tolist()
    assert listed == [[e, int(starts[e]) + r] for e in range(E) for r in range(0, int(counts[e]), tile_rows)] and n <= most
