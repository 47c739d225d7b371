"""The mechanisms Futezen brought to the engine, each alone: the kernel (or the part) against the function of
``plain_futezen`` that states the same mechanism, on hand-made batches whose segments start at position 0, in the
middle of a sequence and on single tokens, over shuffled pages and slots.  Where random numbers would hide a fault
(a token far back in a state or a cache, a norm over the wrong run of channels, a bias that never decides) the inputs
are made so that it shows."""
import math

import pytest
import torch

import plain_futezen as P

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
F64 = torch.float64
EPS = 1e-5
TOL = {torch.float32: 2e-4, torch.bfloat16: 4e-2}
SHOWS = 20 * TOL[torch.float32]     # what a fault has to change in the plain result for the inputs to count as telling


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


def f32_round(t):
    return t.to(torch.float32).to(F64)


def rounding(dtype):
    return bf16_round if dtype == torch.bfloat16 else f32_round


def step_batch(step, slots, done):
    from flyweight_b200.engine import Segment, StepBatch
    return StepBatch([Segment(f"s{s}", slots[s], done[s], [0] * m, []) for s, m in step], [[[0]] * len(step)], DEV)


# ------------------------------------------------------------------ the recurrence
# portions shorter and longer than a run of 64 tokens, than a piece, single tokens alone and beside portions
STATE_CUTS = [[(0, 9), (1, 1), (2, 70)], [(1, 1), (0, 2), (3, 2)], [(0, 1), (1, 1), (2, 1), (3, 1)],
              [(1, 1), (3, 300), (0, 3), (2, 16)], [(1, 2), (3, 1), (0, 1)], [(2, 1), (0, 64), (1, 15)], [(3, 17), (2, 63), (0, 1)]]
SIZES = [(6, 3, 12, 10), (4, 1, 33, 7), (8, 1, 128, 64), (6, 3, 200, 80), (2, 2, 8, 130), (40, 1, 16, 16)]


def scan_inputs(heads, groups, n, e, lengths, seed, rnd):
    """x, b, c, raw step sizes of several sequences; decay rates from one that forgets within a token to one that
    remembers the whole sequence."""
    g = torch.Generator().manual_seed(seed)
    seqs = []
    for length in lengths:
        u = rnd(torch.randn(length, heads * e + 2 * groups * n, generator=g, dtype=F64) / math.sqrt(n))
        u[:, :heads * e] = rnd(u[:, :heads * e] * math.sqrt(n))
        seqs.append((u, f32_round(torch.randn(length, heads, generator=g, dtype=F64) - 1.0)))
    a_log = f32_round(torch.linspace(-7.0, 1.5, heads, dtype=F64))
    bias = f32_round(0.3 * torch.randn(heads, generator=g, dtype=F64))
    skip = f32_round(torch.randn(heads, generator=g, dtype=F64))
    return seqs, a_log, bias, skip


def plain_scan(u, raw, a_log, bias, skip, heads, groups, n, e):
    T = u.shape[0]
    x, b, c = u[:, :heads * e], u[:, heads * e:heads * e + groups * n], u[:, heads * e + groups * n:]
    y, S = P.scalar_decay_scan(x.reshape(T, heads, e), b.reshape(T, groups, n), c.reshape(T, groups, n),
                               P.softplus(raw + bias), torch.exp(a_log), skip)
    return y.reshape(T, heads * e), S


@pytest.mark.parametrize("form", ["scan fp32", "scan bf16", "chosen", "runs"])
@pytest.mark.parametrize("heads,groups,n,e", SIZES)
def test_state_space_over_portions_single_tokens_and_shuffled_slots(form, heads, groups, n, e):
    """Four sequences in shuffled slots; a fifth slot nobody owns must stay as it was, and the states at the end are
    the sequences' own."""
    from flyweight_b200.kernels import state_space as K
    dtype = torch.float32 if form == "scan fp32" else torch.bfloat16
    runs = {"scan fp32": None, "scan bf16": False, "chosen": None, "runs": True}[form]
    lengths = [sum(m for step in STATE_CUTS for s, m in step if s == q) for q in range(4)]
    seqs, a_log, bias, skip = scan_inputs(heads, groups, n, e, lengths, heads + n, rounding(dtype))
    slots = [2, 0, 3, 1]
    size = -(-heads * n * e // 4) * 4
    state = torch.zeros((5, size + 8), dtype=torch.float32, device=DEV)
    state[4] = float("nan")
    done, got = [0] * 4, [[] for _ in range(4)]
    for step in STATE_CUTS:
        batch = step_batch(step, slots, done)
        u = dev(torch.cat([seqs[s][0][done[s]:done[s] + m] for s, m in step]), dtype)
        raw = torch.cat([seqs[s][1][done[s]:done[s] + m] for s, m in step])
        p = dev(torch.cat([torch.full((raw.shape[0], 3), 7.0), raw.float(), torch.full((raw.shape[0], 1), 7.0)], dim=1))
        y = K.state_space(u, p, 3, dev(bias.float()), dev(a_log.float()), dev(skip.float()), state, batch, heads, groups,
                          n, e, runs=runs)
        at = 0
        for s, m in step:
            got[s].append(y[at:at + m].cpu())
            at += m
            done[s] += m
    tol = 5e-5 if form.startswith("scan") else 5e-4        # (runs: fp32 quantities in two bfloat16 halves)
    for s in range(4):
        want, S = plain_scan(*seqs[s], a_log, bias, skip, heads, groups, n, e)
        close(torch.cat(got[s]), want, tol, f"sequence {s}")
        close(state[slots[s], :heads * n * e].cpu().view(heads, n, e), S, tol, f"state of sequence {s}")
    assert torch.isnan(state[4]).all() and (state[:4, heads * n * e:] == 0).all()


@pytest.mark.parametrize("length,alone", [(1500, 0), (1500, 3), (700, 40)])
def test_a_token_far_back_in_the_state(length, alone):
    """One token writes in a direction only the last tokens read, 700 to 1,500 tokens later: a lost piece, a state
    handed on wrongly or a total decay that is off shows, in a portion and in tokens decoded behind it."""
    from flyweight_b200.kernels import state_space as K
    heads, groups, n, e = 4, 2, 32, 64
    seqs, a_log, bias, skip = scan_inputs(heads, groups, n, e, [length], 5, bf16_round)
    a_log = torch.full((heads,), -9.0, dtype=F64)
    u, raw = seqs[0]
    b = u[:, heads * e:heads * e + groups * n].view(length, groups, n)
    c = u[:, heads * e + groups * n:].view(length, groups, n)
    b[:, :, 0] = 0.0
    c[:, :, 0] = 0.0
    b[3, :, 0] = 8.0
    c[-20:, :, 0] = 8.0
    raw[3] = 3.0
    want, _ = plain_scan(u, raw, a_log, bias, skip, heads, groups, n, e)
    without = u.clone()
    without[3, :heads * e] = 0.0
    lost, _ = plain_scan(without, raw, a_log, bias, skip, heads, groups, n, e)
    assert ((lost - want)[-20:].abs().amax(dim=1) > 20.0).all()
    state = torch.zeros((1, heads * n * e), dtype=torch.float32, device=DEV)
    got, done = [], [0]
    for m in [length - alone] + [1] * alone:
        batch = step_batch([(0, m)], [0], done)
        y = K.state_space(dev(u[done[0]:done[0] + m], torch.bfloat16), dev(raw[done[0]:done[0] + m].float()), 0,
                          dev(bias.float()), dev(a_log.float()), dev(skip.float()), state, batch, heads, groups, n, e)
        got.append(y.cpu())
        done[0] += m
    close(torch.cat(got), want, 1e-3, "far token")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,groups", [(60, 1), (60, 6), (4096, 8), (4096, 1), (21, 3), (1032, 2)])
def test_gate_then_norm_over_runs_of_channels(dtype, width, groups):
    from flyweight_b200.kernels import state_space as K
    g = torch.Generator().manual_seed(width + groups)
    y = f32_round(torch.randn(19, width, generator=g, dtype=F64))
    y *= torch.linspace(0.05, 3.0, width, dtype=F64)          # (runs of different size: one mean for all would show)
    y = f32_round(y)
    p = f32_round(torch.randn(19, width + 5, generator=g, dtype=F64))
    w = f32_round(1.0 + 0.3 * torch.randn(width, generator=g, dtype=F64))
    out = K.gate_group_norm(dev(y.float()), dev(p.float()), 4, dev(w.float()), groups, EPS, dtype)
    want = P.gated_group_norm(y, p[:, 4:4 + width], w, groups, EPS)
    close(out.float(), want, 1e-5 if dtype == torch.float32 else 1e-2, "gated norm")
    if groups > 1:
        assert (P.gated_group_norm(y, p[:, 4:4 + width], w, 1, EPS) - want).abs().max() > 0.1


CONV_CUTS = [[(0, 9), (1, 1), (2, 70)], [(1, 1), (0, 2)], [(0, 1), (1, 1), (2, 1)], [(2, 130), (0, 3)], [(1, 2), (0, 64)]]


@pytest.mark.parametrize("dtypes", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16),
                                    (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("channels,taps,col0,behind", [(24, 3, 8, 4), (7, 4, 5, 3), (512, 4, 256, 8), (33, 1, 0, 1), (300, 5, 12, 0)])
def test_convolution_with_bias_and_silu_on_columns_of_a_projection(dtypes, channels, taps, col0, behind):
    from flyweight_b200.kernels import mixing
    g = torch.Generator().manual_seed(channels + taps)
    lengths = [sum(m for step in CONV_CUTS for s, m in step if s == q) for q in range(3)]
    rows = [rounding(dtypes[0])(torch.randn(n, col0 + channels + behind, generator=g, dtype=F64)) for n in lengths]
    w = f32_round(torch.randn(channels, taps, generator=g, dtype=F64))
    bias = f32_round(torch.randn(channels, generator=g, dtype=F64))
    slots = [2, 0, 1]
    state = torch.zeros((3, taps - 1, channels), dtype=torch.float32, device=DEV) if taps > 1 else None
    done, got = [0] * 3, [[] for _ in range(3)]
    for step in CONV_CUTS:
        batch = step_batch(step, slots, done)
        u = dev(torch.cat([rows[s][done[s]:done[s] + m] for s, m in step]), dtypes[0])
        y = mixing.causal_conv(u, dev(w.float()), state, batch, col0=col0, bias=dev(bias.float()), silu=True,
                               out_dtype=dtypes[1])
        assert y.dtype == dtypes[1]
        at = 0
        for s, m in step:
            got[s].append(y[at:at + m].float().cpu())
            at += m
            done[s] += m
    for s in range(3):
        want = P.silu(P.causal_taps(rows[s][:, col0:col0 + channels], w, bias))
        close(torch.cat(got[s]), want, 1e-5 if dtypes[1] == torch.float32 else 1e-2, f"sequence {s}")
        if taps > 1:
            close(state[slots[s]].cpu(), rows[s][-(taps - 1):, col0:col0 + channels], 1e-6, f"state of sequence {s}")


# ------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("tokens", [1, 5, 64, 200, 300])
@pytest.mark.parametrize("experts,top,width,gate", [(12, 3, 512, True), (5, 5, 80, True), (7, 1, 96, False), (40, 8, 1024, True)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_router_with_softmax_over_the_chosen_and_a_row_for_the_shared_expert(tokens, experts, top, width, gate, dtype):
    """The kernel with its own product and, from 256 bfloat16 tokens on, the tensor-core product with the choice
    behind it.  The bias decides some choices and enters the weights; a softmax over all outputs is another one."""
    from flyweight_b200.kernels import experts as K
    g = torch.Generator().manual_seed(experts * tokens + top)
    h = rounding(dtype)(torch.randn(tokens, width, generator=g, dtype=F64))
    router = bf16_round(torch.randn(experts, width, generator=g, dtype=F64) / math.sqrt(width))
    row = bf16_round(torch.randn(1, width, generator=g, dtype=F64) / math.sqrt(width))
    bias = f32_round(torch.randn(experts, generator=g, dtype=F64))
    logits = h @ router.T + bias
    ids, weights = P.chosen_experts(logits, top)
    stacked = torch.cat([router, row]) if gate else router
    got = K.route(dev(h, dtype), dev(stacked.float()), dev(bias.float()), 1, 1, top, "softmax_chosen",
                  dev(stacked, torch.bfloat16) if dtype == torch.bfloat16 else None, gate=gate)
    ordered = logits.sort(dim=1, descending=True).values
    clear = torch.ones(tokens, dtype=torch.bool)
    if experts > 1:
        clear = (ordered[:, :-1] - ordered[:, 1:])[:, :top].min(dim=1).values > 1e-4 if top < experts else \
            (ordered[:, :-1] - ordered[:, 1:]).min(dim=1).values > 1e-4
    assert clear.float().mean() > 0.9
    assert torch.equal(got[0].cpu().long()[clear], ids[clear])
    close(got[1].cpu()[clear], weights[clear], 1e-4, "weights")
    if gate:
        close(got[2].cpu(), torch.sigmoid(h @ row.T)[:, 0], 1e-5, "shared gate")
    else:
        assert len(got) == 2
    if tokens > 60 and top < experts:
        assert not torch.equal(P.chosen_experts(h @ router.T, top)[0], ids)
        assert (torch.gather(torch.softmax(logits, dim=1), 1, ids) - weights).abs().max() > 0.05


def expert_part(seed, dtype, width, ff, experts, top, shared):
    from flyweight_b200.config.futezen import FutezenConfig
    from flyweight_b200.parts import Precision, build_feed_forward
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    mixer = {"heads": 1, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 1.0, "rot": {"base": 10.0, "dims": 0}}
    raw = {"vocab": 8, "width": width, "norm": {"eps": EPS}, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}]}
    part = build_feed_forward(FutezenConfig.from_dict(raw).model_spec().layers[0].parts["feed_forward"])
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, decl in part.declare().items():
        t = torch.randn(decl.shape, generator=g, dtype=F64)
        if name.endswith("router"):
            t = 4.0 * t                                # (choices far apart)
        w[name] = rounding(dtype)(t / math.sqrt(decl.shape[-1]) if len(decl.shape) == 2 else t)
    part.bind(lambda n: w[n].to(dtype), Precision("float32" if dtype == torch.float32 else "bfloat16"), DEV)
    return part, w, mlp


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,experts,top,shared", [(64, 48, 6, 2, 32), (80, 20, 3, 3, 24), (96, 12, 5, 1, 0), (128, 256, 8, 4, 520)])
@pytest.mark.parametrize("tokens", [1, 9, 130, 400])
def test_experts_without_a_gate_beside_a_scaled_shared_one(dtype, width, ff, experts, top, shared, tokens):
    from flyweight_b200.engine import StepContext
    from flyweight_b200.kernels import experts as K
    from flyweight_b200.parts import Precision
    part, w, mlp = expert_part(width + ff, dtype, width, ff, experts, top, shared)
    rnd = rounding(dtype)
    g = torch.Generator().manual_seed(tokens)
    h = rnd(torch.randn(tokens, width, generator=g, dtype=F64))
    logits = h @ w["l0.mlp.router"].T + w["l0.mlp.router.b"]
    ordered = logits.sort(dim=1, descending=True).values
    clear = torch.ones(tokens, dtype=torch.bool) if top == experts else ordered[:, top - 1] - ordered[:, top] > 1e-3
    want = P.routed_experts(h, w, "l0.mlp.", mlp, rnd=rnd)
    ctx = StepContext(step_batch([(0, tokens)], [0], [0]), Precision("float32" if dtype == torch.float32 else "bfloat16"), DEV)
    x = torch.randn(tokens, width, generator=g, dtype=F64).float()
    weight = (1.0 + 0.2 * torch.randn(width, generator=g, dtype=F64)).float()
    for tensor_cores in (True, False):
        K.set_tensor_cores(tensor_cores)
        try:
            close(part.forward(ctx, dev(h, dtype)).cpu()[clear], want[clear], TOL[dtype] / 4, f"sum, tensor cores {tensor_cores}")
            stream = dev(x.clone())
            part.forward_add_normed(ctx, dev(h, dtype), stream, dev(weight), EPS)
            close(stream.cpu()[clear], (x.to(F64) + weight.to(F64) * P.unit(want, EPS))[clear], TOL[dtype], "added")
        finally:
            K.set_tensor_cores(True)
    if shared:
        half = dict(mlp)
        half.pop("shared")
        assert (P.routed_experts(h, w, "l0.mlp.", half, rnd=rnd) - want).abs().max() > SHOWS


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens", [1, 17, 64, 100, 300, 700])
@pytest.mark.parametrize("width,ff", [(64, 40), (128, 384), (96, 1100)])
def test_relu_gate_and_squared_relu_in_the_products(dtype, tokens, width, ff):
    """The dense feed-forward with relu on its gate, and the product whose output leaves through the square of relu,
    at token counts that take every tile and the CTA pairs."""
    from flyweight_b200.config.spec import PartSpec
    from flyweight_b200.engine import StepContext
    from flyweight_b200.kernels import ops
    from flyweight_b200.parts import Precision, build_feed_forward
    rnd = rounding(dtype)
    g = torch.Generator().manual_seed(tokens + ff)
    h = rnd(torch.randn(tokens, width, generator=g, dtype=F64))
    w = {name: rnd(torch.randn(shape, generator=g, dtype=F64) / math.sqrt(shape[1]))
         for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    part = build_feed_forward(PartSpec("swiglu", {"hidden_size": width, "ffn_dim": ff, "activation": "relu"},
                                       {name: name for name in w}))
    precision = Precision("float32" if dtype == torch.float32 else "bfloat16")
    part.bind(lambda n: w[n].to(dtype), precision, DEV)
    ctx = StepContext(step_batch([(0, tokens)], [0], [0]), precision, DEV)
    close(part.forward(ctx, dev(h, dtype)), P.gated_relu(h, w["gate"], w["up"], w["down"], rnd), TOL[dtype] / 4, "dense")
    got = ops.linear_act(dev(h, dtype), dev(w["up"], dtype), "relu_squared", dtype)
    assert got.dtype == dtype
    close(got.float(), torch.relu(h @ w["up"].T) ** 2, 1e-5 if dtype == torch.float32 else 1e-2, "squared relu")


# ------------------------------------------------------------------ mixers whole
def mixer_case(kind, mixer, width, seed, dtype):
    from flyweight_b200.config.futezen import FutezenConfig
    from flyweight_b200.parts import build_mixer
    raw = {"vocab": 8, "width": width, "norm": {"eps": EPS}, "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}
    spec = FutezenConfig.from_dict(raw).model_spec().layers[0].parts["mixer"]
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, decl in build_mixer(spec).declare().items():
        t = torch.randn(decl.shape, generator=g, dtype=F64)
        if name.endswith("A_log"):
            t = torch.linspace(-6.0, 1.0, decl.shape[0], dtype=F64)
        elif len(decl.shape) == 2 and not name.endswith(".conv"):
            t = t / math.sqrt(decl.shape[1])
        elif not name.endswith((".conv", ".b", "bias")):
            t = 1.0 + 0.2 * t
        w[name] = rounding(dtype)(t)
    return spec, w


def run_part(part_spec, w, dtype, h_seqs, cuts, n_pages=40, seed=0):
    """A mixer over several sequences fed in the portions ``cuts``; pages in shuffled order, slot = 3 - s; pools hold
    NaN where nobody wrote.  Returns the outputs by sequence."""
    from flyweight_b200.engine import Segment, StepBatch, StepContext
    from flyweight_b200.parts import Precision, build_mixer
    from flyweight_b200.parts.base import FixedState, PagedKV
    precision = Precision("float32" if dtype == torch.float32 else "bfloat16")
    order = torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
    part = build_mixer(part_spec)
    part.bind(lambda n: w[n].to(dtype), precision, DEV)
    part.prepare(2048, DEV)
    cache = type("Cache", (), {})()
    cache.k_pool = cache.v_pool = cache.state = None
    cache.group = 0
    one = part.state_spec()
    if isinstance(one, PagedKV):
        shape = (n_pages, one.n_kv_heads, 64, one.head_dim)
        cache.k_pool = torch.full(shape, float("nan"), dtype=precision.cache_dtype, device=DEV)
        if one.values:
            cache.v_pool = torch.full(shape, float("nan"), dtype=precision.cache_dtype, device=DEV)
    elif isinstance(one, FixedState):
        cache.state = torch.zeros((4,) + tuple(one.shape), dtype=one.dtype, device=DEV)
    pages = {s: [] for s in range(len(h_seqs))}
    done = {s: 0 for s in range(len(h_seqs))}
    outs = {s: [] for s in range(len(h_seqs))}
    for step in cuts:
        segments = []
        for s, m in step:
            while len(pages[s]) * 64 < done[s] + m:
                pages[s].append(order.pop())
            segments.append(Segment(f"s{s}", 3 - s, done[s], [0] * m, []))
        width = max(len(pages[s]) for s, _ in step)
        table = [pages[s] + [-1] * (width - len(pages[s])) for s, _ in step]
        ctx = StepContext(StepBatch(segments, [table], DEV), precision, DEV)
        h = dev(torch.cat([h_seqs[s][done[s]:done[s] + m] for s, m in step]), precision.act_dtype)
        out = part.forward(ctx, h, cache)
        at = 0
        for s, m in step:
            outs[s].append(out[at:at + m].float().cpu())
            at += m
            done[s] += m
    return {s: torch.cat(parts) for s, parts in outs.items() if parts}


def inputs_with_partners(lengths, width, pairs, seed, dtype, strength):
    """Random rows; for every (sequence, key position, query position) in ``pairs`` both rows get a large share of one
    common direction, so that this query's score on this key can stand out."""
    g = torch.Generator().manual_seed(seed)
    seqs = [torch.randn(n, width, generator=g, dtype=F64) for n in lengths]
    for index, (s, j, i) in enumerate(pairs):
        u = torch.randn(width, generator=torch.Generator().manual_seed(1000 + index), dtype=F64)
        seqs[s][j] += strength * u
        seqs[s][i] -= strength * u
    return [rounding(dtype)(h) for h in seqs]


# sequence 0: positions 0-99, 100-101, 102, 103-139, 140, 141, 142-199 (102, 140 and 141 are decoded alone)
CUTS = [[(0, 100), (1, 3)], [(1, 1), (0, 2), (2, 64)], [(0, 1), (1, 1), (2, 1)], [(2, 63), (0, 37), (1, 60)],
        [(0, 1), (2, 2)], [(0, 1)], [(0, 58), (1, 70)]]
LENGTHS = [200, 135, 130]
FAR = [(0, 2, 95), (0, 63, 102), (0, 64, 141), (0, 0, 199), (1, 0, 134)]
LATENTS = [(3, 8, 8, 20, 12, 24), (2, 16, 4, 8, 40, 40), (8, 32, 16, 32, 64, 48), (4, 64, 32, 64, 96, 96), (2, 32, 32, 48, 20, 160),
           (1, 16, 2, 16, 12, 30), (20, 24, 8, 24, 48, 184), (5, 48, 16, 56, 40, 272), (33, 32, 32, 64, 64, 256),
           (6, 128, 64, 128, 32, 512), (3, 10, 6, 14, 22, 150), (3, 9, 4, 13, 21, 145)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,q_rank,kv_rank", LATENTS)
def test_latent_attention_with_low_rank_queries(dtype, heads, dim, rot_dim, vdim, q_rank, kv_rank, monkeypatch):
    """Cache rows of 32 to 576 entries: the paged kernels, the long rows on their own kernel, prompts over expanded
    keys, the 32-bit kernel.  Keys far back, at a page's last and first place, stand out, asked for from inside a
    portion and by decoded tokens; a plain result that cannot see them must be another one."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": 10.0 / (dim + rot_dim), "rot": {"base": 300.0, "dims": rot_dim}}
    spec, w = mixer_case("latent_attention", m, 64, heads + kv_rank, dtype)
    seqs = inputs_with_partners(LENGTHS, 64, FAR, 9, dtype, strength=2.0)
    rnd = rounding(dtype)
    got = run_part(spec, w, dtype, seqs, CUTS, seed=2)
    wants = []
    for s, h in enumerate(seqs):
        want = P.latent_attention_mixer(h, w, "l0.mix.", m, EPS, torch.arange(h.shape[0]), rnd=rnd)
        close(got[s], want, TOL[dtype], f"sequence {s}")
        wants.append(want)
    # queries without their norm, or a rotation of halves, are felt
    skewed = dict(w, **{"l0.mix.dq.norm": w["l0.mix.dq.norm"] * 1.5})
    off = P.latent_attention_mixer(seqs[0], skewed, "l0.mix.", m, EPS, torch.arange(LENGTHS[0]), rnd=rnd)
    assert (off - wants[0]).abs().max() > SHOWS
    if rot_dim > 2:
        turn = P.turn
        monkeypatch.setattr(P, "turn", lambda x, pos, base, n, neighbours: turn(x, pos, base, n, False))
        off = P.latent_attention_mixer(seqs[0], w, "l0.mix.", m, EPS, torch.arange(LENGTHS[0]), rnd=rnd)
        assert (off - wants[0]).abs().max() > SHOWS


@pytest.mark.parametrize("way", ["expanded", "rows", "fp32 kernel"])
def test_long_latent_rows_by_every_kernel(way):
    """One model's prompts of 500 tokens and single tokens behind them over expanded keys, over the rows themselves and
    through the fp32 kernel: all within the bound of the plain result."""
    from flyweight_b200.kernels import attention as A
    from flyweight_b200.kernels import latent as L
    m = {"heads": 8, "dim": 64, "rot_dim": 32, "vdim": 64, "q_rank": 48, "kv_rank": 256, "scale": 0.1,
         "rot": {"base": 1000.0, "dims": 32}}
    spec, w = mixer_case("latent_attention", m, 64, 3, torch.bfloat16)
    lengths = [520, 300]
    seqs = inputs_with_partners(lengths, 64, [(0, 1, 499), (0, 127, 505), (1, 5, 290)], 4, torch.bfloat16, strength=2.0)
    cuts = [[(0, 500)], [(0, 1), (1, 130)]] + [[(0, 1), (1, 1)]] * 4 + [[(0, 15), (1, 166)]]
    try:
        A.set_tcgen05_enabled(way == "expanded")
        L.set_tensor_cores(way != "fp32 kernel")
        got = run_part(spec, w, torch.bfloat16, seqs, cuts, seed=1)
    finally:
        A.set_tcgen05_enabled(True)
        L.set_tensor_cores(True)
    for s, h in enumerate(seqs):
        want = P.latent_attention_mixer(h, w, "l0.mix.", m, EPS, torch.arange(h.shape[0]), rnd=bf16_round)
        close(got[s], want, TOL[torch.bfloat16], f"{way}, sequence {s}")


@pytest.mark.parametrize("heads,rank,rot,sink", [(1, 144, 16, False), (16, 160, 32, True), (17, 256, 32, False),
                                                 (40, 272, 32, True), (128, 512, 64, False), (10, 500, 20, True)])
@pytest.mark.parametrize("context", [1, 64, 65, 3000])
def test_long_rows_of_single_tokens_over_slices_of_the_context(heads, rank, rot, sink, context):
    """The kernel alone: single tokens of requests with short and long contexts in one step, many slices."""
    from flyweight_b200.engine import Segment, StepBatch
    from flyweight_b200.kernels import latent as L
    row = -(-(rank + rot) // 16) * 16
    g = torch.Generator().manual_seed(heads + context)
    contexts = [context, 1, max(1, context - 63)]
    pages = [-(-c // 64) for c in contexts]
    order = torch.randperm(sum(pages) + 3, generator=g).tolist()
    pool = torch.full((sum(pages) + 3, 1, 64, row), float("nan"), dtype=torch.bfloat16)
    qa = torch.zeros(3, heads, row, dtype=F64)
    qa[:, :, :rank + rot] = bf16_round(torch.randn(3, heads, rank + rot, generator=g, dtype=F64) / math.sqrt(rank + rot))
    sinks = torch.randn(heads, generator=g, dtype=F64).float() if sink else None
    scale, table, want = 3.0, [], []
    for i, (c, n) in enumerate(zip(contexts, pages)):
        rows = torch.zeros(n * 64, row, dtype=F64)
        rows[:c, :rank + rot] = bf16_round(torch.randn(c, rank + rot, generator=g, dtype=F64))
        rows[0, :rank + rot] = bf16_round(6.0 * qa[i, 0, :rank + rot])        # the oldest key stands out
        ids = [order.pop() for _ in range(n)]
        for j, page in enumerate(ids):
            live = min(64, c - 64 * j)
            pool[page, 0, :live] = rows[64 * j:64 * j + live].to(torch.bfloat16)
        table.append(ids + [-1] * (max(pages) - n))
        s = (qa[i] @ rows[:c].T) * scale
        top = s.max(dim=1, keepdim=True).values
        e = torch.exp(s - top)
        total = e.sum(dim=1, keepdim=True) + (torch.exp(sinks.to(F64)[:, None] - top) if sink else 0.0)
        want.append((e / total) @ rows[:c, :rank])
    batch = StepBatch([Segment(f"s{i}", i, c - 1, [0], []) for i, c in enumerate(contexts)], [table], DEV)
    got = L.rows_attention(dev(qa, torch.bfloat16), dev(pool), dev(sinks) if sink else None, batch, batch.block_tables[0],
                           rank, scale, 3)
    close(got.float().view(3, heads, rank), torch.stack(want), 1e-2, "rows")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot_dims", [(4, 2, 16, 24, 8), (3, 1, 20, 12, 20), (8, 2, 64, 64, 64), (6, 6, 128, 64, 32),
                                                        (2, 2, 32, 32, 0), (12, 3, 48, 80, 30)])
def test_attention_with_rotated_halves_of_a_part_of_each_head(dtype, heads, kv, dim, vdim, rot_dims):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 8.0 / dim, "rot": {"base": 500.0, "dims": rot_dims}}
    spec, w = mixer_case("attention", m, 64, heads + dim, dtype)
    # every query head scores as its key head does, with the opposite sign: opposite rows find each other
    w["l0.mix.q"] = -w["l0.mix.k"].view(kv, dim, -1).repeat_interleave(heads // kv, dim=0).reshape(heads * dim, -1).clone()
    seqs = inputs_with_partners(LENGTHS, 64, FAR, 11, dtype, strength=1.5)
    rnd = rounding(dtype)
    got = run_part(spec, w, dtype, seqs, CUTS, seed=4)
    for s, h in enumerate(seqs):
        pos = torch.arange(h.shape[0])
        want = P.attention_mixer(h, w, "l0.mix.", m, EPS, pos, rnd=rnd)
        close(got[s], want, TOL[dtype], f"sequence {s}")
    if 2 < rot_dims:
        other = dict(m, rot={"base": 500.0, "dims": rot_dims - 2})
        off = P.attention_mixer(h, w, "l0.mix.", other, EPS, pos, rnd=rnd)
        assert (off - want).abs().max() > SHOWS


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,vdim,state,groups,conv,norm_groups", [(6, 10, 12, 3, 3, 2), (4, 7, 33, 1, 1, 1), (8, 64, 128, 1, 4, 2),
                                                                      (6, 80, 200, 2, 2, 3), (2, 16, 16, 2, 5, 1)])
def test_state_space_mixer(dtype, heads, vdim, state, groups, conv, norm_groups):
    """Projection, convolution, recurrence, gate, norm and output over portions and single tokens."""
    m = {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}
    spec, w = mixer_case("mamba2", m, 64, heads + state, dtype)
    w["l0.mix.norm"] = w["l0.mix.norm"] * torch.linspace(0.5, 1.5, heads * vdim, dtype=F64)
    w["l0.mix.norm"] = rounding(dtype)(w["l0.mix.norm"])
    g = torch.Generator().manual_seed(3)
    rnd = rounding(dtype)
    seqs = [rnd(torch.randn(n, 64, generator=g, dtype=F64)) for n in LENGTHS]
    got = run_part(spec, w, dtype, seqs, CUTS)
    for s, h in enumerate(seqs):
        want = P.mamba2_mixer(h, w, "l0.mix.", m, EPS, None, rnd=rnd)
        close(got[s], want, TOL[dtype], f"sequence {s}")
    # the convolution, its bias, the skip and the order of gate and norm are felt
    for name in ("conv.b", "D", "dt_bias"):
        off = P.mamba2_mixer(seqs[0], dict(w, **{f"l0.mix.{name}": w[f"l0.mix.{name}"] + 0.5}), "l0.mix.", m, EPS, None, rnd=rnd)
        want = P.mamba2_mixer(seqs[0], w, "l0.mix.", m, EPS, None, rnd=rnd)
        assert (off - want).abs().max() > SHOWS, name
