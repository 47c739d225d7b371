"""A plain, slow implementation of the Futezen design, one function per mechanism, in float64 torch on
the CPU.  It shares no code with the engine: tests compare the engine's parts and whole models with it.

Notation: W the model width, ``unit(y) = y / sqrt(mean(y^2) + eps)`` over the last axis, positions
count from 0 in every sequence, matrices are stored [out][in] and applied as ``y = x @ M.T``.

``rnd`` (optional, in some functions): a function applied where the serving precision rounds (inputs
of matrix products, cached rows); the identity by default.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

F64 = torch.float64


def same(value):
    return value


def bf16(value):
    """To bfloat16 and back: what the serving precision loses where it keeps 16 bits."""
    return value.to(torch.bfloat16).to(value.dtype)


def dither(seed):
    """A stand-in for ``bf16`` that loses as much, but at random: a relative error of up to half a unit in the last
    of bfloat16's places.  Several of them show how far apart two correct 16-bit computations may lie."""
    gen = torch.Generator().manual_seed(seed)

    def lose(value):
        return value * (1.0 + (torch.rand(value.shape, generator=gen, dtype=value.dtype) - 0.5) * 2.0 ** -8)
    return lose


def load_model_dir(path):
    """(config dict, name -> tensor in float64) of a model folder: the file is a little-endian header length,
    a JSON header (dtype, shape, byte range per name) and the data."""
    path = Path(path)
    config = json.loads((path / "config.json").read_text())
    blob = (path / "model.safetensors").read_bytes()
    (header_len,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8:8 + header_len].decode("utf-8"))
    data = memoryview(blob)[8 + header_len:]
    dtypes = {"F64": torch.float64, "F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16}
    weights = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        t = torch.frombuffer(bytearray(data[lo:hi]), dtype=dtypes[entry["dtype"]]).reshape(entry["shape"])
        weights[name] = t.to(F64)
    return config, weights


def unit(y, eps):
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def silu(y):
    return y * torch.sigmoid(y)


def softplus(y):
    """ln(1 + e^y), written so that neither end overflows."""
    return torch.clamp(y, min=0.0) + torch.log1p(torch.exp(-y.abs()))


# ------------------------------------------------------------------ rotation
def turn(x, positions, base, n, neighbours):
    """x: [T][heads][d].  Pair i < n/2 of every head turns by positions * base^(-2i/n): channels (2i, 2i+1) with
    ``neighbours``, else (i, i + n/2); channels from n on pass."""
    if n == 0:
        return x
    f = torch.tensor([float(base) ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * f[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    first, second = (slice(0, n, 2), slice(1, n, 2)) if neighbours else (slice(0, n // 2), slice(n // 2, n))
    a, b = x[..., first], x[..., second]
    out = x.clone()
    out[..., first] = a * cos - b * sin
    out[..., second] = b * cos + a * sin
    return out


# ------------------------------------------------------------------ attention
def causal_softmax(q, k, v, q_pos, k_pos, scale):
    """q: [Tq][H][d], k: [Tk][G][d], v: [Tk][G][e]; query head h reads key/value head h // (H/G); a key at
    position j is visible from position i when j <= i."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros((q.shape[0], H, v.shape[2]), dtype=q.dtype)
    hidden = k_pos[None, :] > q_pos[:, None]
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, -math.inf)
        e = torch.exp(s - s.max(dim=1, keepdim=True).values)
        out[:, h] = (e / e.sum(dim=1, keepdim=True)) @ v[:, g]
    return out


def attention_mixer(h, w, prefix, m, eps, positions, rnd=same):
    """The mixer 'attention': projections, rotation of halves, softmax over every earlier key, output."""
    H, G, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    hr = rnd(h)
    q, k, v = (rnd(hr @ w[prefix + name].T) for name in ("q", "k", "v"))
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, e)
    rot = m.get("rot")
    if rot:
        q, k = (turn(t, positions, rot["base"], int(rot["dims"]), False) for t in (q, k))
    o = causal_softmax(rnd(q), rnd(k), v, positions, positions, float(m["scale"]))
    return rnd(o.reshape(T, H * e)) @ w[prefix + "o"].T


def latent_attention_mixer(h, w, prefix, m, eps, positions, rnd=same):
    """The mixer 'latent_attention': queries from a normed low-rank row; per token a normed latent c and one
    turned key part shared by the heads; head keys U_h c and values V_h c; softmax over every earlier key."""
    H, d, r, e, rank = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    T = h.shape[0]
    hr = rnd(h)
    c_q = rnd(unit(hr @ w[prefix + "dq"].T, eps) * w[prefix + "dq.norm"])
    q = (c_q @ w[prefix + "uq"].T).view(T, H, d + r)
    low = hr @ w[prefix + "dkv"].T
    c = rnd(unit(low[:, :rank], eps) * w[prefix + "dkv.norm"])
    base = float(m["rot"]["base"])
    k_turned = rnd(turn(low[:, None, rank:], positions, base, r, True))              # [T][1][r]
    q_turned = turn(q[:, :, d:], positions, base, r, True)
    k_plain = (c @ w[prefix + "uk"].T).view(T, H, d)
    value = (c @ w[prefix + "uv"].T).view(T, H, e)
    keys = torch.cat([k_plain, k_turned.expand(T, H, r)], dim=-1)
    queries = torch.cat([q[:, :, :d], q_turned], dim=-1)
    o = causal_softmax(rnd(queries), keys, value, positions, positions, float(m["scale"]))
    return rnd(o.reshape(T, H * e)) @ w[prefix + "o"].T


# ------------------------------------------------------------------ state space
def causal_taps(u, taps, bias, history=None):
    """u: [T][C], taps: [C][n], bias [C].  y_t = bias + sum_j taps[:, j] * u_(t - n + 1 + j); what lies before
    the sequence is zero, or ``history`` ([n - 1][C], the rows just before u)."""
    n = taps.shape[1]
    before = torch.zeros((n - 1, u.shape[1]), dtype=u.dtype) if history is None else history
    padded = torch.cat([before, u], dim=0)
    y = bias[None, :].expand_as(u).clone()
    for j in range(n):
        y = y + padded[j:j + u.shape[0]] * taps[:, j][None, :]
    return y


def scalar_decay_scan(x, b, c, dt, a, skip, state=None):
    """x: [T][H][e], b, c: [T][G][n], dt: [T][H] (positive), a: [H] (positive), skip: [H].  Per head, with its
    group g = h // (H/G):  S <- exp(-a dt) S + dt b x^T;  y = S^T c + skip x.  Returns (y, last S [H][n][e])."""
    T, H, e = x.shape
    G, n = b.shape[1], b.shape[2]
    group = torch.arange(H) // (H // G)
    S = torch.zeros((H, n, e), dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        S = torch.exp(-a * dt[t])[:, None, None] * S \
            + dt[t][:, None, None] * b[t][group][:, :, None] * x[t][:, None, :]
        y[t] = (S * c[t][group][:, :, None]).sum(dim=1) + skip[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, weight, groups, eps):
    """unit() of y * silu(z), over each of ``groups`` equal runs of channels on its own, times a weight."""
    T = y.shape[0]
    return unit((y * silu(z)).view(T, groups, -1), eps).reshape(T, -1) * weight


def mamba2_mixer(h, w, prefix, m, eps, positions, rnd=same):
    """The mixer 'mamba2': one projection z | x | B | C | dt, a convolution with bias and silu on x | B | C, the
    recurrence with a scalar decay per head and token, gate, grouped norm, output."""
    H, e, n, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * e
    T = h.shape[0]
    p = rnd(h) @ w[prefix + "in"].T
    z, u, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * n], p[:, 2 * inner + 2 * G * n:]
    u = rnd(silu(causal_taps(u, w[prefix + "conv"], w[prefix + "conv.b"])))
    x, b, c = u[:, :inner], u[:, inner:inner + G * n], u[:, inner + G * n:]
    dt = softplus(dt + w[prefix + "dt_bias"])
    y, _ = scalar_decay_scan(x.view(T, H, e), b.view(T, G, n), c.view(T, G, n), dt,
                             torch.exp(w[prefix + "A_log"]), w[prefix + "D"])
    y = gated_group_norm(y.reshape(T, inner), z, w[prefix + "norm"], int(m["norm_groups"]), eps)
    return rnd(y) @ w[prefix + "o"].T


# ------------------------------------------------------------------ feed-forward
def gated_relu(h, gate, up, down, rnd=same):
    return rnd(torch.relu(h @ gate.T) * (h @ up.T)) @ down.T


def squared_relu(h, up, down, rnd=same):
    return rnd(torch.relu(h @ up.T) ** 2) @ down.T


def chosen_experts(logits, top):
    """The ``top`` largest logits of every row and the softmax over those alone."""
    order = torch.argsort(logits, dim=1, descending=True, stable=True)[:, :top]
    picked = torch.gather(logits, 1, order)
    e = torch.exp(picked - picked.max(dim=1, keepdim=True).values)
    return order, e / e.sum(dim=1, keepdim=True)


def routed_experts(h, w, prefix, mlp, rnd=same):
    """Experts behind a router with a bias, weighted by the softmax over the chosen; beside them a shared expert
    times one sigmoid per token."""
    hr = rnd(h)
    ids, weights = chosen_experts(hr @ w[prefix + "router"].T + w[prefix + "router.b"], int(mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(ids.shape[1]):
            j = int(ids[t, slot])
            out[t] += weights[t, slot] * squared_relu(hr[t:t + 1], w[f"{prefix}e{j}.up"], w[f"{prefix}e{j}.down"], rnd)[0]
    if mlp.get("shared"):
        shared = squared_relu(hr, w[prefix + "shared.up"], w[prefix + "shared.down"], rnd)
        out = out + torch.sigmoid(hr @ w[prefix + "shared.sg"].T) * shared
    return out


def feed_forward(h, w, prefix, mlp, rnd=same):
    if mlp["kind"] == "dense":
        return gated_relu(rnd(h), w[prefix + "gate"], w[prefix + "up"], w[prefix + "down"], rnd)
    return routed_experts(h, w, prefix, mlp, rnd)


# ------------------------------------------------------------------ the model
MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer, "mamba2": mamba2_mixer}


def layer_runs(config):
    """The layers in the order they run: layers start .. stop-1 ``times`` times in a row."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def forward(config, weights, tokens, rnd=same, layers_out=None):
    """Logits [T][vocab] of one sequence from position 0.  ``layers_out``: a list that receives the stream
    behind every layer run."""
    w = weights
    eps = float(config["norm"]["eps"])
    tokens = [int(t) for t in tokens]
    positions = torch.arange(len(tokens))
    x = w["embed"][tokens].clone()
    for index in layer_runs(config):
        layer = config["layers"][index]
        p = f"l{index}."

        def normed(y, name):
            return unit(y, eps) * (1.0 + w[p + name])

        x = x + normed(MIXERS[layer["type"]](normed(x, "norm1"), w, p + "mix.", layer["mixer"], eps, positions, rnd),
                       "norm1b")
        if layer.get("mlp") is not None:
            x = x + normed(feed_forward(normed(x, "norm2"), w, p + "mlp.", layer["mlp"], rnd), "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return rnd(unit(x, eps) * (1.0 + w["final.norm"])) @ rnd(w["embed"]).T


def greedy_generate(config, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(config, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]
