"""A plain, slow implementation of the Vugipel design, one function per mechanism, in float64 torch on
the CPU.  It shares no code with the engine: tests compare the engine's parts and whole models with it.

Notation: W the model width, ``unit(y) = y / sqrt(mean(y^2) + eps)`` over the last axis, positions
count from 0 in every sequence, matrices are stored [out][in] and applied as ``y = x @ M.T``.

``rnd`` (optional, in some functions): a function applied where the serving precision rounds (inputs
of matrix products, cached keys and values); the identity by default.
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
    """(config dict, name -> tensor in float64) of a model folder: the file is a little-endian header
    length, a JSON header (dtype, shape, byte range per name) and the data."""
    path = Path(path)
    config = json.loads((path / "config.json").read_text())
    blob = (path / "model.safetensors").read_bytes()
    (header_len,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8:8 + header_len].decode("utf-8"))
    data = memoryview(blob)[8 + header_len:]
    dtypes = {"F64": torch.float64, "F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16,
              "I32": torch.int32, "I64": torch.int64}
    weights = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        lo, hi = entry["data_offsets"]
        t = torch.frombuffer(bytearray(data[lo:hi]), dtype=dtypes[entry["dtype"]]).reshape(entry["shape"])
        weights[name] = t.to(F64) if t.is_floating_point() else t
    return config, weights


def unit(y, eps):
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ minGRU
def positive_part(u):
    """The candidate of the recurrence: u + 1/2 from zero on, sigmoid(u) below it."""
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def gated_average(z, candidate, state=None):
    """S_t = (1 - z_t) S_(t-1) + z_t candidate_t, channel by channel, from ``state`` (zero)."""
    s = torch.zeros(z.shape[1], dtype=z.dtype) if state is None else state.clone()
    out = torch.empty_like(z)
    for t in range(z.shape[0]):
        s = (1.0 - z[t]) * s + z[t] * candidate[t]
        out[t] = s
    return out


def mingru_mixer(h, w, prefix, rnd=same):
    hr = rnd(h)
    z = torch.sigmoid(hr @ w[prefix + "z"].T + w[prefix + "z.b"])
    u = hr @ w[prefix + "x"].T + w[prefix + "x.b"]
    s = gated_average(z, positive_part(u))
    return rnd(s * silu(hr @ w[prefix + "g"].T)) @ w[prefix + "o"].T


# ------------------------------------------------------------------ rotation
def turn_neighbours(x, positions, base, dims, sign=1.0):
    """x: [T][heads][d].  Channels (2i, 2i+1), i < dims/2, of every head turn by sign * position *
    base^(-2i/dims); the other channels pass."""
    if dims == 0:
        return x
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = sign * positions.to(F64)[:, None] * f[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = a * cos - b * sin
    out[..., 1:dims:2] = b * cos + a * sin
    return out


# ------------------------------------------------------------------ softmax attention
def visible(q_pos, k_pos, size=0, keep_first=0):
    """[Tq][Tk]: a query at i sees a key at j when j <= i and the key is among the last ``size`` positions
    up to i (0: no window) or among the sequence's first ``keep_first``."""
    i, j = q_pos[:, None], k_pos[None, :]
    seen = j <= i
    if size > 0:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def capped_attention(q, k, v, seen, scale, temp=None, softcap=0.0):
    """q: [Tq][H][d], k: [Tk][G][d], v: [Tk][G][e]; query head h reads key/value head h // (H/G).  Scores are
    q.k times ``scale`` times the head's number in ``temp``, then softcap tanh(score / softcap), then an
    ordinary softmax over the visible keys."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros((q.shape[0], H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if temp is not None:
            s = s * temp[h]
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~seen, -math.inf)
        out[:, h] = torch.softmax(s, dim=1) @ v[:, g]
    return out


def turned_attention(h, w, prefix, m, eps, positions, rnd=same):
    """The left half of the parallel mixer: attention with biases, a norm per head of q and k, rotated keys
    and rotated values (each head's sum is turned back by the query's position), a number per head on the
    scores, capped scores, a window with kept first tokens."""
    H, G, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    hr = rnd(h)
    q, k, v = (hr @ w[prefix + name].T + w[prefix + name + ".b"] for name in ("q", "k", "v"))
    q = unit(q.view(T, H, d), eps) * w[prefix + "q.norm"]
    k = unit(k.view(T, G, d), eps) * w[prefix + "k.norm"]
    v = v.view(T, G, e)
    rot = m.get("rot")
    base = float(rot["base"]) if rot else 0.0
    if rot:
        q = turn_neighbours(q, positions, base, int(rot["dims"]))
        k = turn_neighbours(k, positions, base, int(rot["dims"]))
        v = turn_neighbours(v, positions, base, e)
    mask = m.get("mask") or {}
    seen = visible(positions, positions, int(mask.get("size") or 0), int(mask.get("keep_first") or 0))
    o = capped_attention(rnd(q), rnd(k), rnd(v), seen, float(m["scale"]), w[prefix + "temp"],
                         float(m.get("softcap") or 0.0))
    if rot:
        o = turn_neighbours(o, positions, base, e, sign=-1.0)
    return rnd(o.reshape(T, H * e)) @ w[prefix + "o"].T + w[prefix + "o.b"]


# ------------------------------------------------------------------ retention
def decayed_sums(q, k, v, decay, state=None):
    """q, k: [T][H][d], v: [T][H][e], decay: [H].  Per head S <- decay S + k v^T, o = S^T q."""
    T, H, d = q.shape
    s = torch.zeros((H, d, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", s, q[t])
    return out


def retention(h, w, prefix, m, eps, rnd=same):
    """The right half of the parallel mixer."""
    H, d, e = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    hr = rnd(h)
    q = (hr @ w[prefix + "q"].T).view(T, H, d)
    k = (hr @ w[prefix + "k"].T).view(T, H, d) * d ** -0.5
    v = (hr @ w[prefix + "v"].T).view(T, H, e)
    o = decayed_sums(rnd(q), rnd(k), rnd(v), torch.tensor([float(x) for x in m["decay"]], dtype=F64))
    o = unit(o, eps).reshape(T, H * e) * silu(hr @ w[prefix + "g"].T)
    return rnd(o) @ w[prefix + "o"].T


def parallel_mixer(h, w, prefix, m, eps, positions, rnd=same):
    left = turned_attention(h, w, prefix + "left.", m["left"], eps, positions, rnd)
    right = retention(h, w, prefix + "right.", m["right"], eps, rnd)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# ------------------------------------------------------------------ feed-forward
def sigmoid_choice(h, router, top):
    """(ids [T][top], scores [T][top]): the ``top`` largest of s = sigmoid(router h), not renormalised."""
    s = torch.sigmoid(h @ router.T)
    scores, ids = torch.topk(s, top, dim=1)
    return ids, scores


def input_weighted_experts(h, w, prefix, mlp, rnd=same):
    """sum over a token's chosen experts of expert(s h): the score multiplies what the expert reads."""
    top = int(mlp["router"]["top"])
    ids, scores = sigmoid_choice(rnd(h), w[prefix + "router"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(top):
            p = f"{prefix}e{int(ids[t, slot])}."
            x = rnd(rnd(h[t]) * scores[t, slot])
            out[t] += w[p + "down"] @ rnd(silu(w[p + "gate"] @ x) * (w[p + "up"] @ x))
    return out


# ------------------------------------------------------------------ the model
def forward(config, weights, tokens, rnd=same, layers_out=None):
    """Logits [T][vocab] of one sequence from position 0.  ``layers_out``: a list that receives the stream
    behind every layer."""
    w = weights
    eps = float(config["norm"]["eps"])
    tokens = [int(t) for t in tokens]
    positions = torch.arange(len(tokens))
    x = w["embed"][tokens].clone()
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        h = centred_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "mingru":
            x = x + mingru_mixer(h, w, p + "mix.", rnd)
        else:
            x = x + parallel_mixer(h, w, p + "mix.", layer["mixer"], eps, positions, rnd)
        if layer.get("mlp") is not None:
            x = x + input_weighted_experts(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], rnd)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rnd(centred_norm(x, w["final.norm"], eps)) @ w["head"].T


def greedy_generate(config, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(config, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]
