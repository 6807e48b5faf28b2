"""A plain, slow implementation of the Turutar decoder, one function per mechanism, written from the
design's equations with torch on the CPU.  It shares no code with the library: it reads a model folder
with its own safetensors reader, builds every attention mask as a full matrix and keeps no cache between
calls.

Notation.  ``x[t]`` is the residual stream of token t; a layer does, with ``n = norm1(x)``,
``x <- x + a * mixer(n) + b * ff(n)`` (a, b: vectors of the layer) and then adds what the token itself
brings to this layer, behind a norm of its own.  ``precision`` is ``torch.float32`` or ``torch.float64``
for exact arithmetic, or ``torch.bfloat16`` for an emulation of serving precision: operands and results
of matrix products are rounded to bfloat16, everything else stays in float32.
"""

import json
import math
import os
import struct

import numpy as np
import torch

LOGISTIC_SLOPE = 1.702


# ----------------------------------------------------------------------------- reading


def read_safetensors(path):
    with open(path, "rb") as handle:
        (n,) = struct.unpack("<Q", handle.read(8))
        header = json.loads(handle.read(n).decode("utf-8"))
        data = handle.read()
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = np.frombuffer(data[lo:hi], dtype=np.uint8)
        if meta["dtype"] == "BF16":
            t = torch.from_numpy((raw.view("<u2").astype(np.uint32) << 16).view(np.float32).copy())
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(raw.view("<f4").copy())
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        out[name] = t.reshape(meta["shape"])
    return out


def read_model(folder):
    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    return config, read_safetensors(os.path.join(folder, "model.safetensors"))


# ----------------------------------------------------------------------------- precision


class Arithmetic:
    """``work``: the type everything is computed in; ``round_products``: whether operands and
    results of matrix products pass through bfloat16."""

    def __init__(self, precision):
        self.round_products = precision == torch.bfloat16
        self.work = torch.float32 if self.round_products else precision

    def rb(self, t):
        return t.to(torch.bfloat16).to(self.work) if self.round_products else t

    def linear(self, x, w, bias=None, keep=False):
        """``x @ w.T + bias`` for a weight of shape [outputs, inputs]; ``keep``: the result is not rounded."""
        y = self.rb(x) @ self.rb(w.to(self.work)).t()
        if bias is not None:
            y = y + bias.to(self.work)
        return y if keep else self.rb(y)


# ----------------------------------------------------------------------------- small pieces


def logistic(x):
    return 1.0 / (1.0 + torch.exp(-x))


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rms_divide(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """An RMS norm whose weight is stored as the difference from one."""
    return rms_divide(x, eps) * (1.0 + w)


def embed(w, config, tokens, work):
    return norm_around_zero(w["embed"].to(work)[tokens], w["embed.norm"].to(work), config["norm"]["eps"])


def rotate_neighbours(x, positions, base):
    """Turns the whole last axis of ``x`` [tokens, ..., dims]: entry 2i pairs with entry 2i + 1."""
    dims = x.shape[-1]
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * freq
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = torch.cos(angle).to(x.dtype).reshape(shape), torch.sin(angle).to(x.dtype).reshape(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).reshape(x.shape)


def softmax_with_extra(score, visible, extra):
    """Row by row exp(score) / (sum over the visible of exp(score) + exp(extra)): the extra term takes
    weight and brings nothing."""
    s = score.masked_fill(~visible, -math.inf)
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=float(extra))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(extra - top))


# ----------------------------------------------------------------------------- mixers


def window_attention(ar, h, w, prefix, m, eps):
    """No positions in the scores; a norm over all heads together; the values are the keys as projected;
    one added to the softmax's denominator; a logistic gate per head."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = ar.linear(h, w[prefix + "q"], w[prefix + "q.b"])
    k = ar.linear(h, w[prefix + "k"], w[prefix + "k.b"])
    v = k.reshape(T, G, d)
    q = ar.rb(rms_divide(q, eps) * w[prefix + "q.norm"].to(ar.work)).reshape(T, H, d)
    k = ar.rb(rms_divide(k, eps) * w[prefix + "k.norm"].to(ar.work)).reshape(T, G, d)
    place = torch.arange(T)
    behind = place[:, None] - place[None, :]
    visible = (behind >= 0) & (behind < m["mask"]["size"] if m.get("mask") else behind >= 0)
    gate = logistic(ar.linear(h, w[prefix + "g"]))
    out = torch.zeros(T, H, d, dtype=ar.work)
    for head in range(H):
        g = head // (H // G)
        score = (q[:, head] @ k[:, g].t()) * m["scale"]
        out[:, head] = softmax_with_extra(score, visible, torch.tensor(0.0, dtype=ar.work)) @ v[:, g]
    return ar.linear((ar.rb(out) * gate[:, :, None]).reshape(T, H * d), w[prefix + "o"])


def latent_attention(ar, h, w, prefix, m, eps):
    """Queries out of a normalised latent, keys and values of all heads out of another one, one rotated
    key part shared by the heads, a learned term in every head's softmax, a logistic gate per head."""
    T = h.shape[0]
    H, d, r, e, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    place = torch.arange(T)
    cq = ar.rb(rms_divide(ar.linear(h, w[prefix + "dq"]), eps) * w[prefix + "dq.norm"].to(ar.work))
    q = ar.linear(cq, w[prefix + "uq"]).reshape(T, H, d + r)
    down = ar.linear(h, w[prefix + "dkv"])
    latent = ar.rb(rms_divide(down[:, :c], eps) * w[prefix + "dkv.norm"].to(ar.work))
    k_plain = ar.linear(latent, w[prefix + "uk"]).reshape(T, H, d)
    v = ar.linear(latent, w[prefix + "uv"]).reshape(T, H, e)
    q_rot, k_rot = q[:, :, d:], down[:, c:]
    if r:
        q_rot = ar.rb(rotate_neighbours(q_rot, place, m["rot"]["base"]))
        k_rot = ar.rb(rotate_neighbours(k_rot, place, m["rot"]["base"]))
    visible = place[:, None] >= place[None, :]
    sink = w[prefix + "sink"].to(ar.work)
    gate = logistic(ar.linear(h, w[prefix + "g"]))
    out = torch.zeros(T, H, e, dtype=ar.work)
    for head in range(H):
        score = (q[:, head, :d] @ k_plain[:, head].t() + q_rot[:, head] @ k_rot.t()) * m["scale"]
        out[:, head] = softmax_with_extra(score, visible, sink[head]) @ v[:, head]
    return ar.linear((ar.rb(out) * gate[:, :, None]).reshape(T, H * e), w[prefix + "o"])


# ----------------------------------------------------------------------------- feed-forward and token input


def clamped_feed_forward(ar, h, w, prefix, limit):
    g = torch.clamp(ar.linear(h, w[prefix + "gate"]), max=limit)
    u = torch.clamp(ar.linear(h, w[prefix + "up"]), min=-limit, max=limit)
    return ar.linear(g * logistic(LOGISTIC_SLOPE * g) * (u + 1.0), w[prefix + "down"])


def token_side(ar, x, tokens, w, i, dim, eps):
    """What a token itself brings to layer i: its own row of the side table, let through by a gate that
    reads the stream, projected back and normed."""
    p = f"l{i}.side."
    e = w["side.embed"].to(ar.work)[tokens, i * dim:(i + 1) * dim]
    g = gelu_tanh(ar.linear(x, w[p + "gate"])) * e
    return rms_divide(ar.linear(g, w[p + "proj"]), eps) * w[p + "norm"].to(ar.work)


# ----------------------------------------------------------------------------- the model


def layer_runs(config):
    """(layer, whether the start of the stream is added ahead of it) in the order of execution."""
    loop, n = config.get("loop"), len(config["layers"])
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for go in range(loop["times"]):
        runs += [(i, go > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def layer(ar, x, tokens, w, config, i):
    entry, eps, p = config["layers"][i], config["norm"]["eps"], f"l{i}."
    n = ar.rb(norm_around_zero(x, w[p + "norm1"].to(ar.work), eps))
    mixer = window_attention if entry["type"] == "attention" else latent_attention
    total = mixer(ar, n, w, p + "mix.", entry["mixer"], eps) * w[p + "ls1"].to(ar.work)
    if entry.get("mlp") is not None:
        total = total + clamped_feed_forward(ar, n, w, p + "mlp.", entry["mlp"]["limit"]) * w[p + "ls2"].to(ar.work)
    x = x + total
    if config.get("token_side"):
        x = x + token_side(ar, x, tokens, w, i, config["token_side"]["dim"], eps)
    return x


def model_forward(folder, tokens, precision=torch.float64, model=None):
    """(logits [tokens, vocab], the residual stream after every layer run [runs, tokens, width])."""
    config, w = model if model is not None else read_model(folder)
    ar = Arithmetic(precision)
    tokens = torch.as_tensor(tokens, dtype=torch.int64)
    start = x = embed(w, config, tokens, ar.work)
    after = []
    for i, again in layer_runs(config):
        if again:
            x = x + start
        x = layer(ar, x, tokens, w, config, i)
        after.append(x)
    n = ar.rb(norm_around_zero(x, w["final.norm"].to(ar.work), config["norm"]["eps"]))
    return ar.linear(n, w["head"], keep=True), torch.stack(after)


def model_logits(folder, tokens, precision=torch.float64, model=None):
    return model_forward(folder, tokens, precision, model)[0]
