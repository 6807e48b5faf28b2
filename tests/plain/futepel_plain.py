"""A plain, slow implementation of the Futepel decoder, one function per mechanism, written from
the design's equations with torch on the CPU.  It shares no code with the library: it reads a
model folder with its own safetensors reader, walks a sequence token by token where the design has
a recurrence, builds the attention mask as a full matrix and keeps no cache or state between calls.

Notation.  ``x[t]`` is the residual stream of token t; a layer does ``x <- x + mixer(norm(x))`` and,
where it has a feed-forward, ``x <- x + ff(norm'(x))``.  ``precision`` is ``torch.float32`` or
``torch.float64`` for exact arithmetic, or ``torch.bfloat16`` for an emulation of serving precision:
operands and results of matrix products (and the short convolution with its activation) are rounded
to bfloat16, everything else stays in float32.
"""

import json
import math
import os
import struct

import numpy as np
import torch


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

    def linear(self, x, w, keep=False):
        """``x @ w.T`` for a weight of shape [outputs, inputs]; ``keep``: the result is not rounded."""
        y = self.rb(x) @ self.rb(w.to(self.work)).t()
        return y if keep else self.rb(y)


# ----------------------------------------------------------------------------- small pieces


def logistic(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * logistic(x)


def softplus(x):
    return torch.where(x > 30.0, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def rms_divide(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def embed(w, config, tokens, work):
    """Token row times a constant, plus the row of the pair (token before, token), plus the row of the
    position.  A first token has no token before it: it takes the pair table's last row."""
    e = config["embedding"]
    x = w["embed"].to(work)[tokens] * e.get("scale", 1.0)
    if e.get("bigram") is not None:
        g = e["bigram"]
        rows = [g["buckets"]]
        for t in range(1, len(tokens)):
            rows.append((int(tokens[t - 1]) * g["mul_prev"] + int(tokens[t]) * g["mul_cur"]) % g["buckets"])
        x = x + w["bigram"].to(work)[torch.tensor(rows)]
    return x + w["pos"].to(work)[:len(tokens)]


def yarn_frequencies(rot):
    """(frequencies of the pairs, common magnitude of cos and sin), in double."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return plain, 1.0

    def index(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(s["fast"])), 0)
    hi = min(math.ceil(index(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """Turns the whole last axis of ``x`` [tokens, ..., dims]: entry i pairs with entry i + dims/2."""
    if not rot["dims"]:
        return x
    freq, magnitude = yarn_frequencies(rot)
    half = rot["dims"] // 2
    angle = positions.to(torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c = (torch.cos(angle) * magnitude).to(x.dtype).reshape(shape)
    s = (torch.sin(angle) * magnitude).to(x.dtype).reshape(shape)
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


# ----------------------------------------------------------------------------- mixers


def time_mixing(ar, h, w, prefix, m, eps):
    """RWKV-style time mixing: every projection reads its own blend of a token and the one before; a
    matrix state per head with a decay per key channel and a bonus for the current token."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    mixed = {s: h + (before - h) * w[f"{prefix}mu.{s}"].to(ar.work) for s in "rkvgw"}
    r, k, v = (ar.linear(mixed[s], w[prefix + s]).reshape(T, H, d) for s in "rkv")
    gate = silu(ar.linear(mixed["g"], w[prefix + "g"]))
    low = torch.tanh(ar.linear(mixed["w"], w[prefix + "w1"], keep=True))
    z = ar.linear(low, w[prefix + "w2"], keep=True) + w[prefix + "w0"].to(ar.work)
    decay = torch.exp(-torch.exp(z)).reshape(T, H, d)
    u = w[prefix + "u"].to(ar.work)
    S = torch.zeros(H, d, d, dtype=ar.work)
    out = torch.zeros(T, H, d, dtype=ar.work)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    y = rms_divide(out, eps).reshape(T, H * d) * w[prefix + "norm"].to(ar.work) * gate
    return ar.linear(y, w[prefix + "o"])


def latent_attention(ar, h, w, prefix, m, eps, positions):
    """Keys and values of all heads out of one normalised latent per token, one rotated key part
    shared by the heads, one logistic gate per head."""
    T = h.shape[0]
    H, d, r, e, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = ar.linear(h, w[prefix + "q"]).reshape(T, H, d + r)
    down = ar.linear(h, w[prefix + "dkv"])
    latent = ar.rb(rms_divide(down[:, :c], eps) * w[prefix + "dkv.norm"].to(ar.work))
    k_plain = ar.linear(latent, w[prefix + "uk"]).reshape(T, H, d)
    v = ar.linear(latent, w[prefix + "uv"]).reshape(T, H, e)
    rot = m["rot"] if r else {"dims": 0}
    q_rot = ar.rb(rotate(q[:, :, d:], positions, rot))
    k_rot = ar.rb(rotate(down[:, c:], positions, rot))
    visible = positions[:, None] >= positions[None, :]
    out = torch.zeros(T, H, e, dtype=ar.work)
    for head in range(H):
        score = (q[:, head, :d] @ k_plain[:, head].t() + q_rot[:, head] @ k_rot.t()) * m["scale"]
        weight = torch.softmax(score.masked_fill(~visible, -math.inf), dim=-1)
        out[:, head] = weight @ v[:, head]
    gate = logistic(ar.linear(h, w[prefix + "g"]))
    return ar.linear((ar.rb(out) * gate[:, :, None]).reshape(T, H * e), w[prefix + "o"])


def state_space(ar, h, w, prefix, m, eps):
    """Mamba-2: a short causal convolution over x, B and C together, one step size and one decay per
    head, B and C shared by a group of heads, the gate ahead of a grouped norm."""
    T = h.shape[0]
    H, e, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner = H * e
    width = inner + 2 * G * N
    rows = w[prefix + "in"]
    zx = ar.linear(h, rows[:inner + width])
    dt = ar.linear(h, rows[inner + width:], keep=True)
    z, raw = zx[:, :inner], zx[:, inner:]
    kernel, bias = w[prefix + "conv"].to(ar.work), w[prefix + "conv.b"].to(ar.work)
    padded = torch.cat([torch.zeros(taps - 1, width, dtype=ar.work), raw], dim=0)
    conv = sum(padded[j:j + T] * kernel[:, j] for j in range(taps)) + bias
    conv = ar.rb(silu(conv))
    x = conv[:, :inner].reshape(T, H, e)
    B = conv[:, inner:inner + G * N].reshape(T, G, N)
    C = conv[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[prefix + "dt_bias"].to(ar.work))
    rate = torch.exp(w[prefix + "A_log"].to(ar.work))
    D = w[prefix + "D"].to(ar.work)
    group = [i // (H // G) for i in range(H)]
    S = torch.zeros(H, N, e, dtype=ar.work)
    y = torch.zeros(T, H, e, dtype=ar.work)
    for t in range(T):
        b, c = B[t][group], C[t][group]
        S = torch.exp(-rate * dt[t])[:, None, None] * S + (dt[t][:, None] * b)[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hne,hn->he", S, c) + D[:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms_divide(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w[prefix + "norm"].to(ar.work)
    return ar.linear(y, w[prefix + "o"])


# ----------------------------------------------------------------------------- feed-forward


def dense(ar, h, w, prefix):
    u = torch.clamp(ar.linear(h, w[prefix + "up"]), min=0.0)
    return ar.linear(u * u, w[prefix + "down"])


def expert(ar, h, w, prefix):
    g, u = ar.linear(h, w[prefix + "gate"]), ar.linear(h, w[prefix + "up"])
    return ar.linear(silu(g) * u, w[prefix + "down"], keep=True)


def route(ar, h, w, prefix, top):
    """(chosen experts [tokens, top], their weights, all logits): the largest logits, a softmax over
    those alone."""
    z = ar.linear(h, w[prefix + "router"], keep=True)
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1), z


MARGINS = None      # a list, while a caller collects per-token routing margins (routing_margin below)


def mixture(ar, h, w, prefix, mlp):
    T, top = h.shape[0], mlp["router"]["top"]
    chosen, weight, z = route(ar, h, w, prefix, top)
    if MARGINS is not None:
        ordered = torch.sort(z, dim=-1, descending=True).values
        MARGINS.append(ordered[:, top - 1] - ordered[:, top] if top < z.shape[-1] else torch.full((T,), math.inf))
    out = torch.zeros(T, w[prefix + "e0.down"].shape[0], dtype=ar.work)
    for t in range(T):
        for e, c in zip(chosen[t].tolist(), weight[t]):
            out[t] += c * expert(ar, h[t:t + 1], w, f"{prefix}e{e}.")[0]
    if mlp.get("shared") is not None:
        out = out + expert(ar, h, w, prefix + "shared.")
    return ar.rb(out)


# ----------------------------------------------------------------------------- the model


def model_forward(folder, tokens, precision=torch.float64, model=None):
    """(logits [tokens, vocab], the residual stream after every layer [layers, tokens, width])."""
    config, w = model if model is not None else read_model(folder)
    ar = Arithmetic(precision)
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.int64)
    positions = torch.arange(tokens.shape[0])
    x = embed(w, config, tokens, ar.work)
    after = []
    for i, layer in enumerate(config["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        n = ar.rb(rms_divide(x, eps) * w[p + "norm1"].to(ar.work))
        if kind == "wkv":
            x = x + time_mixing(ar, n, w, p + "mix.", m, eps)
        elif kind == "latent_attention":
            x = x + latent_attention(ar, n, w, p + "mix.", m, eps, positions)
        elif kind == "mamba2":
            x = x + state_space(ar, n, w, p + "mix.", m, eps)
        else:
            raise ValueError(f"layer {i}: type {kind!r}")
        mlp = layer.get("mlp")
        if mlp is not None:
            n = ar.rb(rms_divide(x, eps) * w[p + "norm2"].to(ar.work))
            x = x + (dense(ar, n, w, p + "mlp.") if mlp["kind"] == "dense" else mixture(ar, n, w, p + "mlp.", mlp))
        after.append(x)
    n = ar.rb(rms_divide(x, eps) * w["final.norm"].to(ar.work))
    return ar.linear(n, w["head"], keep=True), torch.stack(after)


def model_logits(folder, tokens, precision=torch.float64, model=None):
    return model_forward(folder, tokens, precision, model)[0]


def routing_margin(folder, tokens):
    """Per token, over all routed layers, the smallest distance between the logit of the last expert
    chosen and that of the best one left out, in float64: how sure the routing is."""
    global MARGINS
    MARGINS = []
    try:
        model_forward(folder, tokens, torch.float64)
        return torch.stack(MARGINS).min(0).values if MARGINS else torch.full((len(tokens),), math.inf)
    finally:
        MARGINS = None


def greedy(folder, prompt, n_new, precision=torch.float64):
    model = read_model(folder)
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(model_forward(folder, tokens, precision, model)[0][-1].argmax()))
    return tokens[len(prompt):]
