"""Small Turutar configurations of the tests' own, each unlike the others in every size and option, and
model folders with random weights for them.  Sizes visit the corners: both mixers first, in the middle and
last; heads that share keys, one key head for all, none shared; heads of 9 to 128 entries, sizes that the
tensor-core kernels take, pad and refuse; windows of 1, of less than a page, of exactly one, of one more, and
none; latents larger and smaller than what is read out of them; values smaller than, equal to and larger
than the keys; no rotated part; layers without a feed-forward; limits that nearly always and hardly ever
bite; loops over the first, the last, the middle and a single layer, two to four times, and no loop; a token
part of 5 to 40 columns, and none; widths and vocabularies that are no multiple of eight."""

import json
import os

import torch


def attention(heads, kv_heads, dim, scale, window, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


CONFIGS = {
    # two heads on each key head; a loop that starts behind the first layer and ends with the last; the values
    # of the latent layer are larger than its keys
    "a": dict(vocab=200, width=48, eps=1e-5, loop=(1, 3, 2), side=10, seed=61, layers=[
        attention(4, 2, 12, 0.4, 20, dense(40, 0.6)),
        latent(3, 10, 6, 20, 14, 22, 0.3, dense(56, 2.5)),
        attention(6, 2, 10, 0.35, 33, None),
    ]),
    # sizes that the tensor-core kernels take as they are; one key head for all; a window of one page; three
    # passes over the first two layers, one layer behind them
    "b": dict(vocab=304, width=72, eps=3e-6, loop=(0, 2, 3), side=16, seed=62, layers=[
        attention(4, 1, 32, 0.2, 64, dense(48, 1.5)),
        latent(2, 48, 16, 64, 24, 40, 0.15, None, base=500.0),
        attention(2, 2, 48, 0.15, 5, dense(64, 7.0)),
    ]),
    # nothing a multiple of eight; no loop and no token part; a window of one token, and none; no rotated part
    "c": dict(vocab=333, width=100, eps=2e-5, loop=None, side=0, seed=63, layers=[
        latent(3, 9, 0, 18, 7, 11, 0.25, dense(30, 0.3)),
        attention(3, 3, 9, 0.6, 1, dense(50, 4.0)),
        attention(5, 1, 13, 0.3, None, None),
    ]),
    # heads of 128 (the tcgen05 prompt kernel), a window of one more than a page; latent values that are padded
    # to the keys' size; four passes over one layer in the middle
    "d": dict(vocab=97, width=80, eps=1e-6, loop=(1, 2, 4), side=40, seed=64, layers=[
        latent(2, 96, 32, 96, 50, 16, 0.09, dense(72, 1.0), base=100.0),
        attention(3, 1, 128, 0.09, 65, dense(24, 0.9)),
        attention(2, 2, 96, 0.1, 130, dense(40, 3.0)),
    ]),
    # a token part that is no whole 16-byte piece, and a loop over everything
    "e": dict(vocab=120, width=64, eps=1e-4, loop=(0, 2, 2), side=5, seed=65, layers=[
        latent(4, 16, 16, 16, 16, 16, 0.2, None, base=30.0),
        attention(8, 4, 16, 0.3, 64, dense(64, 1.2)),
    ]),
}


def config_json(name):
    c = CONFIGS[name]
    out = {"architecture": "Turutar", "vocab": c["vocab"], "width": c["width"], "norm": {"eps": c["eps"]}, "layers": c["layers"]}
    if c["loop"] is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), c["loop"]))
    if c["side"]:
        out["token_side"] = {"dim": c["side"]}
    return out


def write_model(folder, name, dtype=torch.bfloat16):
    """Random weights through the library's random-weights mode (stored in bfloat16, as served models
    are), with matrices wide enough that attention weights are far from uniform, layer scales of either
    sign, and biases, sinks and norms inside the mixers of the order of what they stand beside."""
    from thing_htn_2026_b200.config import config_from_dict
    from thing_htn_2026_b200.weights import random_tensors_cpu
    from thing_htn_2026_b200.weights.safetensors_io import write_safetensors
    config = config_from_dict(config_json(name))
    tensors = random_tensors_cpu(config, CONFIGS[name]["seed"], dtype, matrix_std=0.12, gain_std=0.15)
    for i, key in enumerate(sorted(tensors)):
        g = torch.Generator().manual_seed(CONFIGS[name]["seed"] * 1000 + i)
        if key.endswith((".ls1", ".ls2")):
            tensors[key] = (torch.randn(tensors[key].shape, generator=g) * 0.5 + 0.4).to(dtype)
        elif key.endswith((".q.b", ".k.b")):
            tensors[key] = (torch.randn(tensors[key].shape, generator=g) * 0.6).to(dtype)
        elif key.endswith(".sink"):
            tensors[key] = (torch.randn(tensors[key].shape, generator=g) + 3.5).to(dtype)
        elif key == "embed":
            tensors[key] = (torch.randn(tensors[key].shape, generator=g) * torch.rand(tensors[key].shape[0], 1, generator=g)).to(dtype)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(config_json(name), handle, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    return folder


def tokens(name, length, seed):
    g = torch.Generator().manual_seed(9700 + seed)
    return torch.randint(0, CONFIGS[name]["vocab"], (length,), generator=g).tolist()
