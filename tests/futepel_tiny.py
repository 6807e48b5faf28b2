"""Small Futepel configurations of the tests' own, each unlike the others in every size and option,
and model folders with random weights for them.  Sizes visit the corners: every order of the three
mixers; time mixing with heads of 10 to 130, a single head, a rank of 1 to 16; latent attention whose
values are smaller than, equal to and larger than its keys, with sizes that the tensor-core kernels
take, pad and refuse, with and without a rotated part, with and without frequency scaling; state-space
layers with 1 to 5 taps, states of 3 to 130, one group for all heads, one per head and between, a norm
over one part, over parts of several heads and over parts that cut heads; dense feed-forwards, one,
several and all experts per token, with and without a shared one of its own size; layers without a
feed-forward; a model without pairs; widths and vocabularies that are no multiple of eight."""

import json
import os

import torch


def wkv(heads, dim, rank, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank": rank}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, mlp, base=10000.0, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def mamba2(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


CONFIGS = {
    # small odd heads; three groups over six heads; a norm whose parts cut heads; values larger than keys
    "a": dict(vocab=200, width=48, eps=1e-5, scale=6.0, bigram=(31, 7, 5), positions=300, seed=51, layers=[
        wkv(3, 10, 5, moe(5, 2, 24, shared=40)),
        latent(3, 10, 6, 20, 22, 0.3, dense(56)),
        mamba2(6, 5, 7, 3, 4, 2, None),
        wkv(3, 10, 5, dense(56)),
        mamba2(6, 5, 7, 3, 4, 2, moe(5, 2, 24)),
    ]),
    # sizes that the tensor-core kernels take as they are; one group; parts of one head; every expert chosen;
    # scaled frequencies; two taps
    "b": dict(vocab=304, width=72, eps=3e-6, scale=1.0, bigram=(500, 3, 1000003), positions=256, seed=52, layers=[
        mamba2(4, 16, 16, 1, 2, 4, moe(4, 4, 48)),
        latent(2, 48, 16, 64, 40, 0.2, moe(4, 4, 48), base=500.0, scaling=(8.0, 64, 16.0, 1.0)),
        wkv(1, 64, 16, None),
    ]),
    # nothing a multiple of eight; no pairs; no rotated part; heads of 130 and a state of 130; one tap; one group
    # per head; one part; one expert per token; a rank of one
    "c": dict(vocab=333, width=100, eps=2e-5, scale=12.0, bigram=None, positions=299, seed=53, layers=[
        latent(3, 9, 0, 18, 11, 0.25, moe(7, 1, 30, shared=50)),
        wkv(2, 130, 1, moe(7, 1, 30, shared=50)),
        mamba2(2, 33, 130, 2, 1, 1, dense(30)),
    ]),
    # values that are padded to the keys' tensor-core size, and keys of two rotated entries only beside plain
    # ones; scaling whose ramp is one step wide; five taps; a state of three
    "d": dict(vocab=97, width=40, eps=1e-6, scale=3.0, bigram=(1, 1, 1), positions=1000, seed=54, layers=[
        latent(4, 32, 32, 24, 16, 0.15, dense(64), base=100.0, scaling=(2.5, 40, 4.0, 4.0)),
        mamba2(3, 20, 3, 3, 5, 3, moe(3, 2, 16, shared=8)),
        wkv(2, 16, 3, moe(3, 2, 16)),
        latent(1, 14, 2, 16, 8, 0.4, None, base=30.0),
    ]),
}


def config_json(name):
    c = CONFIGS[name]
    embedding = {"scale": c["scale"]}
    if c["bigram"] is not None:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), c["bigram"]))
    return {"architecture": "Futepel", "vocab": c["vocab"], "width": c["width"], "embedding": embedding,
            "max_positions": c["positions"], "norm": {"eps": c["eps"]}, "layers": c["layers"]}


def write_model(folder, name, dtype=torch.bfloat16):
    """Random weights through the library's random-weights mode (stored in bfloat16, as served models
    are), with matrices wide enough that attention weights are far from uniform.  Router matrices are
    wider still, so that a rounding seldom decides which expert is chosen; the tables of pairs and
    positions are of the order of the stream, so that a wrong row shows."""
    from thing_htn_2026_b200.config import config_from_dict
    from thing_htn_2026_b200.weights import random_tensors_cpu
    from thing_htn_2026_b200.weights.safetensors_io import write_safetensors
    config = config_from_dict(config_json(name))
    tensors = random_tensors_cpu(config, CONFIGS[name]["seed"], dtype, matrix_std=0.12, gain_std=0.1)
    for key in tensors:
        if key.endswith(".mlp.router"):
            tensors[key] = (tensors[key].float() * 3.0).to(dtype)
        elif key in ("bigram", "pos"):
            tensors[key] = (tensors[key].float() * 4.0).to(dtype)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(config_json(name), handle, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    return folder


def tokens(name, length, seed):
    g = torch.Generator().manual_seed(9100 + seed)
    return torch.randint(0, CONFIGS[name]["vocab"], (length,), generator=g).tolist()
