"""The Turutar decoder on the device against the plain implementation (tests/plain/turutar_plain.py): each
mechanism alone (the embedding behind a norm; layer scale and added rows in the residual kernel; the token
part; clamped feed-forwards; two latents in one launch; both mixers), single keys made to decide the output
on either side of a window's edge, sinks that take nearly all or nearly nothing, then whole models through the
replay program (whole prompts, token-by-token decoding, prompts cut into portions, batches of unequal
requests, slots and pages used again), and greedy generation through the library's entry point."""

import math
import warnings

import numpy as np
import pytest
import torch

import harness
import turutar_tiny as tiny
from plain import turutar_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("turutar_models")
    return {name: tiny.write_model(str(root / name), name) for name in tiny.CONFIGS}


# ----------------------------------------------------------------------------- comparison

_oracle = {}


def oracle(folder, tokens, precision):
    key = (folder, tuple(tokens), precision)
    if key not in _oracle:
        _oracle[key] = plain.model_logits(folder, list(tokens), precision).numpy()
    return _oracle[key]


def position_error(got, want):
    """Per position: root mean square over the vocabulary of the difference, its mean taken off."""
    d = got.astype(np.float64) - want.astype(np.float64)
    d = d - d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1))


def check_logits(got, folder, tokens, dtype, what):
    """float32: within a few float32 roundings of the plain float32 result.  bfloat16, against exact
    arithmetic and measured by the plain implementation's own bfloat16 emulation: the worst place no
    worse than twice the emulation's worst place, the mean no more than one and a half times its
    mean."""
    assert got.shape[0] == len(tokens), f"{what}: {got.shape[0]} rows for {len(tokens)} places"
    exact = oracle(folder, tokens, torch.float64)
    spread = max(1.0, float(np.abs(exact).max()))
    if dtype == "float32":
        err = position_error(got, oracle(folder, tokens, torch.float32))
        assert err.max() <= 3e-5 * spread, f"{what}: float32 logits differ by {err.max():.3e} at place {int(err.argmax())}"
        return
    noise = position_error(oracle(folder, tokens, torch.bfloat16), exact)
    err = position_error(got, exact)
    worst = int(err.argmax())
    assert err.max() <= 2.0 * noise.max() + 3e-3 * spread, (
        f"{what}: bfloat16 logits are {err[worst]:.3e} from exact at place {worst}, the emulation's worst {noise.max():.3e}")
    assert err.mean() <= 1.5 * noise.mean() + 1.5e-3 * spread, (
        f"{what}: bfloat16 logits are {err.mean():.3e} from exact on average, the emulation {noise.mean():.3e}")


def run_trace(folder, dtype, records, tmp_path, requests, what, max_tokens=None):
    out = harness.replay(folder, dtype, records, str(tmp_path / what.replace(" ", "_")), max_tokens)
    for name, toks in requests.items():
        check_logits(out[name], folder, toks, dtype, f"{what} {name}")
    return out


def trace_portions(requests, sizes):
    """Each request alone, its tokens brought in portions of the given sizes (the last size repeats)."""
    records, step = [], 0
    for name, toks in requests.items():
        at, k = 0, 0
        while at < len(toks):
            n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
            records.append({"step": step, "entries": [{"id": name, "tokens": toks[at:at + n], "want": list(range(n))}],
                            "end": [name] if at + n == len(toks) else []})
            at, k, step = at + n, k + 1, step + 1
    return records


def rand(shape, seed, scale=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, what, loose=1.0):
    got, want = got.float().cpu(), want.float().cpu()
    if dtype == "float32":
        err = (got - want).abs().max().item()
        assert err <= 3e-5 * loose * max(1.0, want.abs().max().item()), f"{what}: float32 differs by {err:.3e}"
    else:
        bad = (got - want).abs() > loose * (3e-2 * max(1.0, want.abs().max().item() / 4) + want.abs() / 16)
        assert bad.sum() <= bad.numel() // 200, f"{what}: {int(bad.sum())} of {bad.numel()} bfloat16 values out of tolerance"


def part_of(folder, layer_index, member, dtype):
    """One member part of a layer of a written model, built as the model builds it."""
    from thing_htn_2026_b200.config import load_config
    from thing_htn_2026_b200.parts import Runtime, part_class
    from thing_htn_2026_b200.weights.loader import load_tensors
    config = load_config(folder)
    spec = config.plan().layers[layer_index].block.params[member]
    cls = part_class(member, spec.kind)
    with warnings.catch_warnings():
        warnings.simplefilter("ignore")
        tensors = load_tensors(folder, cls.tensor_specs(spec), TORCH[dtype], torch.device(DEV), ignored=("*",))
    runtime = Runtime(TORCH[dtype], torch.device(DEV), tensors)
    part = cls(spec, runtime)
    for shared in runtime.shared.values():
        shared.ensure(4096)
    return part, config


class Stepper:
    """Feeds rows to a mixer through a cache of its own, as the step function would."""

    def __init__(self, mixer, dtype, n_slots=3):
        from thing_htn_2026_b200 import ops
        from thing_htn_2026_b200.cache import SequenceCache
        self.ops, self.mixer = ops, mixer
        self.cache = SequenceCache([mixer.cache_need()], max_tokens=64 * 40, dtype=TORCH[dtype], device=DEV, max_slots=n_slots)
        self.err = ops.new_error_word(DEV)

    def step(self, slots, xs):
        from thing_htn_2026_b200.config.base import ScheduleEntry
        from thing_htn_2026_b200.parts import HostBatch, StepContext
        counts = [x.shape[0] for x in xs]
        held = [self.cache.length(s) for s in slots]
        self.cache.prepare(slots, counts)
        cu = [0]
        for c in counts:
            cu.append(cu[-1] + c)
        cu_dev = torch.tensor(cu, dtype=torch.int32, device=DEV)
        slots_dev = torch.tensor(slots, dtype=torch.int32, device=DEV)
        rows = self.ops.step_rows(cu_dev, slots_dev, self.cache.seq_lens, cu[-1], max(counts))
        asked = {}
        self.mixer.step_inputs(HostBatch(slots, counts, held, 64), asked)
        inputs = {k: torch.tensor(v, dtype=torch.int32, device=DEV) for k, v in asked.items()}
        ctx = StepContext(rows=rows, cache=self.cache, err=self.err, inputs=inputs)
        a = self.mixer.forward(torch.cat(xs).to(DEV).contiguous(), ctx, ScheduleEntry(0, 0))
        self.ops.advance(self.cache.seq_lens, slots_dev, cu_dev)
        self.cache.commit(slots, counts)
        assert int(self.err.item()) == 0
        return [a[lo:hi] for lo, hi in zip(cu[:-1], cu[1:])]


# ----------------------------------------------------------------------------- embedding, residual, token part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [7, 48, 256, 2048, 4104, 10000])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_an_embedding_behind_a_norm(dtype, width, offset):
    """Rows of very different lengths; the copy is the same rows in memory of its own."""
    from thing_htn_2026_b200 import ops
    t = TORCH[dtype]
    table, gain = (rand((9, width), 1) * torch.logspace(-3, 2, 9)[:, None]).to(t), rand((width,), 2)
    toks = [8, 0, 3, 3, 7, 1]
    err = ops.new_error_word(DEV)
    args = (table.to(DEV), torch.tensor(toks, dtype=torch.int32, device=DEV), ops.Gain(gain.to(DEV), offset, 1e-4), err)
    once, none = ops.embed_norm(*args)
    out, kept = ops.embed_norm(*args, copy=True)
    want = plain.rms_divide(table.double()[toks], 1e-4) * (offset + gain.double())
    assert none is None and out.data_ptr() != kept.data_ptr() and torch.equal(out, kept) and torch.equal(once, out)
    assert out.dtype == torch.float32 and (out.cpu() - want).abs().max() <= 2e-6 * want.abs().max()
    assert int(err.item()) == 0
    bad, _ = ops.embed_norm(args[0], torch.tensor([1, 9, -1], dtype=torch.int32, device=DEV), *args[2:])
    assert int(err.item()) == ops.ERR_TOKEN_RANGE and torch.isfinite(bad).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [9, 48, 1000, 4096])
def test_layer_scale_and_added_rows_in_the_residual_kernel(dtype, width):
    """Every combination of the outputs with factors, a branch behind a norm and rows to add, each with and
    without a norm of the sum; the factors differ from entry to entry and in sign."""
    from thing_htn_2026_b200 import ops
    t, rows = TORCH[dtype], 5
    h0, rest = rand((rows, width), 1), rand((rows, width), 2)
    a, f, d = (rand((rows, width), s).to(t) for s in (3, 4, 5))
    s1, s2 = rand((width,), 6), rand((width,), 7)
    post = ops.Gain((1 + rand((width,), 8) * 0.1).to(DEV), 0.0, 1e-3)
    gain = ops.Gain((rand((width,), 9) * 0.1).to(DEV), 1.0, 1e-3)
    for with_d in (False, True):
        for with_f in (None, False, True):
            for with_rows in (False, True):
                h = h0.clone().to(DEV)
                want = h0.double()
                if with_f is not None:
                    want = want + a.double() * s1.double() + (f.double() * s2.double() if with_f else 0.0)
                if with_d:
                    want = want + plain.rms_divide(d.double(), 1e-3) * post.weight.cpu().double()
                if with_rows:
                    want = want + rest.double()
                scaled = None if with_f is None else ops.ScaledPair(a.to(DEV), s1.to(DEV), f.to(DEV) if with_f else None,
                                                                    s2.to(DEV) if with_f else None)
                kw = dict(scaled=scaled, add_rows=rest.to(DEV) if with_rows else None)
                branch = d.to(DEV) if with_d else None
                if with_d or with_f is not None or with_rows:
                    _, none = ops.residual_norm(h, branch, post if with_d else None, None, t, **kw)
                    assert none is None and (h.cpu() - want).abs().max() <= 3e-6 * want.abs().max(), (with_d, with_f, with_rows)
                h = h0.clone().to(DEV)
                _, y = ops.residual_norm(h, branch, post if with_d else None, gain, t, **kw)
                assert (h.cpu() - want).abs().max() <= 3e-6 * want.abs().max(), (with_d, with_f, with_rows)
                close(y, plain.rms_divide(want, 1e-3) * (1 + gain.weight.cpu().double()), dtype, "norm of the sum", 0.3)
                h = h0.clone().to(DEV)
                _, y = ops.residual_norm(h, branch, post if with_d else None, ops.STREAM_AS_IS, t, **kw)
                assert torch.equal(y, h.to(t))


def test_what_the_residual_kernel_refuses():
    from thing_htn_2026_b200 import ops
    h, a = torch.zeros(3, 8, device=DEV), torch.zeros(3, 8, device=DEV)
    with pytest.raises(ops.KernelError, match="factors"):
        ops.residual_norm(h, None, None, None, torch.float32, scaled=ops.ScaledPair(a, torch.zeros(7, device=DEV)))
    with pytest.raises(ops.KernelError, match="rows to add"):
        ops.residual_norm(h, None, None, None, torch.float32, add_rows=torch.zeros(2, 8, device=DEV))
    with pytest.raises(ops.KernelError, match="nothing"):
        ops.residual_norm(h, None, None, None, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows, width, dim, column, table_width", [
    (1, 48, 10, 20, 30), (5, 64, 5, 0, 10), (33, 72, 16, 32, 48), (16, 2048, 128, 256, 512), (17, 2048, 128, 0, 128), (3, 100, 7, 3, 11),
    (300, 256, 24, 24, 96), (2, 4096, 256, 256, 2048), (40, 12, 3, 2, 5)])
def test_the_gate_of_the_token_part(dtype, rows, width, dim, column, table_width):
    """Products from far below zero to far above; the columns of this layer only; the kernel with the
    product and the one behind a product."""
    from thing_htn_2026_b200 import ops
    t = TORCH[dtype]
    x, w = rand((rows, width), 1).to(t), rand((dim, width), 2, 3.0 / math.sqrt(width)).to(t)
    table = rand((50, table_width), 3).to(t)
    toks = torch.randint(0, 50, (rows,), generator=torch.Generator().manual_seed(4))
    toks[0] = 49
    z = x.double() @ w.double().t()
    want = torch.nn.functional.gelu(z, approximate="tanh") * table.double()[toks, column:column + dim]
    err = ops.new_error_word(DEV)
    args = (x.to(DEV), w.to(DEV), table.to(DEV), toks.to(torch.int32).to(DEV), column, err)
    for fused in [None, False] + ([True] if dtype == "bfloat16" and width % 8 == 0 else []):
        close(ops.token_gate(*args, fused=fused), want, dtype, f"token gate, fused {fused}", 0.3)
    assert int(err.item()) == 0
    bad = toks.clone()
    bad[-1] = 50
    for fused in [False] + ([True] if dtype == "bfloat16" and width % 8 == 0 else []):
        ops.token_gate(*args[:3], bad.to(torch.int32).to(DEV), column, err, fused=fused)
        assert int(err.item()) == ops.ERR_TOKEN_RANGE
        err.zero_()


@pytest.mark.parametrize("rows, width, dim, second", [(1, 48, 10, True), (8, 2048, 128, True), (16, 72, 16, False), (5, 4096, 256, True),
                                                      (3, 8, 3, True), (2, 16384, 5, True)])
def test_the_gate_of_the_token_part_behind_pending_outputs(rows, width, dim, second):
    """The kernel that adds up the stream and what is pending on it for itself: the same bits as adding
    first, and the stream stays as it is."""
    from thing_htn_2026_b200 import ops
    bf = torch.bfloat16
    h, a, f = rand((rows, width), 1).to(DEV), rand((rows, width), 2).to(bf).to(DEV), rand((rows, width), 3).to(bf).to(DEV)
    s1, s2 = rand((width,), 4).to(DEV), rand((width,), 5).to(DEV)
    w, table = rand((dim, width), 6, 2.0 / math.sqrt(width)).to(bf).to(DEV), rand((20, 2 * dim), 7).to(bf).to(DEV)
    toks = torch.arange(rows, dtype=torch.int32, device=DEV) + 2
    err = ops.new_error_word(DEV)
    pair = ops.ScaledPair(a, s1, f if second else None, s2 if second else None)
    before = h.clone()
    got = ops.token_gate_pending(h, pair, w, table, toks, dim, err)
    assert torch.equal(h, before)
    _, x = ops.residual_norm(h, None, None, ops.STREAM_AS_IS, bf, scaled=pair)
    assert torch.equal(got, ops.token_gate(x, w, table, toks, dim, err, fused=True))
    z = x.cpu().double() @ w.cpu().double().t()
    want = torch.nn.functional.gelu(z, approximate="tanh") * table.cpu().double()[2:2 + rows, dim:]
    close(got, want, "bfloat16", "token gate behind pending outputs", 0.3)
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", [n for n in tiny.CONFIGS if tiny.CONFIGS[n]["side"]])
def test_the_token_part_alone(models, dtype, name):
    """Every layer's part behind a stream of its own, few rows and many, against the plain mechanism."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.parts import StepContext
    data, w = plain.read_model(models[name])
    t, eps = TORCH[dtype], data["norm"]["eps"]
    ar = plain.Arithmetic(torch.float32 if dtype == "float32" else torch.bfloat16)
    for layer in range(len(data["layers"])):
        side, config = part_of(models[name], layer, "side", dtype)
        for rows in (1, 9, 60):
            h = rand((rows, config.width), layer + rows)
            toks = tiny.tokens(name, rows, layer)
            ctx = StepContext(rows=None, cache=None, err=ops.new_error_word(DEV), tokens=torch.tensor(toks, dtype=torch.int32, device=DEV))
            branch = side.forward(h.to(t).to(DEV), ctx)
            got = h.to(DEV)
            ops.residual_norm(got, branch.tensor, branch.norm.as_gain, None, t)
            want = plain.token_side(ar, h, torch.tensor(toks), w, layer, data["token_side"]["dim"], eps)
            close(got.cpu() - h, want, dtype, f"token part of layer {layer}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("first, second, gap", [(14, 22, 0), (64, 16, 3), (1, 700, 8), (1536, 512, 32)])
def test_two_latents_in_one_launch(dtype, first, second, gap):
    from thing_htn_2026_b200 import ops
    t, eps = TORCH[dtype], 1e-3
    proj = (rand((6, first + gap + second + 5), 1) * torch.logspace(-2, 2, 6)[:, None]).to(t)
    g1, g2 = rand((first,), 2), rand((second,), 3)
    a, b = ops.latent_norm(proj.to(DEV), 0, first, g1.to(DEV), eps, second=(first + gap, second, g2.to(DEV)))
    close(a, plain.rms_divide(proj.double()[:, :first], eps) * g1.double(), dtype, "first latent", 0.3)
    close(b, plain.rms_divide(proj.double()[:, first + gap:first + gap + second], eps) * g2.double(), dtype, "second latent", 0.3)
    assert torch.equal(a, ops.latent_norm(proj.to(DEV), 0, first, g1.to(DEV), eps))


FEED_FORWARDS = [(name, i) for name in sorted(tiny.CONFIGS) for i, layer in enumerate(tiny.CONFIGS[name]["layers"])
                 if layer["mlp"] is not None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, layer", FEED_FORWARDS)
def test_feed_forward_alone(models, dtype, name, layer):
    """Inputs so large that both clamps bite on either side."""
    part, config = part_of(models[name], layer, "ffn", dtype)
    mlp = tiny.config_json(name)["layers"][layer]["mlp"]
    _, w = plain.read_model(models[name])
    x = rand((33, config.width), 8 + layer, 4.0).to(TORCH[dtype])
    ar = plain.Arithmetic(torch.float32 if dtype == "float32" else torch.bfloat16)
    prefix = f"l{layer}.mlp."
    up, gate = x.float() @ w[prefix + "up"].t(), x.float() @ w[prefix + "gate"].t()
    assert (up > mlp["limit"]).any() and (up < -mlp["limit"]).any() and (gate > mlp["limit"]).any()
    close(part.forward(x.to(DEV), None), plain.clamped_feed_forward(ar, x.float(), w, prefix, mlp["limit"]), dtype, "feed-forward")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inter, offset, more", [(40, 16, 0), (56, 8, 24), (7, 3, 2), (4096, 2568, 0)])
def test_gates_and_ups_out_of_wider_rows(dtype, inter, offset, more):
    from thing_htn_2026_b200 import ops
    t = TORCH[dtype]
    proj = rand((9, offset + 2 * inter + more), 1, 2.0).to(t)
    g, u = (proj.double()[:, offset + k * inter:offset + (k + 1) * inter] for k in (0, 1))
    g, u = g.clamp(max=1.5), u.clamp(-1.5, 1.5)
    close(ops.clamped_glu(proj.to(DEV), 1.5, 1.702, offset, inter), g * torch.sigmoid(1.702 * g) * (u + 1.0), dtype, "slice", 0.3)
    with pytest.raises(ops.KernelError, match="hold no"):
        ops.clamped_glu(proj.to(DEV), 1.5, 1.702, offset + more + 1, inter)


def test_work_beside_the_current_stream():
    """What a second stream computes from what came before it, read after the join, again and again over the
    same memory; counters of its own; not nested; the same in a captured graph."""
    from thing_htn_2026_b200 import ops
    beside = ops.Beside(DEV)
    x, w1, w2 = rand((8, 4096), 1).to(torch.bfloat16).to(DEV), rand((256, 4096), 2, 0.02).to(torch.bfloat16).to(DEV), rand((384, 4096), 3, 0.02).to(torch.bfloat16).to(DEV)
    err = ops.new_error_word(DEV)

    def both(x):
        y = ops.linear_stream(x, w1, err=err)
        for _ in range(3):
            z = ops.squared_relu(x)
            with beside:
                f = ops.linear_stream(z, w2, err=err)
                with pytest.raises(ops.KernelError, match="nested"):
                    with beside:
                        pass
            y = y + ops.linear_stream(z, w1, err=err)
            beside.join()
            y = y + f[:, :256]
        return y

    with torch.inference_mode():
        z = ops.squared_relu(x)
        want = ops.linear_stream(x, w1)
        for _ in range(3):
            want = want + ops.linear_stream(z, w1) + 0.0
            want = want + ops.linear_stream(z, w2)[:, :256]
        for _ in range(5):
            assert torch.equal(both(x), want)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            out = both(x)
        for _ in range(5):
            graph.replay()
        torch.cuda.synchronize()
        assert torch.equal(out, want) and int(err.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "c", "d"])
def test_one_product_for_both_sublayers(models, dtype, name):
    """A layer whose sublayers share their input product holds every weight once and gives what the
    sublayers give with products of their own, alone and on two streams."""
    from thing_htn_2026_b200.config import load_config
    from thing_htn_2026_b200.engine.loading import load_model
    model = load_model(models[name], dtype, DEV)
    for i, layer in enumerate(load_config(models[name]).to_dict()["layers"]):
        block = model.layers[i]
        if layer["mlp"] is None:
            assert block.w_in is None and block.ffn is None
            continue
        assert block.w_in.shape[0] % 8 == 0 and block.ffn_offset % 8 == 0
        assert block.ffn.w_gate_up.data_ptr() == block.w_in[block.ffn_offset:].data_ptr()
        own = block.mixer.w_qkv if layer["type"] == "attention" else block.mixer.w_in
        assert own.data_ptr() == block.w_in.data_ptr()
        x = rand((5, block.w_in.shape[1]), i).to(TORCH[dtype]).to(DEV)
        from thing_htn_2026_b200 import ops
        proj = ops.linear(x, block.w_in, bias=block.b_in)
        close(block.ffn.forward_rows(proj, block.ffn_offset, None), block.ffn.forward(x, None), dtype, f"layer {i}", 0.3)


# ----------------------------------------------------------------------------- mixers alone


def plain_mixer(folder, layer, x, ar):
    config, w = plain.read_model(folder)
    entry = config["layers"][layer]
    mixer = plain.window_attention if entry["type"] == "attention" else plain.latent_attention
    return mixer(ar, x, w, f"l{layer}.mix.", entry["mixer"], config["norm"]["eps"])


MIXERS = [(name, i) for name in sorted(tiny.CONFIGS) for i in range(len(tiny.CONFIGS[name]["layers"]))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, layer", MIXERS)
def test_mixers_alone_whole_in_portions_and_token_by_token(models, dtype, name, layer):
    """Every mixer of the tiny models against the plain mechanism, for a sequence brought whole, in
    portions of unequal sizes down to two and one (across page borders and window edges), beside another
    sequence, token by token at its end, and in a slot that was used before."""
    folder = models[name]
    mixer, config = part_of(folder, layer, "mixer", dtype)
    ar = plain.Arithmetic(torch.float32 if dtype == "float32" else torch.bfloat16)
    t = TORCH[dtype]
    T = 150
    x, ox = rand((T, config.width), 100 + layer).to(t), rand((31, config.width), 200 + layer).to(t)
    want, want_other = plain_mixer(folder, layer, x.float(), ar), plain_mixer(folder, layer, ox.float(), ar)
    stepper = Stepper(mixer, dtype)
    s0, s1, s2 = stepper.cache.open(3)
    whole = stepper.step([s0], [x])
    close(whole[0], want, dtype, "whole")
    cuts = [0, 1, 3, 5, 63, 64, 66, 128, 130] + list(range(131, T + 1))
    got, got_other, at = [], [], 0
    for lo, hi in zip(cuts[:-1], cuts[1:]):
        if at < ox.shape[0]:
            n = min(hi - lo + 1, ox.shape[0] - at)
            a = stepper.step([s2, s1], [ox[at:at + n], x[lo:hi]])
            got_other.append(a[0]), got.append(a[1])
            at += n
        else:
            got.append(stepper.step([s1], [x[lo:hi]])[0])
    close(torch.cat(got), want, dtype, "in portions and token by token")
    close(torch.cat(got_other), want_other, dtype, "the sequence beside it")
    if dtype == "float32":
        # what a position gets must not depend on the cut beyond rounding
        assert (torch.cat(got) - whole[0]).abs().max() <= 2e-5 * max(1.0, whole[0].abs().max().item())
    stepper.cache.close([s0])
    (again,) = stepper.cache.open(1)
    assert again == s0
    close(stepper.step([again], [ox])[0], want_other, dtype, "a slot used again")


# ----------------------------------------------------------------------------- single keys made to show


def attention_part(t, weights, **params):
    from thing_htn_2026_b200.config.base import PartSpec
    from thing_htn_2026_b200.parts import Runtime, part_class
    names = {"q": "q_proj", "q.b": "q_bias", "k": "k_proj", "k.b": "k_bias", "q.norm": "q_norm", "k.norm": "k_norm", "g": "g_proj",
             "o": "o_proj"}
    spec = PartSpec("attention", {"qk_norm_eps": 1e-5, "qk_norm_scope": "projection", "values": "keys", "biases": ["q", "k"],
                                  "sinks": 0.0, "gate": "head", "softmax_weights": "float32", **params}, {v: k for k, v in names.items()})
    return part_class("mixer", "attention")(spec, Runtime(t, torch.device(DEV), {k: v.to(DEV) for k, v in weights.items()}))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, d, window", [
    (4, 2, 32, 5), (3, 3, 40, 1), (2, 1, 64, 64), (6, 2, 128, 65), (2, 2, 96, 130), (4, 4, 33, 20), (2, 1, 160, 63), (16, 1, 48, 2)])
def test_a_loud_key_just_inside_and_just_outside_the_window(dtype, heads, kv_heads, d, window):
    """One key among many is loud, and the tokens window - 1 and window behind it ask for it: the first gets
    nearly nothing but the loud token's value (its key as projected, with its bias and ahead of the norm),
    the second nothing of it.  The loud key stands at the start, around page borders and beyond; as one
    prompt, with the askers decoded, and in portions of two that leave freed pages behind."""
    t, hidden = TORCH[dtype], 264
    g = torch.Generator().manual_seed(heads * d + window)
    w = {"q": (heads * d, hidden), "q.b": (heads * d,), "k": (kv_heads * d, hidden), "k.b": (kv_heads * d,), "g": (heads, hidden)}
    w = {k: torch.randn(s, generator=g) * 0.1 for k, s in w.items()}
    loud_axis, ask_axis = hidden - 1, hidden - 2
    for k in ("q", "k", "g"):
        w[k][:, ask_axis:] = 0.0
    key = torch.randn(kv_heads, d, generator=g)
    key = key / key.norm(dim=1, keepdim=True) * d ** 0.5
    w["k"][:, loud_axis] = 3.0 * key.reshape(-1)
    w["q"][:, ask_axis] = 3.0 * key.repeat_interleave(heads // kv_heads, dim=0).reshape(-1)
    w["q.norm"], w["k.norm"] = torch.full((heads * d,), 1.5), torch.full((kv_heads * d,), 0.5)
    w["o"] = torch.eye(heads * d)
    w = {k: v.to(t) for k, v in w.items()}
    scale = 20.0 / d
    part = attention_part(t, w, hidden_size=hidden, n_heads=heads, n_kv_heads=kv_heads, head_dim=d, window=window, scale=scale)
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "scale": scale, "mask": {"size": window}}
    wide = {"x." + k: v.double() for k, v in w.items()}
    for loud in (0, 1, 62, 63, 64, 127, 150):
        T = loud + window + 2
        x = torch.randn(T, hidden, generator=g) * 0.1
        x[:, ask_axis:] = 0.0
        x[loud, loud_axis] = 1.0
        for asker in (loud + window - 1, loud + window):
            x[asker, ask_axis] = 1.0
        x = x.to(t)
        exact = plain.window_attention(plain.Arithmetic(torch.float64), x.double(), wide, "x.", m, 1e-5)
        value = (wide["x.k"] @ x[loud].double() + wide["x.k.b"]).reshape(kv_heads, d).repeat_interleave(heads // kv_heads, dim=0)
        gate = torch.sigmoid(x.double() @ wide["x.g"].t())
        inside, outside = loud + window - 1, loud + window
        want = (value * gate[inside][:, None]).reshape(-1)
        assert (exact[inside] - want).abs().max() < 0.02 * want.abs().max()
        assert exact[outside].abs().max() < 0.3 * want.abs().max()
        decoded = [1] * min(T - 1, window + 3)
        for cut in ([T], [T - len(decoded)] + decoded, [2] * (T // 2) + [1] * (T % 2)):
            stepper = Stepper(part, dtype)
            (slot,) = stepper.cache.open(1)
            outs, at = [], 0
            for n in cut:
                outs.append(stepper.step([slot], [x[at:at + n]])[0])
                at += n
            got = torch.cat(outs).double().cpu()
            tol = 2e-4 if dtype == "float32" else 4e-2
            assert (got - exact).abs().max() <= tol * exact.abs().max(), (loud, cut[:2])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, kv_heads", [(9, 3), (64, 1), (128, 3), (96, 3)])
def test_the_added_one_counts_once(dtype, d, kv_heads):
    """Queries of (nearly) nothing: every score is about zero, so a row's weights are one over the tokens
    it sees and the extra one, in prompts and in decoding; with a constant of ln 9 in its place nine more."""
    t, hidden, heads, window, T = TORCH[dtype], 40, 3, 70, 140
    g = torch.Generator().manual_seed(d)
    w = {"q": torch.zeros(heads * d, hidden), "q.b": torch.full((heads * d,), 1e-6), "k": torch.randn(kv_heads * d, hidden, generator=g),
         "k.b": torch.randn(kv_heads * d, generator=g) + 1.0, "q.norm": torch.full((heads * d,), 1e-3), "k.norm": torch.ones(kv_heads * d),
         "g": torch.zeros(heads, hidden), "o": torch.eye(heads * d)}
    w = {k: v.to(t) for k, v in w.items()}
    x = torch.randn(T, hidden, generator=g).to(t)
    v = (x.double() @ w["k"].double().t() + w["k.b"].double()).reshape(T, kv_heads, d).repeat_interleave(heads // kv_heads, dim=1)
    for sink, extra in ((0.0, 1), (math.log(9.0), 9)):
        part = attention_part(t, w, hidden_size=hidden, n_heads=heads, n_kv_heads=kv_heads, head_dim=d, window=window, scale=1e-4, sinks=sink)
        for head in (T, 3):
            stepper = Stepper(part, dtype)
            (slot,) = stepper.cache.open(1)
            outs = [stepper.step([slot], [x[:head]])[0]] + [stepper.step([slot], [x[i:i + 1]])[0] for i in range(head, T)]
            got = torch.cat(outs).double().cpu().reshape(T, heads, d)
            for i in (0, 1, 2, 5, 63, 64, 69, 70, 71, 139):
                seen = v[max(0, i - window + 1):i + 1]
                want = 0.5 * seen.sum(0) / (extra + len(seen))
                assert (got[i] - want).abs().max() <= (1e-5 if dtype == "float32" else 3e-2) * max(1.0, want.abs().max().item()), (sink, head, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, r, e, q_rank", [(4, 10, 6, 20, 12), (4, 32, 32, 64, 40), (2, 48, 16, 24, 8), (3, 16, 0, 16, 5),
                                                    (4, 96, 32, 96, 64), (1, 2, 2, 5, 3)])
def test_one_loud_latent_among_hundreds_beside_its_sink(dtype, heads, d, r, e, q_rank):
    """300 tokens of which one has a rotated key part that meets the last query's (read out of its latent)
    exactly, turned by their places, with a score of 20; the heads' sinks stand at 17, 20, -5 and 22.  The last
    row's read-out is the loud token's value times its share and the head's gate, in places on either side
    of page borders, as one prompt and with the last rows decoded.  Without a rotated part the plain keys are
    loud instead."""
    from thing_htn_2026_b200.config.base import PartSpec
    from thing_htn_2026_b200.parts import Runtime, part_class
    T, t, hidden, rank, score = 300, TORCH[dtype], 408, 24, 20.0
    names = ("q_down", "q_norm", "q_proj", "down_proj", "latent_norm", "up_k", "up_v", "sink", "g_proj", "o_proj")
    position = None if not r else PartSpec("rope", {"head_dim": r, "rotary_dim": r, "theta": 50.0, "layout": "interleaved",
                                                    "frequency_precision": "float64", "angle_precision": "float64"})
    spec = PartSpec("latent_attention", {"hidden_size": hidden, "n_heads": heads, "plain_dim": d, "rot_dim": r, "value_dim": e,
                                         "q_rank": q_rank, "latent_rank": rank, "scale": 1.0, "norm_eps": 1e-9, "position": position,
                                         "sinks": "learned", "gate_scope": "head", "softmax_weights": "float32"}, {n: n for n in names})
    g = torch.Generator().manual_seed(heads * d + r)
    shapes = {"q_down": (q_rank, hidden), "q_norm": (q_rank,), "q_proj": (heads * (d + r), q_rank), "down_proj": (rank + r, hidden),
              "latent_norm": (rank,), "up_k": (heads * d, rank), "up_v": (heads * e, rank), "g_proj": (heads, hidden)}
    w = {n: torch.randn(s, generator=g) * 0.12 for n, s in shapes.items()}
    w["o_proj"] = torch.eye(hidden, heads * e)
    w["sink"] = torch.tensor([17.0, 20.0, -5.0, 22.0])[:heads]
    # the last channel of either latent belongs to the asking and to the loud token alone
    for down, norm in (("q_down", "q_norm"), ("down_proj", "latent_norm")):
        last = (q_rank if down == "q_down" else rank) - 1
        w[down][:, hidden - 2:] = 0.0
        w[down][last] = 0.0
        w[norm][last] = 1.0
    w["g_proj"][:, hidden - 2:] = 0.0
    w["q_down"][q_rank - 1, hidden - 2] = 1.0
    w["down_proj"][rank - 1, hidden - 1] = 1.0
    w["q_proj"][:, q_rank - 1] = 0.0
    loud_direction, ask_direction = torch.eye(hidden)[hidden - 1], torch.eye(hidden)[hidden - 2]
    for loud in (0, 1, 63, 64, 128, 298, 299):
        u = {n: v.clone() for n, v in w.items()}
        if r:
            # the key in the loud direction, turned to its place, meets the asking token's query: turned back by the distance
            key = torch.randn(r, generator=g).double()
            key *= 5.0 / key.norm()
            u["down_proj"][rank:, hidden - 1] = key.float()
            key = u["down_proj"][rank:, hidden - 1].to(t).double()
            query = plain.rotate_neighbours(key[None], torch.tensor([loud - (T - 1)]), 50.0)[0] * score / (key @ key)
            for h in range(heads):
                u["q_proj"][h * (d + r) + d:(h + 1) * (d + r), q_rank - 1] = (query / q_rank ** 0.5).float()
        else:
            u["up_k"][:, rank - 1] *= 8.0
            for h in range(heads):
                k = u["up_k"][h * d:(h + 1) * d, rank - 1] * rank ** 0.5
                u["q_proj"][h * d:(h + 1) * d, q_rank - 1] = k * score / (k @ k) / q_rank ** 0.5
        x = torch.randn(T, hidden, generator=g) * 0.12
        x[:, hidden - 2:] = 0.0
        x[loud] = loud_direction
        x[T - 1] = ask_direction + (loud_direction if loud == T - 1 else 0.0)
        x = x.to(t)
        u = {n: v.to(t) for n, v in u.items()}
        part = part_class("mixer", "latent_attention")(spec, Runtime(t, torch.device(DEV), {n: v.to(DEV) for n, v in u.items()}))
        if part.position is not None:
            part.position.ensure(T)
        f = {n: v.double() for n, v in u.items()}
        c = plain.rms_divide((x.double() @ f["down_proj"].t())[loud, :rank], 1e-9) * f["latent_norm"]
        share = 1.0 / (1.0 + torch.exp(f["sink"] - score))
        gate = torch.sigmoid(x.double()[T - 1] @ f["g_proj"].t())
        value = (f["up_v"] @ c).view(heads, e) * (gate * share)[:, None]
        for first in (T, 290):
            stepper = Stepper(part, dtype)
            (slot,) = stepper.cache.open(1)
            out = stepper.step([slot], [x[:first]])[0]
            for i in range(first, T):
                out = stepper.step([slot], [x[i:i + 1]])[0]
            got = out[-1, :heads * e].double().cpu().view(heads, e)
            assert value.abs().max() > 0.02
            tol = 2e-3 if dtype == "float32" else 8e-2
            assert (got - value).abs().max() <= tol * value.abs().max(), (loud, first)


# ----------------------------------------------------------------------------- whole models


def requests_of(name, lengths, seed):
    return {f"r{n}": tiny.tokens(name, n, seed + n) for n in lengths}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_whole_prompts_and_their_first_tokens(models, tmp_path, dtype, name):
    requests = requests_of(name, [1, 2, 3, 64, 65, 211], 10)
    run_trace(models[name], dtype, harness.trace_whole(requests), tmp_path, requests, "whole")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_decoding_token_by_token_long(models, tmp_path, dtype, name):
    """A prompt of 40 and 190 tokens decoded one by one: the windows pass over decoded tokens, pages behind
    them are given back, every pass of a loop keeps its own keys."""
    requests = requests_of(name, [230], 20)
    run_trace(models[name], dtype, harness.trace_tail(requests, tail=190), tmp_path, requests, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_prompts_in_portions(models, tmp_path, dtype, name):
    requests = requests_of(name, [150], 30)
    for sizes in ([2], [63, 2, 1, 64, 3], [5, 100, 2, 2, 7]):
        run_trace(models[name], dtype, trace_portions(requests, sizes), tmp_path, requests, f"portions {sizes[0]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_batches_of_unequal_requests(models, tmp_path, dtype, name):
    """Two batches, one after the other, in a cache that holds one of them: the second batch takes
    the slots and pages that the first gave back.  Every request also alone."""
    first = requests_of(name, [1, 70, 135, 23], 40)
    second = {k + "x": v for k, v in requests_of(name, [90, 2, 140], 50).items()}
    prompt_lens = {"r1": 1, "r70": 50, "r135": 100, "r23": 23, "r90x": 64, "r2x": 1, "r140x": 128}
    records = harness.trace_batches([first, second], prompt_lens)
    together = run_trace(models[name], dtype, records, tmp_path, {**first, **second}, "batches",
                         max_tokens=harness.max_tokens_of(records))
    alone = harness.replay(models[name], dtype, harness.trace_whole({**first, **second}), str(tmp_path / "alone"))
    if dtype == "float32":
        for key in together:
            err = position_error(together[key], alone[key])
            assert err.max() <= 3e-5 * max(1.0, np.abs(alone[key]).max()), f"{key}: a batch and the request alone differ by {err.max():.3e}"


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_the_stream_after_every_layer_run(models, name):
    """The float32 stream after each execution of a layer (with its pending output added), through the
    model's own layers, schedule and cache."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache import SequenceCache
    from thing_htn_2026_b200.engine.loading import load_model
    from thing_htn_2026_b200.engine.step import StepEntry, StepRunner
    toks = tiny.tokens(name, 37, 5)
    want = plain.model_forward(models[name], toks, torch.float32)[1]
    seen = []
    with torch.inference_mode():
        model = load_model(models[name], "float32", DEV)

        def watched(forward):
            def run(h, d, ctx, entry):
                h, d = forward(h, d, ctx, entry)
                now = h.clone()
                ops.residual_norm(now, d.tensor, d.norm.as_gain if d.norm else None, None, torch.float32, d2=d.second, mult=d.factor,
                                  scaled=d.scaled)
                seen.append(now.cpu())
                return h, d
            return run

        for layer in model.layers:
            layer.forward = watched(layer.forward)
        cache = SequenceCache(model.cache_needs(), max_tokens=128, dtype=torch.float32, device=DEV)
        (slot,) = cache.open(1)
        StepRunner(model, cache).step([StepEntry(slot, toks, [36])])
    assert len(seen) == len(want)
    for k, (got, expected) in enumerate(zip(seen, want)):
        worst = (got - expected).abs().max().item()
        assert worst <= 3e-5 * max(1.0, expected.abs().max().item()), f"after layer run {k}: the stream differs by {worst:.3e}"


def greedy_by_plain(folder, prompt, n_new):
    model = plain.read_model(folder)
    seq, margins = list(prompt), []
    for _ in range(n_new):
        logits = plain.model_forward(folder, seq, torch.float64, model)[0][-1]
        top = logits.topk(2).values
        margins.append(float(top[0] - top[1]))
        seq.append(int(logits.argmax()))
    return seq[len(prompt):], margins


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["a", "c", "d"])
def test_greedy_generation_through_the_engine(models, name, graphs):
    """Engine.generate: the library's own entry point, scheduler, captured decode step and token
    choice, on prompts of unequal lengths, against greedy continuation by the plain implementation
    (up to the first step whose two best logits are closer than rounding)."""
    from thing_htn_2026_b200 import Engine
    prompts = [tiny.tokens(name, n, 50 + n) for n in (5, 70, 23)]
    new = 20
    engine = Engine(models[name], dtype="float32", graphs=graphs)
    got = [[] for _ in prompts]
    for step in engine.generate(prompts, new):
        for i, token in enumerate(step):
            got[i].append(token)
    compared = 0
    for i, prompt in enumerate(prompts):
        want, margins = greedy_by_plain(models[name], prompt, new)
        sure = next((k for k, m in enumerate(margins) if m < 3e-4), new)
        assert got[i][:sure] == want[:sure], f"prompt {i}: {got[i]} against {want} (sure of the first {sure})"
        compared += sure
    assert compared >= 24
    again = [[] for _ in prompts]
    for step in engine.generate(prompts, 6):
        for i, token in enumerate(step):
            again[i].append(token)
    assert [a[:6] for a in again] == [g[:6] for g in got]


def test_a_queue_of_requests_runs_as_batches(models):
    """generate_all: five requests in batches of two, whose slots are used again, give the tokens that
    each gives alone."""
    from thing_htn_2026_b200 import Engine
    prompts = [tiny.tokens("d", n, 80 + n) for n in (9, 66, 1, 30, 130)]
    engine = Engine(models["d"], dtype="float32", max_batch=2)
    together = [c.tokens for c in engine.generate_all(prompts, [6, 3, 9, 1, 5])]
    for prompt, count, tokens in zip(prompts, [6, 3, 9, 1, 5], together):
        alone = Engine(models["d"], dtype="float32")
        assert [step[0] for step in alone.generate([prompt], count)] == tokens


def test_generation_in_bfloat16_runs_and_stays_in_the_vocabulary(models):
    from thing_htn_2026_b200 import Engine
    engine = Engine(models["b"], dtype="bfloat16")
    prompts = [tiny.tokens("b", n, 60 + n) for n in (3, 40)]
    steps = list(engine.generate(prompts, 12, temperature=[0.0, 0.8], seed=3))
    assert len(steps) == 12 and all(0 <= t < 304 for step in steps for t in step)
