"""The Futepel decoder on the device against the plain implementation (tests/plain/futepel_plain.py):
each mechanism alone (pair and position embeddings; the token shift; time mixing; state-space duality
behind its convolution; latent attention with half pairs and a gate per head; the gate ahead of a
grouped norm; routing by a softmax over the chosen; both feed-forwards), single keys made to decide the
output against closed forms, then whole models through the replay program (whole prompts, token-by-token
decoding, prompts cut into portions, batches of unequal requests, slots and pages used again), and
greedy generation through the library's entry point."""

import math
import warnings

import numpy as np
import pytest
import torch

import futepel_tiny as tiny
import harness
from plain import futepel_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("futepel_models")
    return {name: tiny.write_model(str(root / name), name) for name in tiny.CONFIGS}


# ----------------------------------------------------------------------------- comparison

_oracle = {}
_margins = {}


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
    mean.  Places where a router's choice hangs on less than 0.08 in its logits (in exact
    arithmetic) are left out of the bfloat16 comparison, and so are the sixteen places behind each:
    a recurrent layer carries another expert's output on for a while."""
    assert got.shape[0] == len(tokens), f"{what}: {got.shape[0]} rows for {len(tokens)} places"
    exact = oracle(folder, tokens, torch.float64)
    spread = max(1.0, float(np.abs(exact).max()))
    if dtype == "float32":
        err = position_error(got, oracle(folder, tokens, torch.float32))
        assert err.max() <= 3e-5 * spread, f"{what}: float32 logits differ by {err.max():.3e} at place {int(err.argmax())}"
        return
    if (folder, tuple(tokens)) not in _margins:
        _margins[(folder, tuple(tokens))] = plain.routing_margin(folder, list(tokens)).numpy()
    sure = np.ones(len(tokens), dtype=bool)
    for place in np.nonzero(_margins[(folder, tuple(tokens))] <= 0.08)[0]:
        sure[place:place + 17] = False
    if not sure.any():
        return
    noise = position_error(oracle(folder, tokens, torch.bfloat16), exact)[sure]
    err = position_error(got, exact)[sure]
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


class Sequences:
    """Slots and row indices of steps over a cache of the given needs, as the step function makes them."""

    def __init__(self, needs, dtype, n_slots=3, max_tokens=64 * 40):
        from thing_htn_2026_b200 import ops
        from thing_htn_2026_b200.cache import SequenceCache
        self.ops = ops
        self.cache = SequenceCache(needs, max_tokens=max_tokens, dtype=TORCH[dtype], device=DEV, max_slots=n_slots)
        self.err = ops.new_error_word(DEV)

    def rows(self, slots, counts):
        self.cache.prepare(slots, counts)
        self.cu = [0]
        for c in counts:
            self.cu.append(self.cu[-1] + c)
        self.cu_dev = torch.tensor(self.cu, dtype=torch.int32, device=DEV)
        self.slots_dev = torch.tensor(slots, dtype=torch.int32, device=DEV)
        return self.ops.step_rows(self.cu_dev, self.slots_dev, self.cache.seq_lens, self.cu[-1], max(counts))

    def done(self, slots, counts):
        self.ops.advance(self.cache.seq_lens, self.slots_dev, self.cu_dev)
        self.cache.commit(slots, counts)
        assert int(self.err.item()) == 0


# ----------------------------------------------------------------------------- embedding and token shift


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, vocab, buckets, before, token, positions", [
    (48, 50, 7, 3, 5, True), (33, 70000, 1021, 92821, 1000003, True), (256, 9, 1, 1, 1, False), (2048, 300, 64, 0, 1, True)])
def test_embeddings_of_pairs_and_positions(dtype, width, vocab, buckets, before, token, positions):
    """Two sequences of a slot each, one of them in a slot that another used before, brought in steps of
    unequal sizes: the pair of a step's first token reaches back to the step before it (multipliers and
    ids whose products pass 2^32), a first token takes the last row, positions count on."""
    from thing_htn_2026_b200 import ops
    t = TORCH[dtype]
    table, pairs, places = rand((vocab, width), 1).to(t), rand((buckets + 1, width), 2).to(t), rand((40, width), 3).to(t)
    g = torch.Generator().manual_seed(4)
    w = {"embed": table.float(), "bigram": pairs.float(), "pos": places.float() if positions else torch.zeros(40, width)}
    config = {"embedding": {"scale": 3.5, "bigram": {"buckets": buckets, "mul_prev": before, "mul_cur": token}}}
    seqs = Sequences([], dtype)
    cache = seqs.cache
    previous = cache.sequence_state("previous_token")
    pair_table = ops.PairTable(pairs.to(DEV), before, token)
    s0, s1 = cache.open(2)

    def step(slots, toks):
        counts = [len(x) for x in toks]
        rows = seqs.rows(slots, counts)
        out = ops.embed_rows(table.to(DEV), torch.tensor(sum(toks, []), dtype=torch.int32, device=DEV), 3.5, rows, cache.seq_lens,
                             pair_table, previous, places.to(DEV) if positions else None, seqs.err)
        seqs.done(slots, counts)
        return [out[lo:hi].cpu() for lo, hi in zip(seqs.cu[:-1], seqs.cu[1:])]

    for attempt in range(2):
        a = torch.randint(0, vocab, (37,), generator=g).tolist()
        b = torch.randint(0, vocab, (40,), generator=g).tolist()
        a[0] = vocab - 1
        got_a, got_b = [], []
        for lo, hi, lo_b, hi_b in [(0, 3, 0, 1), (3, 4, 1, 2), (4, 6, 2, 36), (6, 7, 36, 37), (7, 37, 37, 40)]:
            x, y = step([s1, s0], [a[lo:hi], b[lo_b:hi_b]])
            got_a.append(x), got_b.append(y)
        for toks, got in ((a, got_a), (b, got_b)):
            want = plain.embed(w, config, torch.tensor(toks), torch.float32)
            assert (torch.cat(got) - want).abs().max() <= 1e-6 * want.abs().max()
        cache.close([s1, s0])
        s0, s1 = cache.open(2)


def test_a_position_beyond_the_table_and_a_token_beyond_the_vocabulary_are_reported(models):
    """The step function refuses before anything runs; the kernel itself reads a row that exists and sets
    its bit."""
    from thing_htn_2026_b200 import Engine, ops
    from thing_htn_2026_b200.cache import SequenceCache
    from thing_htn_2026_b200.engine.loading import load_model
    from thing_htn_2026_b200.engine.step import StepEntry, StepRunner
    with torch.inference_mode():
        model = load_model(models["b"], "float32", DEV)
        assert model.position_limit == 256
        cache = SequenceCache(model.cache_needs(), max_tokens=512, dtype=torch.float32, device=DEV)
        runner = StepRunner(model, cache)
        (slot,) = cache.open(1)
        runner.step([StepEntry(slot, tiny.tokens("b", 255, 1), (254,))])
        with pytest.raises(ValueError, match="positions"):
            runner.step([StepEntry(slot, [1, 2], (0,))])
        runner.step([StepEntry(slot, [1], (0,))])
        with pytest.raises(ValueError, match="positions"):
            runner.step([StepEntry(slot, [1], (0,))])
    engine = Engine(models["b"], dtype="float32")
    with pytest.raises(ValueError, match="positions"):
        list(engine.generate([tiny.tokens("b", 250, 2)], 8))
    assert len(list(engine.generate([tiny.tokens("b", 250, 2)], 7))) == 7
    seqs = Sequences([], "float32")
    (slot,) = seqs.cache.open(1)
    table, places = rand((5, 8), 1).to(DEV), rand((2, 8), 2).to(DEV)
    rows = seqs.rows([slot], [3])
    out = ops.embed_rows(table, torch.tensor([0, 9, 1], dtype=torch.int32, device=DEV), 1.0, rows, seqs.cache.seq_lens,
                         positions=places, err=seqs.err)
    assert torch.isfinite(out).all() and int(seqs.err.item()) == ops.ERR_TOKEN_RANGE | ops.ERR_POSITION_RANGE


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, n_mix", [(48, 5), (33, 5), (256, 1), (2048, 5), (4100, 3)])
def test_token_shift_over_steps_and_slots(dtype, width, n_mix):
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    t = TORCH[dtype]
    mu = rand((n_mix, width), 5)
    seqs = Sequences([StateSpec((width,), t)], dtype)
    shift = seqs.cache.state_view(0)
    s0, s1 = seqs.cache.open(2)
    for attempt in range(2):
        a, b = rand((30, width), 6 + attempt).to(t), rand((12, width), 8 + attempt).to(t)
        got_a, got_b = [], []
        for lo, hi, lo_b, hi_b in [(0, 1, 0, 3), (1, 2, 3, 4), (2, 4, 4, 9), (4, 29, 9, 10), (29, 30, 10, 12)]:
            rows = seqs.rows([s1, s0], [hi - lo, hi_b - lo_b])
            out = ops.token_shift(torch.cat([a[lo:hi], b[lo_b:hi_b]]).to(DEV), mu.to(DEV), shift, rows, seqs.cache.seq_lens)
            seqs.done([s1, s0], [hi - lo, hi_b - lo_b])
            got_a.append(out[:, :hi - lo].cpu()), got_b.append(out[:, hi - lo:].cpu())
        for x, got in ((a.float(), got_a), (b.float(), got_b)):
            before = torch.cat([torch.zeros(1, width), x[:-1]])
            want = x[None] + (before - x)[None] * mu[:, None, :]
            close(torch.cat(got, dim=1), want, dtype, "token shift", 0.2)
        seqs.cache.close([s0, s1])
        s0, s1 = seqs.cache.open(2)


# ----------------------------------------------------------------------------- gates, norms, activations, routing


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, size, columns, offset", [(3, 10, 3, 0), (4, 64, 20, 7), (16, 128, 16, 0), (1, 24, 5, 4), (48, 1, 48, 0)])
def test_a_gate_per_head(dtype, heads, size, columns, offset):
    from thing_htn_2026_b200 import ops
    t = TORCH[dtype]
    a, g = rand((9, heads * size), 1).to(t), rand((9, columns), 2, 3.0).to(t)
    got = ops.logistic_gate(a.to(DEV), g.to(DEV), offset, size)
    want = a.float() * torch.sigmoid(g.float()[:, offset:offset + heads]).repeat_interleave(size, dim=1)
    close(got, want, dtype, "gate per head", 0.2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, parts", [(30, 2), (64, 4), (66, 1), (4096, 1), (4096, 8), (9000, 2), (20000, 1)])
def test_the_gate_ahead_of_a_grouped_norm(dtype, width, parts):
    """Parts of very different sizes of their entries: a statistic taken over the whole row, or the gate
    behind the norm, is far off."""
    from thing_htn_2026_b200 import ops
    t, eps = TORCH[dtype], 1e-5
    scale = torch.logspace(-2, 2, parts).repeat_interleave(width // parts)
    y, gain = rand((5, width), 1) * scale, rand((width,), 2)
    proj = rand((5, width + 7), 3).to(t)
    got = ops.gated_group_norm(y.to(DEV), proj.to(DEV), 3 if width % 4 else 4, gain.to(DEV), eps, parts, t)
    at = 3 if width % 4 else 4
    z = proj.float()[:, at:at + width]
    gated = y * z * torch.sigmoid(z)
    p = gated.reshape(5, parts, -1)
    want = (p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(5, width) * gain
    close(got, want, dtype, "gate, then norm")
    proj4 = rand((5, width + 8), 4).to(t)          # rows that are whole 16-byte pieces
    got = ops.gated_group_norm(y.to(DEV), proj4.to(DEV), 8, gain.to(DEV), eps, parts, t)
    z = proj4.float()[:, 8:]
    p = (y * z * torch.sigmoid(z)).reshape(5, parts, -1)
    close(got, (p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(5, width) * gain, dtype, "aligned rows")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(3, 7), (5, 64), (2, 4096)])
def test_squared_relu(dtype, shape):
    from thing_htn_2026_b200 import ops
    z = rand(shape, 1, 2.0).to(TORCH[dtype])
    close(ops.squared_relu(z.to(DEV)), torch.relu(z.float()) ** 2, dtype, "squared relu", 0.2)


@pytest.mark.parametrize("experts, top", [(8, 1), (5, 5), (7, 3), (64, 6), (2, 1), (40, 4)])
def test_routing_by_a_softmax_over_the_chosen(experts, top):
    from thing_htn_2026_b200 import ops
    z = rand((50, experts), experts + top, 3.0)
    z[0] = 0.0                                          # all equal: the lowest indices win
    z[1] = torch.arange(experts) * -200.0               # a softmax over all experts would lose all but one
    z[2] = torch.arange(experts) * 200.0 + 1e4
    routing = ops.moe_route(z.to(DEV), experts, 1, 1, top, 1.0, scoring="softmax_chosen")
    best = torch.topk(z.double(), top, dim=-1)
    want = torch.zeros(50, experts, dtype=torch.float64).scatter_(1, best.indices, torch.softmax(best.values, -1))
    got = routing.dense.cpu().double()
    assert sorted(routing.chosen[0].tolist()) == list(range(top))
    assert (got[1:] - want[1:]).abs().max() < 1e-6
    assert routing.chosen[2].tolist() == list(range(experts - 1, experts - 1 - top, -1))
    assert torch.allclose(got.sum(-1), torch.ones(50, dtype=torch.float64), atol=1e-6)


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


FEED_FORWARDS = [(name, i) for name in sorted(tiny.CONFIGS) for i, layer in enumerate(tiny.CONFIGS[name]["layers"])
                 if layer["mlp"] is not None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, layer", FEED_FORWARDS)
def test_feed_forward_alone(models, dtype, name, layer):
    part, config = part_of(models[name], layer, "ffn", dtype)
    mlp = tiny.config_json(name)["layers"][layer]["mlp"]
    _, w = plain.read_model(models[name])
    x = rand((33, config.width), 8 + layer, 2.0).to(TORCH[dtype])
    ar = plain.Arithmetic(torch.float32 if dtype == "float32" else torch.bfloat16)
    prefix = f"l{layer}.mlp."
    want = plain.dense(ar, x.float(), w, prefix) if mlp["kind"] == "dense" else plain.mixture(ar, x.float(), w, prefix, mlp)
    got = part.forward(x.to(DEV), None)
    if dtype == "float32":
        close(got, want, dtype, "feed-forward")
    else:
        bad = ((got.float().cpu() - want).abs() > 3e-2 * max(1.0, want.abs().max().item() / 4) + want.abs() / 16).any(dim=1)
        assert bad.sum() <= 2, f"{int(bad.sum())} of {bad.numel()} rows differ"


# ----------------------------------------------------------------------------- mixers alone


class Stepper(Sequences):
    """Feeds rows to a mixer through a cache of its own, as the step function would."""

    def __init__(self, mixer, dtype, n_slots=3):
        super().__init__([mixer.cache_need()], dtype, n_slots)
        self.mixer = mixer

    def step(self, slots, xs):
        from thing_htn_2026_b200.config.base import ScheduleEntry
        from thing_htn_2026_b200.parts import HostBatch, StepContext
        counts = [x.shape[0] for x in xs]
        held = [self.cache.length(s) for s in slots]
        rows = self.rows(slots, counts)
        asked = {}
        if hasattr(self.mixer, "step_inputs"):
            self.mixer.step_inputs(HostBatch(slots, counts, held, 64), asked)
        inputs = {k: torch.tensor(v, dtype=torch.int32, device=DEV) for k, v in asked.items()}
        ctx = StepContext(rows=rows, cache=self.cache, err=self.err, inputs=inputs)
        a = self.mixer.forward(torch.cat(xs).to(DEV).contiguous(), ctx, ScheduleEntry(0, 0))
        self.done(slots, counts)
        return [a[lo:hi] for lo, hi in zip(self.cu[:-1], self.cu[1:])]


def plain_mixer(folder, layer, x, ar):
    config, w = plain.read_model(folder)
    entry = config["layers"][layer]
    prefix, eps = f"l{layer}.mix.", config["norm"]["eps"]
    if entry["type"] == "wkv":
        return plain.time_mixing(ar, x, w, prefix, entry["mixer"], eps)
    if entry["type"] == "mamba2":
        return plain.state_space(ar, x, w, prefix, entry["mixer"], eps)
    return plain.latent_attention(ar, x, w, prefix, entry["mixer"], eps, torch.arange(x.shape[0]))


MIXERS = [(name, i) for name in sorted(tiny.CONFIGS) for i in range(len(tiny.CONFIGS[name]["layers"]))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, layer", MIXERS)
def test_mixers_alone_whole_in_portions_and_token_by_token(models, dtype, name, layer):
    """Every mixer of the tiny models against the plain mechanism, for a sequence brought whole, in
    portions of unequal sizes down to two and one (shorter than the convolution's taps, across page
    borders and the stages of the recurrence), beside another sequence, token by token at its end, and in
    a slot that was used before (state, ring and last row must start from zero again)."""
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

CUTS = ([300], [100, 1, 1, 2, 64, 131, 1], [1] * 30 + [270], [280] + [1] * 20)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [6, 10, 64, 130, 300])
def test_time_mixing_keeps_a_far_key_by_its_decay_and_its_own_by_the_bonus(dtype, d):
    """One loud key 270 tokens back and a query that asks for it: what is left is the product of the
    channel's decays since (the loud token's own decay does not count, the reader's neither); the loud
    token itself reads its own product through the bonus alone.  Over steps of unequal sizes; a slot
    that is opened again starts from nothing."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    T, t, heads, loud, c = 300, TORCH[dtype], 2, 29, d - 1
    r, k, v = torch.zeros(T, heads, d), torch.zeros(T, heads, d), torch.zeros(T, heads, d)
    value = rand((heads, d), d)
    k[loud, :, c], v[loud] = 4.0, value
    r[T - 1, :, c], r[loud, :, c] = 0.5, 0.25
    planes = torch.stack([x.reshape(T, -1) for x in (r, k, v)]).to(t)
    z, w0, u = rand((T, heads * d), 7, 0.5), rand((heads * d,), 8, 0.5).sub(5.0), rand((heads, d), 9)
    decay = torch.exp(-torch.exp(z.double() + w0.double())).view(T, heads, d)
    seqs = Sequences([StateSpec((heads, d, d))], dtype)
    for cut in CUTS[:3]:
        (slot,) = seqs.cache.open(1)
        outs, at = [], 0
        for count in cut:
            rows = seqs.rows([slot], [count])
            outs.append(ops.wkv(planes[:, at:at + count].contiguous().to(DEV), z[at:at + count].contiguous().to(DEV), w0.to(DEV),
                                u.to(DEV), seqs.cache.state_view(0), rows, heads, d))
            seqs.done([slot], [count])
            at += count
        got = torch.cat(outs).cpu().double()
        vt = value.to(t).double()
        fade = decay[loud + 1:T - 1, :, c].prod(0)
        want = fade[:, None] * vt * 4.0 * 0.5
        tol = 1e-4 if dtype == "float32" else 2e-2
        assert want.abs().max() > 0.01
        assert (got[T - 1] - want).abs().max() <= tol * want.abs().max(), cut
        own = u.double()[:, c, None] * vt * 4.0 * 0.25
        assert (got[loud] - own).abs().max() <= tol * own.abs().max(), cut
        assert got[:loud].abs().max() == 0.0 and got[loud + 1:T - 1].abs().max() == 0.0
        seqs.cache.close([slot])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, rank", [(2, 6, 4), (1, 64, 64), (3, 130, 8), (2, 300, 3)])
def test_a_single_step_of_time_mixing_is_one_kernel_and_the_same(dtype, heads, d, rank):
    """The kernel of single-token steps (low-rank decay, recurrence, norm, gain and gate in one) against
    the pieces by hand, for three sequences with states of their own."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    t, eps, n = TORCH[dtype], 1e-5, 3
    planes, low = rand((4, n, heads * d), 1).to(t), rand((n, rank), 2)
    w2, w0, u, gain = rand((heads * d, rank), 3, 0.4).to(t), rand((heads * d,), 4).sub(2.0), rand((heads, d), 5), rand((heads * d,), 6)
    seqs = Sequences([StateSpec((heads, d, d))], dtype, n_slots=5)
    slots = seqs.cache.open(4)[1:]
    S = rand((n, heads, d, d), 7)
    seqs.cache.state_view(0)[torch.tensor(slots)] = S.to(DEV)
    rows = seqs.rows(slots, [1] * n)
    got = ops.wkv_decode(planes.to(DEV), low.to(DEV), w2.to(DEV), w0.to(DEV), u.to(DEV), gain.to(DEV), eps, seqs.cache.state_view(0),
                         rows, heads, d)
    th = torch.tanh(low)
    z = (th.to(t).double() if dtype == "bfloat16" else th.double()) @ w2.double().t() + w0.double()
    w = torch.exp(-torch.exp(z)).view(n, heads, d)
    r, k, v, g = (p.double().view(n, heads, d) for p in planes)
    kv = v[..., :, None] * k[..., None, :]                                        # [value, key]
    o = ((S.double() + u.double()[None, :, None, :] * kv) * r[..., None, :]).sum(-1)
    y = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * gain.double().view(heads, d) * g * torch.sigmoid(g)
    close(got, y.reshape(n, -1), dtype, "one step")
    left = seqs.cache.state_view(0)[torch.tensor(slots)].cpu().double()
    assert (left - (w[..., None, :] * S.double() + kv)).abs().max() <= 2e-5 * left.abs().max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, groups, e, n, taps", [(4, 2, 6, 5, 4), (3, 3, 16, 16, 1), (8, 1, 20, 40, 2), (2, 2, 33, 130, 3), (2, 1, 64, 300, 7)])
def test_state_space_keeps_a_far_input_by_its_decay(dtype, heads, groups, e, n, taps):
    """One token writes, one reads 270 tokens later; all other inputs are zero and silu(0) is 0, so what is
    left is the product of the decays since, times both step sizes' effect; B and C of every group are
    of different sizes, so a head that reads another group's shows.  The convolution passes the current
    token only, except in its first tap, which hands the writer's input to the token taps - 1 later."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    T, t, write, c = 300, TORCH[dtype], 29, n - 1
    inner, channels = heads * e, heads * e + 2 * groups * n
    raw = torch.zeros(T, channels)
    x_in, b_in, c_in = rand((heads, e), 1).abs() + 0.5, torch.arange(1, groups + 1) * 1.5, torch.arange(groups, 0, -1) * 0.75
    raw[write, :inner] = x_in.reshape(-1)
    raw[write].view(-1)[inner:inner + groups * n].view(groups, n)[:, c] = b_in
    raw[T - 1].view(-1)[inner + groups * n:].view(groups, n)[:, c] = c_in
    proj = torch.cat([torch.full((T, 3), 9.0), raw], dim=1).to(t)
    conv_w = torch.zeros(channels, taps)
    conv_w[:, -1] = 1.0
    dt, bias, rate, skip = rand((T, heads), 2), rand((heads,), 3).sub(3.0), torch.rand(heads, generator=torch.Generator().manual_seed(4)) * 0.1 + 0.02, rand((heads,), 5)
    shape = ops.StateSpace(heads, e, n, groups, conv_w.to(DEV), torch.zeros(channels, device=DEV), bias.to(DEV), rate.to(DEV), skip.to(DEV))
    steps = torch.nn.functional.softplus(dt.double() + bias.double())
    seqs = Sequences([(StateSpec((heads, e, n)), StateSpec((taps, channels), t))], dtype)
    silu = lambda v: v * torch.sigmoid(v)
    per = heads // groups
    x1, b1, c1 = (silu(v.to(t).double()) for v in (x_in, b_in, c_in))
    if dtype == "bfloat16":
        x1, b1, c1 = (v.to(torch.float64) for v in (x1, b1, c1))
    for cut in CUTS:
        (slot,) = seqs.cache.open(1)
        outs, at = [], 0
        for count in cut:
            rows = seqs.rows([slot], [count])
            outs.append(ops.state_space(proj[at:at + count].contiguous().to(DEV), 3, dt[at:at + count].contiguous().to(DEV), shape,
                                        seqs.cache.state_view(0, 0), seqs.cache.state_view(0, 1), rows, seqs.cache.seq_lens))
            seqs.done([slot], [count])
            at += count
        got = torch.cat(outs).cpu().double()
        fade = torch.exp(-(rate.double() * steps[write + 1:]).sum(0))
        group = [h // per for h in range(heads)]
        want = (fade * steps[write])[:, None] * (b1[group] * c1[group])[:, None] * x1
        tol = 1e-4 if dtype == "float32" else 2e-2
        assert want.abs().max() > 1e-3
        assert (got[T - 1] - want).abs().max() <= tol * want.abs().max(), cut
        own = skip.double()[:, None] * x1
        assert (got[write] - own).abs().max() <= tol * own.abs().max(), cut
        assert got[:write].abs().max() == 0.0 and got[write + 1:T - 1].abs().max() == 0.0
        seqs.cache.close([slot])


@pytest.mark.parametrize("columns", [1, 2, 4])
@pytest.mark.parametrize("heads, d", [(3, 24), (2, 64), (2, 100), (1, 128)])
def test_every_variant_of_the_recurrence(columns, heads, d):
    """The shared recurrence with 1, 2 and 4 columns of the state in a lane, over prompts of 1, 7, 37 and
    100 tokens side by side (whole stages, groups of eight and what is left), against token by token in
    double, with the states that they leave."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    counts = [1, 37, 100, 7]
    n = sum(counts)
    planes, z = rand((3, n, heads * d), 1), rand((n, heads * d), 2)
    w0, u, S0 = rand((heads * d,), 3).sub(3.0), rand((heads, d), 4), rand((len(counts), heads, d, d), 5, 0.3)
    seqs = Sequences([StateSpec((heads, d, d))], "float32", n_slots=5)
    slots = seqs.cache.open(4)
    seqs.cache.state_view(0)[torch.tensor(slots)] = S0.to(DEV)
    rows = seqs.rows(slots, counts)
    ops.set_recurrence_columns(columns)
    try:
        got = ops.wkv(planes.to(DEV), z.to(DEV), w0.to(DEV), u.to(DEV), seqs.cache.state_view(0), rows, heads, d).cpu().double()
    finally:
        ops.set_recurrence_columns(0)
    left = seqs.cache.state_view(0)[torch.tensor(slots)].cpu().double()
    r, k, v = (p.double().view(n, heads, d) for p in planes)
    w = torch.exp(-torch.exp(z.double() + w0.double())).view(n, heads, d)
    for i, (lo, hi) in enumerate(zip(seqs.cu[:-1], seqs.cu[1:])):
        S = S0[i].double()                                          # [head, value, key]
        for t in range(lo, hi):
            kv = v[t][:, :, None] * k[t][:, None, :]
            want = ((S + u.double()[:, None, :] * kv) * r[t][:, None, :]).sum(-1)
            assert (got[t] - want).abs().max() <= 2e-5 * max(1.0, want.abs().max().item()), (i, t - lo)
            S = w[t][:, None, :] * S + kv
        assert (left[i] - S).abs().max() <= 2e-5 * max(1.0, S.abs().max().item()), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_the_convolution_reaches_back_over_steps_and_no_farther(dtype, taps):
    """Through the skip alone (the state is empty: B is zero): y is the convolved input, so taps in the
    wrong order, a lost ring entry or a neighbour sequence's rows show at once.  Steps from one token to
    runs longer than the kernel's, two sequences side by side, a slot used again."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache.sequence_cache import StateSpec
    t, e, n = TORCH[dtype], 6, 3
    channels = e + 2 * n
    conv_w, conv_b = rand((channels, taps), 1), rand((channels,), 2)
    conv_b[e:] = 0.0
    one = torch.ones(1, device=DEV)
    shape = ops.StateSpace(1, e, n, 1, conv_w.to(DEV), conv_b.to(DEV), one, one, one)
    seqs = Sequences([(StateSpec((1, e, n)), StateSpec((taps, channels), t))], dtype)
    s0, s1 = seqs.cache.open(2)
    for attempt in range(2):
        a, b = rand((61, channels), 3 + attempt).to(t), rand((40, channels), 5 + attempt).to(t)
        a[:, e:], b[:, e:] = 0.0, 0.0
        got_a, got_b = [], []
        for lo, hi, lo_b, hi_b in [(0, 1, 0, 1), (1, 2, 1, 2), (2, 4, 2, 3), (4, 29, 3, 10), (29, 30, 10, 12), (30, 31, 12, 13), (31, 61, 13, 40)]:
            rows = seqs.rows([s1, s0], [hi - lo, hi_b - lo_b])
            x = torch.cat([a[lo:hi], b[lo_b:hi_b]]).to(DEV)
            y = ops.state_space(x, 0, torch.zeros(x.shape[0], 1, device=DEV), shape, seqs.cache.state_view(0, 0),
                                seqs.cache.state_view(0, 1), rows, seqs.cache.seq_lens).cpu()
            seqs.done([s1, s0], [hi - lo, hi_b - lo_b])
            got_a.append(y[:hi - lo, 0]), got_b.append(y[hi - lo:, 0])
        for raw, got in ((a.float(), got_a), (b.float(), got_b)):
            padded = torch.cat([torch.zeros(taps - 1, channels), raw])
            conv = sum(padded[j:j + raw.shape[0]] * conv_w[:, j] for j in range(taps)) + conv_b
            want = (conv * torch.sigmoid(conv))[:, :e]
            assert (torch.cat(got) - want).abs().max() <= 2e-5 * want.abs().max()
        seqs.cache.close([s0, s1])
        s0, s1 = seqs.cache.open(2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, r, e", [(2, 10, 6, 20), (4, 32, 32, 64), (2, 48, 16, 24), (3, 16, 0, 16), (2, 64, 64, 128), (1, 2, 2, 5)])
def test_one_loud_latent_among_hundreds(dtype, heads, d, r, e):
    """300 tokens of which one has a rotated key part that meets the last query's exactly (turned by
    their places), in eight places on either side of page borders: the last row's read-out is the loud
    token's value times the head's gate, as one prompt and with the last rows decoded.  Without a rotated
    part the plain keys are loud instead."""
    from thing_htn_2026_b200.config.base import PartSpec
    from thing_htn_2026_b200.parts import Runtime, part_class
    T, t, hidden, rank = 300, TORCH[dtype], 264, 24
    names = ("q_proj", "down_proj", "latent_norm", "up_k", "up_v", "g_proj", "o_proj")
    rot = {"base": 50.0, "dims": r, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    position = None if not r else PartSpec("rope", {"head_dim": r, "rotary_dim": r, "theta": 50.0, "layout": "half",
                                                    "frequency_precision": "float64", "angle_precision": "float64",
                                                    "scaling": rot["scaling"]})
    spec = PartSpec("latent_attention", {"hidden_size": hidden, "n_heads": heads, "plain_dim": d, "rot_dim": r, "value_dim": e,
                                         "latent_rank": rank, "scale": 1.0, "norm_eps": 1e-5, "position": position,
                                         "gate_scope": "head", "softmax_weights": "float32"}, {n: n for n in names})
    g = torch.Generator().manual_seed(heads * d + r)
    shapes = {"q_proj": (heads * (d + r), hidden), "down_proj": (rank + r, hidden), "latent_norm": (rank,), "up_k": (heads * d, rank),
              "up_v": (heads * e, rank), "g_proj": (heads, hidden)}
    w = {n: torch.randn(s, generator=g) * 0.15 for n, s in shapes.items()}
    w["o_proj"] = torch.eye(hidden, heads * e)
    # the last latent channel is the loud token's own: no other token has anything there
    w["latent_norm"][rank - 1] = 1.0
    w["down_proj"][rank - 1] = 0.0
    loud_direction, ask_direction = torch.eye(hidden)[hidden - 1], torch.eye(hidden)[hidden - 2]
    for weight in ("q_proj", "down_proj", "g_proj"):
        w[weight][:, hidden - 2:] = 0.0
    for case, loud in enumerate([0, 1, 63, 64, 127, 128, 298, 299]):
        u = {n: v.clone() for n, v in w.items()}
        u["down_proj"][rank - 1, hidden - 1] = 1.0
        # the rotated part of a token in the loud direction, turned to its place, meets that of the asking token's query
        if r:
            freq, magnitude = plain.yarn_frequencies(rot)
            key = torch.randn(r, generator=g).double()
            key *= 6.0 / key.norm()
            query = plain.rotate(key[None], torch.tensor([loud - (T - 1)]), rot)[0] / magnitude       # turned back by the distance
            u["down_proj"][rank:, hidden - 1] = key.float()
            for h in range(heads):
                u["q_proj"][h * (d + r) + d:(h + 1) * (d + r), hidden - 2] = (query * 60.0 / (key @ key)).float()
        else:
            u["up_k"][:, rank - 1] *= 8.0
            for h in range(heads):
                k = u["up_k"][h * d:(h + 1) * d, rank - 1] * rank ** 0.5
                u["q_proj"][h * d:(h + 1) * d, hidden - 2] = k * 60.0 / (k @ k)
        x = torch.randn(T, hidden, generator=g) * 0.15
        x[:, hidden - 2:] = 0.0
        x[loud] = loud_direction
        x[T - 1] = ask_direction + (loud_direction if loud == T - 1 else 0.0)
        x = x.to(t)
        u = {n: v.to(t) for n, v in u.items()}
        part = part_class("mixer", "latent_attention")(spec, Runtime(t, torch.device(DEV), {n: v.to(DEV) for n, v in u.items()}))
        if part.position is not None:
            part.position.ensure(T)
        f = {n: v.double() for n, v in u.items()}
        down = x.double() @ f["down_proj"].t()
        c = plain.rms_divide(down[loud, :rank], 1e-5) * f["latent_norm"]
        gate = torch.sigmoid(x.double()[T - 1] @ f["g_proj"].t())
        value = (f["up_v"] @ c).view(heads, e) * gate[:, None]
        for first in (T, 290):
            stepper = Stepper(part, dtype)
            (slot,) = stepper.cache.open(1)
            out = stepper.step([slot], [x[:first]])[0]
            for i in range(first, T):
                out = stepper.step([slot], [x[i:i + 1]])[0]
            got = out[-1, :heads * e].double().cpu().view(heads, e)
            assert value.abs().max() > 0.1
            tol = 2e-4 if dtype == "float32" else 6e-2
            assert (got - value).abs().max() <= tol * max(0.3, value.abs().max().item()), (loud, first)


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
    """A prompt of 40 and 190 tokens decoded one by one: states, rings, last rows, last tokens and keys
    are carried through the cache step after step, over three page borders."""
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
def test_the_stream_after_every_layer(models, name):
    """The float32 stream after each layer of a short prompt (with the layer's pending output added),
    through the model's own layers and cache."""
    from thing_htn_2026_b200 import ops
    from thing_htn_2026_b200.cache import SequenceCache
    from thing_htn_2026_b200.engine.loading import load_model
    from thing_htn_2026_b200.parts import StepContext
    toks = tiny.tokens(name, 37, 5)
    want = plain.model_forward(models[name], toks, torch.float32)[1]
    with torch.inference_mode():
        model = load_model(models[name], "float32", DEV)
        cache = SequenceCache(model.cache_needs(), max_tokens=128, dtype=torch.float32, device=DEV)
        (slot,) = cache.open(1)
        n = len(toks)
        cache.prepare([slot], [n])
        model.ensure_positions(n)
        cu = torch.tensor([0, n], dtype=torch.int32, device=DEV)
        slots = torch.tensor([slot], dtype=torch.int32, device=DEV)
        err = ops.new_error_word(DEV)
        ctx = StepContext(rows=ops.step_rows(cu, slots, cache.seq_lens, n, n, max_context=n), cache=cache, err=err, inputs={})
        h, d = model.embedding.forward(torch.tensor(toks, dtype=torch.int32, device=DEV), err, ctx.rows, cache), None
        for k, entry in enumerate(model.plan.schedule):
            h, d = model.layers[entry.layer].forward(h, d, ctx, entry)
            got = (h + d).cpu()
            worst = (got - want[k]).abs().max().item()
            assert worst <= 3e-5 * max(1.0, want[k].abs().max().item()), f"after layer {k}: the stream differs by {worst:.3e}"
        assert int(err.item()) == 0


def test_what_the_plain_implementation_would_show(models):
    """The plain implementation moves far when positions start at 1 or when the token before the first
    is not the beginning, so the comparisons above would notice either."""
    toks = tiny.tokens("a", 60, 77)
    right = plain.model_logits(models["a"], toks, torch.float64).numpy()
    shifted = plain.model_logits(models["a"], [toks[0]] + toks, torch.float64).numpy()[1:]
    assert position_error(right[:40], shifted[:40]).min() > 1e-3


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
