"""The Midisun design through the engine against the plain implementation (``plain_midisun``): whole prompts, prompts in portions
down to two tokens, token-by-token decoding, batches of unequal requests against each alone, slots, pages and states that are used
again, long decoding past every window, hand-made weights that make one key, a window's edge, a cap, a slope or a sink stand out,
every mechanism and kernel alone, greedy generation through the public entry point and trace replay; in 32-bit and in bfloat16, at
four sets of sizes."""
import math
import tempfile
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import midisun_cases as mc
import plain_midisun as plain
from replay_util import Trace, run_trace

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


@pytest.fixture(scope="module")
def models():
    with tempfile.TemporaryDirectory() as tmp:
        yield {name: mc.Model(name, seed, tmp) for name, seed in (("A", 41), ("B", 42), ("C", 43), ("D", 44))}


def rows(logits, positions):
    a = logits.detach().float().cpu().numpy()
    return {p: a[i].copy() for i, p in enumerate(positions)}


def engine_of(m, dtype, **kw):
    """(engine, recorder of its router choices or None). In bfloat16 a router choice can rest on a gap that rounding closes, so the
    run's own choices are noted (which needs steps that are not replayed from graphs) and the plain implementation takes the same;
    in 32-bit, and where there is no router, the engine runs as it is served, graphs and all, and chooses for itself."""
    routed = any((l.get("mlp") or {}).get("kind") == "moe" for l in m.cfg["layers"])
    if dtype == "bfloat16" and routed:
        engine = m.engine(dtype, graphs=False, **kw)
        return engine, mc.Recorder(engine, m.cfg)
    return m.engine(dtype, **kw), None


def run_cut(engine, tokens, cuts, recorder=None):
    """One sequence fed in portions of the given sizes (the rest one token at a time); logits at every position."""
    slot = engine.new_sequence()
    got, at = {}, 0
    sizes = list(cuts)
    if recorder is not None:
        recorder.choices.pop(0, None)
    while at < len(tokens):
        n = min(sizes.pop(0) if sizes else 1, len(tokens) - at)
        if recorder is not None:
            recorder.rows = [(0, p) for p in range(at, at + n)]
        got.update(rows(engine.step([(slot, tokens[at:at + n])], [list(range(n))]), range(at, at + n)))
        at += n
    engine.free_sequence(slot)
    engine.check_health()
    return got


def rnd(x, T):
    return x.to(T).to(x.dtype)


# ---------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompts_and_prompts_in_portions(models, name, dtype):
    m = models[name]
    engine, rec = engine_of(m, dtype)
    forced = lambda: rec.of(0) if rec is not None else None
    for tokens in mc.prompts(m.vocab, [1, 2, 7, 64, 65, 150, 330], 21):
        got = run_cut(engine, tokens, [len(tokens)], rec)
        mc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} whole {len(tokens)}", forced=forced())
    tokens = mc.prompts(m.vocab, [260], 22)[0]
    # Portions that start and end inside and at page borders and inside and at the windows' edges, two tokens, one token.
    for cuts in ([100, 100, 60], [63, 1, 64, 2, 2, 128], [2, 2, 2, 58, 64, 3, 1, 1, 100, 27], [129, 2, 61, 2, 66], [8, 9, 10, 33, 100, 100]):
        got = run_cut(engine, tokens, cuts, rec)
        mc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} portions {cuts[:4]}", forced=forced())


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_long_decoding_from_a_short_prompt(models, name, dtype):
    """A prompt of three tokens, then 250 single tokens: pages fill up and fall out of the windows while decoding, and the
    recurrent states and the convolution's rows come from the sequence's state at every step."""
    m = models[name]
    engine, rec = engine_of(m, dtype, max_tokens=512, max_seqs=2)
    tokens = mc.prompts(m.vocab, [253], 23)[0]
    got = run_cut(engine, tokens, [3], rec)
    mc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} long decoding", forced=rec.of(0) if rec is not None else None)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_batches_of_unequal_requests_and_reuse_of_slots_pages_and_states(models, name, dtype):
    """Requests of unequal lengths prefilled in one step and decoded together, the shorter ones leaving first; then a second batch
    in the slots, pages and states that the first gave back. Every request is compared with the plain implementation of that
    request alone."""
    m = models[name]
    engine, rec = engine_of(m, dtype, max_tokens=1024, max_seqs=4)
    for seed, lengths, tails in ((31, [1, 40, 129, 300], [0, 12, 40, 3]), (32, [70, 3, 230, 64], [6, 2, 65, 33])):
        reqs = mc.prompts(m.vocab, lengths, seed)
        slots = [engine.new_sequence() for _ in reqs]
        got = [dict() for _ in reqs]
        heads = [len(t) - d for t, d in zip(reqs, tails)]
        if rec is not None:
            rec.choices.clear()
            rec.rows = [(i, p) for i, h in enumerate(heads) for p in range(h)]
        a = engine.step([(s, t[:h]) for s, t, h in zip(slots, reqs, heads)], [list(range(h)) for h in heads]).detach().float().cpu().numpy()
        at = 0
        for i, h in enumerate(heads):
            got[i].update({p: a[at + p].copy() for p in range(h)})
            at += h
        fed = list(heads)
        live = [i for i in range(len(reqs)) if fed[i] < len(reqs[i])]
        for i in range(len(reqs)):
            if i not in live:
                engine.free_sequence(slots[i])
        while live:
            if rec is not None:
                rec.rows = [(i, fed[i]) for i in live]
            out = engine.step([(slots[i], [reqs[i][fed[i]]]) for i in live]).detach().float().cpu().numpy()
            for r, i in enumerate(live):
                got[i][fed[i]] = out[r].copy()
                fed[i] += 1
            for i in [i for i in live if fed[i] == len(reqs[i])]:
                engine.free_sequence(slots[i])
            live = [i for i in live if fed[i] < len(reqs[i])]
        engine.check_health()
        for i, t in enumerate(reqs):
            assert sorted(got[i]) == list(range(len(t)))
            mc.compare(m, t, got[i], DTYPES[dtype], f"{name} {dtype} batch seed {seed} request {i}", forced=rec.of(i) if rec is not None else None)
    assert engine.cache.slots.held == 0


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_steps_that_mix_prompts_portions_and_single_tokens(models, dtype):
    """One step brings a new prompt, a portion of another request and single tokens of two more: the states and the convolution's
    rows of each come from its own slot, and a one-token request takes the many-token kernels."""
    m = models["D"]
    engine, _ = engine_of(m, dtype, max_tokens=1024, max_seqs=4)
    reqs = mc.prompts(m.vocab, [80, 120, 61, 33], 35)
    plan = [[5, 20, 1, 1, 53], [0, 60, 2, 58], [1, 1, 59], [0, 0, 30, 1, 2]]
    slots = [engine.new_sequence() for _ in reqs]
    got, fed = [dict() for _ in reqs], [0] * 4
    for k in range(5):
        entries = [(i, plan[i][k]) for i in range(4) if k < len(plan[i]) and plan[i][k]]
        out = engine.step([(slots[i], reqs[i][fed[i]:fed[i] + n]) for i, n in entries], [list(range(n)) for _, n in entries]).float().cpu().numpy()
        at = 0
        for i, n in entries:
            got[i].update({fed[i] + j: out[at + j].copy() for j in range(n)})
            fed[i] += n
            at += n
    for i, t in enumerate(reqs):
        assert fed[i] == len(t)
        mc.compare(m, t, got[i], DTYPES[dtype], f"{dtype} mixed steps request {i}")


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer(models, name):
    m = models[name]
    engine = m.engine("float32")
    tokens = mc.prompts(m.vocab, [90], 27)[0]
    ref = m.layers(tokens)
    seen = []
    engine.model.observer = lambda occ, x: seen.append((occ, x.detach().float().cpu().clone()))
    slot = engine.new_sequence()
    engine.step([(slot, tokens)])
    engine.model.observer = None
    engine.free_sequence(slot)
    assert [occ for occ, _ in seen] == list(range(len(ref)))
    for occ, x in seen:
        assert float((x - ref[occ]).abs().max()) <= 2e-4 * max(1.0, float(ref[occ].abs().max())), f"layer {occ}"


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_other_arrangements_of_layers(dtype):
    """Each kind of layer alone and twice in a row; windows of one, two and a page and one; many taps;
    one expert per group; every expert chosen; heads of one value; heads and key sizes beyond a block's columns."""
    T = DTYPES[dtype]
    D4 = mc.dense(20)
    one = 1 if T == torch.float32 else 5          # a normed head of one value is a sign, which rounding to bfloat16 may turn
    cases = {
        "attention only": mc.model(50, 24, 1e-4, 4, 5, 0.5, [mc.attention(3, 1, 6, 0.3, D4, cap=2.0, window=1), mc.attention(2, 2, 16, 0.3, None, window=2),
                                                              mc.attention(4, 1, 12, 0.4, mc.moe(8, 4, 2, groups=(4, 3)), cap=50.0, window=65)]),
        "retention only": mc.model(71, 40, 1e-5, 5, 2, 1.1, [mc.retention(2, 4, one, [0.9, 1.0], D4, rot=(2, 30.0)), mc.retention(1, 150, 160, [0.99], None, rot=(90, 50.0))]),
        "mlstm only": mc.model(33, 32, 1e-6, 2, 9, 3.0, [mc.mlstm(2, 6, one, 2.0, mc.moe(12, 3, 3)), mc.mlstm(1, 130, 140, 15.0, D4), mc.mlstm(5, 16, 32, 6.0, None)]),
    }
    with tempfile.TemporaryDirectory() as tmp:
        for name, case in cases.items():
            m = mc.Model(name.replace(" ", "_"), 3, tmp, case)
            engine, rec = engine_of(m, dtype, max_tokens=512, max_seqs=2, max_context=256)
            tokens = mc.prompts(m.vocab, [140], 5)[0]
            for cuts in ([140], [2, 64, 3], [70, 1, 1, 58]):
                got = run_cut(engine, tokens, cuts, rec)
                mc.compare(m, tokens, got, T, f"{name} {dtype} {cuts}", forced=rec.of(0) if rec is not None else None)


# ---------------------------------------------------------------- mixers alone
def _random_tensor(d, g, T):
    name, shape = d.name, tuple(d.shape)
    t = torch.randn(shape, generator=g, dtype=F64)
    if len(shape) == 2:
        t = t * shape[1] ** -0.5
    elif name.endswith(".norm"):
        t = 1 + 0.2 * t
    elif name.endswith(".f.b"):
        t = 2 * t + 2
    elif name.endswith(".b") and not name.endswith(".i.b"):
        t = 0.5 * t
    return rnd(t, T)


def _mixer_of(case, layer, T, tensors=None, seed=0, max_positions=1024):
    """The mixer part of one layer of a configuration, built as the model builds it, with random (or given) tensors.
    Returns (mixer, tensors by checkpoint name in 64-bit, the layer's raw record)."""
    from tileinfer_b200.config import config_from_dict
    from tileinfer_b200.parts import Runtime, lookup
    spec = config_from_dict(case).model_spec().layers[layer].mixer
    cls = lookup("mixer", spec.kind)
    g = torch.Generator().manual_seed(seed)
    if tensors is None:
        tensors = {d.name: _random_tensor(d, g, T) for d in cls.tensors(spec)}
    rt = Runtime(T)
    position = lookup("position", spec.position.kind)(spec.position, rt, max_positions) if spec.position.kind != "none" else None
    return cls(spec, {k: v.to(T) for k, v in tensors.items()}, rt, position), tensors, case["layers"][layer]


def _run_mixer(mixer, T, h, cuts, width, neighbour=None, env=None):
    """One sequence's rows through the mixer in portions (the rest one at a time); with ``neighbour`` another sequence's rows ride
    along in every step, in front."""
    from test_parts_gpu import OneStep
    env = env or OneStep(mixer, T, max_tokens=1024, max_seqs=2)
    slot = env.cache.alloc_slot()
    other = env.cache.alloc_slot() if neighbour is not None else None
    at, out, sizes, k = 0, [], list(cuts), 0
    while at < h.shape[0]:
        n = min(sizes.pop(0) if sizes else 1, h.shape[0] - at)
        entries = [(slot, h[at:at + n].to(T))]
        if other is not None and k < neighbour.shape[0]:
            entries = [(other, neighbour[k:k + 1].to(T))] + entries
        r = env.run(mixer, entries, width)
        out.append(r[len(entries) - 1:] if len(entries) > 1 else r)
        at += n
        k += 1
    env.cache.free_slot(slot)
    if other is not None:
        env.cache.free_slot(other)
    return torch.cat(out)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_every_mixer_alone(dtype):
    """Each layer's mixer of the configurations against the plain mixer: whole, token by token, in portions whose edges fall inside,
    at and outside the windows' edges and the pages' borders, beside another sequence in the batch, and once more in the slot, pages
    and state that the run before gave back."""
    from test_parts_gpu import OneStep
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(3)
    for case in mc.CASES.values():
        width, eps = case["width"], case["norm"]["eps"]
        for layer in range(len(case["layers"])):
            mixer, W, raw = _mixer_of(case, layer, T, seed=layer)
            total = 200
            h = rnd(torch.randn(total, width, generator=g, dtype=F64), T)
            other = rnd(torch.randn(40, width, generator=g, dtype=F64), T)
            ref = plain.MIXERS[raw["type"]](h, W, f"l{layer}.mix.", raw["mixer"], eps).float()
            if raw["type"] == "attention":                          # the output's bias is the block's to add
                ref = ref - W[f"l{layer}.mix.o.b"].float()
            window = (raw["mixer"].get("mask") or {}).get("size", 50)
            env = OneStep(mixer, T, max_tokens=1024, max_seqs=2)
            for cuts in ([total], [1], [window, 2, window + 1, 3], [64, 64, 2, 2, 60], [2, 2, 2, 2]):
                got = _run_mixer(mixer, T, h, cuts, width, neighbour=other if cuts[0] in (1, 64) else None, env=env)
                err = (got - ref).abs().max(-1).values
                tol = (1e-4 if T == torch.float32 else 10 * 2.0 ** -8) * max(1.0, float(ref.abs().max()))
                assert float(err.max()) <= tol, (f"{raw['type']} layer {layer} width {width} cuts {cuts[:3]}: worst {float(err.max()):.3g} at "
                                                 f"{int(err.argmax())} ({tol:.3g}), first bad {int((err > tol).float().argmax())}")


# ---------------------------------------------------------------- weights made by hand
W16 = 16
RAW = 1.5 * 4.0 * math.sqrt(16 / 1.0625)         # the marked key's score: scale, the query's 4 after its norm, the key's e0 after its norm


def _marked_rows(total, mark_at):
    """Ordinary tokens are the unit vector e1; the marked one is e0 with a little e2."""
    h = torch.zeros(total, W16, dtype=F64)
    h[:, 1] = 1.0
    h[mark_at] = 0.0
    h[mark_at, 0], h[mark_at, 2] = 1.0, 0.25
    return h


def _identity_attention(heads, scale, cap=None, window=None, sink=-100.0, q_to_e0=True):
    """Identity projections (every head the same), a gate of one half, no biases; the heads' outputs land in columns of their own
    (head a's e2 in column 2 + 4 a). Queries of ordinary tokens point along e0, so only the marked key scores. The norms run over
    the whole row, which for identical heads is the norm of one."""
    eye = torch.eye(W16, dtype=F64)
    case = mc.model(8, W16, 1e-9, 1, 0, 1.0, [mc.attention(heads, heads, W16, scale, None, cap=cap, window=window)])
    t = {"l0.mix.q": eye.repeat(heads, 1), "l0.mix.k": eye.repeat(heads, 1), "l0.mix.g": torch.zeros(heads, W16, dtype=F64),
         "l0.mix.o": torch.cat([torch.roll(eye, 4 * a, 0) for a in range(heads)], 1), "l0.mix.o.b": torch.zeros(W16, dtype=F64),
         "l0.mix.sink": torch.full((heads,), sink, dtype=F64)}
    for k in "qk":
        t[f"l0.mix.{k}.b"] = torch.zeros(heads * W16, dtype=F64)
        t[f"l0.mix.{k}.norm"] = torch.ones(heads * W16, dtype=F64)
    if q_to_e0:
        for a in range(heads):
            t["l0.mix.q"][a * W16, 1], t["l0.mix.q"][a * W16 + 1, 1] = 1.0, 0.0
    return case, t


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_a_marked_key_is_seen_inside_the_window_and_not_beyond(dtype):
    """One head: every ordinary query scores the marked key 23 (19 with a cap of 30) above the others, so the output's e2 is half the
    marked value's 0.25 (the value is the key as projected: its norm would make it 0.97) for the window's size - 1 queries behind the
    marked one, and exactly zero from then on. Windows of 1, 2, a page, a page and one and no multiple of anything; the edge inside a
    prompt, at a portion's first token and among single tokens; the marker on both sides of a page border and far into the sequence."""
    T = DTYPES[dtype]
    for window, mark_at, cuts, total, cap in ((1, 5, [20], 20, None), (2, 4, [20], 20, 30.0), (2, 63, [64], 70, None), (7, 0, [1], 20, 30.0),
                                              (7, 62, [66, 1, 4], 80, None), (64, 3, [140], 140, 30.0), (64, 64, [100, 27], 200, None),
                                              (65, 64, [65], 140, None), (65, 0, [40, 25, 1, 30], 100, 30.0), (100, 129, [128, 1, 1, 64], 260, None),
                                              (130, 190, [300, 19, 2], 330, 30.0), (100, 227, [230], 335, None), (None, 3, [100, 1], 200, 30.0)):
        case, tensors = _identity_attention(1, 1.5, cap=cap, window=window)
        mixer, _, _ = _mixer_of(case, 0, T, tensors)
        out = _run_mixer(mixer, T, _marked_rows(total, mark_at), cuts, W16)[:, 2]
        last = total if window is None else min(mark_at + window, total)          # the first position that no longer sees the marker
        assert mark_at == 0 or float(out[:mark_at].abs().max()) == 0.0
        what = f"window {window}, marker at {mark_at}, cuts {cuts}"
        if last > mark_at + 1:
            seen = out[mark_at + 1:last]
            assert float((seen - 0.125).abs().max()) <= (1e-4 if T == torch.float32 else 0.01) * 0.125, f"{what}: {seen[:2].tolist()} .. {seen[-2:].tolist()}"
        assert last == total or float(out[last:].abs().max()) == 0.0, f"{what}: seen at {mark_at + int(out[mark_at:].abs().nonzero().max())}, edge {last}"


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_cap_slope_and_sink_against_the_closed_form(dtype):
    """Three heads: the marked key's share seen from n positions behind it is e^(c - slope n) over the sum of that, of e^(-slope j) over
    the other visible keys and of e^sink, c = cap tanh(23.3 / cap), slope = 2^(-8 (a + 1) / 3) for head a: with caps of 1.5 and 4 and
    none (and then a scale of zero, so that slopes and sink alone decide), sinks of 0 and 3, a window and none, in prompts and decoding."""
    T = DTYPES[dtype]
    for cap, scale, sink, window, mark_at, cuts, total in ((1.5, 1.5, 0.0, None, 3, [40, 2], 60), (4.0, 1.5, 3.0, 50, 64, [70, 30], 130), (None, 0.0, 2.0, None, 0, [1], 40),
                                                           (None, 0.0, 0.0, 20, 60, [62, 1, 1, 10], 90), (4.0, 1.5, 3.0, None, 5, [400], 400)):
        case, tensors = _identity_attention(3, scale, cap=cap, window=window, sink=sink, q_to_e0=scale > 0)
        mixer, _, _ = _mixer_of(case, 0, T, tensors)
        out = _run_mixer(mixer, T, _marked_rows(total, mark_at), cuts, W16)
        raw = (RAW if scale else 0.0) * 1.0
        mark = cap * math.tanh(raw / cap) if cap else raw
        for a in range(3):
            slope = 2.0 ** (-8.0 * (a + 1) / 3)
            for i in list(range(mark_at + 1, min(total, mark_at + 24))) + [total - 1]:
                first = 0 if window is None else max(0, i - window + 1)
                weights = {j: math.exp((mark if j == mark_at else 0.0) - slope * (i - j)) for j in range(first, i + 1)}
                want = 0.125 * weights.get(mark_at, 0.0) / (sum(weights.values()) + math.exp(sink))
                got = float(out[i, (2 + 4 * a) % W16])
                assert abs(got - want) <= (1e-4 if T == torch.float32 else 0.02) * want + 1e-7, \
                    f"cap {cap} sink {sink} window {window} head {a} query {i}, marker at {mark_at}: {got} for {want}"


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_a_written_value_fades_by_the_decay_exactly(dtype):
    """Retention with hand-made weights: one token writes, later tokens only read (their key is zero), so the read-out before the norm is
    decay^n times q.k; a large eps makes the norm's divisor nearly constant and the output follows it. Through a prompt, portions and
    single tokens, at two decays, with and without a rotation (whose angle turns q.k by the distance)."""
    T = DTYPES[dtype]
    D, W = 4, 8
    for rot in (None, (2, 10000.0)):
        case = mc.model(8, W, 100.0, 1, 0, 1.0, [mc.retention(2, D, D, [0.5, 0.97], None, rot=rot)])
        t = {f"l0.mix.{k}": torch.zeros(2 * D, W, dtype=F64) for k in "qkvg"}
        t["l0.mix.o"] = torch.eye(W, dtype=F64)
        for a in range(2):
            t["l0.mix.q"][a * D, 1] = t["l0.mix.q"][a * D, 0] = 1.0        # every token asks along the head's first element
            t["l0.mix.k"][a * D, 0] = 1.0                                  # only e0 writes
            t["l0.mix.v"][a * D + 2, 0] = 8.0
            t["l0.mix.g"][a * D + 2, :2] = 4.0
        mixer, _, _ = _mixer_of(case, 0, T, t)
        for mark_at, cuts, total in ((0, [60], 60), (5, [1], 40), (33, [34, 2, 30], 110)):
            h = torch.zeros(total, W, dtype=F64)
            h[:, 1] = 1.0
            h[mark_at, 0], h[mark_at, 1] = 1.0, 0.0
            out = _run_mixer(mixer, T, h, cuts, W)
            for a, decay in enumerate((0.5, 0.97)):
                for i in list(range(mark_at, min(total, mark_at + 12))) + [total - 1]:
                    n = i - mark_at
                    o = decay ** n * 8.0 * D ** -0.5 * (math.cos(n) if rot else 1.0)
                    want = o / math.sqrt(o * o / D + 100.0) * 4.0 / (1 + math.exp(-4.0))
                    assert abs(float(out[i, a * D + 2]) - want) <= (2e-5 if T == torch.float32 else 0.01) * abs(want) + (1e-6 if T == torch.float32 else 1e-3 * decay ** n)


# ---------------------------------------------------------------- kernels alone
def _step(lengths, slots, positions=None):
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    return SimpleNamespace(cu_seqlens=i32(cu), seq_slots=i32(slots), n_seqs=len(lengths), positions=i32(positions) if positions is not None else None)


def test_the_gates_of_the_matrix_memory_alone():
    """keep, add and exp(-m) against a loop in 64-bit: sequences of unequal lengths (beyond the 256 tokens a block takes at once), carried
    from portion to portion; gates that sit at both ends of the cap, so that the maximum is taken by the past and by the new token."""
    from tileinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(9)
    for H, cap, spread in ((1, 6.0, 30.0), (3, 15.0, 3.0), (5, 2.0, 1.0)):
        lengths = [700, 1, 90]
        n = sum(lengths)
        z = (torch.randn(n, 2 * H, generator=g) * spread)
        bias = torch.randn(2 * H, generator=g)
        state = torch.zeros(4, 11 + H, device="cuda")
        keep, add, em = (torch.zeros(n, H, dtype=F64) for _ in range(3))
        ms, at = [], 0
        for L in lengths:
            m = torch.zeros(H, dtype=F64)
            for t in range(at, at + L):
                gi = cap * torch.tanh((z[t, :H].double() + bias[:H]) / cap)
                gf = torch.nn.functional.logsigmoid(cap * torch.tanh((z[t, H:].double() + bias[H:]) / cap))
                new = torch.maximum(gf + m, gi)
                keep[t], add[t], em[t] = torch.exp(gf + m - new), torch.exp(gi - new), torch.exp(-new)
                m = new
            ms.append(m)
            at += L
        starts, fed, slots = [0, 700, 701], [0, 0, 0], [3, 1, 0]
        for portion in (400, 2, 1, 1, 1000):
            live = [b for b in range(3) if fed[b] < lengths[b]]
            take = [min(portion, lengths[b] - fed[b]) for b in live]
            idx = torch.cat([torch.arange(starts[b] + fed[b], starts[b] + fed[b] + k) for b, k in zip(live, take)])
            coef, got_em = torch.zeros(len(idx), H, 2, device="cuda"), torch.zeros(len(idx), H, device="cuda")
            ops.memory_gates(coef, got_em, z[idx].cuda(), bias.cuda(), cap, state, 11, _step(take, [slots[b] for b in live]), H)
            # The maxima themselves may differ by a few roundings of their size; keep and add carry the same error.
            for got, ref in ((coef[..., 0], keep), (coef[..., 1], add), (got_em, em)):
                err = ((got.cpu().double() - ref[idx]).abs() / (ref[idx] + 1e-3)).max()
                assert float(err) <= 1e-4, (H, portion, float(err))
            for b, k in zip(live, take):
                fed[b] += k
        for b in range(3):
            assert float((state[slots[b], 11:].cpu().double() - ms[b]).abs().max()) <= 1e-4
        assert float(state[2].abs().max()) == 0.0 and float(state[:, :11].abs().max()) == 0.0


@pytest.mark.parametrize("H,D,V", [(2, 24, 40), (1, 130, 70), (3, 64, 136), (2, 18, 14), (12, 128, 128), (1, 300, 64)])
def test_matrix_memories_alone(H, D, V):
    """Both recurrences against loops in 64-bit, at sizes that are no multiple of a thread's rows or a block's columns: unequal sequences in
    one launch, continued from the state by portions of 100, 37 and 2 tokens (walked one by one, and in chunks), then one token at a time
    (the one-token kernel, fused with the head's norm and gate where a block holds the head, and where it is not), a slot between them that
    nobody may touch."""
    from tileinfer_b200.kernels import ops
    from tileinfer_b200.parts import Runtime, lookup
    from tileinfer_b200.config import PositionSpec
    g = torch.Generator().manual_seed(D + V)
    for T in (torch.float32, torch.bfloat16):
        lengths = [150, 1, 145]
        n = sum(lengths)
        rot = 16 if D != 300 else 290
        rotation = lookup("position", "rope")(PositionSpec("rope", D, 100.0, None, 256, {"rotary_dim": rot, "table_dtype": "float32", "angles": "float64"}),
                                              Runtime(T), 256).rotation()
        proj = rnd(torch.randn(n, H * (2 * D + 2 * V), generator=g, dtype=F64) * 0.6, T)
        z = (torch.randn(n, 2 * H, generator=g) * 2).double()
        bias = (torch.randn(2 * H, generator=g) + torch.tensor([0.0, 2.0]).repeat_interleave(H)).double()
        cap, eps = 7.0, 1e-6
        norm_w = rnd(1 + 0.2 * torch.randn(H * V, generator=g, dtype=F64), T)
        decay = torch.rand(H, generator=g).double() * 0.3 + 0.7
        offs = (0, H * D, 2 * H * D, 2 * H * D + H * V)
        for gated in (False, True):
            ref, at = torch.zeros(n, H * V, dtype=F64), 0
            for L in lengths:
                part = proj[at:at + L]
                q, k = part[:, :H * D].view(L, H, D), part[:, H * D:2 * H * D].view(L, H, D)
                v, gate = part[:, offs[2]:offs[3]].view(L, H, V), part[:, offs[3]:]
                if gated:
                    soft = lambda x: cap * torch.tanh(x / cap)
                    zz = z[at:at + L] + bias
                    o = plain.mlstm_cell(q * D ** -0.5, k, v, soft(zz[:, :H]), torch.nn.functional.logsigmoid(soft(zz[:, H:])))
                    ref[at:at + L] = plain.rms_divide(o, eps).reshape(L, -1) * norm_w * torch.sigmoid(gate)
                else:
                    pos = torch.arange(L)
                    qr, kr = plain.rotate(q, pos, rot, 100.0), plain.rotate(k, pos, rot, 100.0) * D ** -0.5
                    S = torch.zeros(H, D, V, dtype=F64)
                    o = torch.zeros(L, H, V, dtype=F64)
                    for t in range(L):
                        S = decay[:, None, None] * S + kr[t][:, :, None] * v[t][:, None, :]
                        o[t] = torch.einsum("hdv,hd->hv", S, qr[t])
                    ref[at:at + L] = plain.rms_divide(o, eps).reshape(L, -1) * plain.silu(gate)
                at += L
            for chunked in (False, True):
                floats = -(-(H * D * V + (H * (D + 1) if gated else 0)) // 4) * 4
                state = torch.zeros(4, floats, device="cuda")
                m_off = H * D * (V + 1)
                dev = lambda t, dt=torch.float32: t.to(dt).cuda().contiguous()
                starts, fed, slots = [0, 150, 151], [0, 0, 0], [2, 0, 3]
                got = torch.zeros(n, H * V, dtype=F64)
                for portion in (100, 37, 2) + (1,) * 40:
                    live = [b for b in range(3) if fed[b] < lengths[b]]
                    if not live:
                        break
                    take = [min(portion, lengths[b] - fed[b]) for b in live]
                    idx = torch.cat([torch.arange(starts[b] + fed[b], starts[b] + fed[b] + c) for b, c in zip(live, take)])
                    pos = [fed[b] + j for b, c in zip(live, take) for j in range(c)]
                    step = _step(take, [slots[b] for b in live], pos)
                    rows_, zz = dev(proj[idx], T), dev(z[idx])
                    y = torch.full((len(idx), H * V), float("nan"), dtype=T, device="cuda")
                    o = torch.full((len(idx), H * V), float("nan"), device="cuda")
                    nq, em, mn = (torch.full((len(idx), H), float("nan"), device="cuda") for _ in range(3))
                    cell = dict(z=zz, bias=dev(bias), cap=cap, q_scale=D ** -0.5, w=dev(norm_w, T), gate_sigmoid=True) if gated else \
                        dict(decay=dev(decay), rotation=rotation, k_scale=D ** -0.5)
                    divisor, moves, done = ((nq, em) if gated else None), None, False
                    if all(c == 1 for c in take):
                        if V <= 128 and len(live) % 2:                                   # fused, or raw and finished by the norm's kernel
                            done = ops.memory_token(rows_, offs, state, step, H, D, V, y=y, eps=eps, **cell)
                            fused = done
                        else:
                            done = ops.memory_token(rows_, offs, state, step, H, D, V, o=o, outs=(nq, em, mn) if gated else (None,) * 3, **cell)
                            fused = False
                            moves = (mn, state[:, m_off:m_off + H], step.seq_slots) if gated else None
                        assert done == (V % 4 == 0)
                        moves = moves if done else None
                    else:
                        fused = False
                    if not done and chunked and max(take) > 1:
                        chunks, floats_ws = ops.memory_chunk_sizes(take, H, D, V)
                        ws, tot = torch.full((floats_ws,), float("nan"), device="cuda"), torch.full((chunks, H), float("nan"), device="cuda")
                        kw = dict(k_scale=D ** -0.5, decay=dev(decay), rotation=rotation)
                        if gated:
                            kw = dict(q_scale=D ** -0.5, coef=torch.zeros(len(idx), H, 2, device="cuda"), em=em, w=dev(norm_w, T), gate_sigmoid=True)
                            ops.memory_gates(kw["coef"], em, zz, dev(bias), cap, state, m_off, step, H)
                        fused = V <= 128
                        ops.memory_chunks(rows_, offs, state, step, H, D, V, ws, tot, chunks, y=y if fused else None, o=None if fused else o, nq=nq, eps=eps, **kw)
                    elif not done:
                        if gated:
                            coef = torch.zeros(len(idx), H, 2, device="cuda")
                            ops.memory_gates(coef, em, zz, dev(bias), cap, state, m_off, step, H)
                            ops.memory_scan(o, nq, rows_, *offs[:3], state, coef, D ** -0.5, 1.0, step, H, D, V)
                        else:
                            ops.retention_scan(o, rows_, *offs[:3], state, dev(decay), rotation, 1.0, D ** -0.5, step, H, D, V)
                    if not fused:
                        ops.heads_norm_gate(y, o, rows_[:, offs[3]:], dev(norm_w, T) if gated else None, eps, H, V, gate_sigmoid=gated, divisor=divisor, moves=moves)
                    got[idx] = y.cpu().double()
                    for b, c in zip(live, take):
                        fed[b] += c
                err = (got - ref).abs().max(-1).values
                tol = (1e-4 if T == torch.float32 else 2.0 ** -7) * max(1.0, float(ref.abs().max()))
                assert float(err.max()) <= tol, f"{T} gated {gated} chunked {chunked} {H} heads {D} x {V}: {float(err.max()):.3g} at {int(err.argmax())}"
                assert float(state[1].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("size,groups,taps", [(96, 4, 3), (60, 60, 1), (2560, 8, 4), (33, 3, 2), (1024, 1, 7)])
def test_gated_addition_norm_and_convolution_alone(dtype, size, groups, taps):
    """The stream's update against its formula: the branch as rows, as partial sums and as rows still apart with weights, with and without
    biases and gate (rows or partial sums), the norm in groups; the convolution from the step's rows and from the history, as a kernel of
    its own and inside the update (one-token steps), which must agree bit for bit with one another."""
    from tileinfer_b200.kernels import ops
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(size + taps)
    r = lambda *s: rnd(torch.randn(*s, generator=g, dtype=F64), T)
    dev = lambda t, dt=T: t.to(dt).cuda().contiguous()
    n, eps = 5, 1e-5
    x = torch.randn(n, size, generator=g).double()
    w, b1, b2 = r(size), r(size), r(size)
    apart, index, scores = r(9, size), torch.randint(0, 9, (n, 2), generator=g, dtype=torch.int32), torch.rand(n, 2, generator=g)
    parts, gparts = torch.randn(3, n, size, generator=g), torch.randn(2, n, size, generator=g)
    plain_rows, gate_rows = r(n, size), r(n, size + 8)[:, :size]
    wide = torch.zeros(n, size + 8, dtype=F64)
    wide[:, :size] = gate_rows
    gather = lambda: sum(scores[:, j:j + 1].double() * apart[index[:, j].long()] for j in range(2))
    variants = [(dict(d=dev(plain_rows), gate=dev(wide)[:, :size], d_bias=dev(b1), gate_bias=dev(b2)), plain_rows + b1, gate_rows + b2),
                (dict(d=dev(parts, torch.float32), gate=dev(gparts, torch.float32), gate_bias=dev(b2)), parts.double().sum(0), gparts.double().sum(0) + b2),
                (dict(d=dev(apart), index=index.cuda(), scores=scores.cuda(), gate=dev(wide)[:, :size]), gather(), gate_rows),
                (dict(d=dev(plain_rows), gate=None), plain_rows, None), (dict(d=None, gate=None), None, None)]
    for kw, branch, gate in variants:
        ref = x.clone()
        if branch is not None:
            ref = ref + (branch * torch.sigmoid(gate) if gate is not None else branch)
        want = plain.grouped_norm(ref, w, groups, eps)
        xd, h = x.float().cuda(), torch.full((n, size), float("nan"), dtype=T, device="cuda")
        ops.gated_add_norm32(xd, h=h, w=dev(w), eps=eps, groups=groups, **kw)
        assert float((xd.cpu().double() - ref).abs().max()) <= 1e-5 * max(1.0, float(ref.abs().max()))
        assert float((h.cpu().double() - want).abs().max()) <= (1e-5 if T == torch.float32 else 2.0 ** -7) * float(want.abs().max())
    # The convolution: three sequences in portions; every channel's taps differ.
    conv = r(size, taps)
    cw = dev(conv.t())
    lengths = [13, 1, 9]
    hs = [r(L, size) for L in lengths]
    want = [rnd(h + plain.causal_conv(h, conv), T) for h in hs]
    hist = torch.zeros(4, max(taps - 1, 1) * size, device="cuda")
    slots, fed = [3, 0, 2], [0, 0, 0]
    got = [torch.zeros(L, size, dtype=F64) for L in lengths]
    for portion in (4, 1, 2, 1, 1, 10):
        live = [b for b in range(3) if fed[b] < lengths[b]]
        take = [min(portion, lengths[b] - fed[b]) for b in live]
        rows_ = dev(torch.cat([hs[b][fed[b]:fed[b] + c] for b, c in zip(live, take)]))
        step = _step(take, [slots[b] for b in live])
        out = torch.full_like(rows_, float("nan"))
        before = hist.clone()
        ops.conv_rows(out, rows_, cw, hist if taps > 1 else None, step)
        if taps > 1:
            ops.history_update(hist, rows_, taps, step, size)
        if all(c == 1 for c in take):
            # The same step inside the stream's update: a stream whose norm is the row again would be the easy case; here the norm makes
            # its own row, which the convolution must read as it was rounded.
            xd = torch.randn(len(live), size, generator=g).cuda()
            h, fused, alone = (torch.empty_like(rows_) for _ in range(3))
            other = before.clone()
            ops.gated_add_norm32(xd, None, None, h, dev(w), eps, groups, conv=(cw, before if taps > 1 else None, step.seq_slots, fused))
            ops.conv_rows(alone, h, cw, other if taps > 1 else None, step)
            assert torch.equal(fused, alone)
            if taps > 1:
                ops.history_update(other, h, taps, step, size)
                assert torch.equal(before, other)
        at = 0
        for b, c in zip(live, take):
            got[b][fed[b]:fed[b] + c] = out[at:at + c].cpu().double()
            fed[b] += c
            at += c
    for b in range(3):
        assert float((got[b] - want[b]).abs().max()) <= (1e-5 if T == torch.float32 else 2.0 ** -7) * float(want[b].abs().max())
    assert float(hist[1].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_router_with_groups_scored_by_their_two_best(dtype):
    from tileinfer_b200.kernels import ops
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(6)
    for E, top, groups in ((12, 3, (4, 2)), (8, 2, (2, 1)), (6, 1, (6, 4)), (64, 6, (8, 3)), (5, 5, None), (9, 2, (3, 3))):
        n, width = 80, 40
        h, wr = rnd(torch.randn(n, width, generator=g, dtype=F64), T), rnd(torch.randn(E, width, generator=g, dtype=F64) * width ** -0.5, T)
        corr = rnd(torch.randn(E, generator=g, dtype=F64) - 0.6, T)                  # most choice scores are negative
        z = h @ wr.T
        chosen, margin = plain.choose(z, corr, top, {"count": groups[0], "keep": groups[1]} if groups else None)
        s = torch.sigmoid(z)
        ids, scores = torch.zeros(n, top, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
        for logits in (None, z.float().cuda()):
            ops.router_select(h.to(T).cuda(), wr.to(T).cuda(), logits, E, E, top, ids, scores, softmax=False, correction=corr.float().cuda(),
                              groups=groups[0] if groups else 1, keep=groups[1] if groups else 1, group_best=2)
            sure = 0
            for t in range(n):
                if float(margin[t]) < 1e-5:
                    continue
                sure += 1
                assert ids[t].tolist() == chosen[t].tolist(), (E, groups, t)
                want = s[t, chosen[t]] / (s[t, chosen[t]].sum() + 1e-20)
                assert float((scores[t].cpu().double() - want).abs().max()) <= 1e-5
            assert sure >= 0.9 * n


def _dense_attention(q, k, v, scale, start, window, cap, slope, sink):
    """q [n, H, D] at positions start .. of one sequence with keys k [L, G, D], in 64-bit."""
    n, H, D = q.shape
    L, G, _ = k.shape
    dist = torch.arange(start, start + n)[:, None] - torch.arange(L)[None, :]
    vis = dist >= 0
    if window:
        vis &= dist < window
    out = torch.zeros(n, H, D, dtype=F64)
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        if slope is not None:
            s = s - slope[h].double() * dist
        s = s.masked_fill(~vis, -math.inf)
        e = torch.exp(s)
        den = e.sum(-1) + (torch.exp(sink[h].double()) if sink is not None else 0.0)
        out[:, h] = (e / den[:, None]) @ v[:, h // (H // G)].double()
    return out


@pytest.mark.parametrize("nq,nkv,D,window,cap,sloped", [(8, 2, 64, 100, 9.0, True), (6, 3, 32, 0, 2.0, False), (16, 1, 128, 7, 0.0, True),
                                                        (40, 2, 64, 0, 20.0, True), (4, 4, 96, 333, 5.0, True), (3, 3, 128, 130, 1.0, False)])
def test_capped_and_sloped_attention_kernels_alone(nq, nkv, D, window, cap, sloped):
    """The paged kernels with a cap, slopes by distance, a window and a sink (plain, the prompt kernels on ``mma.sync`` and, for heads of
    64 and 128, on tensor memory, the split-KV decode kernel with 1 to 32 parts) against exact attention: sequences of unequal lengths,
    some continuing from cached positions, shuffled pages, queries scaled so that scores reach several times the cap."""
    from test_kernels_gpu import close, dev, paged
    from tileinfer_b200.kernels import fast, ops
    from tileinfer_b200.kernels.library import check, lib
    torch.manual_seed(19)
    dtype = torch.bfloat16
    r = lambda x: x.to(dtype).float()
    total, fresh = [300, 1, 130, 513, 64], [300, 1, 30, 200, 64]          # cached length after the step, tokens of the step
    B = len(total)
    ks = [r(torch.randn(L, nkv, D)) for L in total]
    vs = [r(torch.randn(L, nkv, D)) for L in total]
    qs = [r(torch.randn(n, nq, D) * (1.0 + 3.0 * (torch.rand(n, nq, 1) > 0.8))) for n in fresh]
    if window:
        ks[3][512 - window] = r(qs[3][-1, 0] * 9.0)[None].expand(nkv, D)          # just outside the last query's window
    slope = torch.tensor([2.0 ** (-8.0 * (h + 1) / nq) for h in range(nq)]) if sloped else None
    sink = torch.randn(nq)
    scale = 1 / math.sqrt(D)
    kp, vp, table = paged(ks, vs, 64, sum(-(-L // 64) for L in total) + 3, 13, dtype)
    want = torch.cat([_dense_attention(qs[b], ks[b], vs[b], scale, total[b] - fresh[b], window, cap, slope, sink) for b in range(B)]).float()
    q = dev(torch.cat(qs), dtype)
    cu = [0]
    for n in fresh:
        cu.append(cu[-1] + n)
    sink_d = dev(sink)
    slope_d, slope2 = (dev(slope), dev(slope * 1.4426950408889634)) if sloped else (None, None)
    p2 = slope2.data_ptr() if sloped else None
    slots, cu_d, lens_d = (dev(torch.arange(1, B + 1, dtype=torch.int32)), dev(torch.tensor(cu, dtype=torch.int32)), dev(torch.tensor(total, dtype=torch.int32)))
    tok_slot = dev(torch.cat([torch.full((n,), b + 1, dtype=torch.int32) for b, n in enumerate(fresh)]))
    positions = dev(torch.cat([torch.arange(total[b] - fresh[b], total[b], dtype=torch.int32) for b in range(B)]))
    empty = lambda n: torch.full((n, nq, D), float("nan"), dtype=dtype, device="cuda")
    out = empty(cu[-1])
    ops.attention_plain(out, q, kp, vp, table, tok_slot, positions, scale, nq, nkv, D, 64, window=window, sink=sink_d, cap=cap, slopes=slope_d)
    close(out, want, dtype, ulps=5.0)
    st = torch.cuda.current_stream().cuda_stream
    tpt = 128 // (nq // nkv)
    out = empty(cu[-1])
    check(lib().ti_attention_prefill_ruled(out.data_ptr(), q.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), table.stride(0), slots.data_ptr(),
                                           cu_d.data_ptr(), lens_d.data_ptr(), B, sum(-(-n // tpt) for n in fresh), scale, nq, nkv, D, 64, window,
                                           sink_d.data_ptr(), 0, None, 0, cap, p2, st), "attention_prefill")
    close(out, want, dtype, ulps=5.0)
    if D in (64, 128):
        out = empty(cu[-1])
        check(lib().ti_attention_prefill_tc_ruled(out.data_ptr(), q.data_ptr(), kp.data_ptr(), vp.data_ptr(), kp.shape[0], table.data_ptr(), table.stride(0),
                                                  slots.data_ptr(), cu_d.data_ptr(), lens_d.data_ptr(), B, cu[-1], sum(-(-n // (2 * tpt)) for n in fresh),
                                                  scale, nq, nkv, D, 64, window, fast.status_word().data_ptr(), sink_d.data_ptr(), 0, None, 0, cap, p2, st),
              "attention_prefill_tc")
        fast.check_status()
        close(out, want, dtype, ulps=5.0)
    last = [c - 1 for c in cu[1:]]                  # one token per sequence: the last query of each
    qd = dev(torch.cat(qs)[last], dtype)
    for splits in (1, 3, 32):
        out = empty(B)
        ws_o, ws_ml = torch.full((B * splits, nq, D), float("nan"), device="cuda"), torch.full((B * splits, nq, 2), float("nan"), device="cuda")
        check(lib().ti_attention_decode_ruled(out.data_ptr(), qd.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), table.stride(0), slots.data_ptr(),
                                              lens_d.data_ptr(), None, None, ws_o.data_ptr(), ws_ml.data_ptr(), scale, B, nq, nkv, D, 64, splits, window,
                                              sink_d.data_ptr(), 0, None, 0, cap, p2, st), "attention_decode")
        close(out, want[last], dtype, ulps=5.0)


def test_bfloat16_steps_take_the_fast_kernels(models):
    """Case B's sizes are ones the fast kernels take: a prompt and a one-token step in bfloat16 go through the tensor-core products, the
    grouped products of the experts and the paged attention kernels with cap and slopes, and a one-token step is one kernel per matrix
    memory of up to 128 values, not through plain stand-ins."""
    from tileinfer_b200.kernels import library
    m = models["B"]
    engine = m.engine("bfloat16", graphs=False)
    slot = engine.new_sequence()
    library.call_counts.clear()
    engine.step([(slot, mc.prompts(m.vocab, [600], 61)[0])])
    prompt = dict(library.call_counts)
    library.call_counts.clear()
    engine.step([(slot, [5])])
    token = dict(library.call_counts)
    engine.free_sequence(slot)
    engine.check_health()
    assert prompt.get("ti_attention_prefill_tc_ruled", 0) == 2 and token.get("ti_attention_decode_ruled", 0) == 2, (prompt, token)
    assert prompt.get("ti_memory_chunks", 0) == 4 and prompt.get("ti_memory_gates", 0) == 2 and prompt.get("ti_conv_rows", 0) == 6, prompt
    assert token.get("ti_memory_token", 0) == 4 and token.get("ti_heads_norm_gate", 0) == 2 and "ti_conv_rows" not in token, token
    for used in (prompt, token):
        assert used.get("ti_gemm_tcgen05_grouped", 0) == 8 and used.get("ti_gated_add_norm32", 0) == 13, used
        assert not any(k.startswith(("ti_attention_plain", "ti_grouped_gemm", "ti_gemm_plain", "ti_expert_combine")) for k in used), used
    assert prompt.get("ti_gemm_tcgen05", 0) > 0 and token.get("ti_gemv_bf16", 0) > 0


# ---------------------------------------------------------------- through the public entry points
def test_greedy_generation_through_the_public_entry_point(models):
    """``generate`` (batches, scheduler, sampler, decode loop) on several prompts at once, more than there are slots, in 32-bit:
    every generated token is the plain implementation's most likely next token for the same prefix."""
    import tileinfer_b200 as ti
    for name in ("A", "B"):
        m = models[name]
        engine = ti.load_model(m.folder, dtype="float32", max_context=256, max_seqs=3)
        reqs = mc.prompts(m.vocab, [3, 41, 90, 17, 1], 41)
        outs = ti.generate(engine, reqs, max_new_tokens=40, stop_ids=[])
        assert [len(o) for o in outs] == [40] * 5
        for p, o in zip(reqs, outs):
            ref, _ = m.reference(p + o)
            for k, tok in enumerate(o):
                row = ref[len(p) + k - 1]
                assert row[tok] >= row.max() - 1e-4 * max(1.0, float(np.abs(row).max())), f"{name} token {k}: generated {tok}, plain argmax {int(row.argmax())}"


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_trace_replay(models, dtype):
    """The same requests through ``bin/trace_run``: whole, with the tail one by one, and in two batches one after the other (the
    second in the first one's slots, pages and states). In bfloat16 on the configuration without routers, whose positions can all
    be compared."""
    m = models["B" if dtype == "float32" else "D"]
    reqs = {f"r{i}": t for i, t in enumerate(mc.prompts(m.vocab, [1, 9, 70, 130, 200], 51))}
    t = Trace()
    t.whole(reqs)
    t.tail_one_by_one(reqs, tail=20)
    names = list(reqs)
    t.batch({r: reqs[r] for r in names[:3]}, {r: min(len(reqs[r]) - 1, 4 + 3 * i) for i, r in enumerate(names[:3])}, tag="x")
    t.batch({r: reqs[r] for r in names[2:]}, {r: min(len(reqs[r]) - 1, 30) for r in names[2:]}, tag="y")
    with tempfile.TemporaryDirectory() as out:
        got = run_trace(m.folder, dtype, t, out, sum(-(-len(x) // 64) * 64 for x in reqs.values()), m.vocab)
    by_request = {}
    for (rid, pos), row in got.items():
        by_request.setdefault(rid, {})[pos] = row
    assert len(by_request) == 5 + 5 + 3 + 3
    for rid, g in by_request.items():
        mc.compare(m, reqs[rid[1:]], g, DTYPES[dtype], f"replay {dtype} {rid}", need=0.0)
