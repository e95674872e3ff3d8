"""The Pemarax design through the engine against the plain implementation (``plain_pemarax``): whole prompts, prompts in portions down to
two tokens, token-by-token decoding, batches of unequal requests against each alone, slots, pages and states that are used again, long
decoding past every window, hand-made weights that make one key, a window's edge, a kept position, a sink or a decay stand out, every
mechanism and kernel alone, greedy generation through the public entry point and trace replay; in 32-bit and in bfloat16, at three sets of
sizes."""
import math
import tempfile

import numpy as np
import pytest
import torch

import pemarax_cases as pc
import plain_pemarax as plain
from replay_util import Trace, run_trace
from test_midisun_gpu import _run_mixer, _step, rnd, rows, run_cut

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


@pytest.fixture(scope="module")
def models():
    with tempfile.TemporaryDirectory() as tmp:
        yield {name: pc.Model(name, seed, tmp) for name, seed in (("A", 51), ("B", 52), ("C", 53))}


def engine_of(m, dtype, **kw):
    """(engine, recorder of its router choices or None). In bfloat16 a router choice can rest on a gap that rounding closes, so the
    run's own choices are noted (which needs steps that are not replayed from graphs) and the plain implementation takes the same;
    in 32-bit the engine runs as it is served, graphs and all, and chooses for itself."""
    if dtype == "bfloat16":
        engine = m.engine(dtype, graphs=False, **kw)
        return engine, pc.Recorder(engine, m.cfg)
    return m.engine(dtype, **kw), None


# ---------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts_and_prompts_in_portions(models, name, dtype):
    m = models[name]
    engine, rec = engine_of(m, dtype)
    forced = lambda: rec.of(0) if rec is not None else None
    for tokens in pc.prompts(m.vocab, [1, 2, 7, 64, 65, 150, 400], 21):
        got = run_cut(engine, tokens, [len(tokens)], rec)
        pc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} whole {len(tokens)}", forced=forced())
    tokens = pc.prompts(m.vocab, [280], 22)[0]
    # Portions that start and end inside and at page borders and inside and at the windows' edges, two tokens, one token.
    for cuts in ([100, 100, 80], [63, 1, 64, 2, 2, 148], [2, 2, 2, 58, 64, 3, 1, 1, 100, 47], [129, 2, 61, 2, 86], [5, 4, 1, 57, 3, 100, 110]):
        got = run_cut(engine, tokens, cuts, rec)
        pc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} portions {cuts[:4]}", forced=forced())


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_from_a_short_prompt(models, name, dtype):
    """A prompt of three tokens, then 330 single tokens: pages fill up and fall out of the windows while decoding, kept ones stay, and
    the recurrent states and the convolutions' rows come from the sequence's state at every step."""
    m = models[name]
    engine, rec = engine_of(m, dtype, max_tokens=512, max_seqs=2)
    tokens = pc.prompts(m.vocab, [333], 23)[0]
    got = run_cut(engine, tokens, [3], rec)
    pc.compare(m, tokens, got, DTYPES[dtype], f"{name} {dtype} long decoding", forced=rec.of(0) if rec is not None else None)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_batches_of_unequal_requests_and_reuse_of_slots_pages_and_states(models, name, dtype):
    """Requests of unequal lengths prefilled in one step and decoded together, the shorter ones leaving first; then a second batch
    in the slots, pages and states that the first gave back. Every request is compared with the plain implementation of that
    request alone."""
    m = models[name]
    engine, rec = engine_of(m, dtype, max_tokens=1024, max_seqs=4)
    for seed, lengths, tails in ((31, [1, 40, 129, 300], [0, 12, 40, 3]), (32, [70, 3, 230, 64], [6, 2, 65, 33])):
        reqs = pc.prompts(m.vocab, lengths, seed)
        slots = [engine.new_sequence() for _ in reqs]
        heads = [len(t) - d for t, d in zip(reqs, tails)]
        if rec is not None:
            rec.choices.clear()
            rec.rows = [(i, p) for i, h in enumerate(heads) for p in range(h)]
        a = engine.step([(s, t[:h]) for s, t, h in zip(slots, reqs, heads)], [list(range(h)) for h in heads]).detach().float().cpu().numpy()
        ends = np.cumsum(heads)
        got = [{p: a[e - h + p].copy() for p in range(h)} for e, h in zip(ends, heads)]
        fed = list(heads)
        live = list(range(len(reqs)))
        while live:
            for i in [i for i in live if fed[i] == len(reqs[i])]:
                engine.free_sequence(slots[i])
                live.remove(i)
            if not live:
                break
            if rec is not None:
                rec.rows = [(i, fed[i]) for i in live]
            out = engine.step([(slots[i], [reqs[i][fed[i]]]) for i in live]).detach().float().cpu().numpy()
            for r, i in enumerate(live):
                got[i][fed[i]] = out[r].copy()
                fed[i] += 1
        engine.check_health()
        for i, t in enumerate(reqs):
            assert sorted(got[i]) == list(range(len(t)))
            pc.compare(m, t, got[i], DTYPES[dtype], f"{name} {dtype} batch seed {seed} request {i}", forced=rec.of(i) if rec is not None else None)
    assert engine.cache.slots.held == 0


@pytest.mark.parametrize("name", ["A", "B"])
def test_steps_that_mix_prompts_portions_and_single_tokens(models, name):
    """One step brings a new prompt, a portion of another request and single tokens of two more: the states and the convolutions' rows
    of each come from its own slot, and a one-token request takes the many-token kernels."""
    m = models[name]
    engine, _ = engine_of(m, "float32", max_tokens=1024, max_seqs=4)
    reqs = pc.prompts(m.vocab, [80, 120, 61, 33], 35)
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
        pc.compare(m, t, got[i], torch.float32, f"{name} mixed steps request {i}")


def test_a_long_step_runs_in_chunks(models):
    """A step longer than the engine takes at once is cut inside it; pages of the windows come and go between the chunks."""
    m = models["B"]
    engine = m.engine("float32", max_step_tokens=128, max_seqs=2)
    tokens = pc.prompts(m.vocab, [500], 36)[0]
    slot = engine.new_sequence()
    got = rows(engine.step([(slot, tokens)], [list(range(500))]), range(500))
    assert engine.cache.groups[0].pages.held < 8
    pc.compare(m, tokens, got, torch.float32, "chunks")


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer(models, name):
    m = models[name]
    engine = m.engine("float32")
    tokens = pc.prompts(m.vocab, [90], 27)[0]
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
    """Each kind of layer alone and twice in a row; windows of one, two and a page and one, kept positions inside, beside and beyond the
    window; many taps; one expert, every expert; values and states of one and beyond a block's columns."""
    T = DTYPES[dtype]
    D4 = pc.moe(20, 2, 1)
    one = 1 if T == torch.float32 else 5          # rows of very few values normed are little more than signs, which rounding to bfloat16 may turn
    cases = {
        "attention only": pc.model(50, 24, 1e-4, 0.3, [pc.attention(3, 1, 6, 5, 0.3, D4, window=1, keep=1, conv=5), pc.attention(2, 2, 16, None, 0.5, None, window=2, keep=130),
                                                        pc.attention(4, 1, 12, 20, 0.4, pc.moe(8, 4, 4), window=65, keep=64, rot=(4, 9.0)),
                                                        pc.attention(16, 4, 32, 48, 0.3, None, window=40, keep=9, conv=4, rot=(30, 9.0))]),
        "latent only": pc.model(71, 40, 1e-5, 1.3, [pc.latent(2, 4, 2, 3, 5, 0.5, 30.0, D4, window=1), pc.latent(1, 50, 14, 60, 90, 0.2, 50.0, None),
                                                     pc.latent(5, 16, 8, 1, 250, 0.1, 10.0, pc.moe(12, 1, 1), window=128)]),
        "parallel only": pc.model(33, 32, 1e-6, 0.6, [pc.parallel((2, 1, 6, 5, 0.4, 3), (3, one, 1, 1, 9, 1), D4), pc.parallel((1, 1, 40, 8, 0.2, 100), (1, 150, 140, 1, 2, 1), None),
                                                       pc.parallel((3, 3, 8, 16, 0.3, None), (8, 16, 32, 8, 4, 8), pc.moe(12, 3, 3)),
                                                       pc.parallel((20, 5, 36, 16, 0.3, 30), (4, 8, 16, 2, 4, 1), None)]),
    }
    with tempfile.TemporaryDirectory() as tmp:
        for name, case in cases.items():
            m = pc.Model(name.replace(" ", "_"), 3, tmp, case)
            engine, rec = engine_of(m, dtype, max_tokens=512, max_seqs=2, max_context=256)
            tokens = pc.prompts(m.vocab, [220], 5)[0]
            for cuts in ([220], [2, 64, 3], [70, 1, 1, 58]):
                got = run_cut(engine, tokens, cuts, rec)
                pc.compare(m, tokens, got, T, f"{name} {dtype} {cuts}", forced=rec.of(0) if rec is not None else None)


# ---------------------------------------------------------------- mixers alone
def _random_tensor(d, g, T):
    name, shape = d.name, tuple(d.shape)
    t = torch.randn(shape, generator=g, dtype=F64)
    if name.endswith(".conv"):
        t = 0.4 * t + 0.3
    elif len(shape) == 2:
        t = t * shape[1] ** -0.5
    elif name.endswith((".norm", ".out", ".D")):
        t = 1 + 0.2 * t
    elif name.endswith(".dt_bias"):
        t = t - 2
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


def _window(raw):
    m = raw["mixer"].get("left", raw["mixer"])
    return (m.get("mask") or {}).get("size", 50)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_every_mixer_alone(dtype):
    """Each layer's mixer of the configurations against the plain mixer: whole, token by token, in portions whose edges fall inside,
    at and outside the windows' edges and the pages' borders, beside another sequence in the batch, and once more in the slot, pages
    and state that the run before gave back."""
    from test_parts_gpu import OneStep
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(3)
    for case in pc.CASES.values():
        width, eps = case["width"], case["norm"]["eps"]
        for layer in range(len(case["layers"])):
            mixer, W, raw = _mixer_of(case, layer, T, seed=layer)
            total = 220
            h = rnd(torch.randn(total, width, generator=g, dtype=F64), T)
            other = rnd(torch.randn(40, width, generator=g, dtype=F64), T)
            ref = plain.MIXERS[raw["type"]](h, W, f"l{layer}.mix.", raw["mixer"], eps).float()
            window = _window(raw)
            env = OneStep(mixer, T, max_tokens=1024, max_seqs=2)
            for cuts in ([total], [1], [window, 2, window + 1, 3], [64, 64, 2, 2, 60], [2, 2, 2, 2]):
                got = _run_mixer(mixer, T, h, cuts, width, neighbour=other if cuts[0] in (1, 64) else None, env=env)
                err = (got - ref).abs().max(-1).values
                tol = (1e-4 if T == torch.float32 else 10 * 2.0 ** -8) * max(1.0, float(ref.abs().max()))
                assert float(err.max()) <= tol, (f"{raw['type']} layer {layer} width {width} cuts {cuts[:3]}: worst {float(err.max()):.3g} at "
                                                 f"{int(err.argmax())} ({tol:.3g}), first bad {int((err > tol).float().argmax())}")


# ---------------------------------------------------------------- weights made by hand
W16 = 16


def _marked_rows(total, mark_at):
    """Ordinary tokens are the unit vector e1; the marked one is e0 with a little e2."""
    h = torch.zeros(total, W16, dtype=F64)
    h[:, 1] = 1.0
    h[mark_at] = 0.0
    h[mark_at, 0], h[mark_at, 2] = 1.0, 0.25
    return h


def _identity_attention(scale, window, keep, latent=False, normed=False):
    """One head with identity projections whose queries point along e0 for ordinary tokens, so that only the marked key scores; latent: the
    latent is the row, keys and values are it; normed: the parallel mixer's attention. Returns (mixer's raw layer, tensors by name)."""
    eye = torch.eye(W16, dtype=F64)
    q = eye.clone()
    q[0, 1], q[1, 1] = 1.0, 0.0
    if latent:
        layer = pc.latent(1, W16, 2, W16, W16, scale, 10.0, None, window=window)
        t = {"q": torch.cat([q, torch.zeros(2, W16, dtype=F64)]), "dkv": torch.cat([eye, torch.zeros(2, W16, dtype=F64)]), "dkv.norm": torch.ones(W16, dtype=F64),
             "uk": eye, "uv": eye, "o": eye}
        return pc.model(8, W16, 1e-9, 1.0, [layer]), {"l0.mix." + k: v for k, v in t.items()}
    t = {"q": q, "k": eye, "v": eye, "o": eye}
    if normed:
        layer = pc.parallel((1, 1, W16, W16, scale, window), (1, 4, 4, 1, 1, 1), None)
        t.update({"q.norm": torch.ones(W16, dtype=F64), "k.norm": torch.ones(W16, dtype=F64)})
        return pc.model(8, W16, 1e-9, 1.0, [layer]), {"l0.mix.left." + k: v for k, v in t.items()}
    return pc.model(8, W16, 1e-9, 1.0, [pc.attention(1, 1, W16, W16, scale, None, window=window, keep=keep)]), {"l0.mix." + k: v for k, v in t.items()}


def _identity_mixer(kind, T, scale, window, keep):
    from tileinfer_b200.config import config_from_dict
    from tileinfer_b200.parts import Runtime, lookup
    case, tensors = _identity_attention(scale, window, keep, latent=kind == "latent", normed=kind == "normed")
    if kind != "normed":
        return _mixer_of(case, 0, T, tensors)[0]
    spec = config_from_dict(case).model_spec().layers[0].mixer.options["left"]
    return lookup("mixer", spec.kind)(spec, {k: v.to(T) for k, v in tensors.items()}, Runtime(T), None)


PLACES = ((1, 0, 5, [20], 20), (2, 0, 4, [20], 20), (2, 1, 0, [1], 30), (7, 3, 2, [1], 40), (7, 3, 3, [30, 2], 40), (9, 64, 63, [66, 2], 200),
          (9, 64, 64, [200], 260), (64, 1, 0, [140], 300), (64, 65, 64, [100, 27], 330), (64, 65, 65, [65], 200), (65, 128, 127, [129, 1, 60], 400),
          (100, 130, 129, [400], 420), (100, 130, 130, [128, 2, 64], 300), (130, 20, 190, [300, 19, 2], 330), (100, 300, 227, [230], 340),
          (None, 0, 3, [100, 1], 200))


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("kind", ["attention", "latent", "normed"])
def test_a_marked_key_is_seen_inside_the_window_and_where_it_is_kept(kind, dtype):
    """Every ordinary query scores the marked key 20 or more above the others, so the output's e2 is the marked value for the window's size - 1
    queries behind it, and exactly zero from then on; a marked key among the kept first positions is seen by every later query, the first one
    behind them is not. Edges inside prompts, at portions' first tokens and among single tokens, markers on both sides of page borders."""
    T = DTYPES[dtype]
    for window, keep, mark_at, cuts, total in PLACES:
        if kind != "attention":
            keep = 0
        mixer = _identity_mixer(kind, T, 1.5 if kind != "latent" else 6.0, window, keep)
        out = _run_mixer(mixer, T, _marked_rows(total, mark_at), cuts, W16)[:, 2]
        value = 0.25 if kind != "latent" else 0.25 / math.sqrt((1 + 0.0625) / W16)
        last = total if window is None or mark_at < keep else min(mark_at + window, total)      # the first position that no longer sees the marker
        what = f"{kind} window {window}, {keep} kept, marker at {mark_at}, cuts {cuts}"
        assert mark_at == 0 or float(out[:mark_at].abs().max()) == 0.0, what
        if last > mark_at + 1:
            seen = out[mark_at + 1:last]
            assert float((seen - value).abs().max()) <= (1e-4 if T == torch.float32 else 0.01) * value, f"{what}: {seen[:2].tolist()} .. {seen[-2:].tolist()}"
        assert last == total or float(out[last:].abs().max()) == 0.0, f"{what}: seen at {mark_at + int(out[mark_at:].abs().nonzero().max())}, edge {last}"


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("kind", ["attention", "latent", "normed"])
def test_how_many_keys_are_seen(kind, dtype):
    """With a scale of zero every visible key weighs the same: the ordinary value's share is n / (n + 1) of n visible keys where one is added
    to the denominator, and the marked value's share is one in n where nothing is."""
    T = DTYPES[dtype]
    for window, keep, mark_at, cuts, total in PLACES:
        if kind != "attention":
            keep = 0
        mixer = _identity_mixer(kind, T, 0.0, window, keep)
        rows_ = _marked_rows(total, mark_at)
        if kind == "attention":
            rows_[:] = 0.0
            rows_[:, 1] = 1.0
        out = _run_mixer(mixer, T, rows_, cuts, W16)
        ok = plain.visible(total, {"size": window, "keep_first": keep})
        n = ok.sum(-1).double()
        if kind == "attention":
            want = n / (n + 1)
            got = out[:, 1].double()
        else:
            value = 0.25 if kind != "latent" else 0.25 / math.sqrt((1 + 0.0625) / W16)
            want, got = ok[:, mark_at].double() * value / n, out[:, 2].double()
        err = (got - want).abs() / (want + 1e-9)
        assert float(err.max()) <= (2e-5 if T == torch.float32 else 0.01), f"{kind} window {window} keep {keep}: {float(err.max())} at {int(err.argmax())}"


# ---------------------------------------------------------------- kernels alone
def _dense_attention(q, k, v, scale, start, window, keep, sink):
    """q [n, H, D] at positions start .. of one sequence with keys k [L, G, D], in 64-bit."""
    n, H, D = q.shape
    L, G, _ = k.shape
    ok = plain.visible(L, {"size": window, "keep_first": keep})[start:start + n]
    out = torch.zeros(n, H, D, dtype=F64)
    for h in range(H):
        s = ((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale).masked_fill(~ok, -math.inf)
        e = torch.exp(s)
        out[:, h] = (e / (e.sum(-1) + torch.exp(sink[h].double()))[:, None]) @ v[:, h // (H // G)].double()
    return out


@pytest.mark.parametrize("nq,nkv,D,window,keep", [(8, 2, 64, 100, 20), (6, 3, 32, 7, 64), (16, 1, 128, 64, 65), (40, 2, 64, 130, 1), (4, 4, 96, 200, 300),
                                                  (3, 3, 128, 1, 128), (12, 4, 64, 90, 700), (5, 1, 256, 70, 129), (32, 8, 128, 300, 130)])
def test_attention_kernels_with_kept_positions_alone(nq, nkv, D, window, keep):
    """The paged kernels with a window beside kept first positions and a sink (plain, the prompt kernels on ``mma.sync`` and, for heads of 64
    and 128, on tensor memory, the split-KV decode kernel with 1 to 32 parts) against exact attention: sequences of unequal lengths, some
    continuing from cached positions. The block tables name a page full of NaN keys wherever no query may look, as after the pages between
    the kept ones and the window were given back and taken by someone else (whose values are finite)."""
    from test_kernels_gpu import close, dev, paged
    from tileinfer_b200.kernels import fast, ops
    from tileinfer_b200.kernels.library import check, lib
    torch.manual_seed(19)
    dtype = torch.bfloat16
    r = lambda x: x.to(dtype).float()
    total, fresh = [300, 1, 130, 613, 64, 1100], [300, 1, 30, 200, 64, 40]          # cached length after the step, tokens of the step
    B = len(total)
    ks = [r(torch.randn(L, nkv, D)) for L in total]
    vs = [r(torch.randn(L, nkv, D)) for L in total]
    qs = [r(torch.randn(n, nq, D)) for n in fresh]
    ks[3][612 - window] = r(qs[3][-1, 0] * 9.0)[None].expand(nkv, D)                # just outside the last query's window
    ks[5][min(keep, 1099)] = r(qs[5][-1, 0] * 9.0)[None].expand(nkv, D)             # just behind the kept positions
    ks[5][keep - 1] = r(qs[5][-1, 0] * 3.0)[None].expand(nkv, D)                    # the last kept position
    sink = torch.randn(nq)
    scale = 1 / math.sqrt(D)
    kp, vp, table = paged(ks, vs, 64, sum(-(-L // 64) for L in total) + 3, 13, dtype)
    used = set(table[1:B + 1].flatten().tolist()) if table.shape[0] > B else set(table.flatten().tolist())
    spare = next(p for p in range(kp.shape[0]) if p not in used)
    kp[spare] = float("nan")
    for b in range(B):
        start = total[b] - fresh[b]
        for page in range(-(-total[b] // 64)):                                       # pages come and go in units of two
            unit = page // 2 * 2 * 64
            if unit >= keep and unit + 128 <= max(0, start - window + 1):
                table[b + 1, page] = spare
    want = torch.cat([_dense_attention(qs[b], ks[b], vs[b], scale, total[b] - fresh[b], window, keep, sink) for b in range(B)]).float()
    q = dev(torch.cat(qs), dtype)
    cu = np.concatenate([[0], np.cumsum(fresh)]).tolist()
    sink_d = dev(sink)
    slots, cu_d, lens_d = (dev(torch.arange(1, B + 1, dtype=torch.int32)), dev(torch.tensor(cu, dtype=torch.int32)), dev(torch.tensor(total, dtype=torch.int32)))
    tok_slot = dev(torch.cat([torch.full((n,), b + 1, dtype=torch.int32) for b, n in enumerate(fresh)]))
    positions = dev(torch.cat([torch.arange(total[b] - fresh[b], total[b], dtype=torch.int32) for b in range(B)]))
    empty = lambda n: torch.full((n, nq, D), float("nan"), dtype=dtype, device="cuda")
    out = empty(cu[-1])
    ops.attention_plain(out, q, kp, vp, table, tok_slot, positions, scale, nq, nkv, D, 64, window=window, sink=sink_d, keep=keep)
    close(out, want, dtype, ulps=5.0)
    st = torch.cuda.current_stream().cuda_stream
    tpt = 128 // (nq // nkv)
    out = empty(cu[-1])
    check(lib().ti_attention_prefill_kept(out.data_ptr(), q.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), table.stride(0), slots.data_ptr(),
                                          cu_d.data_ptr(), lens_d.data_ptr(), B, sum(-(-n // tpt) for n in fresh), scale, nq, nkv, D, 64, window,
                                          sink_d.data_ptr(), 0, None, 0, 0.0, None, keep, st), "attention_prefill")
    close(out, want, dtype, ulps=5.0)
    if D in (64, 128):
        out = empty(cu[-1])
        check(lib().ti_attention_prefill_tc_kept(out.data_ptr(), q.data_ptr(), kp.data_ptr(), vp.data_ptr(), kp.shape[0], table.data_ptr(), table.stride(0),
                                                 slots.data_ptr(), cu_d.data_ptr(), lens_d.data_ptr(), B, cu[-1], sum(-(-n // (2 * tpt)) for n in fresh),
                                                 scale, nq, nkv, D, 64, window, fast.status_word().data_ptr(), sink_d.data_ptr(), 0, None, 0, 0.0, None, keep,
                                                 st), "attention_prefill_tc")
        fast.check_status()
        close(out, want, dtype, ulps=5.0)
    last = [c - 1 for c in cu[1:]]                  # one token per sequence: the last query of each
    qd = dev(torch.cat(qs)[last], dtype)
    for splits in (1, 3, 32):
        out = empty(B)
        ws_o, ws_ml = torch.full((B * splits, nq, D), float("nan"), device="cuda"), torch.full((B * splits, nq, 2), float("nan"), device="cuda")
        check(lib().ti_attention_decode_kept(out.data_ptr(), qd.data_ptr(), kp.data_ptr(), vp.data_ptr(), table.data_ptr(), table.stride(0), slots.data_ptr(),
                                             lens_d.data_ptr(), None, None, ws_o.data_ptr(), ws_ml.data_ptr(), scale, B, nq, nkv, D, 64, splits, window,
                                             sink_d.data_ptr(), 0, None, 0, 0.0, None, keep, st), "attention_decode")
        close(out, want[last], dtype, ulps=5.0)


def _ssm_reference(rows_, lengths, conv, bias, dt_bias, a_log, skip, H, G, N, V, T):
    """(y before gate and norm, final states) of unequal sequences in 64-bit; the convolution's output is rounded to T, as kernels store it."""
    inner, C = H * V, H * V + 2 * G * N
    ys, states, at = [], [], 0
    for L in lengths:
        part = rows_[at:at + L]
        xbc = rnd(plain.silu(plain.causal_conv(part[:, inner:inner + C], conv) + bias), T)
        x, B, Cm = torch.split(xbc, [inner, G * N, G * N], -1)
        dt = plain.softplus(part[:, inner + C:inner + C + H] + dt_bias)
        ys.append(plain.state_space_cell(x.reshape(L, H, V), B.reshape(L, G, N), Cm.reshape(L, G, N), dt, a_log, skip).reshape(L, inner))
        S = torch.zeros(H, N, V, dtype=F64)
        for t in range(L):
            b = B[t].view(G, N).repeat_interleave(H // G, 0)
            S = torch.exp(-torch.exp(a_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t].view(H, V)[:, None, :]
        states.append(S)
        at += L
    return torch.cat(ys), states


@pytest.mark.parametrize("H,G,N,V,taps", [(6, 2, 20, 36, 4), (2, 1, 130, 70, 2), (4, 4, 18, 14, 3), (8, 2, 128, 64, 4), (3, 3, 64, 136, 1), (12, 3, 16, 48, 6),
                                          (4, 1, 64, 64, 4), (2, 2, 256, 128, 3), (5, 1, 48, 80, 4), (1, 1, 1, 1, 2), (4, 2, 32, 96, 5), (3, 1, 96, 32, 1)])
def test_the_state_space_kernels_alone(H, G, N, V, taps):
    """Inputs, chunks and the one-token step against loops in 64-bit: unequal sequences in one launch, continued from the state by portions
    of 130, 64, 37 and 2 tokens, then one token at a time; step sizes and decays over several orders of magnitude (a head that forgets within
    a token, one that keeps everything); work space full of NaN and a slot between the sequences that nobody may touch."""
    from tileinfer_b200.kernels import ops
    from tileinfer_b200.parts import Runtime
    from tileinfer_b200.parts.state_space import chunk_step
    g = torch.Generator().manual_seed(N + V)
    inner, C = H * V, H * V + 2 * G * N
    ld = inner + C + H + (-(inner + C + H)) % 16
    for T in (torch.float32, torch.bfloat16):
        lengths = [330, 1, 145]
        n = sum(lengths)
        rows_ = rnd(torch.randn(n, ld, generator=g, dtype=F64), T)
        conv, bias = rnd(torch.randn(C, taps, generator=g, dtype=F64) * 0.5, T), rnd(torch.randn(C, generator=g, dtype=F64) * 0.3, T)
        dt_bias = torch.linspace(-4, 1, H, dtype=F64).float().double()
        a_log = torch.linspace(4, -7, H, dtype=F64).float().double() if H > 1 else torch.tensor([-3.0], dtype=F64)
        skip = torch.randn(H, generator=g).double()
        ref, states = _ssm_reference(rows_, lengths, conv, bias, dt_bias, a_log, skip, H, G, N, V, T)
        dev = lambda t, dt=torch.float32: t.to(dt).cuda().contiguous()
        hist_off = -(-H * N * V // 4) * 4
        state = torch.zeros(4, hist_off + -(-max(taps - 1, 1) * C // 4) * 4, device="cuda")
        rt = Runtime(T)
        starts, fed, slots = [0, 330, 331], [0, 0, 0], [2, 0, 3]
        got = torch.zeros(n, inner, dtype=F64)
        for portion in (130, 64, 37, 2) + (1,) * 97:
            live = [b for b in range(3) if fed[b] < lengths[b]]
            if not live:
                break
            take = [min(portion, lengths[b] - fed[b]) for b in live]
            idx = torch.cat([torch.arange(starts[b] + fed[b], starts[b] + fed[b] + c) for b, c in zip(live, take)])
            step = _step(take, [slots[b] for b in live], [fed[b] + j for b, c in zip(live, take) for j in range(c)])
            step.is_decode, step.host_q_lens = all(c == 1 for c in take), take
            r = dev(rows_[idx], T)
            xbc, coef = torch.full((len(idx), C), float("nan"), dtype=T, device="cuda"), torch.full((len(idx), H, 2), float("nan"), device="cuda")
            hist = state[:, hist_off:] if taps > 1 else None
            ops.ssm_inputs(xbc, coef, r, inner, inner + C, dev(conv.t(), T), dev(bias, T), hist, dev(dt_bias), dev(a_log), step)
            y = torch.full((len(idx), inner), float("nan"), device="cuda")
            if step.is_decode:
                ops.ssm_token(y, xbc, coef, dev(skip), state, step, H, G, N, V)
            else:
                if taps > 1:
                    ops.history_update(hist, r[:, inner:], taps, step, C)
                chunk_step(rt, y, xbc, coef, dev(skip), state, step, H, G, N, V)
                for name, buf in rt._buffers.items():                              # the next step must not read what this one left there
                    if buf.is_floating_point():
                        buf.fill_(float("nan"))
            got[idx] = y.cpu().double()
            for b, c in zip(live, take):
                fed[b] += c
        # An element of the convolution's output may round the other way in 32-bit: one unit of bfloat16 in one factor.
        tol = (2e-5 if T == torch.float32 else 2.0 ** -8) * max(1.0, float(ref.abs().max()))
        err = (got - ref).abs().max(-1).values
        assert float(err.max()) <= tol, f"{T}: {float(err.max()):.3g} at {int(err.argmax())}, {tol:.3g}"
        for b in range(3):
            S = state[slots[b], :H * N * V].view(H, N, V).cpu().double()
            assert float((S - states[b]).abs().max()) <= tol * max(1.0, float(states[b].abs().max())) , (T, b)
            if taps > 1:
                ends = starts[b] + lengths[b]
                past = torch.zeros(taps - 1, C, dtype=F64)
                have = min(taps - 1, lengths[b])
                past[taps - 1 - have:] = rows_[ends - have:ends, inner:inner + C]
                assert torch.equal(state[slots[b], hist_off:hist_off + (taps - 1) * C].view(taps - 1, C).cpu().double(), past)
        assert float(state[1].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("size,parts", [(96, 4), (60, 60), (2560, 8), (33, 3), (1024, 1), (4096, 2)])
def test_gate_and_norm_in_parts_alone(dtype, size, parts):
    from tileinfer_b200.kernels import ops
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(size)
    y, z, w = torch.randn(7, size, generator=g).double(), rnd(torch.randn(7, size + 24, generator=g, dtype=F64), T), rnd(torch.randn(size, generator=g, dtype=F64), T)
    y[:, :size // parts] *= 20.0                                                   # parts of different sizes
    want = plain.parts_norm(y * plain.silu(z[:, 8:8 + size]), w, parts, 1e-5)
    out = torch.full((7, size), float("nan"), dtype=T, device="cuda")
    ops.ssm_gate_norm(out, y.float().cuda(), z.to(T).cuda()[:, 8:8 + size], w.to(T).cuda(), 1e-5, parts)
    assert float((out.cpu().double() - want).abs().max()) <= (1e-5 if T == torch.float32 else 2.0 ** -8) * float(want.abs().max())


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_the_stream_update_with_a_multiplier_and_a_gain_around_zero(dtype):
    from tileinfer_b200.kernels import ops
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(8)
    for size in (60, 33, 1024):
        x, d = torch.randn(5, size, generator=g).double(), rnd(torch.randn(5, size, generator=g, dtype=F64), T)
        parts, w = torch.randn(3, 5, size, generator=g), rnd(0.3 * torch.randn(size, generator=g, dtype=F64), T)
        apart, index, scores = rnd(torch.randn(9, size, generator=g, dtype=F64), T), torch.randint(0, 9, (5, 2), generator=g, dtype=torch.int32), torch.rand(5, 2, generator=g)
        gathered = sum(scores[:, j:j + 1].double() * apart[index[:, j].long()] for j in range(2))
        for mult in (0.37, 1.0):
            for kw, branch in ((dict(d=d.to(T).cuda()), d), (dict(d=parts.cuda()), parts.double().sum(0)),
                               (dict(d=apart.to(T).cuda(), index=index.cuda(), scores=scores.cuda()), gathered)):
                ref = x + mult * branch
                want = plain.offset_norm(ref, w, 1e-5)
                xd, h = x.float().cuda(), torch.full((5, size), float("nan"), dtype=T, device="cuda")
                ops.gated_add_norm32(xd, gate=None, h=h, w=w.to(T).cuda(), eps=1e-5, mult=mult, offset=True, **kw)
                assert float((xd.cpu().double() - ref).abs().max()) <= 1e-5 * max(1.0, float(ref.abs().max()))
                assert float((h.cpu().double() - want).abs().max()) <= (1e-5 if T == torch.float32 else 2.0 ** -7) * float(want.abs().max())


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_the_stream_update_by_two_normed_sublayers(dtype):
    """Both sides as rows and as partial sums, of very different sizes, against the formula and against the sum made by a kernel of its own."""
    from tileinfer_b200.kernels import ops
    from tileinfer_b200.parts import Runtime
    from tileinfer_b200.parts.norm import PairRows
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(8)
    for size in (60, 33, 1024, 5000):
        x, w = torch.randn(5, size, generator=g).double(), rnd(0.3 * torch.randn(size, generator=g, dtype=F64), T)
        wa, wb = rnd(torch.randn(size, generator=g, dtype=F64), T), rnd(torch.randn(size, generator=g, dtype=F64), T)
        a, b, parts = rnd(50 * torch.randn(5, size, generator=g, dtype=F64), T), rnd(0.02 * torch.randn(5, size, generator=g, dtype=F64), T), torch.randn(3, 5, size, generator=g)
        for left, right, lv, rv in ((a.to(T).cuda(), b.to(T).cuda(), a, b), (parts.cuda(), b.to(T).cuda(), parts.double().sum(0), b),
                                    (b.to(T).cuda(), parts.cuda(), b, parts.double().sum(0))):
            pair = 0.7 * plain.rms_divide(lv, 1e-4) * wa + 0.4 * plain.rms_divide(rv, 1e-4) * wb
            ref = x + 0.6 * pair
            want = plain.offset_norm(ref, w, 1e-5)
            xd, h = x.float().cuda(), torch.full((5, size), float("nan"), dtype=T, device="cuda")
            wad, wbd = wa.to(T).cuda(), wb.to(T).cuda()
            ops.pair_add_norm32(xd, left, right, wad, wbd, 0.7, 0.4, 1e-4, 0.6, h, w.to(T).cuda(), 1e-5, offset=True)
            assert float((xd.cpu().double() - ref).abs().max()) <= 1e-5 * max(1.0, float(ref.abs().max()))
            assert float((h.cpu().double() - want).abs().max()) <= (1e-5 if T == torch.float32 else 2.0 ** -7) * float(want.abs().max())
            apart = PairRows(left, right, wad, wbd, 1e-4, 0.7, 0.4).combined(Runtime(T))
            assert float((apart[0].cpu().double() - pair).abs().max()) <= 1e-5 * max(1.0, float(pair.abs().max()))


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_router_that_chooses_on_biased_logits(dtype):
    """Biases that decide the choice, logits so far apart that a softmax over all of them would be zero for most, equal logits (the smaller
    index first), one expert and all of them."""
    from tileinfer_b200.kernels import ops
    T = DTYPES[dtype]
    g = torch.Generator().manual_seed(6)
    for E, top, spread in ((12, 3, 1.0), (8, 8, 1.0), (6, 1, 1.0), (64, 6, 1.0), (1, 1, 1.0), (40, 5, 300.0)):
        n, width = 80, 40
        h, wr = rnd(torch.randn(n, width, generator=g, dtype=F64), T), rnd(spread * torch.randn(E, width, generator=g, dtype=F64) * width ** -0.5, T)
        bias = rnd(2 * torch.randn(E, generator=g, dtype=F64), T)
        h[0] = 0.0
        bias[:2] = bias[0]
        z = h @ wr.T + bias
        chosen, margin = plain.choose(z, top)
        ids, scores = torch.zeros(n, top, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
        for logits in (None, (h @ wr.T).float().cuda()):
            ops.router_select(h.to(T).cuda(), wr.to(T).cuda(), logits, E, E, top, ids, scores, logit_bias=bias.float().cuda(), on_logits=True)
            sure = 0
            for t in range(n):
                if float(margin[t]) < 1e-4 * spread:
                    continue
                sure += 1
                assert sorted(ids[t].tolist()) == sorted(chosen[t].tolist()), (E, t)
                want = torch.softmax(z[t][ids[t].cpu().long()], -1)
                assert float((scores[t].cpu().double() - want).abs().max()) <= 1e-5 * spread
            assert sure >= 0.9 * n
            if E > 2 and float(bias[0]) >= float(bias.sort(descending=True).values[min(top, E - 1)]):
                order = ids[0].tolist()
                assert 1 not in order or 0 in order and order.index(0) < order.index(1)


def test_bfloat16_steps_take_the_fast_kernels(models):
    """Case B's sizes are ones the fast kernels take: a prompt and a one-token step in bfloat16 go through the tensor-core products, the
    grouped products of the experts, the paged attention kernels with kept positions and the state-space kernels, not through plain stand-ins."""
    from tileinfer_b200.kernels import library
    m = models["B"]
    engine = m.engine("bfloat16", graphs=False)
    slot = engine.new_sequence()
    library.call_counts.clear()
    engine.step([(slot, pc.prompts(m.vocab, [600], 61)[0])])
    prompt = dict(library.call_counts)
    library.call_counts.clear()
    engine.step([(slot, [5])])
    token = dict(library.call_counts)
    engine.free_sequence(slot)
    engine.check_health()
    assert prompt.get("ti_attention_prefill_tc_kept", 0) == 3 and token.get("ti_attention_decode_kept", 0) == 3, (prompt, token)
    assert prompt.get("ti_attention_prefill_tc", 0) == 3 and prompt.get("ti_attention_prefill", 0) == 1, prompt
    assert prompt.get("ti_ssm_inputs", 0) == 2 and prompt.get("ti_ssm_chunks_tc", 0) == 2 and "ti_ssm_chunks" not in prompt and token.get("ti_ssm_token", 0) == 2, (prompt, token)
    for used in (prompt, token):
        assert used.get("ti_gemm_tcgen05_grouped", 0) == 12 and used.get("ti_gated_add_norm32", 0) == 11 and used.get("ti_pair_add_norm32", 0) == 2, used
        assert not any(k.startswith(("ti_attention_plain", "ti_grouped_gemm", "ti_gemm_plain", "ti_expert_combine", "ti_head_gemm")) for k in used), used
    assert prompt.get("ti_gemm_tcgen05", 0) > 0 and token.get("ti_gemv_bf16", 0) > 0


# ---------------------------------------------------------------- through the public entry points
def test_greedy_generation_through_the_public_entry_point(models):
    """``generate`` (batches, scheduler, sampler, decode loop) on several prompts at once, more than there are slots, in 32-bit:
    every generated token is the plain implementation's most likely next token for the same prefix."""
    import tileinfer_b200 as ti
    for name in ("A", "B"):
        m = models[name]
        engine = ti.load_model(m.folder, dtype="float32", max_context=256, max_seqs=3)
        reqs = pc.prompts(m.vocab, [3, 41, 90, 17, 1], 41)
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
    second in the first one's slots, pages and states)."""
    m = models["B" if dtype == "float32" else "C"]
    reqs = {f"r{i}": t for i, t in enumerate(pc.prompts(m.vocab, [1, 9, 70, 130, 200], 51))}
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
        pc.compare(m, reqs[rid[1:]], g, DTYPES[dtype], f"replay {dtype} {rid}", need=0.0)
