"""The Pemarax configuration on the CPU: keys read and refused, the round trip, the records and tensors it lowers to, the books of a window
with kept first positions, and pieces of the plain implementation against closed forms."""
import copy
import json
import math

import pytest
import torch

import pemarax_cases as pc
import plain_pemarax as plain
from tileinfer_b200.cache import Cache
from tileinfer_b200.config import ConfigError, config_from_dict
from tileinfer_b200.engine.model import tensor_declarations
from tileinfer_b200.parts import CacheRequest


@pytest.mark.parametrize("name", sorted(pc.CASES))
def test_round_trip_and_registry(name):
    case = pc.CASES[name]
    cfg = config_from_dict(case)
    assert type(cfg).__name__ == "PemaraxConfig"
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    spec = cfg.model_spec()
    assert spec.architecture == "Pemarax" and len(spec.layers) == len(case["layers"]) and spec.order == tuple(range(len(case["layers"])))
    assert spec.options["residual_dtype"] == "float32"
    for layer, raw in zip(spec.layers, case["layers"]):
        assert layer.block == "gated" and layer.options["residual_mult"] == case["residual_mult"] and layer.mixer_norm.options["offset"]
        assert (layer.feed_forward is None) == (raw["mlp"] is None)
        assert layer.mixer.kind == {"attention": "conv_attention", "parallel": "pair"}.get(raw["type"], raw["type"])
        if raw["type"] == "attention":
            m = raw["mixer"].get("mask") or {}
            assert layer.mixer.window == m.get("size") and layer.mixer.options["keep_first"] == m.get("keep_first", 0)
        if raw["type"] == "parallel":
            assert layer.mixer.options["right"].head_dim == raw["mixer"]["right"]["state"]


def test_what_is_refused():
    for path, value in ((("layers", 0, "type"), "convolution"), (("layers", 0, "mixer", "heads"), 5), (("layers", 0, "mlp", "router", "top"), 9),
                        (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "dims"), 12), (("layers", 0, "mixer", "mask", "size"), -1),
                        (("layers", 0, "mixer", "mask", "keep_first"), -2), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0),
                        (("layers", 1, "mixer", "right", "groups"), 4), (("layers", 1, "mixer", "right", "norm_groups"), 4),
                        (("layers", 1, "mixer", "left", "mask", "keep_first"), 3), (("layers", 1, "mixer", "right", "state"), 0),
                        (("layers", 2, "mixer", "rot_dim"), 8), (("layers", 2, "mixer", "mask", "keep_first"), 3), (("layers", 0, "mlp", "kind"), "dense"), (("vocab",), 0)):
        bad = copy.deepcopy(pc.CASE_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)
    for path in (("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "right", "state"), ("layers", 1, "mixer", "left"), ("layers", 2, "mixer", "kv_rank"),
                 ("layers", 0, "mixer", "rot", "scaling", "slow"), ("layers", 0, "mlp", "expert"), ("norm", "eps"), ("width",)):
        bad = copy.deepcopy(pc.CASE_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_declared_tensors():
    names = {d.name: d.shape for d in tensor_declarations(config_from_dict(pc.CASE_A).model_spec())}
    assert names["l0.mix.q"] == (60, 60) and names["l0.mix.k"] == (20, 60) and names["l0.mix.v"] == (28, 60) and names["l0.mix.o"] == (60, 84)
    assert names["l0.mix.v.conv"] == (28, 3) and "l0.mix.q.norm" not in names and "l0.mix.sink" not in names and "l0.mix.q.b" not in names
    assert names["l0.mlp.router.b"] == (6,) and names["l0.mlp.e5.up"] == (20, 60) and "l0.mlp.e0.gate" not in names
    assert names["l1.mix.left.q.norm"] == (12,) and names["l1.mix.left.o"] == (60, 66) and names["l1.mix.left.out"] == (60,)
    assert names["l1.mix.right.in"] == (2 * 42 + 2 * 30 + 6, 60) and names["l1.mix.right.conv"] == (102, 4) and names["l1.mix.right.conv.b"] == (102,)
    assert names["l1.mix.right.A_log"] == names["l1.mix.right.D"] == names["l1.mix.right.dt_bias"] == (6,) and names["l1.mix.right.norm"] == (42,)
    assert names["l2.mix.q"] == (48, 60) and names["l2.mix.dkv"] == (24, 60) and names["l2.mix.uk"] == (30, 18) and names["l2.mix.uv"] == (42, 18)
    assert "l2.norm2" not in names and "l2.mlp.router" not in names and names["final.norm"] == (60,)
    absent = {d.name for d in tensor_declarations(config_from_dict(pc.CASE_C).model_spec())}
    assert not any(n.endswith("q.conv") for n in absent) and "l1.mix.right.conv" in absent


def test_the_command_line_writes_a_model_folder(tmp_path):
    from tileinfer_b200.cli import cli
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(pc.CASE_C))
    out = tmp_path / "model"
    assert cli(["random", str(cfg), str(out), "--seed", "4"]) == 0
    raw, W = pc.load_folder(str(out))
    assert config_from_dict(raw) == config_from_dict(pc.CASE_C) and W["l1.mix.right.conv"].shape == (64, 1) and W["l2.mix.dkv"].shape == (32, 64)


def _windowed(window, keep, **kw):
    args = dict(max_tokens=64 * 40, max_seqs=2, max_step_tokens=256)
    args.update(kw)
    return Cache([CacheRequest("paged_kv", kv_heads=1, head_dim=8, window=window, keep_first=keep)], torch.float32, "cpu", **args)


@pytest.mark.parametrize("window,keep", [(100, 1), (64, 128), (10, 200), (300, 64)])
def test_kept_pages_stay_while_the_window_moves_on(window, keep):
    cache = _windowed(window, keep)
    group = cache.groups[0]
    unit = 64 * group.release_granule
    slot, other = cache.alloc_slot(), cache.alloc_slot()
    length = 0
    for n in [200, 1, 1, 250, 63, 65, 128, 1, 256, 256]:
        cache.reserve([(slot, n)])
        cache.prepare([(slot, n)])
        cache.advance(slot, n)
        length += n
        table = group.table(slot)
        needed = {p // 64 for p in range(length) if p < keep or p > length - window}
        assert all(table[p] is not None for p in needed), (length, table)
        held = [p for p in table if p is not None]
        assert len(held) == len(set(held)) == group.pages.held
        bound = -(-keep // unit) * group.release_granule + -(-(window - 1) // 64) + group.release_granule + 1
        assert len(held) <= bound, (length, len(held), bound)
    kept = [table[p] for p in range(-(-keep // 64))]
    assert None not in kept
    cache.reserve([(other, 100)])
    assert not set(kept) & {p for p in group.table(other) if p is not None}
    with pytest.raises(ValueError):
        cache.truncate(slot, keep + 1)                               # pages behind the kept ones were given back
    cache.free_slot(slot)
    cache.free_slot(other)
    assert group.pages.held == 0


def test_a_pool_of_kept_pages_holds_every_sequence():
    """The pool that a group with a window sizes for itself has room for all sequences' windows, kept pages and one step."""
    cache = _windowed(70, 130, max_tokens=64 * 400, max_seqs=5, max_seq_len=64 * 60, max_step_tokens=128)
    slots = [cache.alloc_slot() for _ in range(5)]
    assert cache.groups[0].num_pages < 5 * 60
    for round_ in range(40):
        growth = [(s, 20 + 3 * i) for i, s in enumerate(slots)]
        cache.reserve(growth, chunk_tokens=128)
        for s, n in growth:
            cache.prepare([(s, n)])
            cache.advance(s, n)
    assert all(cache.groups[0].table(s)[2] is not None for s in slots)


# ---------------------------------------------------------------- the plain implementation against closed forms
def test_plain_masks():
    ok = plain.visible(7, {"size": 2, "keep_first": 1})
    assert ok[5].tolist() == [True, False, False, False, True, True, False] and ok[0].tolist() == [True] + [False] * 6
    assert plain.visible(3, None).tolist() == [[True, False, False], [True, True, False], [True, True, True]]


def test_plain_softmax_with_one_more():
    q, k = torch.zeros(3, 1, 2, dtype=torch.float64), torch.zeros(3, 1, 2, dtype=torch.float64)
    v = torch.ones(3, 1, 1, dtype=torch.float64)
    out = plain.attend(q, k, v, 1.0, plain.visible(3, None), one_more=True)
    assert torch.allclose(out[:, 0], torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=torch.float64))


def test_plain_rotation():
    x = torch.tensor([[[1.0, 0.0, 5.0]], [[1.0, 0.0, 5.0]]], dtype=torch.float64)
    y = plain.rotate(x, torch.tensor([0, 1]), {"dims": 2, "base": 100.0}, True)
    assert torch.allclose(y[1, 0], torch.tensor([math.cos(1), math.sin(1), 5.0], dtype=torch.float64))
    # a factor of one changes no frequency and multiplies by one; beyond the ramp a frequency is divided by the factor
    rot = {"factor": 1.0, "original": 64, "fast": 8.0, "slow": 1.0}
    assert plain.frequencies(8, 100.0, rot) == (plain.frequencies(8, 100.0)[0], 1.0)
    f, mult = plain.frequencies(64, 10.0, {"factor": 4.0, "original": 8, "fast": 1.0, "slow": 0.9})
    base, _ = plain.frequencies(64, 10.0)
    assert abs(mult - (0.1 * math.log(4.0) + 1)) < 1e-15 and abs(f[-1] - base[-1] / 4) < 1e-15 and f[0] == base[0]


def test_plain_state_space():
    """One head, one state: what a token writes comes back times the decay to the power of the distance, beside the skip."""
    t, dt, a = 6, 0.3, 0.4
    x = torch.zeros(t, 1, 1, dtype=torch.float64)
    x[1] = 2.0
    one = torch.ones(t, 1, 1, dtype=torch.float64)
    y = plain.state_space_cell(x, one, one, torch.full((t, 1), dt, dtype=torch.float64), torch.tensor([math.log(a)], dtype=torch.float64),
                               torch.tensor([5.0], dtype=torch.float64))[:, 0, 0]
    want = [0.0] + [dt * 2.0 * math.exp(-a * dt) ** n for n in range(t - 1)]
    want[1] += 10.0
    assert torch.allclose(y, torch.tensor(want, dtype=torch.float64))
    assert abs(float(plain.softplus(torch.tensor(-30.0, dtype=torch.float64))) - math.exp(-30.0)) < 1e-25


def test_plain_router():
    z = torch.tensor([[1.0, 3.0, 2.0, -1.0]], dtype=torch.float64)
    chosen, margin = plain.choose(z, 2)
    assert chosen.tolist() == [[1, 2]] and float(margin) == 1.0
    assert plain.choose(z, 4)[1].tolist() == [math.inf]
