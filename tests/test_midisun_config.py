"""The Midisun configuration on the CPU: keys read and refused, the round trip, the records and tensors it lowers to, and pieces of
the plain implementation against closed forms."""
import copy
import json
import math

import pytest
import torch

import midisun_cases as mc
import plain_midisun as plain
from tileinfer_b200.config import ConfigError, config_from_dict
from tileinfer_b200.engine.model import tensor_declarations


@pytest.mark.parametrize("name", sorted(mc.CASES))
def test_round_trip_and_registry(name):
    case = mc.CASES[name]
    cfg = config_from_dict(case)
    assert type(cfg).__name__ == "MidisunConfig"
    assert config_from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    spec = cfg.model_spec()
    assert spec.architecture == "Midisun" and len(spec.layers) == len(case["layers"]) and spec.order == tuple(range(len(case["layers"])))
    assert spec.options["residual_dtype"] == "float32" and spec.options["embed_scale"] == case["embedding"]["scale"]
    for layer, raw in zip(spec.layers, case["layers"]):
        assert layer.block == "gated" and layer.mixer_norm.options["groups"] == case["norm"]["groups"]
        assert (layer.feed_forward is None) == (raw["mlp"] is None)
        assert layer.mixer.kind == {"attention": "conv_attention"}.get(raw["type"], raw["type"])


def test_what_is_refused():
    for path, value in ((("layers", 0, "type"), "convolution"), (("layers", 0, "mixer", "heads"), 5), (("layers", 0, "mixer", "vdim"), 12),
                        (("layers", 0, "mlp", "router", "top"), 9), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
                        (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 2, "mixer", "rot", "dims"), 7),
                        (("layers", 2, "mixer", "decay"), [0.5, 0.9]), (("layers", 1, "mixer", "gate_cap"), 0.0), (("layers", 0, "mlp", "kind"), "other"),
                        (("norm", "groups"), 7), (("layers", 3, "mixer", "mask", "size"), -1), (("canon", "taps"), 100)):
        bad = copy.deepcopy(mc.CASE_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError):
            config_from_dict(bad)
    for path in (("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "gate_cap"), ("layers", 2, "mixer", "decay"), ("norm", "eps"), ("width",)):
        bad = copy.deepcopy(mc.CASE_A)
        at = bad
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_declared_tensors():
    names = {d.name: d.shape for d in tensor_declarations(config_from_dict(mc.CASE_A).model_spec())}
    assert names["l0.mix.q"] == (60, 60) and names["l0.mix.k"] == (20, 60) and "l0.mix.v" not in names
    assert names["l0.mix.q.b"] == (60,) and names["l0.mix.k.norm"] == (20,) and names["l0.mix.o.b"] == (60,) and names["l0.mix.sink"] == (6,)
    assert names["l0.mix.g"] == (6, 60) and names["l0.canon1"] == (60, 4) and names["l0.rg2"] == (60, 60) and names["l0.rg1.b"] == (60,)
    assert names["l1.mix.i"] == (3, 60) and names["l1.mix.f.b"] == (3,) and names["l1.mix.norm"] == (42,) and names["l1.mix.v"] == (42, 60)
    assert names["l2.mix.g"] == (66, 60) and "l2.mix.norm" not in names and "l2.norm2" not in names and "l2.rg2" not in names and "l2.rg1" in names
    assert names["l0.mlp.correction"] == (6,) and names["l1.mlp.e4.down"] == (60, 12) and names["l3.mlp.gate"] == (36, 60)
    assert not any("canon" in d.name for d in tensor_declarations(config_from_dict(mc.CASE_D).model_spec()))


def test_the_command_line_writes_a_model_folder(tmp_path):
    from tileinfer_b200.cli import cli
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(mc.CASE_C))
    out = tmp_path / "model"
    assert cli(["random", str(cfg), str(out), "--seed", "4"]) == 0
    raw, W = mc.load_folder(str(out))
    assert config_from_dict(raw) == config_from_dict(mc.CASE_C) and W["l1.mix.q"].shape == (16, 64) and W["l0.canon1"].shape == (64, 1)


# ---------------------------------------------------------------- the plain implementation against closed forms
def test_plain_norm_and_convolution():
    x = torch.tensor([[3.0, -3.0, 0.5, 0.5]], dtype=torch.float64)
    y = plain.grouped_norm(x, torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=torch.float64), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[1.0, -2.0, 3.0, 4.0]], dtype=torch.float64))
    rows = torch.arange(1, 6, dtype=torch.float64)[:, None]
    y = plain.causal_conv(rows, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64))
    assert y[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]


def test_plain_slopes_and_window():
    assert plain.slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625] and abs(plain.slopes(3)[0] - 2 ** (-8 / 3)) < 1e-15
    # One head whose scores are all zero: with a window of 2 and no sink to speak of, a token's weights are 1 and exp(-slope).
    W = {"l.q": torch.zeros(4, 4), "l.k": torch.eye(4), "l.q.b": torch.zeros(4), "l.k.b": torch.zeros(4), "l.q.norm": torch.ones(4),
         "l.k.norm": torch.ones(4), "l.sink": torch.tensor([-1e9]), "l.g": torch.zeros(1, 4), "l.o": torch.eye(4), "l.o.b": torch.zeros(4)}
    W = {k: v.double() for k, v in W.items()}
    h = torch.eye(4, dtype=torch.float64)
    m = {"heads": 1, "dim": 4, "scale": 1.0, "mask": {"size": 2}, "softcap": 5.0}
    y = plain.attention(h, W, "l.", m, 1e-6) * 2.0                    # the gate is sigmoid(0)
    e = math.exp(-2.0 ** -8)
    for i in range(1, 4):
        want = torch.zeros(4, dtype=torch.float64)
        want[i], want[i - 1] = 1 / (1 + e), e / (1 + e)
        assert torch.allclose(y[i], want)


def test_plain_matrix_memories():
    # Retention of one key: what a token wrote comes back times the decay to the power of the distance.
    W = {"l.q": torch.ones(1, 2), "l.k": torch.tensor([[1.0, 0.0]]), "l.v": torch.tensor([[1.0, 0.0]]), "l.g": torch.ones(1, 2), "l.o": torch.ones(1, 1)}
    S = torch.zeros(5, dtype=torch.float64)
    h = torch.tensor([[1.0, 0.0]] + [[0.0, 1.0]] * 4, dtype=torch.float64)
    y = plain.retention(h, {k: v.double() for k, v in W.items()}, "l.", {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, 1.0)
    for t in range(5):
        o = 0.5 ** t
        S[t] = o / math.sqrt(o * o + 1.0) * (1 / (1 + math.exp(-1.0)))
    assert torch.allclose(y[:, 0], S)
    # The mLSTM cell against the same sums without the running maximum (small gates, so that nothing overflows).
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(6, 1, n, generator=g, dtype=torch.float64) for n in (3, 3, 2))
    ig, fg = torch.randn(6, 1, generator=g, dtype=torch.float64), torch.nn.functional.logsigmoid(torch.randn(6, 1, generator=g, dtype=torch.float64))
    o = plain.mlstm_cell(q, k, v, ig, fg)
    for t in range(6):
        w = torch.stack([ig[j, 0] + fg[j + 1:t + 1, 0].sum() for j in range(t + 1)]).exp()
        num = sum(w[j] * (k[j, 0] @ q[t, 0]) * v[j, 0] for j in range(t + 1))
        den = sum(w[j] * (k[j, 0] @ q[t, 0]) for j in range(t + 1)).abs()
        m = max(max(float(ig[j, 0] + fg[j + 1:t + 1, 0].sum()) for j in range(t + 1)), float(fg[:t + 1, 0].sum()))
        want = num / (max(float(den), 1.0) + 1e-6 * math.exp(m))
        assert torch.allclose(o[t, 0], want, rtol=1e-9)


def test_plain_router_groups():
    """A group with two good experts beats one with a single better expert; a choice score may be negative; the margin is the smaller gap."""
    score = torch.tensor([[0.9, 0.1, 0.6, 0.5, 0.2, 0.3]], dtype=torch.float64)
    z = torch.log(score / (1 - score))
    zero = torch.zeros(6, dtype=torch.float64)
    chosen, margin = plain.choose(z, zero, 2, {"count": 3, "keep": 1})
    assert sorted(chosen[0].tolist()) == [2, 3] and abs(float(margin) - 0.1) < 1e-12
    chosen, _ = plain.choose(z, torch.tensor([0.2, 0, 0, 0, 0, 0], dtype=torch.float64), 2, {"count": 3, "keep": 1})
    assert sorted(chosen[0].tolist()) == [0, 1]
    chosen, _ = plain.choose(z, zero - 2.0, 2, {"count": 3, "keep": 1})
    assert sorted(chosen[0].tolist()) == [2, 3]
    assert plain.choose(z, zero, 1)[0].tolist() == [[0]]
