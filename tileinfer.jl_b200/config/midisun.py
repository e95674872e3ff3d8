"""Typed configuration of the Midisun design and its lowering to per-layer records.

A Midisun model is a decoder whose config.json lists its layers one by one (``layers``: ``type``, ``mixer``, ``mlp``), so every layer
may have sizes of its own. What the design fixes lives here and in the parts; what config.json gives is read from it and nowhere else:

* the embedding is multiplied by ``embedding.scale``; the stream is 32-bit; norms are RMS norms in ``norm.groups`` equal parts of the row;
* a layer is x += mixer(h + conv(h)) * sigmoid(R1 h + b1), then x += ff(h) * sigmoid(R2 h + b2), h the norm of x, conv a causal
  convolution over time of ``canon.taps`` taps per channel;
* mixer ``attention``: grouped-query attention with biases on q, k and the output, RMS norms of q and k over their whole rows, the keys as
  projected for values, scores capped at ``softcap``, a slope 2^(-8 (h + 1) / heads) by distance taken off them, a window of ``mask.size``
  positions, a sink in the softmax and one sigmoid gate per head;
* mixer ``retention``: linear attention with a fixed ``decay`` per head and a rotation of q and k, every head normed, a SiLU gate;
* mixer ``mlstm``: a matrix memory with exponential gates capped at ``gate_cap``, every head normed, a sigmoid gate;
* feed-forward ``dense``: down(silu(gate h) * (up h)); ``moe``: a sigmoid router with a correction for the choice and ``groups`` scored by
  their two best choices, the ``top`` best of ``experts`` such units, weights divided by their sum.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .apertus import ConfigError, _require
from .spec import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec

DEFAULT_MAX_POSITIONS = 131072       # config.json gives no limit; tables are sized by the engine's max_context below this


def _need(m: Mapping[str, Any], key: str, where: str):
    if not isinstance(m, Mapping) or key not in m or m[key] is None:
        raise ConfigError(f"config.json: {where} has no \"{key}\"")
    return m[key]


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: Optional[float] = None
    window: Optional[int] = None         # mask.size

    @classmethod
    def from_dict(cls, m, where):
        mask, heads, dim = m.get("mask"), int(_need(m, "heads", where)), int(_need(m, "dim", where))
        out = cls(heads, int(m.get("kv_heads") or heads), dim, float(_need(m, "scale", where)), None if not m.get("softcap") else float(m["softcap"]),
                  None if not mask else int(_need(mask, "size", where + ".mask")))
        if min(out.heads, out.kv_heads, out.dim) < 1 or out.heads % out.kv_heads:
            raise ConfigError(f"{where}: {out.heads} query heads do not divide into {out.kv_heads} key/value heads")
        if int(m.get("vdim") or dim) != dim:
            raise ConfigError(f"{where}: values are the keys as projected, so vdim {m['vdim']} must be dim {dim}")
        if (out.window is not None and out.window < 1) or (out.softcap is not None and out.softcap <= 0):
            raise ConfigError(f"{where}: mask.size and softcap must be positive")
        return out

    def to_dict(self):
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.dim}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        return d

    def slopes(self):
        return tuple(2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads))


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def from_dict(cls, m, where):
        rot, dim = m.get("rot"), int(_need(m, "dim", where))
        out = cls(int(_need(m, "heads", where)), dim, int(m.get("vdim") or dim), tuple(float(a) for a in _need(m, "decay", where)),
                  0 if not rot else int(_need(rot, "dims", where + ".rot")), 10000.0 if not rot else float(_need(rot, "base", where + ".rot")))
        if min(out.heads, out.dim, out.vdim) < 1 or len(out.decay) != out.heads:
            raise ConfigError(f"{where}: {len(out.decay)} decays for {out.heads} heads")
        if out.rot_dims < 0 or out.rot_dims % 2 or out.rot_dims > out.dim:
            raise ConfigError(f"{where}.rot.dims {out.rot_dims} must be even and at most dim {out.dim}")
        return out

    def to_dict(self):
        d = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return d


@dataclass(frozen=True)
class MLstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, m, where):
        dim = int(_need(m, "dim", where))
        out = cls(int(_need(m, "heads", where)), dim, int(m.get("vdim") or dim), float(_need(m, "gate_cap", where)))
        if min(out.heads, out.dim, out.vdim) < 1 or out.gate_cap <= 0:
            raise ConfigError(f"{where}: heads, dim, vdim and gate_cap must be positive")
        return out

    def to_dict(self):
        return {"dim": self.dim, "gate_cap": self.gate_cap, "heads": self.heads, "vdim": self.vdim}


MIXERS = {"attention": AttentionConfig, "retention": RetentionConfig, "mlstm": MLstmConfig}


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    top: int
    groups: Optional[Tuple[int, int]] = None      # (count, keep)

    def to_dict(self):
        r = {"experts": self.experts, "top": self.top}
        if self.groups:
            r["groups"] = {"count": self.groups[0], "keep": self.groups[1]}
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": r}


def _mlp_from_dict(m, where):
    if m is None:
        return None
    kind = _need(m, "kind", where)
    if kind == "dense":
        out = DenseConfig(int(_need(m, "ff", where)))
        if out.ff < 1:
            raise ConfigError(f"{where}.ff must be positive")
        return out
    if kind != "moe":
        raise ConfigError(f"{where}.kind \"{kind}\" is not a feed-forward of this design (dense, moe)")
    r = _need(m, "router", where)
    g = r.get("groups")
    out = MoeConfig(int(_need(_need(m, "expert", where), "ff", where + ".expert")), int(_need(r, "experts", where + ".router")),
                    int(_need(r, "top", where + ".router")),
                    None if not g else (int(_need(g, "count", where + ".router.groups")), int(_need(g, "keep", where + ".router.groups"))))
    if out.ff < 1 or not 1 <= out.top <= out.experts:
        raise ConfigError(f"{where}.router: top {out.top} of {out.experts} experts")
    if out.groups:
        count, keep = out.groups
        if count < 1 or out.experts % count or not 1 <= keep <= count or keep * (out.experts // count) < out.top:
            raise ConfigError(f"{where}.router.groups: {keep} of {count} groups of {out.experts} experts for top {out.top}")
    return out


@dataclass(frozen=True)
class MidisunLayerConfig:
    type: str                          # "attention" | "retention" | "mlstm"
    mixer: Any
    mlp: Any                           # DenseConfig | MoeConfig | None


@dataclass(frozen=True)
class MidisunConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    canon_taps: int                    # 0: the mixers read the norm's output itself
    embedding_scale: float
    layers: Tuple[MidisunLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Midisun"
    model_type = "midisun"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, c: Mapping[str, Any]) -> "MidisunConfig":
        layers = []
        for i, l in enumerate(_require(c, "layers")):
            where = f"layers[{i}]"
            kind = _need(l, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}.type \"{kind}\" is not a mixer of this design ({', '.join(MIXERS)})")
            layers.append(MidisunLayerConfig(kind, MIXERS[kind].from_dict(_need(l, "mixer", where), where + ".mixer"),
                                             _mlp_from_dict(l.get("mlp"), where + ".mlp")))
        eos = c.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        norm = _require(c, "norm")
        out = cls(vocab=int(_require(c, "vocab")), width=int(_require(c, "width")), norm_eps=float(_need(norm, "eps", "norm")),
                  norm_groups=int(norm.get("groups") or 1), canon_taps=int((c.get("canon") or {}).get("taps") or 0),
                  embedding_scale=float((c.get("embedding") or {}).get("scale", 1.0)), layers=tuple(layers),
                  max_positions=int(c.get("max_positions") or DEFAULT_MAX_POSITIONS), eos_token_ids=eos)
        if out.vocab < 1 or out.width < 1 or not layers:
            raise ConfigError("vocab and width must be positive and layers not empty")
        if out.norm_groups < 1 or out.width % out.norm_groups:
            raise ConfigError(f"norm.groups {out.norm_groups} does not divide width {out.width}")
        if not 0 <= out.canon_taps <= 64:
            raise ConfigError(f"canon.taps {out.canon_taps}: up to 64 taps are built")
        return out

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
             "layers": [{"mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict(), "type": l.type} for l in self.layers],
             "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "vocab": self.vocab, "width": self.width}
        if self.canon_taps:
            d["canon"] = {"taps": self.canon_taps}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- lowering
    def _mixer_spec(self, kind: str, m, prefix: str) -> MixerSpec:
        W, eps = self.width, self.norm_eps
        if kind == "attention":
            return MixerSpec(kind="conv_attention", prefix=prefix, hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                             qk_norm=True, qk_norm_eps=eps, scale=m.scale, window=m.window,
                             tensor_names={"q": "q", "k": "k", "g": "g", "o": "o", "sink": "sink", "bias_suffix": ".b", "norm_suffix": ".norm"},
                             options={"value_dim": m.dim, "conv_taps": 0, "bias": True, "out_bias": True, "row_norm": True, "sink": True,
                                      "gate": "head", "shared_kv": True, "softcap": m.softcap, "slopes": m.slopes()})
        names = {k: k for k in ("q", "k", "v", "g", "o")}
        if kind == "retention":
            position = PositionSpec(kind="none")
            if m.rot_dims:
                position = PositionSpec(kind="rope", head_dim=m.dim, theta=m.rot_base, max_positions=self.max_positions,
                                        options={"rotary_dim": m.rot_dims, "pairing": "half", "table_dtype": "float32", "angles": "float64"})
            return MixerSpec(kind="retention", prefix=prefix, hidden_size=W, num_heads=m.heads, head_dim=m.dim, position=position,
                             tensor_names=names, options={"value_dim": m.vdim, "decay": m.decay, "norm_eps": eps})
        return MixerSpec(kind="mlstm", prefix=prefix, hidden_size=W, num_heads=m.heads, head_dim=m.dim,
                         tensor_names={**names, "i": "i", "f": "f", "norm": "norm", "bias_suffix": ".b"},
                         options={"value_dim": m.vdim, "gate_cap": m.gate_cap, "norm_eps": eps})

    def _feed_forward_spec(self, x, prefix: str) -> FeedForwardSpec:
        if isinstance(x, DenseConfig):
            return FeedForwardSpec("gated_mlp", prefix, self.width, x.ff, {"gate": "gate", "up": "up", "down": "down"}, {"activation": "silu"})
        return FeedForwardSpec("routed_experts", prefix, self.width, x.ff,
                               {"router": "router", "correction": "correction", "expert": "e{}.", "gate": "gate", "up": "up", "down": "down"},
                               {"experts": x.experts, "top": x.top, "limit": None, "score": "sigmoid", "correction": True, "groups": x.groups,
                                "group_best": 2, "renormalize": True, "scale_input": False})

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = lambda name: NormSpec("rmsnorm32", W, eps, name, {"init_std": 0.1, "groups": self.norm_groups})
        layers = []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            ffn = None if l.mlp is None else self._feed_forward_spec(l.mlp, p + "mlp.")
            layers.append(LayerSpec("gated", self._mixer_spec(l.type, l.mixer, p + "mix."), norm(p + "norm1"), ffn,
                                    None if ffn is None else norm(p + "norm2"),
                                    options={"taps": self.canon_taps, "conv": p + "canon1", "gates": (p + "rg1", p + "rg2"), "bias_suffix": ".b"}))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers), order=tuple(range(len(layers))),
            final_norm=norm("final.norm"), embed_name="embed", lm_head_name="head", max_positions=self.max_positions,
            eos_token_ids=self.eos_token_ids, init_std=W ** -0.5, embedding_kind="scaled_pair32", head_kind="linear",
            options={"residual_dtype": "float32", "embed_init_std": 1.0, "embed_scale": self.embedding_scale})
