"""Typed configuration of the Pemarax design and its lowering to per-layer records.

A Pemarax model is a decoder whose config.json lists its layers one by one (``layers``: ``type``, ``mixer``, ``mlp``), so every layer
may have sizes of its own. What the design fixes lives here and in the parts; what config.json gives is read from it and nowhere else:

* the stream is 32-bit; a layer is x += m mixer(norm(x)), then x += m ff(norm(x)), m = ``residual_mult``; norms are RMS norms whose weight
  is stored around zero;
* mixer ``attention``: grouped-query attention behind short convolutions of q, k and v, neighbouring pairs rotated (``rot``, with YaRN
  ``scaling``), then every query and key head divided by its root mean square; a window of ``mask.size`` beside the first
  ``mask.keep_first`` positions; a one in the softmax's denominator;
* mixer ``latent_attention``: keys and values from a normed latent of ``kv_rank`` that is all the cache keeps, beside one rotated key part
  of ``rot_dim`` elements shared by the heads (half-split pairs); queries straight from the input; a window;
* mixer ``parallel``: grouped-query attention with weighted RMS norms of the heads, no rotation and a window (``left``), beside a
  state-space recurrence (``right``); each output is RMS-normed over the model's width and the result is half their sum;
* feed-forward ``moe``: a router with a bias whose ``top`` largest logits choose among ``experts`` units down(max(up h, 0)^2), weighted by
  the softmax over the chosen logits.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .apertus import ConfigError, _require
from .spec import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, YarnRopeScaling

DEFAULT_MAX_POSITIONS = 131072       # config.json gives no limit; tables are sized by the engine's max_context below this


def _need(m: Mapping[str, Any], key: str, where: str):
    if not isinstance(m, Mapping) or key not in m or m[key] is None:
        raise ConfigError(f"config.json: {where} has no \"{key}\"")
    return m[key]


@dataclass(frozen=True)
class MaskConfig:
    size: Optional[int] = None           # keys of the window, the query's own included; None: every earlier position
    keep_first: int = 0                  # positions at the sequence's start that stay visible beside the window

    @classmethod
    def from_dict(cls, m, where, keeps: bool = False):
        if not m:
            return cls()
        size = m.get("size")
        out = cls(None if size is None else int(size), int(m.get("keep_first") or 0))
        if (out.size is not None and out.size < 1) or out.keep_first < 0:
            raise ConfigError(f"{where}: size must be positive and keep_first not negative")
        if out.keep_first and not keeps:
            raise ConfigError(f"{where}.keep_first: only the attention mixer keeps first positions")
        return out

    def to_dict(self):
        d = {} if self.size is None else {"size": self.size}
        return {**d, "keep_first": self.keep_first} if self.keep_first else d


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: Optional[YarnRopeScaling] = None

    @classmethod
    def from_dict(cls, r, where):
        s, scaling = r.get("scaling"), None
        if s:
            w = where + ".scaling"
            scaling = YarnRopeScaling(*(float(_need(s, k, w)) for k in ("factor", "original", "fast", "slow")))
            if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0:
                raise ConfigError(f"{w}: factor, original, fast and slow must be positive")
        out = cls(int(_need(r, "dims", where)), float(_need(r, "base", where)), scaling)
        if out.dims < 2 or out.dims % 2:
            raise ConfigError(f"{where}.dims {out.dims} must be even and at least 2")
        return out

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            s = self.scaling
            d["scaling"] = {"factor": s.factor, "fast": s.fast, "original": s.original, "slow": s.slow}
        return d


@dataclass(frozen=True)
class AttentionConfig:
    """The attention mixer, and the left half of the parallel mixer (no rotation and no convolution there)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    mask: MaskConfig
    rot: Optional[RotationConfig] = None
    conv: int = 0                        # taps of the short convolutions; 0: none

    @classmethod
    def from_dict(cls, m, where, left: bool = False):
        heads, rot = int(_need(m, "heads", where)), None if left else m.get("rot")
        out = cls(heads, int(m.get("kv_heads") or heads), int(_need(m, "dim", where)), int(m.get("vdim") or _need(m, "dim", where)),
                  float(_need(m, "scale", where)), MaskConfig.from_dict(m.get("mask"), where + ".mask", keeps=not left),
                  None if not rot else RotationConfig.from_dict(rot, where + ".rot"), 0 if left else int(m.get("conv") or 0))
        if min(out.heads, out.kv_heads, out.dim, out.vdim) < 1 or out.heads % out.kv_heads or out.conv < 0:
            raise ConfigError(f"{where}: {out.heads} query heads do not divide into {out.kv_heads} key/value heads")
        if out.rot is not None and out.rot.dims > out.dim:
            raise ConfigError(f"{where}.rot.dims {out.rot.dims} exceeds dim {out.dim}")
        return out

    def to_dict(self):
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.mask.to_dict():
            d["mask"] = self.mask.to_dict()
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.conv:
            d["conv"] = self.conv
        return d


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                             # unrotated query/key size of a head
    rot_dim: int                         # rotated query/key size (the key's part is shared by the heads); 0: none
    vdim: int
    kv_rank: int
    scale: float
    mask: MaskConfig
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, m, where):
        rot = m.get("rot")
        out = cls(int(_need(m, "heads", where)), int(_need(m, "dim", where)), int(m.get("rot_dim") or 0), int(m.get("vdim") or _need(m, "dim", where)),
                  int(_need(m, "kv_rank", where)), float(_need(m, "scale", where)), MaskConfig.from_dict(m.get("mask"), where + ".mask"),
                  None if not rot else RotationConfig.from_dict(rot, where + ".rot"))
        if min(out.heads, out.dim, out.vdim, out.kv_rank) < 1 or out.rot_dim < 0:
            raise ConfigError(f"{where}: heads, dim, vdim and kv_rank must be positive")
        if (out.rot_dim > 0) != (out.rot is not None) or (out.rot is not None and out.rot.dims != out.rot_dim):
            raise ConfigError(f"{where}: the rotated part of {out.rot_dim} elements needs a rotation of as many (rot.dims)")
        return out

    def to_dict(self):
        d = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "scale": self.scale, "vdim": self.vdim}
        if self.mask.to_dict():
            d["mask"] = self.mask.to_dict()
        if self.rot_dim:
            d.update({"rot": self.rot.to_dict(), "rot_dim": self.rot_dim})
        return d


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, m, where):
        out = cls(int(_need(m, "heads", where)), int(_need(m, "vdim", where)), int(_need(m, "state", where)), int(m.get("groups") or 1),
                  int(_need(m, "conv", where)), int(m.get("norm_groups") or 1))
        if min(out.heads, out.vdim, out.state, out.groups, out.conv, out.norm_groups) < 1:
            raise ConfigError(f"{where}: heads, vdim, state, groups, conv and norm_groups must be positive")
        if out.heads % out.groups or (out.heads * out.vdim) % out.norm_groups:
            raise ConfigError(f"{where}: {out.heads} heads in {out.groups} groups, {out.heads * out.vdim} channels normed in {out.norm_groups} parts")
        return out

    def to_dict(self):
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: StateSpaceConfig

    @classmethod
    def from_dict(cls, m, where):
        return cls(AttentionConfig.from_dict(_need(m, "left", where), where + ".left", left=True),
                   StateSpaceConfig.from_dict(_need(m, "right", where), where + ".right"))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    top: int

    @classmethod
    def from_dict(cls, m, where):
        kind = _need(m, "kind", where)
        if kind != "moe":
            raise ConfigError(f"{where}.kind \"{kind}\" is not a feed-forward of this design (moe)")
        r = _need(m, "router", where)
        out = cls(int(_need(_need(m, "expert", where), "ff", where + ".expert")), int(_need(r, "experts", where + ".router")),
                  int(_need(r, "top", where + ".router")))
        if out.ff < 1 or not 1 <= out.top <= out.experts:
            raise ConfigError(f"{where}.router: top {out.top} of {out.experts} experts")
        return out

    def to_dict(self):
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}


_MIXERS = {"attention": AttentionConfig, "latent_attention": LatentAttentionConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class PemaraxLayerConfig:
    type: str                            # "attention" | "latent_attention" | "parallel"
    mixer: Any
    mlp: Optional[MoeConfig]


@dataclass(frozen=True)
class PemaraxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[PemaraxLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Pemarax"
    model_type = "pemarax"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, c: Mapping[str, Any]) -> "PemaraxConfig":
        layers = []
        for i, l in enumerate(_require(c, "layers")):
            where = f"layers[{i}]"
            kind = _need(l, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type \"{kind}\" is not a mixer of this design ({', '.join(_MIXERS)})")
            mlp = l.get("mlp")
            layers.append(PemaraxLayerConfig(kind, _MIXERS[kind].from_dict(_need(l, "mixer", where), where + ".mixer"),
                                             None if mlp is None else MoeConfig.from_dict(mlp, where + ".mlp")))
        eos = c.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        mult = c.get("residual_mult")
        out = cls(vocab=int(_require(c, "vocab")), width=int(_require(c, "width")), norm_eps=float(_need(_require(c, "norm"), "eps", "norm")),
                  residual_mult=1.0 if mult is None else float(mult), layers=tuple(layers),
                  max_positions=int(c.get("max_positions") or DEFAULT_MAX_POSITIONS), eos_token_ids=eos)
        if out.vocab < 1 or out.width < 1 or not layers:
            raise ConfigError("vocab and width must be positive and layers not empty")
        return out

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture,
             "layers": [{"mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict(), "type": l.type} for l in self.layers],
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- lowering
    def _position(self, rot: Optional[RotationConfig], head_dim: int, pairing: str) -> PositionSpec:
        if rot is None:
            return PositionSpec(kind="none")
        return PositionSpec(kind="rope", head_dim=head_dim, theta=rot.base, scaling=rot.scaling, max_positions=self.max_positions,
                            options={"rotary_dim": rot.dims, "pairing": pairing, "table_dtype": "float32", "angles": "float64"})

    def _attention_spec(self, m: AttentionConfig, prefix: str, left: bool) -> MixerSpec:
        options = {"value_dim": m.vdim, "conv_taps": m.conv, "bias": False, "gate": False, "row_norm": True, "head_norm": True,
                   "norm_weight": left, "norm_last": not left, "sink": False if left else "zero", "keep_first": m.mask.keep_first}
        return MixerSpec(kind="conv_attention", prefix=prefix, hidden_size=self.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                         qk_norm=True, qk_norm_eps=self.norm_eps, scale=m.scale, window=m.mask.size, position=self._position(m.rot, m.dim, "interleaved"),
                         tensor_names={"q": "q", "k": "k", "v": "v", "o": "o", "conv_suffix": ".conv", "norm_suffix": ".norm"}, options=options)

    def _mixer_spec(self, kind: str, m, prefix: str) -> MixerSpec:
        W, eps = self.width, self.norm_eps
        if kind == "attention":
            return self._attention_spec(m, prefix, left=False)
        if kind == "latent_attention":
            return MixerSpec(kind="latent_attention", prefix=prefix, hidden_size=W, num_heads=m.heads, num_kv_heads=1, head_dim=m.dim, scale=m.scale,
                             window=m.mask.size, position=self._position(m.rot, m.rot_dim, "half"),
                             tensor_names={"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"},
                             options={"value_dim": m.vdim, "q_rank": 0, "kv_rank": m.kv_rank, "latent_norm_eps": eps, "rot_dim": m.rot_dim})
        left, r = self._attention_spec(m.left, prefix + "left.", left=True), m.right
        right = MixerSpec(kind="state_space", prefix=prefix + "right.", hidden_size=W, num_heads=r.heads, head_dim=r.state,
                          tensor_names={"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
                                        "norm": "norm", "o": "o"},
                          options={"value_dim": r.vdim, "groups": r.groups, "conv_taps": r.conv, "norm_groups": r.norm_groups, "norm_eps": eps})
        return MixerSpec(kind="pair", prefix=prefix, hidden_size=W, position=left.position,
                         tensor_names={"left_out": "left.out", "right_out": "right.out"},
                         options={"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5, "out_norm": True, "norm_eps": eps})

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = lambda name: NormSpec("rmsnorm32", W, eps, name, {"init_std": 0.1, "offset": True})
        layers = []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            ffn = n2 = None
            if l.mlp is not None:
                ffn = FeedForwardSpec("routed_experts", p + "mlp.", W, l.mlp.ff,
                                      {"router": "router", "logit_bias": "router.b", "expert": "e{}.", "up": "up", "down": "down"},
                                      {"experts": l.mlp.experts, "top": l.mlp.top, "limit": None, "score": "chosen", "logit_bias": True,
                                       "scale_input": False, "gated": False, "activation": "relu2"})
                n2 = norm(p + "norm2")
            layers.append(LayerSpec("gated", self._mixer_spec(l.type, l.mixer, p + "mix."), norm(p + "norm1"), ffn, n2,
                                    options={"residual_mult": self.residual_mult}))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=W, layers=tuple(layers), order=tuple(range(len(layers))),
            final_norm=norm("final.norm"), embed_name="embed", lm_head_name="head", max_positions=self.max_positions,
            eos_token_ids=self.eos_token_ids, init_std=W ** -0.5, embedding_kind="lookup32", head_kind="linear",
            options={"residual_dtype": "float32", "embed_init_std": 1.0})
