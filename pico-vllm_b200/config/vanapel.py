"""Configuration of the Vanapel decoder, read from its config.json keys.

config.json names the model in ``architecture`` and describes the stack layer by layer: ``layers[i] = {"type": mixer kind,
"mixer": its sizes and constants, "mlp": its feed-forward or null}``.  Model-wide keys: ``vocab``, ``width``, ``norm.eps``,
``norm.groups`` (equal runs of the vector that are normed separately; 1 when absent).  Mixer kinds:

* ``attention`` - ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the window; no mask: all keys),
  ``v_mix`` (the values are mixed with those of the first layer that has it; false when absent).
* ``latent_attention`` - ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated query/key size per head), ``vdim``,
  ``q_rank``, ``kv_rank``, ``scale``, ``rot`` = ``{"base", "dims", "scaling": {"factor", "original", "fast", "slow"} or absent}``.

Feed-forward: ``{"kind": "dense", "ff", "limit"}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..errors import ConfigError
from .base import KeyReader

ARCHITECTURE = "Vanapel"
MIXER_KINDS = ("attention", "latent_attention")


def _object(raw, at: str) -> KeyReader:
    if not isinstance(raw, dict):
        raise ConfigError(f"{at}: must be an object")
    return KeyReader(raw, at)


@dataclass(frozen=True)
class WindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    v_mix: bool

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "v_mix": self.v_mix}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class FrequencyScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class RotaryLatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    scaling: Optional[FrequencyScaling]

    def to_dict(self) -> Dict[str, Any]:
        rot = {"base": self.rot_base, "dims": self.rot_dims}
        if self.scaling is not None:
            rot["scaling"] = self.scaling.to_dict()
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": rot}


@dataclass(frozen=True)
class FeedForwardSpec:
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: Optional[FeedForwardSpec]

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class VanapelConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    layers: Tuple[LayerSpec, ...]
    torch_dtype: str = "bfloat16"
    bos_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None
    max_position_embeddings: int = 1 << 20      # nothing in the design bounds a request's length

    architecture = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], where: str = "config.json") -> "VanapelConfig":
        r = KeyReader(raw, where)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        norm = _object(r.any("norm"), f"{where}: norm")
        eps, groups = norm.number("eps", positive=True), norm.integer("groups", default=1, minimum=1)
        if width % groups:
            raise ConfigError(f"{where}: norm: 'groups' {groups} does not divide 'width' {width} evenly")
        layers_raw = r.any("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: key 'layers' must be a non-empty list")
        layers, shared = [], None
        for i, item in enumerate(layers_raw):
            at = f"{where}: layers[{i}]"
            lr = _object(item, at)
            kind = lr.string("type")
            if kind == "attention":
                mixer = _read_attention(lr.any("mixer"), f"{at}.mixer")
                if mixer.v_mix:
                    if shared is not None and (mixer.kv_heads, mixer.vdim) != shared[:2]:
                        raise ConfigError(f"{at}.mixer: 'v_mix' needs the 'kv_heads' and 'vdim' of layer {shared[2]}, whose values are mixed in")
                    shared = shared or (mixer.kv_heads, mixer.vdim, i)
            elif kind == "latent_attention":
                mixer = _read_latent(lr.any("mixer"), f"{at}.mixer")
            else:
                raise ConfigError(f"{at}: 'type' {kind!r} is not a mixer of {ARCHITECTURE} (have {list(MIXER_KINDS)})")
            layers.append(LayerSpec(kind, mixer, _read_ff(lr.any("mlp"), f"{at}.mlp")))
        dtype = r.string("torch_dtype", default=None) or r.string("dtype", default="bfloat16")
        return cls(vocab=vocab, width=width, norm_eps=eps, norm_groups=groups, layers=tuple(layers), torch_dtype=dtype,
                   bos_token_id=r.integer("bos_token_id", default=None), eos_token_id=r.integer("eos_token_id", default=None))

    def to_dict(self) -> Dict[str, Any]:
        """config.json content that :meth:`from_dict` reads back to an equal object."""
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "layers": [l.to_dict() for l in self.layers]}
        for k in ("bos_token_id", "eos_token_id"):
            if getattr(self, k) is not None:
                d[k] = getattr(self, k)
        return d


def _read_attention(raw, at: str) -> WindowAttentionSpec:
    m = _object(raw, at)
    heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{at}: 'heads' {heads} must be a multiple of 'kv_heads' {kv_heads}")
    window = None
    if m.any("mask") is not None:
        window = _object(m.any("mask"), f"{at}.mask").integer("size", minimum=1)
    return WindowAttentionSpec(heads, kv_heads, m.integer("dim", minimum=1), m.integer("vdim", minimum=1), m.number("scale"), window,
                               bool(m.boolean("v_mix", default=False)))


def _read_latent(raw, at: str) -> RotaryLatentSpec:
    m = _object(raw, at)
    rot_dim = m.integer("rot_dim", minimum=2)
    rot = _object(m.any("rot"), f"{at}.rot")
    dims = rot.integer("dims", minimum=2)
    if dims % 2 or dims > rot_dim:
        raise ConfigError(f"{at}.rot: 'dims' {dims} must be even and at most 'rot_dim' {rot_dim}")
    scaling = None
    if rot.any("scaling") is not None:
        s = _object(rot.any("scaling"), f"{at}.rot.scaling")
        scaling = FrequencyScaling(*(s.number(k, positive=True) for k in ("factor", "original", "fast", "slow")))
    return RotaryLatentSpec(m.integer("heads", minimum=1), m.integer("dim", minimum=1), rot_dim, m.integer("vdim", minimum=1),
                            m.integer("q_rank", minimum=1), m.integer("kv_rank", minimum=1), m.number("scale"),
                            rot.number("base", positive=True), dims, scaling)


def _read_ff(raw, at: str) -> Optional[FeedForwardSpec]:
    if raw is None:
        return None
    f = _object(raw, at)
    kind = f.string("kind")
    if kind != "dense":
        raise ConfigError(f"{at}: 'kind' {kind!r} is not a feed-forward of {ARCHITECTURE} (have ['dense'])")
    return FeedForwardSpec(f.integer("ff", minimum=1), f.number("limit", positive=True))
