"""Configuration of the Zegorax decoder, read from its config.json keys.

config.json names the model in ``architecture`` and describes the stack layer by layer: ``layers[i] = {"type": mixer kind,
"mixer": its sizes and constants, "mlp": its feed-forward or null}``.  Model-wide keys: ``vocab``, ``width``, ``norm.eps`` (of
the norms inside the mixers), ``max_positions`` (rows of the learned position table: no request can be longer), ``loop`` =
``{"start", "stop", "times"}`` (layers start .. stop - 1 run ``times`` times in a row; absent: every layer runs once).  Mixer kinds:

* ``attention`` - ``heads``, ``kv_heads``, ``dim`` (per map), ``vdim``, ``scale``, ``diff``, ``rot``.
* ``latent_attention`` - ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated query/key size per head), ``vdim``, ``q_rank``,
  ``kv_rank``, ``scale``, ``rot``, ``mask.size`` (the window; no mask: all keys).
* ``delta`` - ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps).

``rot`` = ``{"base", "dims", "scaling": {"factor", "low", "high", "original"} or absent}``.
Feed-forward: ``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..errors import ConfigError
from .base import KeyReader

ARCHITECTURE = "Zegorax"
MIXER_KINDS = ("attention", "latent_attention", "delta")


def _object(raw, at: str) -> KeyReader:
    if not isinstance(raw, dict):
        raise ConfigError(f"{at}: must be an object")
    return KeyReader(raw, at)


@dataclass(frozen=True)
class BandScaling:
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    scaling: Optional[BandScaling]

    def to_dict(self) -> Dict[str, Any]:
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: RotarySpec

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "diff": self.diff, "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class WindowLatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    window: Optional[int]

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
             "kv_rank": self.kv_rank, "scale": self.scale, "rot": self.rot.to_dict()}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class HeadDecayDeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class FeedForwardSpec:
    kind: str                        # "dense" or "moe"
    ff: int
    experts: int = 0
    top: int = 0

    def to_dict(self) -> Dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: Optional[FeedForwardSpec]

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int

    def to_dict(self) -> Dict[str, Any]:
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class ZegoraxConfig:
    vocab: int
    width: int
    norm_eps: float
    max_positions: int
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec] = None
    torch_dtype: str = "bfloat16"
    bos_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None

    architecture = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    def layer_runs(self) -> List[int]:
        """The layers in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b = self.loop.start, self.loop.stop
        return list(range(a)) + list(range(a, b)) * self.loop.times + list(range(b, n))

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], where: str = "config.json") -> "ZegoraxConfig":
        r = KeyReader(raw, where)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        eps = _object(r.any("norm"), f"{where}: norm").number("eps", positive=True)
        layers_raw = r.any("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: key 'layers' must be a non-empty list")
        readers = {"attention": _read_differential, "latent_attention": _read_latent, "delta": _read_delta}
        layers = []
        for i, item in enumerate(layers_raw):
            at = f"{where}: layers[{i}]"
            lr = _object(item, at)
            kind = lr.string("type")
            if kind not in readers:
                raise ConfigError(f"{at}: 'type' {kind!r} is not a mixer of {ARCHITECTURE} (have {list(MIXER_KINDS)})")
            layers.append(LayerSpec(kind, readers[kind](lr.any("mixer"), f"{at}.mixer"), _read_ff(lr.any("mlp"), f"{at}.mlp")))
        loop = None
        if r.any("loop") is not None:
            lp = _object(r.any("loop"), f"{where}: loop")
            loop = LoopSpec(lp.integer("start", minimum=0), lp.integer("stop", minimum=0), lp.integer("times", minimum=1))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"{where}: loop: 'start' {loop.start} and 'stop' {loop.stop} must name a run of the {len(layers)} layers")
        dtype = r.string("torch_dtype", default=None) or r.string("dtype", default="bfloat16")
        return cls(vocab=vocab, width=width, norm_eps=eps, max_positions=r.integer("max_positions", minimum=1), layers=tuple(layers),
                   loop=loop, torch_dtype=dtype, bos_token_id=r.integer("bos_token_id", default=None),
                   eos_token_id=r.integer("eos_token_id", default=None))

    def to_dict(self) -> Dict[str, Any]:
        """config.json content that :meth:`from_dict` reads back to an equal object."""
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "max_positions": self.max_positions, "layers": [l.to_dict() for l in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        for k in ("bos_token_id", "eos_token_id"):
            if getattr(self, k) is not None:
                d[k] = getattr(self, k)
        return d


def _read_rot(raw, at: str, limit: int, of: str) -> RotarySpec:
    rot = _object(raw, at)
    dims = rot.integer("dims", minimum=0)
    if dims % 2 or dims > limit:
        raise ConfigError(f"{at}: 'dims' {dims} must be even and at most '{of}' {limit}")
    scaling = None
    if rot.any("scaling") is not None:
        s = _object(rot.any("scaling"), f"{at}.scaling")
        scaling = BandScaling(*(s.number(k, positive=True) for k in ("factor", "low", "high", "original")))
        if scaling.high < scaling.low:
            raise ConfigError(f"{at}.scaling: 'high' {scaling.high} must not be below 'low' {scaling.low}")
    return RotarySpec(rot.number("base", positive=True), dims, scaling)


def _grouped(m: KeyReader, at: str) -> Tuple[int, int]:
    heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{at}: 'heads' {heads} must be a multiple of 'kv_heads' {kv_heads}")
    return heads, kv_heads


def _read_differential(raw, at: str) -> DifferentialSpec:
    m = _object(raw, at)
    heads, kv_heads = _grouped(m, at)
    dim = m.integer("dim", minimum=1)
    return DifferentialSpec(heads, kv_heads, dim, m.integer("vdim", minimum=1), m.number("scale"), m.number("diff"),
                            _read_rot(m.any("rot"), f"{at}.rot", dim, "dim"))


def _read_latent(raw, at: str) -> WindowLatentSpec:
    m = _object(raw, at)
    rot_dim = m.integer("rot_dim", minimum=1)
    window = None
    if m.any("mask") is not None:
        window = _object(m.any("mask"), f"{at}.mask").integer("size", minimum=1)
    return WindowLatentSpec(m.integer("heads", minimum=1), m.integer("dim", minimum=1), rot_dim, m.integer("vdim", minimum=1),
                            m.integer("q_rank", minimum=1), m.integer("kv_rank", minimum=1), m.number("scale"),
                            _read_rot(m.any("rot"), f"{at}.rot", rot_dim, "rot_dim"), window)


def _read_delta(raw, at: str) -> HeadDecayDeltaSpec:
    m = _object(raw, at)
    return HeadDecayDeltaSpec(*_grouped(m, at), m.integer("dim", minimum=1), m.integer("vdim", minimum=1),
                              m.integer("conv", default=1, minimum=1))


def _read_ff(raw, at: str) -> Optional[FeedForwardSpec]:
    if raw is None:
        return None
    f = _object(raw, at)
    kind = f.string("kind")
    if kind == "dense":
        return FeedForwardSpec("dense", f.integer("ff", minimum=1))
    if kind != "moe":
        raise ConfigError(f"{at}: 'kind' {kind!r} is not a feed-forward of {ARCHITECTURE} (have ['dense', 'moe'])")
    router = _object(f.any("router"), f"{at}.router")
    experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
    if top > experts:
        raise ConfigError(f"{at}.router: 'top' {top} exceeds the {experts} experts")
    return FeedForwardSpec("moe", _object(f.any("expert"), f"{at}.expert").integer("ff", minimum=1), experts, top)
