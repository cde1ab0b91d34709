"""The Zegorax decoder put together from parts.

Embedding plus a learned vector per position; layers with ONE squashing norm each, h = norm1(x), x += mixer(h) + feed_forward(h);
a run of layers may be gone through several times in a row with the same weights, each pass with cache entries of its own.
Mixers: differential attention with rotation and a gate per head, latent attention over a window with a rotated key part and
a gate on every number, the gated delta rule with a decay per head.  Feed-forward: dense with biases and the tanh form of gelu,
routed experts (softmax over the chosen), or none.  Last norm; the head is the embedding table.
Tensor names: ``embed``, ``pos``, ``<norm>``, ``<norm>.b`` and ``<norm>.alpha`` for ``<norm>`` = ``l<i>.norm1`` and ``final.norm``,
``l<i>.mix.<q|k|v|g|o|lq1|lk1|lq2|lk2>`` or ``l<i>.mix.<dq|dq.norm|uq|dkv|dkv.norm|uk|uv|g|o>`` or ``l<i>.mix.<q|k|v|q.conv|k.conv|
v.conv|b|a|A_log|dt_bias|norm|g|o>``, ``l<i>.mlp.<gate|up|down>`` with ``.b`` or ``l<i>.mlp.<router|router.b|e<k>.gate|e<k>.up|
e<k>.down>``.
"""
from __future__ import annotations

from ..config.zegorax import ZegoraxConfig
from ..parts import (BandScaledRotary, DifferentialAttention, GatedDeltaRule, GatedMLP, LatentAttention, LearnedPositions, OutputHead,
                     ParallelBlock, RoutedExperts, TanhNorm, TokenEmbedding)
from .decoder import Binding, DecoderModel, LayerCall


def _rotary(rot, dim: int, pairing: str) -> BandScaledRotary:
    s = rot.scaling
    bands = {} if s is None else dict(factor=s.factor, low=s.low, high=s.high, original=s.original)
    return BandScaledRotary(dim, rot.base, rot.dims, pairing=pairing, **bands)


def _mixer(kind: str, m, D: int, eps: float, p: str):
    if kind == "attention":
        mixer = DifferentialAttention(D, m.heads, m.kv_heads, m.dim, m.vdim, eps, m.scale, m.diff, _rotary(m.rot, m.dim, "rot_half"))
        names = {f"{n}.weight": p + n for n in ("q", "k", "v", "g", "o")}
        names.update({n: p + n for n in ("lq1", "lk1", "lq2", "lk2")})
    elif kind == "latent_attention":
        mixer = LatentAttention(D, m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank, m.scale, eps, window=m.window, gate="elements",
                                rot_dim=m.rot_dim, position=_rotary(m.rot, m.rot_dim, "neighbours"))
        names = {f"{n}.weight": p + n for n in ("dq", "uq", "dkv", "uk", "uv", "g", "o")}
        names.update({n: p + n for n in ("dq.norm", "dkv.norm")})
    else:
        mixer = GatedDeltaRule(D, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, head_decay=True, full_gate=True, gate_act="silu")
        names = {f"{n}.weight": p + n for n in ("q", "k", "v", "g", "b", "a", "o")}
        names.update({n: p + n for n in ("q.conv", "k.conv", "v.conv", "A_log", "dt_bias", "norm")})
    return mixer, names


def _feed_forward(f, D: int, p: str):
    if f.kind == "dense":
        names = {f"{n}.weight": p + n for n in ("gate", "up", "down")}
        names.update({f"{n}.bias": f"{p}{n}.b" for n in ("gate", "up", "down")})
        return GatedMLP(D, f.ff, "gelu_tanh", bias=True), names
    names = {"router.weight": p + "router", "router.bias": p + "router.b"}
    for e in range(f.experts):
        names.update({f"e{e}.{n}.weight": f"{p}e{e}.{n}" for n in ("gate", "up", "down")})
    return RoutedExperts(D, f.ff, f.experts, f.top), names


def _norm(D: int, name: str):
    norm = TanhNorm(D)
    return norm, Binding(norm, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})


def build_zegorax(cfg: ZegoraxConfig) -> DecoderModel:
    D, eps = cfg.width, cfg.norm_eps
    embed, position = TokenEmbedding(cfg.vocab, D), LearnedPositions(cfg.max_positions, D)
    bindings = [Binding(embed, {"weight": "embed"}), Binding(position, {"weight": "pos"})]
    blocks = []
    for i, layer in enumerate(cfg.layers):
        norm1, norm_binding = _norm(D, f"l{i}.norm1")
        mixer, names = _mixer(layer.type, layer.mixer, D, eps, f"l{i}.mix.")
        bindings += [norm_binding, Binding(mixer, names)]
        ff = None
        if layer.mlp is not None:
            ff, ff_names = _feed_forward(layer.mlp, D, f"l{i}.mlp.")
            bindings.append(Binding(ff, ff_names))
        blocks.append(ParallelBlock(norm1, mixer, ff))
    order, entries = [], 0
    for i in cfg.layer_runs():                     # every run of a layer has cache entries of its own
        spec = blocks[i].mixer.cache_spec()
        n = len(spec) if isinstance(spec, tuple) else 1
        ids = tuple(range(entries, entries + n))
        entries += n
        order.append(LayerCall(block=i, cache=ids if isinstance(spec, tuple) else ids[0]))
    final_norm, norm_binding = _norm(D, "final.norm")
    bindings.append(norm_binding)
    return DecoderModel(cfg, embed, blocks, order, final_norm, OutputHead(cfg.vocab, D, tied_to=embed), bindings, embed_position=position)
