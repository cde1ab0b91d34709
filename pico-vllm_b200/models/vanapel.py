"""The Vanapel decoder put together from parts.

Layer i: grouped RMS norm -> mixer -> grouped RMS norm of its output -> add; then, unless the layer has no feed-forward, the
same around a dense feed-forward of the capped form.  Mixers: softmax attention over a window with unit queries and keys, a
learned logarithmic distance bias, a learned sink and - in layers with ``v_mix`` - values mixed with those of the first such
layer; latent attention with a query latent, a rotated key part shared by the heads (stretched frequencies) and a learned
sink.  Last grouped norm, an untied head.
Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.<q|k|v|r1|r2|sink|vmix|o>`` or ``l<i>.mix.<dq|dq.norm|
uq|dkv|dkv.norm|uk|uv|sink|o>``, ``l<i>.mlp.<gate|up|down>``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.vanapel import VanapelConfig
from ..parts import (DistanceBiasAttention, GatedMLP, GroupedRMSNorm, LatentAttention, OutputHead, SandwichBlock, TokenEmbedding,
                     YarnRotary)
from .decoder import Binding, DecoderModel, LayerCall


def _window_attention(m, D: int, eps: float, p: str, value_mix):
    mixer = DistanceBiasAttention(D, m.heads, m.kv_heads, m.dim, m.vdim, eps, scale=m.scale, whole_qk_norm=False, value_norm=False,
                                  distance_bias=False, sink=None, window=m.window, head_qk_norm=True, log_bias=True,
                                  learned_sink=True, value_mix=value_mix)
    names = {f"{n}.weight": p + n for n in ("q", "k", "v", "o")}
    names.update({n: p + n for n in ("r1", "r2", "sink")})
    if value_mix:
        names["vmix"] = p + "vmix"
    return mixer, names


def _latent_attention(m, D: int, eps: float, p: str):
    s = m.scaling
    stretch = {} if s is None else dict(factor=s.factor, original=s.original, fast=s.fast, slow=s.slow)
    mixer = LatentAttention(D, m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank, m.scale, eps, gate=False, rot_dim=m.rot_dim,
                            position=YarnRotary(m.rot_dim, m.rot_base, m.rot_dims, **stretch), sink=True)
    names = {f"{n}.weight": p + n for n in ("dq", "uq", "dkv", "uk", "uv", "o")}
    names.update({n: p + n for n in ("dq.norm", "dkv.norm", "sink")})
    return mixer, names


def build_vanapel(cfg: VanapelConfig) -> DecoderModel:
    D, eps = cfg.width, cfg.norm_eps

    def norm():
        return GroupedRMSNorm(D, eps, cfg.norm_groups)
    embed = TokenEmbedding(cfg.vocab, D)
    bindings = [Binding(embed, {"weight": "embed"})]
    blocks, order = [], []
    mixing = False                     # a layer before this one has handed its values on
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.type == "attention":
            mixer, names = _window_attention(m, D, eps, p + "mix.", ("mix" if mixing else "first") if m.v_mix else None)
            mixing = mixing or m.v_mix
        else:
            mixer, names = _latent_attention(m, D, eps, p + "mix.")
        norm1, norm1b = norm(), norm()
        bindings += [Binding(norm1, {"weight": p + "norm1"}), Binding(mixer, names), Binding(norm1b, {"weight": p + "norm1b"})]
        norm2 = ff = norm2b = None
        if layer.mlp is not None:
            norm2, norm2b = norm(), norm()
            ff = GatedMLP(D, layer.mlp.ff, "capped", limit=layer.mlp.limit)
            bindings += [Binding(norm2, {"weight": p + "norm2"}),
                         Binding(ff, {f"{n}.weight": f"{p}mlp.{n}" for n in ("gate", "up", "down")}),
                         Binding(norm2b, {"weight": p + "norm2b"})]
        blocks.append(SandwichBlock(norm1, mixer, norm1b, norm2, ff, norm2b))
        order.append(LayerCall(block=i, cache=i))
    final_norm, head = norm(), OutputHead(cfg.vocab, D)
    bindings += [Binding(final_norm, {"weight": "final.norm"}), Binding(head, {"weight": "head"})]
    return DecoderModel(cfg, embed, blocks, order, final_norm, head, bindings)
