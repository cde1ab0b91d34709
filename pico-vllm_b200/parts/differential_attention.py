"""Differential attention: every head runs two softmax attentions ("maps") over the same values and takes one off the other.

With mixer input h (width D), H query heads, G key/value heads (query head a reads key/value head a // (H / G)), query/key size d
per map, value size d_v:

    q = W_q h  (H x 2 x d),  k = W_k h  (G x 2 x d),  v = W_v h  (G x d_v)         each head's maps lie side by side
    q, k: rotated by the position encoding, the first ``rot_dim`` numbers of each map
    A_m(i) = sum_(j <= i) softmax_j( scale * q_m(i) . k_m(j) ) v(j)                m = 1, 2
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff                                one number for the layer
    o = A_1 - lambda A_2;   o <- o / sqrt(mean(o^2) + eps) * (1 - diff)            per head
    out = W_o concat_heads( o * sigmoid(W_g h)_head )                               (``gate``)

(Ye, Dong, Xia, Sun, Zhu, Huang, Wei: "Differential Transformer", with a gate per head beside it.)

The cache holds one key row [k_1 | k_2] and one value row per token and key/value head.  The paged attention kernels see 2 H query
heads over G key/value heads: the query row of map m is zero but for q_m in the place of k_m, so its product with the key
row is q_m . k_m, and keys and values are read once for both maps and all heads of the group.  The maps' outputs come back side
by side and one kernel takes their difference, its norm and the gate.

Launches: one product for q, k, v and the gate logits -> rotation, spreading of the queries and cache store (one kernel) -> paged
attention -> difference, norm and gate (one kernel) -> output product.  Angles, scores, softmax, difference and norm are float32.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..errors import ConfigError
from .attention import AttentionPlan, _linear, decode_splits
from .base import CacheView, PagedKV, Param, Part, Piece, StepShape
from .registry import register

MAPS = 2


@register("mixer", "differential_attention")
class DifferentialAttention(Part):
    def __init__(self, width: int, n_heads: int, n_kv_heads: int, dim: int, vdim: int, eps: float, scale: float, diff: float,
                 position: Part, gate: bool = True):
        if n_heads % n_kv_heads:
            raise ConfigError("differential_attention: heads must be a multiple of kv_heads")
        if getattr(position, "pairing", "rot_half") != "rot_half" or position.rot_dim > dim:
            raise ConfigError("differential_attention: the position encoding must pair dimension i with i + rot_dim / 2 within a map")
        self.width, self.n_heads, self.n_kv_heads, self.dim, self.vdim = width, n_heads, n_kv_heads, dim, vdim
        self.row = -(-max(MAPS * dim, vdim) // 16) * 16          # a head in the cache and the kernels: padded with zeros
        self.eps, self.scale, self.diff, self.position, self.has_gate = float(eps), float(scale), float(diff), position, gate
        self.proj_weight = self.lambdas = self.o_weight = self.lam = None

    def params(self) -> List[Param]:
        H, G, D = self.n_heads, self.n_kv_heads, self.width
        proj = [Piece("q.weight", (H * MAPS * self.dim, D)), Piece("k.weight", (G * MAPS * self.dim, D)),
                Piece("v.weight", (G * self.vdim, D))]
        if self.has_gate:
            proj.append(Piece("g.weight", (H, D)))
        return [Param("proj_weight", tuple(proj)),
                Param("lambdas", tuple(Piece(n, (self.dim,)) for n in ("lq1", "lk1", "lq2", "lk2")), kind="vector"),
                Param("o_weight", (Piece("o.weight", (D, H * self.vdim)),))]

    def assign(self, attr: str, tensor: torch.Tensor) -> None:
        if attr == "proj_weight" and tensor.shape[0] % 16:       # the weight-streaming product wants whole tiles of 16 rows
            tensor = torch.cat([tensor, tensor.new_zeros((16 - tensor.shape[0] % 16, tensor.shape[1]))], 0).contiguous()
        elif attr == "lambdas":                                  # weights alone decide it: worked out once
            q1, k1, q2, k2 = tensor.detach().to("cpu", torch.float32).view(4, self.dim)
            self.lam = float(torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum()) + self.diff)
        setattr(self, attr, tensor)

    def materialize(self, device, dtype):
        self.position.materialize(device, dtype)

    def cache_spec(self):
        return PagedKV(self.n_kv_heads, self.row)

    def plan_key(self):
        return ("differential_attention", self.n_heads, self.n_kv_heads, self.row)

    def plan(self, shape: StepShape) -> AttentionPlan:
        splits = decode_splits(shape, self.n_kv_heads)
        scratch = ops.attention_scratch_floats(shape.num_tokens, MAPS * self.n_heads, self.row, splits)
        return AttentionPlan(key=(splits, 0), scratch_floats=scratch, splits=splits, pair_min_keys=0)

    def forward(self, h: torch.Tensor, batch, cache: CacheView) -> torch.Tensor:
        gb = batch.groups[cache.group]
        H, G, d, dv, row = self.n_heads, self.n_kv_heads, self.dim, self.vdim, self.row
        k_off, v_off = H * MAPS * d, (H + G) * MAPS * d
        g_off = v_off + G * dv
        proj = _linear(h, self.proj_weight)                      # [T, q | k | v | gate logits]
        q = ops.map_rope_store(proj, 0, k_off, v_off, batch.positions, self.position.inv_freq, getattr(self.position, "mult", 1.0),
                               gb.slots if cache.store else None, cache.k, cache.v, H, G, MAPS, d, dv, row, cache.page_size)
        heads = MAPS * H
        out = torch.empty((h.shape[0], heads * row), dtype=h.dtype, device=h.device)
        plan = batch.plan(self)
        splits = plan.splits if plan is not None else 1
        if ops.mma_attention_takes(h.dtype, heads, G, row):
            ops.paged_attention_mma(q, cache.k, cache.v, out, batch.tok_seg, batch.positions, gb.block_table, batch.cu_q,
                                    batch.prefill_segs, batch.num_prefill_segs, batch.max_prefill_q, batch.decode_tokens,
                                    batch.num_decode_tokens, heads, G, row, cache.page_size, None, self.scale, splits,
                                    batch.scratch, cache.k_map, cache.v_map, cache.k_map2d, cache.v_map2d, 0)
        else:       # float32, or sizes the tensor-core kernels do not take
            ops.paged_attention(q, cache.k, cache.v, out, batch.tok_seg, batch.positions, gb.block_table, heads, G, row,
                                cache.page_size, None, self.scale, splits, batch.scratch)
        y = ops.map_difference(out, H, row, dv, self.lam, self.eps, 1.0 - self.diff,
                               proj[:, g_off:g_off + H] if self.has_gate else None)
        return _linear(y, self.o_weight)
