"""The Zegorax design in the engine against the plain implementation of tests/plain_zegorax.py: the new kernels against torch
arithmetic, each mechanism alone (models of one layer), whole models of several small shapes in every cutting of requests into
steps, batches against each request alone, keys just inside and just outside a window and far back, a memory that must survive
from step to step, looped layers, long decoding through pages and slots that are used again, and greedy generation through
the entry points.

Routers: the float32 runs route by the data.  In bfloat16 the router's input differs from the float64 oracle's by the rounding of
the layers before it, enough to send some tokens to other experts than the oracle does; so the bfloat16 runs of whole models
choose all experts of a layer (the weights still differ from token to token)."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fake_ops
import helpers
import plain_zegorax as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
REL = {"float32": 5e-5, "bfloat16": 6e-2}      # max |difference| / max |logit| over a step; float32 is the sharp test
STD = 0.12


def _rot(base, dims, scaling=None):
    rot = dict(base=base, dims=dims)
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def _att(heads, kv_heads, dim, vdim, scale, diff, rot):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, rot=rot))


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window=None, base=10000.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=_rot(base, rot_dim))
    if window:
        m["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=m)


def _delta(heads, kv_heads, dim, vdim, conv):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv))


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def _layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def _model(vocab, width, layers, loop=None, eps=1e-5, positions=640):
    d = dict(architecture="Zegorax", vocab=vocab, width=width, norm=dict(eps=eps), max_positions=positions, layers=layers)
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


SHAPES = {
    # key and value sizes differ everywhere; a rotation of half of every map with all three bands of scaled frequencies; a window
    # of 24, no multiple of a page, over rows of 40 + 8; query/key heads shared by two heads of the delta rule; a loop over three
    # kinds of layer, twice, in the middle; layers without feed-forward
    "a": _model(211, 96, [_layer(_delta(4, 2, 16, 24, 3), _dense(64)),
                          _layer(_att(4, 2, 24, 40, 0.3, 0.4, _rot(500.0, 12, (4.0, 1.0, 4.0, 96))), _moe(24, 6, 2)),
                          _layer(_lat(3, 16, 8, 24, 20, 40, 0.3, 24, 300.0)),
                          _layer(_delta(2, 2, 40, 16, 2), _moe(40, 5, 3)),
                          _layer(_att(3, 1, 20, 12, 0.4, 0.2, _rot(100.0, 20)), _dense(40))], loop=(1, 4, 2)),
    # rows of 64 and 128, which the TMA and tcgen05 kernels take (two maps of 32 and of 64; a latent of 96 + 32); a loop from the
    # first layer on, to the last; one tap; a window of a page and one over three quarters of a tile
    "b": _model(304, 128, [_layer(_att(4, 1, 32, 64, 0.2, 0.8, _rot(10000.0, 16, (8.0, 1.0, 2.0, 64))), _dense(96)),
                           _layer(_lat(4, 64, 32, 64, 64, 96, 0.12, 16), _moe(64, 8, 4)),
                           _layer(_att(8, 4, 64, 128, 0.12, 0.5, _rot(1000.0, 64)), None),
                           _layer(_delta(3, 1, 64, 32, 1), _dense(48)),
                           _layer(_lat(2, 32, 16, 16, 32, 48, 0.2, 48), _moe(32, 4, 1))], loop=(0, 5, 2), eps=1e-6),
    # awkward sizes: a width that is a multiple of 2 only, an odd vocabulary, maps of 10 and 18, a rotation of two numbers, inner sizes
    # that are no multiples of 8, a window of 7, five taps; no loop
    "c": _model(203, 102, [_layer(_att(6, 2, 10, 12, 0.5, 0.6, _rot(50.0, 2)), _moe(28, 9, 3)),
                           _layer(_delta(6, 3, 20, 12, 5), _dense(52)),
                           _layer(_lat(5, 20, 6, 12, 22, 36, 0.3, 7, 50.0), _moe(12, 2, 2)),
                           _layer(_att(5, 1, 18, 50, 0.3, 0.1, _rot(200.0, 18, (2.0, 0.5, 8.0, 40))))], eps=1e-4),
    # more than sixteen map rows on one key/value head, rows beyond 256, a layer three times, latent attention without a window
    "d": _model(150, 160, [_layer(_att(9, 1, 32, 16, 0.25, 0.5, _rot(1000.0, 8)), _dense(72)),
                           _layer(_lat(18, 24, 64, 16, 48, 208, 0.15), _moe(72, 3, 2)),
                           _layer(_att(2, 1, 136, 80, 0.1, 0.9, _rot(10000.0, 32, (1.0, 1.0, 1.0, 50))))], loop=(1, 2, 3)),
}
SEEDS = {"a": 11, "b": 22, "c": 33, "d": 44}
LENGTHS = {"a": [1, 9, 33, 70, 150, 230], "b": [2, 17, 48, 97, 200], "c": [3, 40, 129, 75], "d": [5, 31, 90]}


def _raw(name, dtype):
    """The shape as tested in ``dtype``: in bfloat16 every routed layer chooses all of its experts."""
    raw = copy.deepcopy(SHAPES[name] if isinstance(name, str) else name)
    if dtype == "bfloat16":
        for layer in raw["layers"]:
            if layer["mlp"] and layer["mlp"]["kind"] == "moe":
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


def _tensors(raw, seed, std=STD):
    from pico_vllm_b200.registry import config_from_dict
    from pico_vllm_b200.weights import random_tensors
    t = random_tensors(config_from_dict(raw), seed, std=std, dtype=torch.bfloat16)
    for n in t:
        x = t[n].float()
        if n.endswith(".alpha"):
            x = 0.5 + 4.0 * (x - 0.5)                       # from nearly linear to well into the bend
        elif n in ("embed", "pos"):
            x = x * 4.0
        elif n.endswith("norm1.b") or n == "final.norm.b":
            x = x * 2.0
        elif n.endswith(".norm1") or n.endswith(".norm"):
            x = 1.0 + 4.0 * (x - 1.0)                       # weights around one, some well away from it
        elif n.rsplit(".", 1)[-1] in ("lq1", "lk1", "lq2", "lk2"):
            x = x * 2.5
        elif n.endswith(".A_log"):
            x = x * 10.0 - 2.0                              # decays from fast to slow
        elif n.endswith(".conv"):
            x = x * 1.5
        elif n.endswith(".b") and n.count(".") == 3:        # biases of the feed-forward and the router
            x = x * 3.0
        t[n] = x.to(torch.bfloat16)
    return t


def _runner(raw, tensors, dtype, max_tokens, graph=False, page_size=16, max_num_seqs=4):
    from pico_vllm_b200.config import EngineConfig
    from pico_vllm_b200.engine import ModelRunner, make_cache, model_from_tensors
    from pico_vllm_b200.registry import config_from_dict
    ecfg = EngineConfig(dtype=dtype, page_size=page_size, max_cache_tokens=max_tokens, max_num_seqs=max_num_seqs,
                        use_cuda_graph=graph, device=DEV)
    model = model_from_tensors(config_from_dict(raw), tensors, ecfg)
    return ModelRunner(model, make_cache(model, ecfg, poison_freed=True), ecfg)


def _oracle(raw, tensors, reqs):
    return {rid: plain.forward(raw, tensors, ids) for rid, ids in reqs.items()}


def _compare(steps, reqs, got, logits, dtype, what):
    """float32, the sharp test: every step within REL of the plain implementation.  bfloat16: every wanted row's largest
    difference is measured against the largest logit of its step; all rows but a few (2% of the trace's, or one) stay within
    REL, and none is beyond three times that."""
    want = helpers.expected_logits(steps, reqs, logits)
    errs = []
    for i, (g, w) in enumerate(zip(got, want)):
        assert (g is None) == (w is None), f"{what} step {i}"
        if w is None:
            continue
        assert g.shape == w.shape and torch.isfinite(g).all(), f"{what} step {i}: shape or a value that is not finite"
        if dtype == "float32":
            helpers.assert_close_logits(g, w.float(), REL[dtype], f"{what} step {i}")
        else:
            errs += [(float(e), i) for e in (g.double() - w.double()).abs().amax(1) / float(w.abs().max())]
    if errs:
        over = [(e, i) for e, i in errs if e > REL[dtype]]
        assert len(over) <= max(1, len(errs) * 2 // 100), f"{what}: {len(over)} of {len(errs)} rows over {REL[dtype]}: {over[:8]}"
        assert max(errs)[0] <= 3 * REL[dtype], f"{what}: a row is off by {max(errs)}"


def _shows(diff, scale, dtype):
    """Whether a difference between two oracles is large enough that the comparison in ``dtype`` would catch it."""
    return diff > max(20 * REL["float32"], 3.5 * REL[dtype] if dtype == "bfloat16" else 0.0) * scale


def _status():
    from pico_vllm_b200 import ops
    ops.check_kernel_status()


def _close(got, want, tol, what):
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, what
    err = float((got - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), f"{what}: off by {err}"


# ------------------------------------------------------------------------------------------------ the kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,T", [(96, 9), (102, 9), (8, 1), (7, 3), (2048, 9), (4100, 5), (1536, 400)])
def test_squashing_norm_with_the_adds_before_it(dtype, H, T):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(H)
    x = torch.randn(T, H, generator=g) * 2
    ds = [torch.randn(T, H, generator=g).to(dtype) for _ in range(3)]
    w, b, alpha = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.tensor(0.8)
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
    for terms in ([], [(ds[0], 1.0)], [(ds[0], 1.0), (ds[1], 0.5)], [(ds[2], -1.5), (ds[1], 1.0), (ds[0], 2.0)]):
        for r, with_out in ((None, True), (rows, True), (None, False)):
            if not terms and not with_out:
                continue
            xw, xg = x.clone(), x.to(DEV)
            n = T if r is None else 3
            ow, og = torch.zeros(n, H).to(dtype), torch.zeros(n, H).to(dtype).to(DEV)
            fake_ops.tanh_norm(xw, terms, alpha, w, b, ow if with_out else None, r)
            ops.tanh_norm(xg, [(d.to(DEV), s) for d, s in terms], alpha.to(DEV), w.to(DEV), b.to(DEV), og if with_out else None,
                          None if r is None else r.to(DEV))
            _close(xg, xw, 1e-6, "stream")
            _close(og, ow, 2e-6 if dtype == torch.float32 else 1e-2, "squashed")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,M,d,dv,rot,shift", [(4, 2, 2, 32, 48, 16, 0), (8, 1, 2, 64, 128, 64, 0), (3, 1, 2, 20, 12, 20, 1), (2, 2, 2, 16, 64, 0, 0),
                                                  (5, 1, 2, 24, 96, 8, 0), (6, 3, 1, 40, 30, 10, 0), (2, 1, 3, 16, 16, 4, 0), (1, 1, 2, 160, 8, 32, 0),
                                                  (12, 2, 2, 32, 64, 24, 0)])
def test_maps_rotated_spread_and_stored(dtype, H, G, M, d, dv, rot, shift):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(d + H)
    T, ps, row = 11, 4, -(-max(M * d, dv) // 16) * 16
    x = torch.randn(T, shift + (H + G) * M * d + G * dv + 16 + 3 * shift, generator=g).to(dtype)
    pos = torch.tensor([0, 1, 2, 300, 1117, -1, 7, 8, 9, 10, 11], dtype=torch.int32)
    slots = torch.tensor([0, 5, 6, 7, 9, -1, 13, -1, 20, 2, 31], dtype=torch.int32)
    inv = (37.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float()
    offs = (shift, shift + H * M * d, shift + (H + G) * M * d)
    fill = lambda: torch.full((8, G, ps, row), float("nan")).to(dtype)
    dev = lambda t: t.to(DEV)
    tol = 3e-4 if dtype == torch.float32 else 1e-2       # float32: the angle of position 1117 is rounded before sin and cos
    for sl in (slots, None):
        kp, vp, kg, vg = fill(), fill(), fill().to(DEV), fill().to(DEV)
        want = fake_ops.map_rope_store(x, *offs, pos, inv, 1.3, sl, kp, vp, H, G, M, d, dv, row, ps)
        got = ops.map_rope_store(dev(x), *offs, dev(pos), dev(inv), 1.3, None if sl is None else dev(sl), kg, vg, H, G, M, d, dv, row, ps)
        _close(got, want, tol, "queries")
        assert torch.equal(got.cpu() == 0, want == 0)     # zeros beside a map stay zeros
        for a, b, what in ((kg, kp, "keys"), (vg, vp, "values")):
            assert torch.equal(torch.isnan(a.float().cpu()), torch.isnan(b.float()))      # nothing stored where nothing belongs
            _close(torch.nan_to_num(a.float()), torch.nan_to_num(b.float()), tol, what)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,row,dv", [(4, 64, 64), (3, 48, 40), (6, 128, 96), (5, 32, 12), (2, 272, 80), (1, 256, 256), (9, 32, 16), (2, 320, 300)])
def test_difference_of_maps(dtype, H, row, dv):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(row + dv)
    T = 13
    a = torch.randn(T, H * 2 * row, generator=g).to(dtype)
    a[:, dv:row] = float("nan")                           # numbers beyond a head's values do not count
    wide = (torch.randn(T, H + 5, generator=g) * 3).to(dtype)
    for gate in (wide[:, 2:2 + H], None):
        want = fake_ops.map_difference(a, H, row, dv, 0.7, 1e-5, 0.35, gate)
        got = ops.map_difference(a.to(DEV), H, row, dv, 0.7, 1e-5, 0.35, None if gate is None else wide.to(DEV)[:, 2:2 + H])
        _close(got, want, 2e-6 if dtype == torch.float32 else 1e-2, "difference")


def _segments(lens, pad_at=None):
    """cu_q, positions, tok_seg, seg_slots for segments of the given lengths (a segment ``pad_at`` is padding)."""
    cu, pos, seg = [0], [], []
    for s, n in enumerate(lens):
        cu.append(cu[-1] + n)
        pos += [-1] * n if s == pad_at else list(range(5 * s, 5 * s + n))
        seg += [s] * n
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    return i32(cu), i32(pos), i32(seg), i32(list(range(len(lens) - 1, -1, -1)))


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 24), (2, 2, 40, 8), (3, 1, 64, 64), (2, 1, 200, 130), (1, 1, 128, 16), (6, 3, 10, 20)])
@pytest.mark.parametrize("lens,pad_at", [([1, 70, 5, 2], 2), ([1, 1, 1], None), ([33], None), ([3, 2, 3], None), ([4, 1, 15, 16, 17], None)])
def test_delta_rule_kernels_with_a_decay_per_head(H, G, d, dv, lens, pad_at):
    """Both forms: a pass over the memory for every token, and for every four (steps that hold a segment of four or more)."""
    from pico_vllm_b200 import ops
    for longest in (1, max(lens)):
        _delta_rule_case(ops, H, G, d, dv, lens, pad_at, longest)


def _delta_rule_case(ops, H, G, d, dv, lens, pad_at, longest):
    g = torch.Generator().manual_seed(d + dv + len(lens))
    cu, pos, seg, slots = _segments(lens, pad_at)
    T, S = int(cu[-1]), len(lens)
    xc = torch.randn(T, 2 * G * d + H * dv + 3, generator=g)
    proj = torch.randn(T, 2 * H + 5, generator=g) * 2
    dt_bias, a_log = torch.randn(H, generator=g), torch.randn(H, generator=g) - 1.0
    for dtype in (torch.float32, torch.bfloat16):
        p = proj.to(dtype)
        want = fake_ops.delta_prepare(xc, 2, 2 + G * d, p, 3, p[:, 3 + H:3 + 2 * H], dt_bias, a_log, H, G, d, per_head=True, max_q_len=longest)
        pg = p.to(DEV)
        got = ops.delta_prepare(xc.to(DEV), 2, 2 + G * d, pg, 3, pg[:, 3 + H:3 + 2 * H], dt_bias.to(DEV), a_log.to(DEV), H, G, d, per_head=True,
                                max_q_len=longest).cpu()
        pair, dots = got[:, 2 * G * d:2 * G * d + 4 * H].view(T, H, 4), got[:, 2 * G * d + 4 * H:].view(T, G, 8)
        pair[:, :, 2:] = 0                             # numbers nobody reads
        dots[:, :, 7 if longest >= ops.DELTA_BLOCK_MIN_TOKENS else 1:] = 0
        _close(got, want, 2e-6, "delta_prepare")
    prep = want
    state = torch.randn(S + 1, H, dv, d, generator=g) * 0.3
    v = xc[:, 2 + 2 * G * d:]
    st_want = state.clone()
    o_want = fake_ops.gated_delta_rule(prep, v, st_want, slots, cu, pos, H, G, d, dv, per_head=True, max_q_len=longest)
    st_got = state.to(DEV)
    o_got = ops.gated_delta_rule(prep.to(DEV), v.to(DEV), st_got, slots.to(DEV), cu.to(DEV), pos.to(DEV), H, G, d, dv, per_head=True,
                                 max_q_len=longest)
    live = pos >= 0
    _close(o_got.cpu()[live], o_want[live], 2e-5, "delta rule outputs")
    _close(st_got, st_want, 2e-5, "delta rule states")
    _status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,n", [(4, 24), (3, 700), (12, 64)])
def test_group_norm_with_a_silu_gate(dtype, groups, n):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(7, groups * n, generator=g), torch.rand(groups * n, generator=g) + 0.5
    gate = (torch.randn(7, groups * n + 9, generator=g) * 3).to(dtype)
    for act in ("sigmoid", "silu"):
        want = fake_ops.group_rms_norm(x, groups, n, n, w, 1e-5, dtype, post_gate=gate[:, 5:], post_act=act)
        got = ops.group_rms_norm(x.to(DEV), groups, n, n, w.to(DEV), 1e-5, dtype, post_gate=gate.to(DEV)[:, 5:], post_act=act)
        _close(got, want, 2e-6 if dtype == torch.float32 else 1e-2, act)


@pytest.mark.parametrize("M,K,I", [(1, 96, 40), (9, 64, 24), (16, 1536, 256), (130, 128, 72), (300, 352, 416), (700, 1536, 1000)])
def test_biased_gelu_inside_the_products(M, K, I):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(M)
    x = torch.randn(M, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(2 * I, K, generator=g) * 2.0 * K ** -0.5).to(torch.bfloat16)
    gu = x.float() @ w.float().t()
    for bias in (torch.randn(2 * I, generator=g) * 2, None):
        want = fake_ops._biased(gu, bias, "gelu_tanh")
        bg = None if bias is None else bias.to(DEV)
        if ops.skinny_takes(x.to(DEV), w.to(DEV)):
            _close(ops.skinny_gate_up_gelu(x.to(DEV), w.to(DEV), bg), want, 1e-2, "few tokens")
        if ops.tc_takes(x.to(DEV), w.to(DEV)):
            for rows in (None, 256, 512):
                _close(ops.tc_gate_up_gelu(x.to(DEV), w.to(DEV), bg, rows=rows), want, 1e-2, f"tcgen05 {rows}")
    _status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,I", [(5, 24), (40, 52), (3, 7), (600, 96)])
def test_biased_activations_and_products_with_a_bias(dtype, T, I):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(T)
    gu, bias = (torch.randn(T, 2 * I, generator=g) * 4).to(dtype), torch.randn(2 * I, generator=g)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for act in ("silu", "gelu_tanh"):
        for b in (bias, None):
            _close(ops.bias_glu(gu.to(DEV), None if b is None else b.to(DEV), act), fake_ops.bias_glu(gu, b, act), tol, act)
    x, w = torch.randn(T, 48, generator=g).to(dtype), torch.randn(64, 48, generator=g).to(dtype)
    b = torch.randn(64, generator=g).to(torch.bfloat16).float()
    _close(ops.linear_bias(x.to(DEV), w.to(DEV), b.to(DEV)), fake_ops.linear_bias(x, w, b), tol, "product")


# ------------------------------------------------------------------------------------------------ whole models
_CUTS = {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_tail_decode(r, 32),
         "portions": helpers.trace_portions, "mixed": lambda r: helpers.trace_mixed(r, max_live=4, seed=3)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SHAPES))
@pytest.mark.parametrize("cut,graph", [("whole", False), ("tail", False), ("tail", True), ("portions", False),
                                       ("mixed", False), ("mixed", True)])
def test_every_cutting_matches_plain(dtype, name, cut, graph):
    raw = _raw(name, dtype)
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 500 + i) for i, n in enumerate(LENGTHS[name])}
    steps = _CUTS[cut](reqs)
    tensors = _tensors(raw, SEEDS[name])
    runner = _runner(raw, tensors, dtype, helpers.live_token_peak(steps), graph=graph)
    _compare(steps, reqs, helpers.replay(runner, steps), _cached_oracle(name, dtype, raw, tensors, reqs), dtype, f"{name}/{cut}/{dtype}")
    if graph:
        assert runner.graph_replays > 0
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)      # every page came back
    _status()


_LOGITS = {}


def _cached_oracle(name, dtype, raw, tensors, reqs):
    """The plain implementation's logits of a named shape: the same for every cutting."""
    if (name, dtype) not in _LOGITS:
        _LOGITS[name, dtype] = _oracle(raw, tensors, reqs)
    return _LOGITS[name, dtype]


def _random_shape(seed):
    """A model whose every size, count, constant, order of layers and loop is drawn from ``seed``."""
    import random
    rnd = random.Random(seed)
    pick = rnd.choice
    layers = []
    n = rnd.randint(3, 6)
    for _ in range(n):
        kind = pick(["attention", "latent", "delta"])
        if kind == "attention":
            G = pick([1, 2, 3])
            d, dv = pick([16, 32, 64, 24, 40]), pick([16, 32, 64, 128, 40])
            scaling = None if rnd.random() < 0.3 else (pick([2.0, 8.0, 32.0]), pick([1.0, 0.5]), pick([4.0, 2.0]), pick([16, 128, 2048]))
            mixer = _att(G * pick([1, 2, 3, 8]), G, d, dv, pick([0.7, 1.0, 1.4]) * d ** -0.5, pick([0.2, 0.5, 0.8]),
                         _rot(pick([100.0, 10000.0, 500000.0]), pick([d, d // 2 // 2 * 2, 8]), scaling))
        elif kind == "latent":
            d, dr = pick([16, 32, 64, 24]), pick([2, 8, 16, 32])
            mixer = _lat(rnd.randint(1, 12), d, dr, pick([16, 32, 64, 8]), pick([32, 48, 128, 20]), pick([32, 64, 96, 112, 40, 224]),
                         pick([0.7, 1.0, 1.4]) * (d + dr) ** -0.5, pick([None, 1, 5, 16, 33, 72, 100, 130]), pick([100.0, 10000.0, 500000.0]))
        else:
            G = pick([1, 2, 4])
            mixer = _delta(G * pick([1, 2, 3]), G, pick([16, 32, 64, 48, 128]), pick([16, 32, 64, 24, 128]), rnd.randint(1, 5))
        f = rnd.random()
        experts = pick([2, 4, 8, 5])
        layers.append(_layer(mixer, None if f < 0.15 else _dense(pick([48, 64, 100, 384])) if f < 0.45
                             else _moe(pick([16, 24, 64]), experts, rnd.randint(1, experts))))
    loop = None
    if rnd.random() < 0.75:
        a = rnd.randrange(n)
        loop = (a, min(n, a + rnd.randint(1, 2)), rnd.randint(1, 3))
    return _model(pick([97, 211, 448, 1000]), pick([64, 72, 96, 160, 256]), layers, loop, pick([1e-5, 1e-6, 1e-4]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(14)))
def test_drawn_shapes_in_mixed_batches(dtype, seed):
    """Models drawn at random - sizes, head counts, order of layers, loops, windows, constants - each with four live requests,
    portions beside single tokens, pages and slots used again, against the plain implementation."""
    raw = _raw(_random_shape(seed), dtype)
    tensors = _tensors(raw, 100 + seed)
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 40 * seed + i) for i, n in enumerate([110, 3, 41, 77, 60, 18])}
    steps = helpers.trace_mixed(reqs, max_live=4, seed=seed)
    runner = _runner(raw, tensors, dtype, helpers.live_token_peak(steps), graph=seed % 2 == 0)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), dtype, f"drawn {seed}/{dtype}")
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)
    _status()


ALONE = {
    "two maps": [_layer(_att(4, 2, 24, 40, 0.5, 0.5, _rot(300.0, 8, (4.0, 1.0, 4.0, 64))))],
    "two maps, TMA rows": [_layer(_att(6, 2, 32, 64, 0.4, 0.3, _rot(1000.0, 32)))],
    "latent": [_layer(_lat(3, 24, 12, 40, 30, 56, 0.3, 20, 300.0))],
    "latent, no window": [_layer(_lat(2, 16, 16, 16, 20, 24, 0.3))],
    "delta": [_layer(_delta(4, 2, 24, 40, 4))],
    "delta, one tap": [_layer(_delta(2, 2, 32, 16, 1))],
    "dense": [_layer(_delta(1, 1, 8, 8, 1), _dense(44))],
    "experts": [_layer(_lat(1, 8, 2, 8, 8, 16, 0.3), _moe(36, 8, 3))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("times", [None, 3])
@pytest.mark.parametrize("what", sorted(ALONE))
def test_each_mechanism_alone(dtype, times, what):
    """A model of one layer, run once and three times in a row: a whole prompt, then the same prompt token by token, then in
    portions down to two tokens."""
    raw = _raw(_model(157, 72, copy.deepcopy(ALONE[what]), loop=(0, 1, times) if times else None), dtype)
    tensors = _tensors(raw, 5)
    reqs = {"p": helpers.random_ids(75, raw["vocab"], 21)}
    logits = _oracle(raw, tensors, reqs)
    for cut, steps in (("whole", helpers.trace_whole(reqs)), ("single", helpers.trace_tail_decode(reqs, 74)),
                       ("portions", helpers.trace_portions(reqs, sizes=(2, 5, 2, 21, 3)))):
        runner = _runner(raw, tensors, dtype, 128)
        _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"{what}/{cut}/{dtype}/{times}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size", [4, 16, 64])
def test_other_page_sizes_and_batches_against_each_alone(dtype, page_size):
    """Unequal requests in one batch give what each gives alone (the same engine, one request per step), and both agree
    with the plain implementation."""
    raw = _raw("a", dtype)
    tensors = _tensors(raw, SEEDS["a"])
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 900 + i) for i, n in enumerate([6, 50, 17, 120])}
    together = [dict(entries=[dict(id=r, tokens=ids[:-4], want=list(range(len(ids) - 4))) for r, ids in reqs.items()], end=[])]
    for k in range(4, 0, -1):
        together.append(dict(entries=[dict(id=r, tokens=[ids[-k]], want=[0]) for r, ids in reqs.items()],
                             end=list(reqs) if k == 1 else []))
    alone = helpers.trace_tail_decode(reqs, 4)
    logits = _oracle(raw, tensors, reqs)
    outs = {}
    for what, steps in (("together", together), ("alone", alone)):
        runner = _runner(raw, tensors, dtype, helpers.live_token_peak(steps), page_size=page_size)
        got = helpers.replay(runner, steps)
        _compare(steps, reqs, got, logits, dtype, f"{what}/page {page_size}/{dtype}")
        at, rows = {r: 0 for r in reqs}, {}
        for st, g in zip(steps, got):
            i = 0
            for e in st["entries"]:
                for w in e["want"]:
                    rows[(e["id"], at[e["id"]] + w)] = g[i]
                    i += 1
                at[e["id"]] += len(e["tokens"])
        outs[what] = rows
    assert outs["together"].keys() == outs["alone"].keys()
    scale = max(float(v.abs().max()) for v in outs["alone"].values())
    worst = max(float((outs["together"][k] - outs["alone"][k]).abs().max()) for k in outs["alone"])
    assert worst <= (2e-5 if dtype == "float32" else 6e-2) * scale


def _without_positions(tensors):
    """No learned positions and no biases in the norms, so that what a layer reads is the tokens alone."""
    for n in tensors:
        if n == "pos" or n.endswith("norm1.b"):
            tensors[n] = torch.zeros_like(tensors[n])
    return tensors


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [48, 112])           # 112 + 16 numbers a row: the TMA and tcgen05 kernels
@pytest.mark.parametrize("window", [48, 50])
def test_keys_just_inside_and_just_outside_a_window(dtype, window, rank):
    """A window of three pages and one that ends in the middle of a page, scores made sharp by a large factor on q.k.  The
    oracle with a window one longer or one shorter gives other logits by far more than the tolerance, so a window that is
    one token off shows; the engine must agree with the right one from a whole prompt, from single tokens and from portions cut
    at the window's length and at page borders."""
    raw = _model(97, 64, [_layer(_lat(4, 32, 16, 32, 48, rank, 1.2, window, 10000.0))])
    tensors = _without_positions(_tensors(raw, 91))
    tensors["l0.mix.o"] = tensors["l0.mix.o"] * 16
    ids = helpers.random_ids(4 * window + 9, raw["vocab"], 6)
    reqs = {"r": ids}
    logits = _oracle(raw, tensors, reqs)
    scale = float(logits["r"].abs().max())
    for other in (window - 1, window + 1):
        wrong = copy.deepcopy(raw)
        wrong["layers"][0]["mixer"]["mask"]["size"] = other
        diff = (plain.forward(wrong, tensors, ids) - logits["r"]).abs().amax(1)
        assert _shows(float(diff[window:].max()), scale, dtype), (other, float(diff[window:].max()) / scale)
    cuts = {"whole": helpers.trace_whole(reqs), "single": helpers.trace_tail_decode(reqs, 3 * window + 5),
            "edges": helpers.trace_portions(reqs, sizes=(window - 1, 2, window - 2, 3, window, window + 1, 2)),
            "pages": helpers.trace_portions(reqs, sizes=(16, 32, 15, 2, 48, 17))}
    for what, steps in cuts.items():
        runner = _runner(raw, tensors, dtype, 256)
        _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"{what}/{dtype}/window {window}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["latent", "attention"])
def test_a_far_key_among_hundreds_and_the_first_tokens(dtype, kind):
    """420 equal tokens but one, at position 3, chosen so that the last queries notice it: losing it would show.  Read from a
    whole prompt, token by token, and in portions."""
    layer = _lat(2, 48, 16, 32, 32, 48, 1.0) if kind == "latent" else _att(2, 1, 32, 64, 6.0, 0.3, _rot(10000.0, 8, (8.0, 1.0, 4.0, 64)))
    raw = _model(97, 64, [_layer(layer)])
    tensors = _without_positions(_tensors(raw, 17))
    if kind == "attention":      # equal values cancel in the difference of the maps: one map has to prefer the odd token clearly
        for n in ("q", "k"):
            tensors[f"l0.mix.{n}"] = tensors[f"l0.mix.{n}"] * 3
    tensors["l0.mix.o"] = tensors["l0.mix.o"] * (16 if kind == "attention" else 4)
    base = [11] * 420
    plain_last = plain.forward(raw, tensors, base)[-1]
    best, best_diff = None, 0.0
    for cand in range(20, 36):
        ids = list(base)
        ids[3] = cand
        d = float((plain.forward(raw, tensors, ids)[-1] - plain_last).abs().max())
        if d > best_diff:
            best, best_diff = cand, d
    ids = list(base)
    ids[3] = best
    reqs = {"r": ids}
    logits = _oracle(raw, tensors, reqs)
    assert _shows(best_diff, float(logits["r"].abs().max()), dtype), best_diff / float(logits["r"].abs().max())
    cuts = {"whole": helpers.trace_whole(reqs), "single": helpers.trace_tail_decode(reqs, 200),
            "portions": helpers.trace_portions(reqs, sizes=(2, 2, 3, 64, 130, 2, 17))}
    for what, steps in cuts.items():
        runner = _runner(raw, tensors, dtype, 448)
        _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"{what}/{dtype}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_memory_that_remembers_the_first_tokens(dtype):
    """The delta rule set to forget slowly, with keys of 64, run twice in a row: the output at the end of 400 tokens still holds
    the first 200, so a memory that is lost, zeroed or handed to another request or pass shows.  Two requests take turns, in
    portions down to two tokens and single tokens, in slots that were used before; then whole prompts and long portions."""
    raw = _model(120, 64, [_layer(_delta(3, 1, 64, 40, 4))], loop=(0, 1, 2))
    tensors = _without_positions(_tensors(raw, 8))
    tensors["l0.mix.A_log"] = torch.full_like(tensors["l0.mix.A_log"], -9.0)
    tensors["l0.mix.o"] = tensors["l0.mix.o"] * 3
    reqs = {"w": helpers.random_ids(40, raw["vocab"], 1), "x": helpers.random_ids(400, raw["vocab"], 2),
            "y": helpers.random_ids(300, raw["vocab"], 3)}
    logits = _oracle(raw, tensors, reqs)
    late = plain.forward(raw, tensors, [0] * 200 + reqs["x"][200:])     # other tokens in the first 200 places
    assert _shows(float((late[-1] - logits["x"][-1]).abs().max()), float(logits["x"].abs().max()), dtype)
    steps = helpers.trace_whole({"w": reqs["w"]})                         # uses a slot and gives it back
    steps += helpers.trace_mixed({"x": reqs["x"], "y": reqs["y"]}, max_live=2, seed=5, chunk_sizes=(2, 7, 64, 3, 2, 33))
    runner = _runner(raw, tensors, dtype, 1024, max_num_seqs=2)
    _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"memory/{dtype}")
    steps = helpers.trace_whole({"x": reqs["x"], "y": reqs["y"]}) + helpers.trace_portions({"x": reqs["x"]}, sizes=(300, 2, 98))
    _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"long portions/{dtype}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_reused_slots(dtype):
    """300 single-token steps after a short prompt, twice, through a pool that holds one request."""
    raw = _raw("a", dtype)
    tensors = _tensors(raw, SEEDS["a"])
    reqs = {"x": helpers.random_ids(330, raw["vocab"], 41), "y": helpers.random_ids(330, raw["vocab"], 42)}
    steps = helpers.trace_tail_decode(reqs, 300)
    runner = _runner(raw, tensors, dtype, 384, graph=True, max_num_seqs=1)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), dtype, f"long decode/{dtype}")
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)
    _status()


def test_batches_of_many_tokens_and_many_requests():
    """bfloat16: a prompt long enough for the tcgen05 products with the gelu epilogue, beside 40 requests that decode (more than
    the weight-streaming products take), wanted rows here and there."""
    raw = _raw(_model(300, 128, [_layer(_att(4, 2, 32, 64, 0.2, 0.5, _rot(10000.0, 32)), _dense(96)), _layer(_lat(4, 32, 32, 32, 64, 96, 0.15, 70), _moe(64, 4, 2)),
                                 _layer(_delta(2, 2, 64, 64, 4), _dense(64))], loop=(1, 3, 2)), "bfloat16")
    tensors = _tensors(raw, 3)
    reqs = {f"r{i}": helpers.random_ids(14 + (i * 7) % 30, raw["vocab"], 700 + i) for i in range(40)}
    reqs["long"] = helpers.random_ids(420, raw["vocab"], 699)
    steps = helpers.trace_many_decoders(reqs, tail=5, per_step=14)
    runner = _runner(raw, tensors, "bfloat16", helpers.live_token_peak(steps), graph=True, max_num_seqs=44)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), "bfloat16", "many")
    _status()


# ------------------------------------------------------------------------------------------------ the entry points
def _greedy(raw, tensors, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(plain.forward(raw, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]


def _write_model(raw, tensors, folder):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def test_greedy_generation_through_the_scheduler_and_the_command_line(tmp_path, capsys):
    """float32, so that the greedy choice is the oracle's: several requests of unequal length through ``LLM.generate`` (its
    scheduler cuts prompts into portions and batches them beside decoding requests), then one through the command line."""
    from pico_vllm_b200 import LLM, SamplingParams
    raw = SHAPES["c"]
    tensors = _tensors(raw, SEEDS["c"])
    folder = _write_model(raw, tensors, str(tmp_path / "model"))
    prompts = [helpers.random_ids(n, raw["vocab"], 70 + n) for n in (3, 41, 18, 77)]
    llm = LLM(folder, dtype="float32", page_size=16, max_cache_tokens=512, max_num_seqs=3, max_num_batched_tokens=32, device=DEV)
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=10, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert list(o.token_ids) == _greedy(raw, tensors, p, 10)
    from pico_vllm_b200.cli import main
    capsys.readouterr()
    rc = main(["run", "--model", folder, "--dtype", "float32", "--prompt-ids", ",".join(map(str, prompts[2])),
               "--prompt-ids", "9,9", "--max-new-tokens", "8", "--temperature", "0", "--num-gpu-blocks", "32", "--ignore-eos"])
    assert rc == 0
    lines = [l for l in capsys.readouterr().out.splitlines() if l.startswith("[")]
    printed = {int(l[1:l.index("]")]): [int(t) for t in l.split("] ")[1].split()] for l in lines}
    for rid, p in enumerate([prompts[2], [9, 9]]):       # prompt and generated tokens are printed together
        assert printed[rid] == p + _greedy(raw, tensors, p, 8)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    """bin/trace_run on a model folder: four live requests, portions beside single tokens, pages and slots used again."""
    raw = _raw("a", dtype)
    tensors = _tensors(raw, SEEDS["a"])
    folder = _write_model(raw, tensors, str(tmp_path / "model"))
    reqs = {f"q{i}": helpers.random_ids(n, raw["vocab"], 300 + i) for i, n in enumerate([70, 5, 130, 33, 64, 90])}
    steps = helpers.trace_mixed(reqs, max_live=4, seed=9)
    out_dir = str(tmp_path / "out")
    lines = "".join(json.dumps(dict(step=i, **s)) + "\n" for i, s in enumerate(steps))
    run = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out_dir,
                          "--max-tokens", str(helpers.live_token_peak(steps))], input=lines, capture_output=True, text=True,
                         cwd=ROOT, timeout=1500)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    logits = _oracle(raw, tensors, reqs)
    got = [None if w is None else torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(-1, raw["vocab"]))
           for i, w in enumerate(helpers.expected_logits(steps, reqs, logits))]
    _compare(steps, reqs, got, logits, dtype, f"trace_run/{dtype}")
