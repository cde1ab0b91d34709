"""The Vanapel design in the engine against the plain implementation of tests/plain_vanapel.py: the new kernels against torch
arithmetic, each mechanism alone (models of one to three layers), whole models of several small shapes in every cutting of
requests into steps, batches against each request alone, keys just inside and just outside a window and far back, the first
tokens of a request, long decoding through pages and slots that are used again, and greedy generation through the entry
points."""
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
import plain_vanapel as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
REL = {"float32": 5e-5, "bfloat16": 6e-2}      # max |difference| / max |logit| over a step; float32 is the sharp test
STD = 0.12


def _att(heads, kv_heads, dim, vdim, scale, window=None, v_mix=False):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if window:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m)


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, scaling=None):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
                                                    scale=scale, rot=rot))


def _layer(mixer, ff=None, limit=1.0):
    return dict(mixer, mlp=None if ff is None else dict(kind="dense", ff=ff, limit=limit))


def _model(vocab, width, layers, groups=1, eps=1e-5):
    return dict(architecture="Vanapel", vocab=vocab, width=width, norm=dict(eps=eps, groups=groups), layers=layers)


SHAPES = {
    # three groups of 32; key and value sizes differ everywhere (heads padded to 48 in the cache); windows of 24 and 9, no
    # multiples of a page; a latent of 40 and 8 rotated numbers in a row of 48; layers without feed-forward; an attention layer
    # that sees everything and keeps its own values; three layers that share values
    "a": _model(211, 96, [_layer(_att(4, 2, 32, 48, 0.2, 24, True), 64, 0.9),
                          _layer(_lat(3, 16, 8, 24, 24, 40, 0.3, 500.0, (4.0, 64, 8.0, 0.5))),
                          _layer(_att(6, 2, 16, 48, 0.3, 9, True)),
                          _layer(_att(3, 1, 40, 20, 0.15), 40, 2.0),
                          _layer(_att(2, 2, 24, 48, 0.25, 33, True), 24, 0.5)], groups=3),
    # one group; a latent layer first; rows of 128 (96 + 32) and heads of 64 and 128, which the TMA and tcgen05 kernels take;
    # a rotation without stretching; windows of a page and of three quarters of a tile
    "b": _model(300, 128, [_layer(_lat(4, 64, 32, 64, 64, 96, 0.1)),
                           _layer(_att(4, 1, 64, 64, 0.125, 16, True), 96, 3.0),
                           _layer(_att(8, 4, 128, 128, 0.09, 48, False), 64, 1.0),
                           _layer(_att(2, 1, 64, 64, 0.2, 100, True), None),
                           _layer(_lat(8, 32, 16, 32, 32, 48, 0.2, 100.0, (2.0, 32, 16.0, 2.0)), 48, 0.7)], eps=1e-6),
    # awkward sizes: groups of 34, which no vector of four fits into evenly, an odd vocabulary, heads of 20, 12 and 10, inner
    # sizes that are no multiples of 8, a window of 7
    "c": _model(203, 102, [_layer(_att(5, 1, 20, 12, 0.3, 7, True), 28, 1.3),
                           _layer(_lat(5, 20, 6, 12, 22, 36, 0.3, 50.0, (8.0, 100, 4.0, 0.25)), 12, 0.6),
                           _layer(_att(6, 1, 10, 12, 0.5, 20, True), 52, 4.0)], groups=3, eps=1e-4),
    # more than sixteen query heads on one key/value head, a cached row beyond 256, a window of one position
    "d": _model(150, 160, [_layer(_lat(18, 24, 64, 16, 48, 256, 0.15, 1000.0, (1.0, 512, 32.0, 1.0)), 72, 1.0),
                           _layer(_att(20, 1, 32, 16, 0.2, 30, False)),
                           _layer(_att(2, 1, 32, 32, 0.2, 1, True), 32, 0.4),
                           _layer(_att(4, 1, 16, 32, 0.2, 64, True))], groups=5),
}
SEEDS = {"a": 11, "b": 22, "c": 33, "d": 44}
LENGTHS = {"a": [1, 9, 33, 70, 150, 230], "b": [2, 17, 48, 97, 200], "c": [3, 40, 129, 75], "d": [5, 31, 90]}


def _tensors(raw, seed, std=STD):
    from pico_vllm_b200.registry import config_from_dict
    from pico_vllm_b200.weights import random_tensors
    t = random_tensors(config_from_dict(raw), seed, std=std, dtype=torch.bfloat16)
    for n in t:
        x = t[n].float()
        if n.endswith(".norm") or ".norm" in n:
            x = 1.0 + 4.0 * (x - 1.0)                       # weights around one, some well away from it
        elif n.endswith(".sink"):
            x = x * 15.0                                    # sinks that take much, and some that take little
        elif n.endswith(".r1"):
            x = 0.4 + 3.0 * (x - 0.5).abs()
        elif n.endswith(".r2"):
            x = 0.05 + 5.0 * (x - 0.5).abs()
        elif n.endswith(".mlp.gate") or n.endswith(".mlp.up"):
            x = x * 2.0                                     # so that the caps cut
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
    REL, and none is beyond twice that."""
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
        assert max(errs)[0] <= 2 * REL[dtype], f"{what}: a row is off by {max(errs)}"


def _shows(diff, scale, dtype):
    """Whether a difference between two oracles is large enough that the comparison in ``dtype`` would catch it."""
    return diff > max(20 * REL["float32"], 3 * REL[dtype] if dtype == "bfloat16" else 0.0) * scale


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
@pytest.mark.parametrize("H,groups,post_groups", [(96, 3, 3), (102, 3, 2), (288, 4, 2), (2048, 4, 4), (1536, 1, 2), (512, 8, 1),
                                                  (4100, 5, 5), (6144, 2, 3), (100, 10, 10)])
def test_norms_in_groups(dtype, H, groups, post_groups):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(H + groups)
    T = 9
    x = torch.randn(T, H, generator=g) * torch.linspace(0.1, 3.0, H)       # the groups' root mean squares differ
    d = (torch.randn(T, H, generator=g) * torch.linspace(2.0, 0.2, H)).to(dtype)
    w, pw = torch.rand(H, generator=g) + 0.5, torch.rand(H, generator=g) + 0.5
    rows = torch.tensor([7, 0, 3], dtype=torch.int32)
    for r in (None, rows):
        for delta in (d, None):
            xw, xg = x.clone(), x.to(DEV)
            n = T if r is None else 3
            ow, og = torch.zeros(n, H).to(dtype), torch.zeros(n, H).to(dtype).to(DEV)
            fake_ops.post_add_norm(xw, delta, pw, 1, 1e-5, w, 1, 1e-4, ow, r, post_groups, groups)
            ops.post_add_norm(xg, None if delta is None else delta.to(DEV), pw.to(DEV), 1, 1e-5, w.to(DEV), 1, 1e-4, og,
                              None if r is None else r.to(DEV), post_groups, groups)
            _close(xg, xw, 1e-5, "stream")
            _close(og, ow, 1e-5 if dtype == torch.float32 else 1e-2, "normed")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,norm,mix,shift", [(4, 2, 32, 48, True, True, 0), (8, 1, 64, 40, True, False, 0), (3, 1, 20, 12, True, True, 1),
                                                     (2, 2, 128, 128, True, True, 0), (5, 1, 256, 16, False, True, 0), (6, 3, 10, 30, True, True, 0),
                                                     (1, 1, 300, 8, True, False, 0), (40, 4, 16, 16, True, True, 0)])
def test_head_norm_store(dtype, H, G, d, dv, norm, mix, shift):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(d + H)
    T, ps, row = 11, 4, -(-max(d, dv) // 16) * 16
    x = (torch.randn(T, shift + (H + G) * d + G * dv + 3 * shift, generator=g) * 2).to(dtype)
    slots = torch.tensor([0, 5, 6, 7, 9, -1, 13, -1, 20, 2, 31], dtype=torch.int32)
    lam = torch.tensor(0.3) if mix else None
    wide = torch.randn(T, G * dv + 16, generator=g).to(dtype)
    first = wide[:, 8:8 + G * dv] if mix else None
    fill = lambda: torch.full((8, G, ps, row), float("nan")).to(dtype)
    kp, vp, kg, vg = fill(), fill(), fill().to(DEV), fill().to(DEV)
    offs = (shift, shift + H * d, shift + (H + G) * d)
    want = fake_ops.head_norm_store(x, *offs, norm, 1e-5, slots, kp, vp, H, G, d, dv, row, ps, lam, first)
    got = ops.head_norm_store(x.to(DEV), *offs, norm, 1e-5, slots.to(DEV), kg, vg, H, G, d, dv, row, ps, lam.to(DEV) if mix else None,
                              wide.to(DEV)[:, 8:8 + G * dv] if mix else None)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    _close(got, want, tol, "queries")
    for a, b, what in ((kg, kp, "keys"), (vg, vp, "values")):
        assert torch.equal(torch.isnan(a.float().cpu()), torch.isnan(b.float()))      # nothing stored where nothing belongs
        _close(torch.nan_to_num(a.float()), torch.nan_to_num(b.float()), tol, what)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("r,dr,rot,H,d,qr", [(40, 8, 8, 3, 16, 24), (36, 6, 6, 5, 20, 0), (96, 32, 16, 2, 64, 64), (64, 80, 80, 4, 8, 10)])
def test_rotated_key_part_and_rotated_queries(dtype, r, dr, rot, H, d, qr):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(r)
    T, row = 11, -(-(r + dr) // 16) * 16
    p = torch.randn(T, qr + r + dr + 2, generator=g).to(dtype)
    pos = torch.tensor([0, 1, 2, 300, 1117, -1, 7, 8, 9, 10, 11], dtype=torch.int32)
    slots = torch.tensor([3, 0, 9, 1, 7, -1, 8, 2, 30, 31, 12], dtype=torch.int32)
    qw, kw = torch.rand(max(qr, 1), generator=g) + 0.5, torch.rand(r, generator=g) + 0.5
    inv = (37.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)).float()
    dev = lambda t: t.to(DEV)
    cw, cg = torch.full((2, 1, 16, row), float("nan")).to(dtype), torch.full((2, 1, 16, row), float("nan")).to(dtype).to(DEV)
    off = qr + r
    want, _ = fake_ops.latent_norm_store(p, 0, qr, qw if qr else None, qr, r, kw, slots, cw, 0, 0, 1e-5, rot=(off, dr, pos, inv, 1.2))
    got, gate = ops.latent_norm_store(dev(p), 0, qr, dev(qw) if qr else None, qr, r, dev(kw), dev(slots), cg, 0, 0, 1e-5,
                                      rot=(off, dr, dev(pos), dev(inv), 1.2))
    tol = 3e-4 if dtype == torch.float32 else 1e-2       # float32: the angle of position 1117 is rounded before sin and cos
    assert gate is None and (got is None) == (qr == 0)
    if qr:
        _close(got, want, tol, "query latent")
    assert torch.equal(torch.isnan(cg.float().cpu()), torch.isnan(cw.float()))
    _close(torch.nan_to_num(cg.float()), torch.nan_to_num(cw.float()), tol, "cache rows")
    x = torch.randn(T, H * (d + dr), generator=g).to(dtype)
    xg = dev(x)
    ops.rotate_tail(xg, H, dr, dev(pos), dev(inv), 1.2)
    _close(xg, fake_ops.rotate_tail(x.clone(), H, dr, pos, inv, 1.2), tol, "queries")


def _attention_case(H, G, hd, dv, ps, lens, starts, seed):
    """Queries, pages with the keys and values of segments of the given lengths behind ``starts`` earlier tokens, and the
    index arrays of a step; pages in mixed order, NaN wherever nothing belongs."""
    g = torch.Generator().manual_seed(seed)
    T, S = sum(lens), len(lens)
    blocks = [-(-(st + n) // ps) for st, n in zip(starts, lens)]
    perm = torch.randperm(sum(blocks) + 3, generator=g)
    kp = torch.full((sum(blocks) + 3, G, ps, hd), float("nan"))
    vp = kp.clone()
    table = torch.zeros(S, max(blocks) + 1, dtype=torch.int32)
    at = 0
    for s in range(S):
        table[s, :blocks[s]] = perm[at:at + blocks[s]].to(torch.int32)
        for n in range(starts[s] + lens[s]):
            pg = int(table[s, n // ps])
            kp[pg, :, n % ps] = torch.randn(G, hd, generator=g)
            v = torch.zeros(G, hd)
            v[:, :dv] = torch.randn(G, dv, generator=g)
            vp[pg, :, n % ps] = v
        at += blocks[s]
    q = torch.randn(T, H * hd, generator=g)
    cu, pos, seg = [0], [], []
    for s, (n, st) in enumerate(zip(lens, starts)):
        cu.append(cu[-1] + n)
        pos += list(range(st, st + n))
        seg += [s] * n
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    pf = i32([s for s, n in enumerate(lens) if n > 1])
    dec = i32([cu[s] for s, n in enumerate(lens) if n == 1])
    return q, kp, vp, table, i32(cu), i32(pos), i32(seg), pf, dec, max(lens)


@pytest.mark.parametrize("H,G,hd,dv", [(4, 2, 48, 48), (7, 1, 64, 56), (16, 1, 128, 96), (6, 2, 128, 128), (3, 1, 80, 64), (4, 1, 64, 64)])
@pytest.mark.parametrize("ps,window,splits", [(16, None, 1), (16, 150, 4), (8, 70, 3), (64, 300, 8), (16, None, 2)])
@pytest.mark.parametrize("bias,sink", [(True, True), (True, False), (False, True)])
def test_attention_kernels_with_distance_bias_and_sink(H, G, hd, dv, ps, window, splits, bias, sink):
    """Every paged attention kernel (tcgen05 and mma.sync portions, TMA and mma.sync single tokens with their parts in clusters
    and through scratch, the float32 kernel) with a logarithmic bias and sinks that differ by head."""
    from pico_vllm_b200 import ops
    lens, starts = [1, 70, 2, 1, 37, 1], [500, 130, 0, 0, 300, 77]
    q, kp, vp, table, cu, pos, seg, pf, dec, mx = _attention_case(H, G, hd, dv, ps, lens, starts, hd + ps)
    g = torch.Generator().manual_seed(7)
    slopes = torch.rand(H, generator=g) * 1.5 if bias else None
    rates = torch.rand(H, generator=g) * 2 + 0.01 if bias else None
    sinks = torch.randn(H, generator=g) * 3 if sink else None
    dev = lambda t: None if t is None else t.to(DEV)
    scale = 0.8 * hd ** -0.5
    for dtype in (torch.float32, torch.bfloat16):
        qd, kd, vd = q.to(dtype), kp.to(dtype), vp.to(dtype)
        want = torch.zeros(q.shape).to(torch.float32)
        fake_ops.paged_attention(qd.float(), kd.float(), vd.float(), want, seg, pos, table, H, G, hd, ps, window, scale, slopes=slopes,
                                 sinks=sinks, rates=rates)
        T = q.shape[0]
        scratch = torch.empty(max(1, ops.attention_scratch_floats(T, H, hd, splits)), device=DEV)
        kg, vg = kd.to(DEV), vd.to(DEV)
        tol = 1e-5 if dtype == torch.float32 else 2e-2
        out = torch.zeros(T, H * hd, dtype=dtype, device=DEV)
        ops.paged_attention(dev(qd), kg, vg, out, dev(seg), dev(pos), dev(table), H, G, hd, ps, window, scale, splits, scratch,
                            slopes=dev(slopes), sinks=dev(sinks), rates=dev(rates))
        _close(out, want, tol, f"generic {dtype}")
        if dtype == torch.float32:
            continue
        for maps in (False, True):
            m1 = (ops.make_kv_tensor_map(kg), ops.make_kv_tensor_map(vg)) if maps else (None, None)
            m2 = (ops.make_kv_tensor_map_2d(kg), ops.make_kv_tensor_map_2d(vg, values=True)) if maps else (None, None)
            if maps and m1[0] is None:
                continue
            out = torch.zeros(T, H * hd, dtype=dtype, device=DEV)
            ops.paged_attention_mma(dev(qd), kg, vg, out, dev(seg), dev(pos), dev(table), dev(cu), dev(pf), len(pf), mx, dev(dec), len(dec),
                                    H, G, hd, ps, window, scale, splits, scratch, *m1, *m2, 0, slopes=dev(slopes), sinks=dev(sinks),
                                    rates=dev(rates))
            _close(out, want, tol, f"tensor cores, TMA {maps}")
    _status()


def test_attention_over_a_latent_that_is_key_and_value_with_sinks():
    """One tensor read as keys and as values, rows of 128 (tensor maps) and of 80, 320 and 640 (the widest)."""
    from pico_vllm_b200 import ops
    for hd, H in ((128, 12), (80, 8), (320, 3), (640, 2)):
        lens, starts = [1, 33, 1], [260, 70, 3]
        q, kp, _, table, cu, pos, seg, pf, dec, mx = _attention_case(H, 1, hd, hd, 16, lens, starts, hd)
        g = torch.Generator().manual_seed(hd)
        sinks = torch.randn(H, generator=g) * 2
        dev = lambda t: t.to(DEV)
        scale = hd ** -0.5
        for dtype in (torch.float32, torch.bfloat16):
            qd, kd = q.to(dtype), kp.to(dtype)
            want = torch.zeros(q.shape)
            fake_ops.paged_attention(qd.float(), kd.float(), kd.float(), want, seg, pos, table, H, 1, hd, 16, None, scale, sinks=sinks)
            kg, T = kd.to(DEV), q.shape[0]
            out = torch.zeros(T, H * hd, dtype=dtype, device=DEV)
            scratch = torch.empty(ops.attention_scratch_floats(T, H, hd, 2), device=DEV)
            ops.paged_attention(dev(qd), kg, kg, out, dev(seg), dev(pos), dev(table), H, 1, hd, 16, None, scale, 2, scratch, sinks=dev(sinks))
            _close(out, want, 1e-5 if dtype == torch.float32 else 2e-2, f"generic {hd}")
            if ops.mma_attention_takes(dtype, H, 1, hd):
                m1, m2, m3 = ops.make_kv_tensor_map(kg), ops.make_kv_tensor_map_2d(kg), ops.make_kv_tensor_map_2d(kg, values=True)
                out = torch.zeros(T, H * hd, dtype=dtype, device=DEV)
                ops.paged_attention_mma(dev(qd), kg, kg, out, dev(seg), dev(pos), dev(table), dev(cu), dev(pf), len(pf), mx, dev(dec),
                                        len(dec), H, 1, hd, 16, None, scale, 2, scratch, m1, m1, m2, m3, 0, sinks=dev(sinks))
                _close(out, want, 2e-2, f"tensor cores {hd}")
    _status()


@pytest.mark.parametrize("M,K,I", [(1, 96, 40), (9, 64, 24), (16, 1536, 256), (130, 128, 72), (300, 352, 416), (700, 1536, 1000)])
def test_capped_gate_and_up_inside_the_products(M, K, I):
    from pico_vllm_b200 import ops
    g = torch.Generator().manual_seed(M)
    x = torch.randn(M, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(2 * I, K, generator=g) * 2.0 * K ** -0.5).to(torch.bfloat16)
    gu = x.float() @ w.float().t()
    for limit in (0.7, 3.0):
        want = fake_ops._capped(gu[:, :I], gu[:, I:], limit)
        if ops.skinny_takes(x.to(DEV), w.to(DEV)):
            _close(ops.skinny_gate_up_swiglu(x.to(DEV), w.to(DEV), limit=limit), want, 1e-2, "few tokens")
            xf, nw = torch.randn(M, K, generator=g), torch.rand(K, generator=g) + 0.5
            if ops.skinny_norm_takes(xf.to(DEV), w.to(DEV)):
                y = xf / torch.sqrt((xf * xf).mean(-1, keepdim=True) + 1e-5) * nw
                gn = y.to(torch.bfloat16).float() @ w.float().t()
                _close(ops.skinny_gate_up_swiglu(xf.to(DEV), w.to(DEV), nw.to(DEV), 1e-5, limit=limit),
                       fake_ops._capped(gn[:, :I], gn[:, I:], limit), 2e-2, "few tokens, norm inside")
        if ops.tc_takes(x.to(DEV), w.to(DEV)):
            for rows in (None, 256, 512):
                _close(ops.tc_gate_up_swiglu(x.to(DEV), w.to(DEV), rows=rows, limit=limit), want, 1e-2, f"tcgen05 {rows}")
    _status()


# ------------------------------------------------------------------------------------------------ whole models
_CUTS = {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_tail_decode(r, 32),
         "portions": helpers.trace_portions, "mixed": lambda r: helpers.trace_mixed(r, max_live=4, seed=3)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SHAPES))
@pytest.mark.parametrize("cut,graph", [("whole", False), ("tail", False), ("tail", True), ("portions", False),
                                       ("mixed", False), ("mixed", True)])
def test_every_cutting_matches_plain(dtype, name, cut, graph):
    raw = SHAPES[name]
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 500 + i) for i, n in enumerate(LENGTHS[name])}
    steps = _CUTS[cut](reqs)
    tensors = _tensors(raw, SEEDS[name])
    runner = _runner(raw, tensors, dtype, helpers.live_token_peak(steps), graph=graph)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), dtype, f"{name}/{cut}/{dtype}")
    if graph:
        assert runner.graph_replays > 0
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)      # every page came back
    _status()


def _random_shape(seed):
    """A model whose every size, count, constant and order of layers is drawn from ``seed``."""
    import random
    rnd = random.Random(seed)
    pick = rnd.choice
    width, groups = pick([(64, 1), (64, 4), (72, 3), (96, 2), (160, 5), (320, 4), (256, 8)])
    share = (pick([1, 2, 4]), pick([16, 32, 64, 40, 128]))            # key/value heads and value size of the layers that mix
    layers = []
    for _ in range(rnd.randint(3, 6)):
        if rnd.random() < 0.6:
            mix = rnd.random() < 0.7
            G, dv = share if mix else (pick([1, 2, 3]), pick([16, 24, 48, 64]))
            d = pick([16, 32, 64, 40, 128])
            mixer = _att(G * pick([1, 2, 3, 8]), G, d, dv, pick([0.7, 1.0, 1.4]) * d ** -0.5, pick([None, 1, 5, 16, 33, 72, 100, 130]), mix)
        else:
            scaling = None if rnd.random() < 0.2 else (pick([1.0, 2.0, 8.0]), pick([16, 128, 2048]), pick([32.0, 4.0]), pick([1.0, 0.25]))
            d, dr = pick([16, 32, 64, 24]), pick([2, 8, 16, 32])
            mixer = _lat(rnd.randint(1, 12), d, dr, pick([16, 32, 64, 8]), pick([32, 48, 128, 20]), pick([32, 64, 96, 112, 40, 224]),
                         pick([0.7, 1.0, 1.4]) * (d + dr) ** -0.5, pick([100.0, 10000.0, 500000.0]), scaling)
        layers.append(_layer(mixer, pick([None, 48, 64, 100, 384]), pick([0.5, 1.0, 3.0, 7.0])))
    return _model(pick([97, 211, 448, 1000]), width, layers, groups, pick([1e-5, 1e-6, 1e-4]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(14)))
def test_drawn_shapes_in_mixed_batches(dtype, seed):
    """Models drawn at random - sizes, head counts, order of layers, groups, windows, constants - each with four live requests,
    portions beside single tokens, pages and slots used again, against the plain implementation.  (Scales near the size's
    own: scores of tens turn the 16-bit rounding of queries and keys into a tenth of a logit, in torch as in the kernels.)"""
    raw = _random_shape(seed)
    tensors = _tensors(raw, 100 + seed)
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 40 * seed + i) for i, n in enumerate([150, 3, 41, 77, 120, 18])}
    steps = helpers.trace_mixed(reqs, max_live=4, seed=seed)
    runner = _runner(raw, tensors, dtype, helpers.live_token_peak(steps), graph=seed % 2 == 0)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), dtype, f"drawn {seed}/{dtype}")
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)
    _status()


_RELAY = [_layer(_att(2, 1, 16, 24, 0.3, 12, True)), _layer(_lat(2, 8, 4, 8, 12, 16, 0.3)), _layer(_att(4, 1, 24, 24, 0.3, 30, True))]
ALONE = {
    "window": [_layer(_att(4, 2, 24, 40, 0.3, 20))],
    "no window": [_layer(_att(3, 3, 32, 16, 0.3))],
    "latent": [_layer(_lat(3, 24, 12, 40, 30, 56, 0.3, 300.0, (4.0, 64, 8.0, 0.5)))],
    "latent, plain frequencies": [_layer(_lat(2, 16, 16, 16, 20, 24, 0.3))],
    "mixed values": _RELAY,
    "feed-forward": [_layer(_att(1, 1, 8, 8, 0.3, 8), 44, 0.8)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("groups", [1, 3])
@pytest.mark.parametrize("what", sorted(ALONE))
def test_each_mechanism_alone(dtype, groups, what):
    """A model of one layer (three where values are mixed): a whole prompt, then the same prompt token by token, then in
    portions down to two tokens."""
    raw = _model(157, 72, copy.deepcopy(ALONE[what]), groups)
    tensors = _tensors(raw, 5)
    reqs = {"p": helpers.random_ids(75, raw["vocab"], 21)}
    logits = _oracle(raw, tensors, reqs)
    for cut, steps in (("whole", helpers.trace_whole(reqs)), ("single", helpers.trace_tail_decode(reqs, 74)),
                       ("portions", helpers.trace_portions(reqs, sizes=(2, 5, 2, 21, 3)))):
        runner = _runner(raw, tensors, dtype, 128)
        _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"{what}/{cut}/{dtype}/{groups}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size", [4, 16, 64])
def test_other_page_sizes_and_batches_against_each_alone(dtype, page_size):
    """Unequal requests in one batch give what each gives alone (the same engine, one request per step), and both agree
    with the plain implementation."""
    raw = SHAPES["a"]
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
    assert worst <= (2e-5 if dtype == "float32" else 4e-2) * scale


def _weak_bias(tensors, sink=-6.0):
    """Distance penalties small enough for a far key to count, sinks that take little."""
    for n in tensors:
        if n.endswith(".r1"):
            tensors[n] = torch.full_like(tensors[n], 0.02)
        if n.endswith(".sink"):
            tensors[n] = torch.full_like(tensors[n], sink)
    return tensors


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [32, 64])           # 64: the TMA and tcgen05 kernels
@pytest.mark.parametrize("window", [48, 50])
def test_keys_just_inside_and_just_outside_a_window(dtype, window, dim):
    """A window of three pages and one that ends in the middle of a page, scores made sharp by a large factor on q.k.  The
    oracle with a window one longer or one shorter gives other logits by far more than the tolerance, so a window that is
    one token off shows; the engine must agree with the right one from a whole prompt, from single tokens and from portions cut
    at the window's length and at page borders."""
    raw = _model(97, 64, [_layer(_att(4, 1, dim, dim, 0.4, window))], 2)
    tensors = _weak_bias(_tensors(raw, 91))
    ids = helpers.random_ids(4 * window + 9, raw["vocab"], 6)
    reqs = {"r": ids}
    logits = _oracle(raw, tensors, reqs)
    scale = float(logits["r"].abs().max())
    for other in (window - 1, window + 1):
        wrong = copy.deepcopy(raw)
        wrong["layers"][0]["mixer"]["mask"]["size"] = other
        diff = (plain.forward(wrong, tensors, ids) - logits["r"]).abs().amax(1)
        assert _shows(float(diff[window:].max()), scale, dtype)
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
    layer = _lat(2, 48, 16, 32, 32, 48, 0.5, 10000.0, (8.0, 64, 8.0, 0.5)) if kind == "latent" else _att(2, 1, 64, 32, 0.3)
    raw = _model(97, 64, [_layer(layer)], 2)
    tensors = _weak_bias(_tensors(raw, 17))
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
    assert _shows(best_diff, float(logits["r"].abs().max()), dtype), best_diff
    cuts = {"whole": helpers.trace_whole(reqs), "single": helpers.trace_tail_decode(reqs, 200),
            "portions": helpers.trace_portions(reqs, sizes=(2, 2, 3, 64, 130, 2, 17))}
    for what, steps in cuts.items():
        runner = _runner(raw, tensors, dtype, 448)
        _compare(steps, reqs, helpers.replay(runner, steps), logits, dtype, f"{what}/{dtype}")
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_reused_slots(dtype):
    """300 single-token steps after a short prompt, twice, through a pool that holds one request."""
    raw = SHAPES["a"]
    tensors = _tensors(raw, SEEDS["a"])
    reqs = {"x": helpers.random_ids(330, raw["vocab"], 41), "y": helpers.random_ids(330, raw["vocab"], 42)}
    steps = helpers.trace_tail_decode(reqs, 300)
    runner = _runner(raw, tensors, dtype, 384, graph=True, max_num_seqs=1)
    _compare(steps, reqs, helpers.replay(runner, steps), _oracle(raw, tensors, reqs), dtype, f"long decode/{dtype}")
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)
    _status()


def test_batches_of_many_tokens_and_many_requests():
    """bfloat16: a prompt long enough for the tcgen05 products with the capped epilogue, beside 40 requests that decode (more
    than the weight-streaming products take), wanted rows here and there."""
    raw = _model(300, 128, [_layer(_att(4, 2, 64, 64, 0.125, 70, True), 96, 1.0), _layer(_lat(4, 32, 32, 32, 64, 96, 0.15), 128, 0.8),
                            _layer(_att(2, 2, 64, 64, 0.2, 40, True), 64, 2.0)], 4)
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
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=12, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert list(o.token_ids) == _greedy(raw, tensors, p, 12)
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
    raw = SHAPES["a"]
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
