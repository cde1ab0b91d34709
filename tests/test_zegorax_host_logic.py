"""The Zegorax design through the step function, the cache and the batch building on the CPU, with the kernels replaced by torch
doubles (tests/fake_ops.py): looped layers with cache entries and states of their own for every pass, windows whose pages come
back, page and slot reuse and wanted rows, in every way of cutting requests into steps."""
import pytest

import fake_ops
import helpers
import plain_zegorax as plain
from test_zegorax_gpu import SEEDS, SHAPES, _tensors


def _runner(raw, tensors, max_tokens, page_size, max_num_seqs=4):
    from pico_vllm_b200.config import EngineConfig
    from pico_vllm_b200.engine import ModelRunner, make_cache, model_from_tensors
    from pico_vllm_b200.registry import config_from_dict
    ecfg = EngineConfig(dtype="float32", page_size=page_size, max_cache_tokens=max_tokens, max_num_seqs=max_num_seqs,
                        use_cuda_graph=False, device="cpu")
    model = model_from_tensors(config_from_dict(raw), tensors, ecfg)
    return ModelRunner(model, make_cache(model, ecfg, poison_freed=True), ecfg)


@pytest.fixture
def on_cpu(monkeypatch):
    fake_ops.install(monkeypatch)
    import pico_vllm_b200.engine.core as core
    monkeypatch.setattr(core, "_require_device", lambda device: None)


@pytest.mark.parametrize("name,page_size", [("a", 8), ("b", 16), ("c", 4)])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_every_cutting_matches_plain(on_cpu, name, page_size, cut):
    raw = SHAPES[name]
    tensors = _tensors(raw, SEEDS[name])
    reqs = {f"r{i}": helpers.random_ids(n, raw["vocab"], 40 + i) for i, n in enumerate([1, 7, 30, 36, 18])}
    steps = {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_tail_decode(r, 12),
             "portions": helpers.trace_portions, "mixed": lambda r: helpers.trace_mixed(r, max_live=3, seed=2)}[cut](reqs)
    runner = _runner(raw, tensors, helpers.live_token_peak(steps), page_size, max_num_seqs=3)
    logits = {rid: plain.forward(raw, tensors, ids) for rid, ids in reqs.items()}
    want = helpers.expected_logits(steps, reqs, logits)
    got = helpers.replay(runner, steps)
    for i, (g, w) in enumerate(zip(got, want)):
        assert (g is None) == (w is None)
        if w is not None:
            helpers.assert_close_logits(g, w.float(), 5e-5, f"{name}/{cut} step {i}")
    assert all(g.pool.in_use == 0 for g in runner.cache.groups)


def test_pages_a_window_has_passed_come_back(on_cpu):
    """While a request decodes, a window's pages are given back as soon as no later query can see them - in every pass of a looped
    layer, whose entries share the group's block table; layers without a window keep theirs."""
    raw = SHAPES["a"]
    tensors = _tensors(raw, SEEDS["a"])
    runner = _runner(raw, tensors, 128, 8, max_num_seqs=1)
    ids = helpers.random_ids(90, raw["vocab"], 3)
    steps = helpers.trace_tail_decode({"r": ids}, 40)[:-1]       # the request stays
    helpers.replay(runner, steps)
    by_window = {g.spec.window: g for g in runner.cache.groups if g.spec.window}
    assert by_window[24].pool.in_use <= 24 // 8 + 1 and len(by_window[24].entries) == 2
    assert all(g.pool.in_use == 12 for g in runner.cache.groups if g.spec.window is None)


def test_a_request_cannot_outgrow_the_position_table(on_cpu):
    from pico_vllm_b200.errors import ScheduleError
    raw = dict(SHAPES["c"], max_positions=20)
    runner = _runner(raw, _tensors(raw, 1), 64, 4, max_num_seqs=1)
    with pytest.raises(ScheduleError):
        helpers.replay(runner, helpers.trace_whole({"r": helpers.random_ids(21, raw["vocab"], 3)}))
