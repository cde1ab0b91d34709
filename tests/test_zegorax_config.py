"""The Zegorax configuration reader, the builder's tensor names, order and cache layout, the parts' own rules, the random-weights
folder, and what the plain implementation of the tests notices (CPU)."""
import copy
import json
import math

import pytest
import torch

import helpers
import plain_zegorax as plain
from test_zegorax_gpu import SEEDS, SHAPES, _shows, _tensors


def _cfg(raw):
    from pico_vllm_b200.registry import config_from_dict
    return config_from_dict(raw)


@pytest.mark.parametrize("name", sorted(SHAPES))
def test_reads_back_what_it_writes(name):
    cfg = _cfg(SHAPES[name])
    assert cfg.architecture == "Zegorax" and _cfg(cfg.to_dict()) == cfg
    assert _cfg(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert cfg.layer_runs() == plain.layer_runs(SHAPES[name])


def test_absent_keys_have_the_documented_meaning():
    raw = copy.deepcopy(SHAPES["a"])
    del raw["loop"], raw["layers"][1]["mixer"]["rot"]["scaling"], raw["layers"][2]["mixer"]["mask"]
    cfg = _cfg(raw)
    assert cfg.loop is None and cfg.layer_runs() == [0, 1, 2, 3, 4] and cfg.layers[1].mixer.rot.scaling is None
    assert cfg.layers[2].mixer.window is None and cfg.layers[2].mlp is None and cfg.max_position_embeddings == 640


@pytest.mark.parametrize("change,word", [
    (lambda r: r["norm"].pop("eps"), "eps"),
    (lambda r: r.pop("max_positions"), "max_positions"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=26), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda r: r["layers"][2]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda r: r["layers"][1].update(type="mamba2"), "type"),
    (lambda r: r["layers"][0]["mlp"].update(kind="other"), "kind"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda r: r["loop"].update(stop=6), "stop"),
    (lambda r: r["loop"].update(start=4), "start"),
    (lambda r: r["loop"].update(times=0), "times"),
    (lambda r: r.pop("vocab"), "vocab"),
])
def test_errors_name_the_key(change, word):
    from pico_vllm_b200.errors import ConfigError
    raw = copy.deepcopy(SHAPES["a"])
    change(raw)
    with pytest.raises(ConfigError) as e:
        _cfg(raw)
    assert word in str(e.value)


def test_tensor_names_order_and_cache_entries():
    from pico_vllm_b200.errors import WeightError
    from pico_vllm_b200.parts import FixedState, PagedKV, PagedLatent
    from pico_vllm_b200.registry import build_model
    from pico_vllm_b200.weights.loader import check_tensors, wanted_tensors
    raw = SHAPES["a"]
    model = build_model(_cfg(raw))
    want = wanted_tensors(model)
    assert want["pos"] == (640, 96) and want["l0.norm1.alpha"] == () and want["final.norm.b"] == (96,) and "head" not in want
    assert want["l0.mix.q"] == (32, 96) and want["l0.mix.v.conv"] == (96, 3) and want["l0.mix.a"] == (4, 96) and want["l0.mix.dt_bias"] == (4,)
    assert want["l0.mix.norm"] == (24,) and want["l0.mix.g"] == (96, 96) and want["l0.mlp.down.b"] == (96,)
    assert want["l1.mix.q"] == (192, 96) and want["l1.mix.k"] == (96, 96) and want["l1.mix.lq1"] == (24,) and want["l1.mix.g"] == (4, 96)
    assert want["l1.mlp.router.b"] == (6,) and "l1.mlp.e0.gate.b" not in want
    assert want["l2.mix.dkv"] == (48, 96) and want["l2.mix.uq"] == (72, 20) and want["l2.mix.g"] == (72, 96) and "l2.mlp.router" not in want
    delta = lambda H, dv, d, taps, C: [FixedState((H, dv, d)), FixedState((taps - 1, C))]
    att, lat, late = PagedKV(2, 48), PagedLatent(48, 24), PagedKV(1, 48)
    one_pass = [att, lat] + delta(2, 16, 40, 2, 192)
    assert model.cache_entries == delta(4, 24, 16, 3, 160) + one_pass + one_pass + [late]
    assert [c.block for c in model.order] == [0, 1, 2, 3, 1, 2, 3, 4]
    have = {n: tuple(t.shape) for n, t in _tensors(raw, 1).items()}
    check_tensors(model, have, "test")
    have["l0.mix.q"] = (7, 96)
    del have["l1.mix.lk2"]
    with pytest.raises(WeightError) as e:
        check_tensors(model, have, "test")
    assert e.value.missing == ["l1.mix.lk2"] and e.value.wrong_shape == ["l0.mix.q"]


def test_random_weights_folder(tmp_path):
    from pico_vllm_b200.config.base import read_config_json
    from pico_vllm_b200.weights import write_random_model
    from safetensors.torch import load_file
    cfg = _cfg(SHAPES["c"])
    folder = write_random_model(cfg, 3, str(tmp_path / "m"))
    assert _cfg(read_config_json(folder)) == cfg
    t = load_file(folder + "/model.safetensors")
    assert t["l2.mix.uk"].shape == (100, 36) and t["l0.norm1.alpha"].shape == () and t["l0.mix.q"].dtype == torch.bfloat16


@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 64), (8.0, 0.5, 2.0, 700), (3.0, 1.0, 1.0, 30)])
def test_frequencies_in_three_bands(scaling):
    from pico_vllm_b200.parts import BandScaledRotary
    rot = dict(base=500.0, dims=24)
    kw = {}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        kw = rot["scaling"]
    got = BandScaledRotary(32, 500.0, 24, **kw).frequencies()
    want = torch.tensor(plain.scaled_frequencies(rot), dtype=torch.float64)
    assert torch.allclose(got.double(), want, rtol=1e-6, atol=0)
    if scaling and scaling[2] > scaling[1]:
        base = torch.tensor(plain.scaled_frequencies(dict(base=500.0, dims=24)))
        share = want / base
        assert (share == 1).any() and (share < 1).any()


def test_reordered_rows_turn_neighbours_into_halves():
    """Latent attention loads the rows of the rotated part in another order; the same order on both sides keeps every score."""
    from pico_vllm_b200.parts import BandScaledRotary, LatentAttention
    H, d, dr, r, qr, D = 2, 6, 8, 10, 5, 12
    mixer = LatentAttention(D, H, d, 4, qr, r, 1.0, 1e-5, gate="elements", rot_dim=dr, position=BandScaledRotary(dr, 100.0, 6, pairing="neighbours"))
    g = torch.Generator().manual_seed(0)
    uq, down = torch.randn(H * (d + dr), qr, generator=g), torch.randn(qr + r + dr + H * 4, D, generator=g)
    mixer.assign("uq_weight", uq)
    mixer.assign("down_weight", down)
    order = [0, 2, 4, 1, 3, 5, 6, 7]
    a, b = uq.view(H, d + dr, qr), mixer.uq_weight.view(H, d + dr, qr)
    assert torch.equal(b[:, :d], a[:, :d]) and torch.equal(b[:, d:], a[:, d:][:, order])
    at = qr + r
    assert torch.equal(mixer.down_weight[:at], down[:at]) and torch.equal(mixer.down_weight[at:at + dr], down[at:at + dr][order])
    assert torch.equal(mixer.down_weight[at + dr:at + dr + H * 4], down[at + dr:])


def test_parts_refuse_what_is_not_built():
    from pico_vllm_b200.errors import ConfigError, KernelError
    from pico_vllm_b200.parts import (BandScaledRotary, DifferentialAttention, GatedDeltaRule, GatedMLP, LatentAttention, NormedDelta,
                                      RMSNorm, SumDelta, TanhNorm)
    x = torch.zeros(1, 96)
    for delta in (NormedDelta(x, RMSNorm(96, 1e-5)), SumDelta([(x, RMSNorm(96, 1e-5), 1.0)])):
        with pytest.raises(KernelError):
            TanhNorm(96).add_norm(x, delta)
    assert not getattr(TanhNorm(96), "plain_rms", False)
    with pytest.raises(ConfigError):
        GatedMLP(64, 64, "capped", limit=2.0, bias=True)
    with pytest.raises(ConfigError):
        GatedDeltaRule(64, 2, 2, 16, 16, 4, 1e-5, head_decay=True)
    with pytest.raises(ConfigError):
        GatedDeltaRule(64, 2, 2, 16, 16, 4, 1e-5, gate_act="relu")
    with pytest.raises(ConfigError):
        BandScaledRotary(16, 100.0, 7)
    with pytest.raises(ConfigError):
        DifferentialAttention(64, 2, 1, 16, 16, 1e-5, 0.25, 0.5, BandScaledRotary(16, 100.0, 8, pairing="neighbours"))
    with pytest.raises(ConfigError):
        LatentAttention(64, 2, 16, 16, 8, 16, 1.0, 1e-5, gate="rows")


CHANGES = {
    "loop": lambda r: r["loop"].update(times=3),
    "window": lambda r: r["layers"][2]["mixer"]["mask"].update(size=23),
    "diff": lambda r: r["layers"][1]["mixer"].update(diff=0.5),
    "bands": lambda r: r["layers"][1]["mixer"]["rot"].pop("scaling"),
    "scale": lambda r: r["layers"][2]["mixer"].update(scale=0.33),
    "rotated numbers": lambda r: r["layers"][4]["mixer"]["rot"].update(dims=18),
    "top": lambda r: r["layers"][1]["mlp"]["router"].update(top=3),
}
TENSORS = {"positions": "pos", "norm bias": "l1.norm1.b", "alpha": "l2.norm1.alpha", "lambda": "l1.mix.lq2", "gate per head": "l1.mix.g",
           "gate per number": "l2.mix.g", "delta gate": "l0.mix.g", "decay": "l3.mix.a", "decay bias": "l0.mix.dt_bias", "step size": "l3.mix.b",
           "first tap": None, "gate bias": "l0.mlp.gate.b", "up bias": "l0.mlp.up.b", "down bias": "l4.mlp.down.b", "router bias": "l1.mlp.router.b"}


@pytest.mark.parametrize("what", sorted(CHANGES) + sorted(TENSORS) + ["pairing"])
def test_the_oracle_notices(what, monkeypatch):
    """Left out or changed, each mechanism moves the logits of a test shape by far more than the tolerance, so the whole-model
    comparisons would notice."""
    raw = SHAPES["a"]
    tensors = _tensors(raw, SEEDS["a"])
    ids = helpers.random_ids(48, raw["vocab"], 21)
    base = plain.forward(raw, tensors, ids)
    other, changed = copy.deepcopy(raw), dict(tensors)
    if what in CHANGES:
        CHANGES[what](other)
    elif what == "pairing":
        monkeypatch.setattr(plain, "rotate_neighbours", plain.rotate_halves)
    elif what == "first tap":
        changed["l0.mix.k.conv"] = tensors["l0.mix.k.conv"].clone()
        changed["l0.mix.k.conv"][:, 0] = 0
    else:
        changed[TENSORS[what]] = tensors[TENSORS[what]] * 0
    diff = float((plain.forward(other, changed, ids) - base).abs().max())
    assert _shows(diff, float(base.abs().max()), "float32"), diff


def test_softplus_and_gelu_of_the_oracle():
    z = torch.linspace(-40, 40, 81, dtype=torch.float64)
    assert torch.allclose(plain.softplus(z), torch.nn.functional.softplus(z, threshold=60.0), rtol=1e-12, atol=1e-14)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), rtol=1e-12, atol=1e-14)
    assert math.isclose(float(plain.map_weight({k: torch.zeros(3, dtype=torch.float64) for k in ("lq1", "lk1", "lq2", "lk2")}, 0.3)), 0.3)
