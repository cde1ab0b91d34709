"""The Vanapel configuration reader, the builder's tensor names and cache layout, the random-weights folder, and what the plain
implementation of the tests notices (CPU)."""
import copy
import json

import pytest
import torch

import helpers
import plain_vanapel as plain
from test_vanapel_gpu import SEEDS, SHAPES, _shows, _tensors


def _cfg(raw):
    from pico_vllm_b200.registry import config_from_dict
    return config_from_dict(raw)


@pytest.mark.parametrize("name", sorted(SHAPES))
def test_reads_back_what_it_writes(name):
    cfg = _cfg(SHAPES[name])
    assert cfg.architecture == "Vanapel" and _cfg(cfg.to_dict()) == cfg
    assert _cfg(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_absent_keys_have_the_documented_meaning():
    raw = copy.deepcopy(SHAPES["a"])
    del raw["norm"]["groups"], raw["layers"][3]["mixer"]["v_mix"], raw["layers"][1]["mixer"]["rot"]["scaling"]
    cfg = _cfg(raw)
    assert cfg.norm_groups == 1 and cfg.layers[3].mixer.v_mix is False and cfg.layers[3].mixer.window is None
    assert cfg.layers[1].mixer.scaling is None and cfg.layers[1].mlp is None


@pytest.mark.parametrize("change,word", [
    (lambda r: r["norm"].update(groups=5), "groups"),
    (lambda r: r["norm"].pop("eps"), "eps"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][2]["mixer"].update(vdim=16), "v_mix"),
    (lambda r: r["layers"][0]["mixer"].update(v_mix=1), "v_mix"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda r: r["layers"][1].update(type="mamba2"), "type"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda r: r["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda r: r.pop("vocab"), "vocab"),
])
def test_errors_name_the_key(change, word):
    from pico_vllm_b200.errors import ConfigError
    raw = copy.deepcopy(SHAPES["a"])
    change(raw)
    with pytest.raises(ConfigError) as e:
        _cfg(raw)
    assert word in str(e.value)


def test_tensor_names_cache_entries_and_who_mixes_values():
    from pico_vllm_b200.errors import WeightError
    from pico_vllm_b200.parts import PagedKV, PagedLatent
    from pico_vllm_b200.registry import build_model
    from pico_vllm_b200.weights.loader import check_tensors, wanted_tensors
    raw = SHAPES["a"]
    model = build_model(_cfg(raw))
    want = wanted_tensors(model)
    assert want["l0.mix.v"] == (96, 96) and want["l0.mix.vmix"] == () and want["l2.mix.r1"] == (6,) and want["l1.mix.sink"] == (3,)
    assert want["l1.mix.dkv"] == (48, 96) and want["l1.mix.uq"] == (72, 24) and want["l1.mix.uk"] == (48, 40) and want["l1.mix.dkv.norm"] == (40,)
    assert want["l0.mlp.gate"] == (64, 96) and want["head"] == (211, 96) and "l0.norm2b" in want
    assert "l3.mix.vmix" not in want and "l1.norm2" not in want and "l2.mlp.gate" not in want
    assert model.cache_entries == [PagedKV(2, 48, 24), PagedLatent(48, None), PagedKV(2, 48, 9), PagedKV(1, 48, None), PagedKV(2, 48, 33)]
    assert [getattr(b.mixer, "value_mix", None) for b in model.blocks] == ["first", None, "mix", None, "mix"]
    have = {n: tuple(t.shape) for n, t in _tensors(raw, 1).items()}
    check_tensors(model, have, "test")
    have["l0.mix.q"] = (7, 96)
    del have["l2.mix.sink"]
    with pytest.raises(WeightError) as e:
        check_tensors(model, have, "test")
    assert e.value.missing == ["l2.mix.sink"] and e.value.wrong_shape == ["l0.mix.q"]


def test_random_weights_folder(tmp_path):
    from pico_vllm_b200.config.base import read_config_json
    from pico_vllm_b200.weights import write_random_model
    from safetensors.torch import load_file
    cfg = _cfg(SHAPES["c"])
    folder = write_random_model(cfg, 3, str(tmp_path / "m"))
    assert _cfg(read_config_json(folder)) == cfg
    t = load_file(folder + "/model.safetensors")
    assert t["l1.mix.uk"].shape == (100, 36) and t["l0.mix.vmix"].shape == () and t["l0.mix.q"].dtype == torch.bfloat16


def test_parts_refuse_what_is_not_built():
    from pico_vllm_b200.errors import ConfigError, KernelError
    from pico_vllm_b200.parts import DistanceBiasAttention, GatedMLP, GroupedRMSNorm, LatentAttention, RMSNorm, SumDelta
    with pytest.raises(ConfigError):
        GroupedRMSNorm(96, 1e-5, 5)
    with pytest.raises(ConfigError):
        GatedMLP(64, 64, "capped")
    with pytest.raises(ConfigError):
        GatedMLP(64, 64, "silu", limit=2.0)
    with pytest.raises(ConfigError):
        DistanceBiasAttention(64, 2, 1, 16, 16, 1e-5, log_bias=True)             # beside the fixed slopes
    with pytest.raises(ConfigError):
        LatentAttention(64, 2, 16, 16, 8, 16, 1.0, 1e-5, rot_dim=8)              # no position encoding for the rotated part
    x = torch.zeros(1, 96)
    with pytest.raises(KernelError):
        SumDelta([(x, GroupedRMSNorm(96, 1e-5, 3), 1.0)]).flat()
    assert RMSNorm(96, 1e-5).plain_rms and GroupedRMSNorm(96, 1e-5).plain_rms and not GroupedRMSNorm(96, 1e-5, 3).plain_rms


CHANGES = {
    "groups": lambda r: r["norm"].update(groups=1),
    "window": lambda r: r["layers"][0]["mixer"]["mask"].update(size=23),
    "cap": lambda r: r["layers"][0]["mlp"].update(limit=50.0),
    "stretch": lambda r: r["layers"][1]["mixer"]["rot"].pop("scaling"),
    "value mixing": lambda r: r["layers"][4]["mixer"].update(v_mix=False),
    "scale": lambda r: r["layers"][1]["mixer"].update(scale=0.3 * 1.14),
}


@pytest.mark.parametrize("what", sorted(CHANGES) + ["sink", "latent sink", "r1", "r2"])
def test_the_oracle_notices(what):
    """Left out or changed, each mechanism moves the logits of a test shape by far more than the tolerance, so the whole-model
    comparisons would notice."""
    raw = SHAPES["a"]
    tensors = _tensors(raw, SEEDS["a"])
    ids = helpers.random_ids(60, raw["vocab"], 21)
    base = plain.forward(raw, tensors, ids)
    other, changed = copy.deepcopy(raw), dict(tensors)
    if what in CHANGES:
        CHANGES[what](other)
    elif what == "sink":
        changed["l2.mix.sink"] = torch.full_like(tensors["l2.mix.sink"], -50.0)
    elif what == "latent sink":
        changed["l1.mix.sink"] = torch.full_like(tensors["l1.mix.sink"], -50.0)
    else:
        changed[f"l0.mix.{what}"] = tensors[f"l0.mix.{what}"] * 1.25
    diff = float((plain.forward(other, changed, ids) - base).abs().max())
    assert _shows(diff, float(base.abs().max()), "float32"), diff
