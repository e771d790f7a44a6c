"""Lemunex without a GPU: the configuration reader, expected tensors, random models on disk, and the
plain implementation's own consistency."""
import copy
import math

import pytest
import torch

import plain_lemunex as P
from pretrained_rstr_b200.config.base import ConfigError
from pretrained_rstr_b200.config.registry import lookup, named_sizes, read_config
from pretrained_rstr_b200.weights import load_weights, make_random_model
from pretrained_rstr_b200.weights.safetensors_io import save_file

RAW = {"architecture": "Lemunex", "vocab": 90, "width": 32, "norm": {"eps": 1e-5},
       "layers": [
           {"type": "mamba2", "mlp": {"kind": "dense", "ff": 40},
            "mixer": {"heads": 4, "vdim": 6, "state": 5, "groups": 2, "conv": 3, "norm_groups": 3}},
           {"type": "parallel",
            "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.4, "mask": {"size": 9},
                               "rot": {"base": 300.0, "dims": 6,
                                       "scaling": {"factor": 3.0, "original": 50, "fast": 8.0, "slow": 1.0}}},
                      "right": {"heads": 3, "dim": 4, "vdim": 8, "tau": 5.0},
                      "left_scale": 0.7, "right_scale": 1.3},
            "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "identity": 2, "top": 3},
                    "shared": {"ff": 20}}},
           {"type": "mamba2", "mlp": None,
            "mixer": {"heads": 2, "vdim": 8, "state": 16, "groups": 1, "conv": 1, "norm_groups": 1}}]}


def test_registry_and_structure():
    arch = lookup(RAW)
    cfg = arch.config_class.from_dict(RAW)
    assert arch.name == "Lemunex" and arch.config_class.from_dict(cfg.to_dict()) == cfg
    assert [(e.layer, e.cache_layer) for e in cfg.run_order()] == [(0, 0), (1, 1), (2, 2)]
    specs = cfg.layer_specs()
    assert [s.mixer.kind for s in specs] == ["state_space", "side_by_side", "state_space"]
    assert [s.feed_forward.kind for s in specs] == ["act_mlp", "gated_moe", "none"]
    assert all(s.arrangement == "parallel" and set(s.norms) == {"shared"} for s in specs)
    assert specs[0].norms["shared"].params["offset"] == 1.0
    left, right = specs[1].mixer.params["left"], specs[1].mixer.params["right"]
    assert left.kind == "window_attention" and right.kind == "gated_linear_attention"
    assert left.params["window"] == 9 and left.params["rot_layout"] == "interleaved"
    assert left.params["rot_yarn"]["original"] == 50 and left.params["head_gate"] and left.params["out_bias"]
    assert right.params["tau"] == 5.0 and specs[1].mixer.params["right_scale"] == 1.3
    moe = specs[1].feed_forward.params
    assert moe["identity"] == 2 and moe["top"] == 3 and moe["shared_inner"] == 20 and not moe["renormalize"]
    exp = {k: tuple(v.shape) for k, v in arch.expected_tensors(cfg).items()}
    assert exp["l0.mix.in"] == (24 + 24 + 20 + 4, 32) and exp["l0.mix.conv"] == (44, 3)
    assert exp["l1.mix.left.o"] == (32, 24) and exp["l1.mix.right.norm"] == (8,)
    assert exp["l1.mlp.router"] == (7, 32) and exp["l1.mlp.e4.down"] == (32, 12) and "l1.mlp.e5.down" not in exp
    assert exp["l1.mlp.shared.sg"] == (1, 32) and exp["head"] == (90, 32) and "l2.mlp.up" not in exp
    plain = copy.deepcopy(RAW)
    del plain["layers"][1]["mlp"]["router"]["identity"], plain["layers"][1]["mixer"]["left"]["rot"]["scaling"]
    plain["layers"][1]["mlp"]["shared"] = None
    cfg = arch.config_class.from_dict(plain)
    assert arch.expected_tensors(cfg)["l1.mlp.correction"].shape == (5,)
    assert "l1.mlp.shared.sg" not in arch.expected_tensors(cfg)
    assert cfg.layer_specs()[1].mixer.params["left"].params["rot_yarn"] is None
    assert "lemunex-small" in named_sizes()


@pytest.mark.parametrize("change", [
    lambda r: r["layers"][0].__setitem__("type", "mamba"),
    lambda r: r["layers"][0]["mixer"].__setitem__("groups", 3),
    lambda r: r["layers"][0]["mixer"].__setitem__("norm_groups", 5),
    lambda r: r["layers"][0]["mixer"].__delitem__("state"),
    lambda r: r["layers"][0]["mixer"].__setitem__("conv", 0),
    lambda r: r["layers"][0]["mlp"].__delitem__("ff"),
    lambda r: r["layers"][1]["mixer"]["left"].__setitem__("kv_heads", 3),
    lambda r: r["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 5),
    lambda r: r["layers"][1]["mixer"]["left"]["rot"]["scaling"].__delitem__("slow"),
    lambda r: r["layers"][1]["mixer"]["right"].__setitem__("tau", 0.0),
    lambda r: r["layers"][1]["mixer"].__delitem__("left_scale"),
    lambda r: r["layers"][1]["mixer"].__setitem__("right", None),
    lambda r: r["layers"][1]["mlp"]["router"].__setitem__("top", 8),
    lambda r: r["layers"][1]["mlp"].__setitem__("kind", "sparse"),
    lambda r: r.__setitem__("layers", [])])
def test_bad_configurations_are_refused(change):
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError):
        lookup(raw).config_class.from_dict(raw)


def test_the_file_decides_the_decays_rank(tmp_path):
    """The low-rank matrix has as many rows as its tensor says."""
    arch = lookup(RAW)
    cfg = arch.config_class.from_dict(RAW)
    tensors = dict(arch.random_tensors(cfg, 1))
    tensors["l1.mix.right.a1"], tensors["l1.mix.right.a2"] = torch.randn(3, 32), torch.randn(12, 3)
    cfg.save(str(tmp_path))
    save_file(tensors, str(tmp_path / "model.safetensors"))
    store = load_weights(str(tmp_path), arch.expected_tensors(cfg), torch.device("cpu"))
    assert tuple(store.get("l1.mix.right.a1").shape) == (3, 32)


def test_random_folder_round_trip_and_plain_consistency(tmp_path):
    """A random model written by the package is read by the plain implementation's own reader;
    the plain model is causal, and every mechanism it has moves its logits."""
    arch = lookup(RAW)
    cfg = arch.config_class.from_dict(RAW)
    folder = str(tmp_path / "m")
    make_random_model(folder, cfg, 3, torch.float32)
    assert read_config(folder)[1].to_dict() == cfg.to_dict()
    raw, W = P.read_folder(folder)
    assert set(W) == set(arch.expected_tensors(cfg))
    ids = [(7 * i + 3) % 90 for i in range(30)]
    taps, margins = [], []
    full = P.forward(ids, W, raw, taps=taps, margins=margins)
    assert len(taps) == 3 and full.shape == (30, 90) and len(margins) == 1 and bool((margins[0] >= 0).all())
    assert torch.allclose(P.forward(ids[:17], W, raw), full[:17], atol=1e-10)        # causal

    def moved(change_raw=None, change_w=None):
        r, w = copy.deepcopy(raw), dict(W)
        if change_raw:
            change_raw(r)
        if change_w:
            change_w(w)
        return float((P.forward(ids, w, r)[-1] - full[-1]).abs().max())

    parallel = lambda r: r["layers"][1]
    assert moved(lambda r: parallel(r)["mixer"].__setitem__("right_scale", 1.0)) > 1e-3
    assert moved(lambda r: parallel(r)["mixer"]["right"].__setitem__("tau", 2.0)) > 1e-3
    assert moved(lambda r: parallel(r)["mixer"]["left"]["mask"].__setitem__("size", 8)) > 1e-4
    assert moved(lambda r: parallel(r)["mixer"]["left"]["rot"].__delitem__("scaling")) > 1e-4
    assert moved(lambda r: parallel(r)["mlp"]["router"].__setitem__("top", 2)) > 1e-4
    assert moved(lambda r: r["layers"][0]["mixer"].__setitem__("norm_groups", 1)) > 1e-5
    for name in ("embed.norm", "l1.mix.left.k.b", "l1.mix.left.o.b", "l1.mix.left.g", "l1.mix.right.a2.b",
                 "l1.mix.right.norm", "l0.mix.conv", "l0.mix.conv.b", "l0.mix.dt_bias", "l0.mix.A_log", "l0.mix.D",
                 "l1.mlp.shared.sg", "l1.mlp.router", "l2.mix.norm", "head"):
        bend = 1.0 + 0.5 * torch.sin(torch.arange(W[name].numel(), dtype=torch.float64) + 1.0).reshape(W[name].shape)
        assert moved(None, lambda w: w.__setitem__(name, w[name] * bend)) > 1e-4, name
    shift = torch.linspace(-3.0, 3.0, 7, dtype=torch.float64)                        # (another choice of experts)
    assert moved(None, lambda w: w.__setitem__("l1.mlp.correction", shift)) > 1e-4
    one = W["l1.mlp.correction"] + 1.0                                               # (the same choice: nothing)
    assert moved(None, lambda w: w.__setitem__("l1.mlp.correction", one)) < 1e-12


def test_yarn_frequencies():
    """Kept, blended and interpolated pairs, and the magnitude, against the plain implementation."""
    from pretrained_rstr_b200.parts.positions_rotary import yarn_frequencies
    for base, dims, factor, original in ((10000.0, 64, 8.0, 512), (500.0, 12, 2.5, 40)):
        rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": 32.0, "slow": 1.0}}
        freq, mag = P.angle_table(rot)
        (hi, lo), got = yarn_frequencies(base, dims, factor, original, 32.0, 1.0, "cpu", with_lo=True)
        assert got == pytest.approx(mag) == pytest.approx(0.1 * math.log(factor) + 1.0)
        assert torch.allclose(hi.double() + lo.double(), freq, rtol=1e-12)
        plain = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
        assert float(freq[-1] / plain[-1]) == pytest.approx(1.0 / factor)
