"""Musilorn without a GPU: the configuration reader, the run order with its caches and joins,
expected tensors, random models on disk, frequencies, and the plain implementation's own
consistency."""
import copy
import math

import pytest
import torch

import plain_musilorn as P
from pretrained_rstr_b200.config.base import ConfigError
from pretrained_rstr_b200.config.registry import lookup, named_sizes, read_config
from pretrained_rstr_b200.weights import make_random_model

RAW = {"architecture": "Musilorn", "vocab": 90, "width": 32, "norm": {"eps": 1e-6}, "residual_mult": 0.4,
       "logit_softcap": 7.0, "loop": {"start": 1, "stop": 3, "times": 3},
       "layers": [
           {"type": "retention", "mlp": None,
            "mixer": {"heads": 2, "dim": 8, "vdim": 12, "decay": [0.9, 0.99], "rot": {"base": 100.0, "dims": 4}}},
           {"type": "attention", "mlp": {"kind": "dense", "ff": 24},
            "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "conv": 4, "scale": 0.4, "softcap": 3.0,
                      "rot": {"base": 50.0, "dims": 6,
                              "scaling": {"factor": 2.0, "low": 1.0, "high": 3.0, "original": 40}}}},
           {"type": "attention", "mlp": None,
            "mixer": {"heads": 3, "kv_heads": 3, "dim": 8, "vdim": 8, "conv": 1, "scale": 0.3, "softcap": 9.0,
                      "rot": {"base": 50.0, "dims": 2}}},
           {"type": "retention", "mlp": {"kind": "dense", "ff": 16},
            "mixer": {"heads": 1, "dim": 16, "vdim": 8, "decay": [0.95], "rot": {"base": 100.0, "dims": 16}}}]}


def test_registry_and_structure():
    arch = lookup(RAW)
    cfg = arch.config_class.from_dict(RAW)
    assert arch.name == "Musilorn" and arch.config_class.from_dict(cfg.to_dict()) == cfg
    order = cfg.run_order()
    assert [e.layer for e in order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [e.cache_layer for e in order] == [0, 1, 2, 4, 5, 6, 7, 3]         # a cache per pass
    assert [e.join_embedding for e in order] == [False, True, False, True, False, True, False, False]
    assert not any(e.add_embedding for e in order)
    assert P.run_list(RAW) == [(e.layer, e.join_embedding) for e in order]
    assert cfg.stream_join_spec().params["weights"] == "loop.in"
    specs = cfg.layer_specs()
    assert [s.mixer.kind for s in specs] == ["retention", "window_attention", "window_attention", "retention"]
    assert [s.feed_forward.kind for s in specs] == ["none", "gated_mlp", "none", "gated_mlp"]
    assert set(specs[0].norms) == {"mixer", "mixer_after"} and len(specs[1].norms) == 4
    mx = specs[1].mixer.params
    assert mx["conv"] == 4 and mx["softcap"] == 3.0 and mx["keys_are_values"] and mx["sink_score"] == 0.0
    assert mx["rot_layout"] == "interleaved" and mx["rot_bands"]["original"] == 40
    assert specs[2].mixer.params["rot_bands"] is None and specs[2].mixer.params["rot_dims"] == 2
    assert specs[3].mixer.params["k_scale"] == pytest.approx(0.25)
    exp = {k: tuple(v.shape) for k, v in arch.expected_tensors(cfg).items()}
    assert exp["loop.in"] == (32, 64) and exp["l1.mix.k.conv"] == (12, 4) and exp["l1.mix.q.norm"] == (6,)
    assert exp["l1.norm2b.b"] == (32,) and exp["l0.mix.g"] == (24, 32) and exp["l3.mlp.down"] == (32, 16)
    assert "l1.mix.v" not in exp and "l0.norm2" not in exp and "l2.norm2b" not in exp
    plain = copy.deepcopy(RAW)
    del plain["loop"], plain["logit_softcap"], plain["layers"][1]["mixer"]["softcap"]
    cfg = arch.config_class.from_dict(plain)
    assert [e.cache_layer for e in cfg.run_order()] == [0, 1, 2, 3] and cfg.stream_join_spec() is None
    assert "loop.in" not in arch.expected_tensors(cfg) and cfg.head_spec().params["softcap"] is None
    assert "musilorn-small" in named_sizes()


@pytest.mark.parametrize("change", [
    lambda r: r["layers"][0].__setitem__("type", "convolution"),
    lambda r: r["layers"][0]["mixer"].__setitem__("decay", [0.9]),
    lambda r: r["layers"][0]["mixer"].__setitem__("rot", None),
    lambda r: r["layers"][1]["mixer"].__setitem__("kv_heads", 3),
    lambda r: r["layers"][1]["mixer"].__setitem__("vdim", 8),
    lambda r: r["layers"][1]["mixer"].__setitem__("conv", 0),
    lambda r: r["layers"][1]["mixer"]["rot"].__setitem__("dims", 5),
    lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].__delitem__("low"),
    lambda r: r["layers"][1]["mlp"].__setitem__("kind", "moe"),
    lambda r: r["loop"].__setitem__("stop", 9),
    lambda r: r.__delitem__("residual_mult"),
    lambda r: r.__setitem__("logit_softcap", 0.0)])
def test_bad_configurations_are_refused(change):
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError):
        lookup(raw).config_class.from_dict(raw)


@pytest.mark.parametrize("base,dims,factor,low,high,original", [
    (10000.0, 64, 8.0, 1.0, 4.0, 512), (500000.0, 16, 3.5, 1.0, 2.0, 100), (77.0, 6, 2.0, 2.0, 8.0, 4096)])
def test_banded_frequencies(base, dims, factor, low, high, original):
    """Every band (kept, blended, divided), against the plain implementation; the blend meets the
    two others at the band's edges."""
    from pretrained_rstr_b200.parts.positions_rotary import banded_frequencies, split_frequencies
    got = banded_frequencies(base, dims, factor, low, high, original)
    plain = P.plain_frequencies(base, dims)
    want = P.banded_frequencies(plain, factor, low, high, original)
    assert got == pytest.approx(want, rel=1e-14)
    kinds = {("kept" if g == f else "divided" if g == pytest.approx(f / factor, rel=1e-14) else "blended")
             for g, f in zip(got, plain)}
    assert len(kinds) >= (3 if dims == 64 else 1)
    for edge, value in ((original / high, 1.0), (original / low, 1.0 / factor)):
        f = 2.0 * math.pi / edge
        for nudge in (1.0 - 1e-9, 1.0 + 1e-9):
            assert P.banded_frequencies([f * nudge], factor, low, high, original)[0] == \
                pytest.approx(f * value, rel=1e-6)
    hi, lo = split_frequencies(got, "cpu")
    assert torch.allclose(hi.double() + lo.double(), torch.tensor(got, dtype=torch.float64), rtol=1e-13)


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
    taps = []
    full = P.forward(ids, W, raw, taps=taps)
    assert len(taps) == 8 and full.shape == (30, 90) and float(full.abs().max()) < 7.0
    assert torch.allclose(P.forward(ids[:17], W, raw), full[:17], atol=1e-10)        # causal

    def moved(change_raw=None, change_w=None):
        r, w = copy.deepcopy(raw), dict(W)
        if change_raw:
            change_raw(r)
        if change_w:
            change_w(w)
        return float((P.forward(ids, w, r)[-1] - full[-1]).abs().max())

    assert moved(lambda r: r.__setitem__("residual_mult", 0.5)) > 1e-3
    assert moved(lambda r: r["loop"].__setitem__("times", 2)) > 1e-3
    assert moved(lambda r: r["layers"][1]["mixer"].__setitem__("softcap", 1.0)) > 1e-4
    assert moved(lambda r: r["layers"][1]["mixer"]["rot"].__delitem__("scaling")) > 1e-4
    assert moved(lambda r: r["layers"][0]["mixer"].__setitem__("decay", [0.5, 0.99])) > 1e-4
    for name in ("loop.in", "l1.mix.k.conv", "l1.mix.q.norm", "l2.mix.k.conv", "l1.norm2b", "l0.norm1b.b"):
        bend = 1.0 + 0.5 * torch.sin(torch.arange(W[name].numel(), dtype=torch.float64)).reshape(W[name].shape)
        assert moved(None, lambda w: w.__setitem__(name, w[name] * bend)) > 1e-4, name
