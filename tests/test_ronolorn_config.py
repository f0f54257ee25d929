"""Ronolorn off the device: the configuration reader, the caches and states it makes, the checkpoint's tensor
names, and the plain implementation against closed forms of its own mechanisms."""
import math

import pytest
import torch

import plain_ronolorn as plain
from ronolorn_configs import RONOLORN_TINY, make_ronolorn_dir, random_ronolorn_config_dict, ronolorn_config, ronolorn_config_dict


def test_registry_reads_the_architecture_key_and_round_trips():
    from tinyserve_b200.config import RonolornConfig, architecture_of, config_from_dict
    raw = ronolorn_config_dict("P")
    assert architecture_of(raw) == "Ronolorn"
    cfg = config_from_dict(raw)
    assert isinstance(cfg, RonolornConfig) and cfg.vocab == 180 and cfg.width == 64 and cfg.streams == 3 and cfg.embedding_scale == 5.0
    assert config_from_dict(cfg.to_dict()) == cfg
    for seed in range(30):
        drawn = config_from_dict(random_ronolorn_config_dict(seed))
        assert config_from_dict(drawn.to_dict()) == drawn


@pytest.mark.parametrize("damage,text", [
    (lambda r: r.pop("width"), "width"),
    (lambda r: r.pop("streams"), "streams"),
    (lambda r: r.update(streams=0), "streams"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r["norm"].update(eps=0), "eps"),
    (lambda r: r["embedding"].update(scale="big"), "scale"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["layers"][0].update(type="attention_3"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].update(dim=0), "dim"),
    (lambda r: r["layers"][2]["mixer"].update(vdim=16), "vdim"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].update(factor=-1.0), "factor"),
    (lambda r: r["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda r: r["layers"][1]["mlp"].pop("ff"), "ff"),
])
def test_a_damaged_configuration_is_refused(damage, text):
    from tinyserve_b200.config import ConfigError, config_from_dict
    raw = ronolorn_config_dict("P")
    damage(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_caches_states_and_streams():
    from tinyserve_b200.parts import build_model
    p = build_model(ronolorn_config("P"))
    assert p.spec.streams == 3 and p.lm_head is None and p.capturable and p.blocks[3].ffn is None
    kinds = [(g.kind, g.num_kv_heads, g.head_dim, g.window) for g in p.cache_groups]
    assert sorted(kinds) == [("window", 2, 32, 9), ("window", 2, 32, 20)]      # rows as wide as the wider size, in sixteens
    # a memory per head, and the convolution's last inputs of q, k and v
    assert [tuple(s.shape) for s in p.state_entries] == [(4, 20, 12), (2, 2 * 2 * 20 + 4 * 12), (3, 12, 40), (4, 2 * 3 * 12 + 3 * 40)]
    assert all(s.dtype == "float32" for s in p.state_entries)
    q = build_model(ronolorn_config("Q"))
    assert [tuple(s.shape) for s in q.state_entries] == [(6, 36, 10)], "one tap needs no state"
    assert q.blocks[2].mixer.position is None and q.blocks[1].mixer.v_size == 0
    assert sorted(g.window for g in q.cache_groups) == [1, 33, 50]


def test_streams_are_the_business_of_every_layer():
    import dataclasses
    from tinyserve_b200.parts import DecoderModel
    spec = ronolorn_config("P").model_spec()
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(dataclasses.replace(spec, streams=2))
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(dataclasses.replace(spec, streams=0))


def test_checkpoint_names(tmp_path):
    from safetensors import safe_open
    folder = make_ronolorn_dir(tmp_path, "P", seed=3)
    with safe_open(f"{folder}/model.safetensors", "pt") as fh:
        names = {k: tuple(fh.get_slice(k).get_shape()) for k in fh.keys()}
    assert names["embed"] == (180, 64) and names["final.norm"] == (64,) and "head" not in names
    assert names["l0.mix.q.b"] == (64,) and names["l0.mix.v"] == (64, 64) and names["l0.mix.o.b"] == (64,)
    assert names["l1.mix.q.conv"] == (40, 3) and names["l1.mix.v.conv"] == (48, 3) and names["l1.mix.a"] == (4, 64)
    assert names["l1.mix.A_log"] == (4,) and names["l1.mix.dt_bias"] == (4,) and names["l1.mix.norm"] == (12,)
    assert names["l2.mix.q.norm"] == (144,) and names["l2.mix.k.norm"] == (48,)
    assert "l2.mix.v" not in names and "l2.mix.o.b" not in names
    assert names["l1.hc2.mix"] == (3, 3) and names["l3.hc1.in"] == (3,)
    assert not any(k.startswith(("l3.mlp", "l3.norm2", "l3.hc2")) for k in names)


def test_what_a_layer_without_feed_forward_does_not_read_may_be_in_the_checkpoint(tmp_path):
    from safetensors.torch import load_file, save_file
    from tinyserve_b200.parts import build_model
    from tinyserve_b200.weights.loader import WeightError, load_weights
    folder = make_ronolorn_dir(tmp_path, "P", seed=3)
    path = f"{folder}/model.safetensors"
    w = load_file(path)
    w.update({"l3.norm2": torch.ones(64), "l3.hc2.mix": torch.eye(3), "l3.hc2.in": torch.ones(3)})
    save_file(w, path)
    load_weights(build_model(ronolorn_config("P")), folder, torch.float32, "cpu")
    w["l3.mlp.up"] = torch.ones(2, 2)
    save_file(w, path)
    with pytest.raises(WeightError, match="l3.mlp.up"):
        load_weights(build_model(ronolorn_config("P")), folder, torch.float32, "cpu")


# ----------------------------------------------------------------------------- the plain implementation
def test_a_memory_gives_back_what_was_written_and_replaces_it():
    """With orthogonal keys, no fading and full strength the memory is a dictionary; a second write under a key
    replaces the first; half a strength goes half the way."""
    eye = torch.eye(4, dtype=torch.float64)
    v = torch.randn(4, 3, dtype=torch.float64)
    keys = eye[[0, 1, 0, 1]]
    one = torch.ones(4, dtype=torch.float64)
    out, S = plain.delta_memory(eye[[0, 0, 1, 0]], keys, v, one, one)
    assert torch.allclose(out, torch.stack([v[0], v[0], v[1], v[2]]))
    assert torch.allclose(S[:2], v[2:]) and S[2:].abs().max() == 0
    out, _ = plain.delta_memory(eye[[0, 0, 0, 0]], eye[[0, 0, 0, 0]], v[:1].repeat(4, 1), one, 0.5 * one)
    assert torch.allclose(out, v[:1] * torch.tensor([[0.5], [0.75], [0.875], [0.9375]], dtype=torch.float64))
    out, _ = plain.delta_memory(eye[[0, 0, 0, 0]], eye[[0, 1, 1, 1]], v, 0.5 * one, one)
    assert torch.allclose(out, v[:1] * torch.tensor([[1.0], [0.5], [0.25], [0.125]], dtype=torch.float64))


def test_a_stretched_rotation_keeps_fast_pairs_and_slows_the_others():
    rot = {"base": 100.0, "dims": 32, "scaling": {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 0.5}}
    f, magnitude = plain.pair_frequencies(rot)
    g, one = plain.pair_frequencies({"base": 100.0, "dims": 32})
    ratio = f / g
    assert one == 1.0 and abs(magnitude - (0.1 * math.log(4.0) + 1)) < 1e-12
    assert abs(ratio[0] - 1) < 1e-12 and (ratio[1:] <= ratio[:-1] + 1e-12).all() and 0.25 <= ratio[-1] < 0.9
    from tinyserve_b200.parts.rotary import Rotary
    cos, sin = Rotary.tables(32, 100.0, 50, ("ramp", 4.0, 256.0, 8.0, 0.5))
    a = torch.arange(50, dtype=torch.float64)[:, None] * f[None]
    assert (cos.double() - a.cos() * magnitude).abs().max() < 1e-6 and (sin.double() - a.sin() * magnitude).abs().max() < 1e-6


def test_one_more_in_the_softmax_sum_and_the_window():
    s = torch.randn(5, 5, dtype=torch.float64)
    seen = plain.window_mask(5, 2)
    assert [int(x) for x in seen.sum(-1)] == [1, 2, 2, 2, 2] and not seen[4, 2] and seen[4, 3]
    p = plain.softmax_over(s, seen, True)
    e = torch.exp(s) * seen
    assert torch.allclose(p, e / (1 + e.sum(-1, keepdim=True)))
    assert torch.allclose(plain.softmax_over(s, seen, False).sum(-1), torch.ones(5, dtype=torch.float64))


def test_streams_mix_from_to():
    X = torch.randn(2, 3, 4, dtype=torch.float64)
    y = torch.randn(3, 4, dtype=torch.float64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 5.0]], dtype=torch.float64)
    out = torch.tensor([0.5, -1.0], dtype=torch.float64)
    new = plain.streams_out(X, y, mix, out)
    assert torch.allclose(new[0], X[0] + 3 * X[1] + 0.5 * y) and torch.allclose(new[1], 2 * X[0] + 5 * X[1] - y)
    assert torch.allclose(plain.streams_in(X, out), 0.5 * X[0] - X[1])


@pytest.mark.parametrize("name", sorted(RONOLORN_TINY))
def test_the_plain_model_is_causal(name, tmp_path):
    folder = make_ronolorn_dir(tmp_path, name, seed=1)
    cfg, W = plain.load_folder(folder)
    ids = [(7 * i + 3) % cfg["vocab"] for i in range(40)]
    whole = plain.logits(cfg, W, ids)
    assert torch.isfinite(whole).all()
    assert (plain.logits(cfg, W, ids[:23]) - whole[:23]).abs().max() < 1e-9 * whole.abs().max()
