"""Gunulorn off the device: the configuration reader, the run order and cache entries it makes, the
checkpoint's tensor names, and the plain implementation against closed forms of its own mechanisms."""
import math

import pytest
import torch

import plain_gunulorn as plain
from gunulorn_configs import (GUNULORN_TINY, gunulorn_config, gunulorn_config_dict, make_gunulorn_dir,
                              random_gunulorn_config_dict)


def test_registry_reads_the_architecture_key_and_round_trips():
    from tinyserve_b200.config import GunulornConfig, architecture_of, config_from_dict
    raw = gunulorn_config_dict("P")
    assert architecture_of(raw) == "Gunulorn"
    cfg = config_from_dict(raw)
    assert isinstance(cfg, GunulornConfig) and cfg.vocab == 180 and cfg.width == 64 and cfg.logit_scale == 0.7
    assert config_from_dict(cfg.to_dict()) == cfg
    for seed in range(30):
        drawn = config_from_dict(random_gunulorn_config_dict(seed))
        assert config_from_dict(drawn.to_dict()) == drawn


@pytest.mark.parametrize("damage,text", [
    (lambda r: r.pop("width"), "width"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r["norm"].update(eps=0), "eps"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["layers"][0].update(type="attention_3"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].update(vdim=31), "vdim"),
    (lambda r: r["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda r: r["layers"][1]["mixer"].update(conv=-2), "conv"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(vdim=24), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(heads=2), "kv_from"),
    (lambda r: r["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda r: r["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(identity=1.5), "identity"),
    (lambda r: r.update(logit_softcap=-1.0), "softcap"),
])
def test_a_damaged_configuration_is_refused(damage, text):
    from tinyserve_b200.config import ConfigError, config_from_dict
    raw = gunulorn_config_dict("P")
    damage(raw)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(raw)


def test_run_order_caches_and_states():
    from tinyserve_b200.parts import build_model
    p = build_model(gunulorn_config("P"))
    # the last layer reads the second one's entry and writes none
    assert [(c.layer, c.cache, c.writes_cache) for c in p.calls] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 1, False)]
    kinds = [(g.kind, g.num_kv_heads, g.head_dim, g.window, g.keep_first) for g in p.cache_groups]
    assert sorted(kinds) == [("full", 2, 32, 0, 0), ("window", 2, 32, 9, 1), ("window", 2, 32, 20, 3)]      # rows as wide as the wider, in sixteens
    # convolution state: the writer keeps q, k and v rows, the reader its queries' only
    assert [tuple(s.shape) for s in p.state_entries] == [(2, 4 * 24 + 2 * 24 + 2 * 16), (4, 4 * 24)]
    assert [c.state for c in p.calls] == [-1, 0, -1, 1]
    assert p.blocks[2].ffn is None and p.lm_head is not None and p.spec.logit_softcap == 7.0
    q = build_model(gunulorn_config("Q"))
    assert q.spec.logit_scale == 1.0 and q.spec.logit_softcap == 0.0
    assert [tuple(s.shape) for s in q.state_entries] == [(7, 4 * 36), (1, 6 * 20)], "one tap needs no state"
    r = build_model(gunulorn_config("R"))
    assert [(c.cache, c.writes_cache) for c in r.calls] == [(0, True), (0, False), (1, True), (2, True), (0, False)]
    assert p.capturable and q.capturable and r.capturable


def test_checkpoint_names(tmp_path):
    from safetensors import safe_open
    folder = make_gunulorn_dir(tmp_path, "P", seed=3)
    with safe_open(f"{folder}/model.safetensors", "pt") as fh:
        names = set(fh.keys())
        shapes = {k: tuple(fh.get_slice(k).get_shape()) for k in names}
    for name in ("embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mix.k", "l0.mix.v", "l0.mix.o",
                 "l0.mlp.router", "l0.mlp.correction", "l0.mlp.e1.gate", "l0.mlp.e1.up", "l0.mlp.e1.down", "l1.mix.q.conv",
                 "l1.mix.k.conv", "l1.mix.v.conv", "l1.mix.temp", "l1.mix.sink", "l1.mlp.up", "l1.mlp.up.b", "l1.mlp.down",
                 "l1.mlp.down.b", "l1.mlp.act", "l3.mix.q.conv", "l3.mix.temp", "l3.mix.sink"):
        assert name in names, name
    for name in ("l0.mix.q.conv", "l0.mix.sink", "l0.mlp.e2.up", "l2.norm2", "l3.mix.k", "l3.mix.v", "l3.mix.k.conv"):
        assert name not in names, name
    assert not any(n.endswith((".weight", ".bias")) for n in names)
    assert shapes["l0.mix.v"] == (2 * 32, 64) and shapes["l0.mix.o"] == (64, 4 * 32) and shapes["l0.mlp.router"] == (5, 64)
    assert shapes["l1.mix.q.conv"] == (4 * 24, 3) and shapes["l1.mix.v.conv"] == (2 * 16, 3) and shapes["l3.mix.q.conv"] == (4 * 24, 5)
    assert shapes["l1.mlp.act"] == (4,) and shapes["l1.mlp.up.b"] == (72,) and shapes["l1.mix.temp"] == (4,)
    # a checkpoint may hold the norm of a feed-forward that a layer does not have
    from tinyserve_b200.parts import build_model
    from tinyserve_b200.weights.loader import check_checkpoint
    index = {k: ("f", v, "BF16") for k, v in shapes.items()}
    index["l2.norm2"] = ("f", (64,), "BF16")
    check_checkpoint(build_model(gunulorn_config("P")), index)


def test_parts_refuse_what_they_do_not_combine():
    from tinyserve_b200.config import PartSpec
    from tinyserve_b200.parts import Attention, MixtureOfExperts
    turn = lambda dims, pairing="interleaved": PartSpec("rotary", {"rotary_dim": dims, "theta": 1e4, "pairing": pairing})
    for bad in (dict(conv_taps=9), dict(conv_taps=2, position=turn(8)), dict(value_rotation=turn(8)),
                dict(value_rotation=turn(16, "half")), dict(sinks=True, sink_score=0.0), dict(value_rotation=turn(16), chunk=4)):
        with pytest.raises(ValueError):
            Attention(32, 4, 2, 16, **bad)
    for bad in (dict(identity=2), dict(identity=2, router="softmax_corrected", activation="relu_squared"),
                dict(identity=-1, router="softmax_corrected", activation="silu_gated")):
        with pytest.raises(ValueError):
            MixtureOfExperts(32, 16, 4, 2, **bad)
    with pytest.raises(ValueError):
        MixtureOfExperts(32, 16, 4, 7, router="softmax_corrected", activation="silu_gated", identity=2)


# ----------------------------------------------------------------------------- the plain implementation itself
@pytest.mark.parametrize("name", sorted(GUNULORN_TINY))
def test_plain_model_is_causal_and_sees_far_tokens(name, tmp_path):
    cfg, W = plain.load_folder(make_gunulorn_dir(tmp_path, name, seed=1))
    ids = torch.randint(0, cfg["vocab"], (50,), generator=torch.Generator().manual_seed(5)).tolist()
    full, layers = plain.forward(cfg, W, ids, return_layers=True)
    assert layers.shape == (len(cfg["layers"]), 50, cfg["width"])
    assert (plain.logits(cfg, W, ids[:31]) - full[:31]).abs().max() < 1e-9, "a position does not see what follows"
    other = list(ids)
    other[0] = (ids[0] + 1) % cfg["vocab"]
    assert (plain.logits(cfg, W, other)[-1] - full[-1]).abs().max() > 1e-6, "the last position sees the first token"
    if cfg.get("logit_softcap"):
        assert full.abs().max() < cfg["logit_softcap"]


def test_plain_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(0)
    draw = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # convolution: the last tap is the token itself, nothing before the first row
    u, w = draw(6, 3), draw(3, 4)
    y = plain.past_convolution(u, w)
    assert (y[0] - w[:, 3] * u[0]).abs().max() < 1e-12
    assert (y[4] - (w[:, 3] * u[4] + w[:, 2] * u[3] + w[:, 1] * u[2] + w[:, 0] * u[1])).abs().max() < 1e-12
    assert (plain.past_convolution(u[:2], w) - y[:2]).abs().max() < 1e-12
    # a turn there and back is nothing; a turn keeps every pair's length
    v, pos, rot = draw(7, 2, 10), torch.arange(7) + 3, {"base": 50.0, "dims": 4}
    t = plain.rotate_values(v, pos, rot)
    assert (plain.rotate_values(t, pos, rot, back=True) - v).abs().max() < 1e-12
    assert (t.view(7, 2, 5, 2).pow(2).sum(-1) - v.view(7, 2, 5, 2).pow(2).sum(-1)).abs().max() < 1e-12
    r = plain.rotate_first(v, pos, rot)
    assert (r[..., 4:] == v[..., 4:]).all() and (r[..., :4] - v[..., :4]).abs().max() > 0.1
    # attention to a token's own turned value alone gives that value back
    assert (plain.rotate_values(plain.rotate_values(v[3:4], pos[3:4], rot), pos[3:4], rot, back=True) - v[3:4]).abs().max() < 1e-12
    # the sink: weights that sum to less than one by exactly its share
    s = draw(5, 5)
    p = plain.softmax_with_sink(s, plain.causal_mask(5), torch.tensor(0.7, dtype=torch.float64))
    share = torch.tensor([math.exp(0.7) / (math.exp(0.7) + float(s[i, :i + 1].exp().sum())) for i in range(5)], dtype=torch.float64)
    assert (1 - p.sum(-1) - share).abs().max() < 1e-12
    # the window: the query's own key and size - 1 before it, and the first keys
    m = plain.window_mask(9, 3, 2)
    assert m[8].tolist() == [True, True, False, False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 8
    assert plain.window_mask(4, 1, 0).tolist() == torch.eye(4, dtype=torch.bool).tolist()
    # the polynomial: on a row of ones every normed power is one
    one = torch.ones(1, 6, dtype=torch.float64)
    assert (plain.poly_norm(one, torch.tensor([0.5, 2.0, -1.0, 0.25], dtype=torch.float64), 0.0) - 1.75).abs().max() < 1e-12
    # the router: a correction moves the choice and not the weights
    h = draw(4, 5)
    W = {"router": draw(6, 5), "correction": torch.tensor([0.0, 0, 0, 0, 9, 0], dtype=torch.float64)}
    idx, wt = plain.route(h, W, "", {"top": 2})
    sc = torch.softmax(h @ W["router"].T, -1)
    assert (idx[:, 0] == 4).all() and (wt.sum(-1) - 1).abs().max() < 1e-12
    assert (wt[:, 0] / wt[:, 1] - sc.gather(1, idx)[:, 0] / sc.gather(1, idx)[:, 1]).abs().max() < 1e-9
    # identity experts alone: the output is the input
    W["correction"] = torch.tensor([0.0, 0, 0, 0, 9, 9], dtype=torch.float64)
    assert (plain.experts(h, W, "", {"router": {"experts": 4, "identity": 2, "top": 2}}) - h).abs().max() < 1e-12
