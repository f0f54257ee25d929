"""Tiny Gunulorn configurations for the tests; they differ from one another in every size, in the order
of the layers and in which options are there at all."""
from __future__ import annotations


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, identity, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def _conv(heads, kv_heads, dim, vdim, scale, conv, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _turned(heads, kv_heads, dim, vdim, scale, base, dims, size, keep_first):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims},
            "mask": {"size": size, "keep_first": keep_first}}


GUNULORN_TINY = {
    # a window first; values wider than keys and narrower; a reader of the second layer's keys and values with
    # another number of taps; experts of which a token takes one, identity experts more than experts
    "P": {
        "vocab": 180, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.7, "logit_softcap": 7.0,
        "layers": [
            {"type": "attention_2", "mlp": _moe(40, 2, 3, 1), "mixer": _turned(4, 2, 16, 32, 0.4, 1e4, 8, 20, 3)},
            {"type": "attention", "mlp": _dense(72), "mixer": _conv(4, 2, 24, 16, 0.3, 3)},
            {"type": "attention_2", "mlp": None, "mixer": _turned(2, 2, 24, 16, 0.35, 100.0, 24, 9, 1)},
            {"type": "attention", "mlp": _moe(24, 3, 1, 4), "mixer": _conv(4, 2, 24, 16, 0.5, 5, kv_from=1)},
        ]},
    # no cap on the logits and a scale of one; one tap; no identity experts; a window of one key, a window
    # without kept tokens; keys without a rotated part; sizes that are no power of two
    "Q": {
        "vocab": 301, "width": 96, "norm": {"eps": 1e-6},
        "layers": [
            {"type": "attention", "mlp": _moe(56, 5, 0, 2), "mixer": _conv(6, 3, 20, 12, 0.3, 1)},
            {"type": "attention_2", "mlp": _dense(104), "mixer": _turned(3, 1, 48, 16, 0.2, 5e5, 0, 33, 0)},
            {"type": "attention_2", "mlp": _moe(48, 1, 1, 1), "mixer": _turned(5, 5, 20, 10, 0.45, 3e3, 20, 1, 5)},
            {"type": "attention", "mlp": _dense(40), "mixer": _conv(2, 1, 36, 36, 0.2, 8)},
            {"type": "attention", "mlp": None, "mixer": _conv(6, 3, 20, 12, 0.6, 2, kv_from=0)},
        ]},
    # head sizes the tensor-core kernels take; two readers of one layer, one of them the layer right behind it
    "R": {
        "vocab": 384, "width": 128, "norm": {"eps": 1e-5}, "logit_scale": 1.5, "logit_softcap": 20.0,
        "layers": [
            {"type": "attention", "mlp": _dense(192), "mixer": _conv(8, 2, 64, 64, 0.125, 2)},
            {"type": "attention", "mlp": _moe(64, 8, 2, 3), "mixer": _conv(8, 2, 64, 64, 0.2, 6, kv_from=0)},
            {"type": "attention_2", "mlp": _moe(32, 10, 3, 5), "mixer": _turned(6, 3, 64, 64, 0.15, 1e4, 48, 40, 2)},
            {"type": "attention_2", "mlp": _dense(96), "mixer": _turned(2, 1, 32, 64, 0.2, 2.5e5, 16, 64, 17)},
            {"type": "attention", "mlp": _moe(64, 4, 4, 2), "mixer": _conv(8, 2, 64, 64, 0.125, 3, kv_from=0)},
        ]},
}


def gunulorn_config_dict(name: str) -> dict:
    import copy
    return dict(copy.deepcopy(GUNULORN_TINY[name]), architecture="Gunulorn")


def gunulorn_config(name: str):
    from tinyserve_b200.config import config_from_dict
    return config_from_dict(gunulorn_config_dict(name))


def decisive(folder: str, seed: int = 0, sharp: float = 6.0) -> str:
    """A random model made to show its parts.  With weights of 0.02 every router scores all experts alike
    (which of them a token takes would hang on the last bit of a sum) and every head looks at all keys
    alike; here the routers are ten times as large, queries and keys ``sharp`` times, and the factors on
    the heads' scores spread over [-1.2, 1.2] away from zero."""
    import os
    import torch
    from safetensors.torch import load_file, save_file
    path = os.path.join(folder, "model.safetensors")
    weights = load_file(path)
    g = torch.Generator().manual_seed(1000 + seed)
    for name in list(weights):
        w = weights[name]
        if name.endswith(".router"):
            w = w.float() * 10.0
        elif name.endswith((".mix.q", ".mix.k")):
            w = w.float() * sharp
        elif name.endswith((".mix.v", ".mix.o", ".mlp.up", ".mlp.down")):
            w = w.float() * 2.0
        elif name.endswith(".temp"):
            w = (0.4 + 0.8 * torch.rand(w.shape, generator=g)) * torch.sign(torch.rand(w.shape, generator=g) - 0.3)
        else:
            continue
        weights[name] = w.to(weights[name].dtype)
    save_file(weights, path)
    return folder


def make_gunulorn_dir(folder, name: str, seed: int = 0, sharp: float = 6.0) -> str:
    from tinyserve_b200.weights import write_random_model
    return decisive(write_random_model(gunulorn_config(name), str(folder), seed=seed), seed, sharp)


def random_gunulorn_config_dict(seed: int) -> dict:
    """A configuration drawn from a seed: sizes that are no power of two and no multiple of 16 among them,
    any order of layer kinds, readers of an earlier layer, layers without feed-forward, windows of one key
    and wider than the prompts, rotation over all, a part or none of a head."""
    import random
    r = random.Random(seed)
    even = lambda lo, hi: 2 * r.randint(lo // 2, hi // 2)
    width = 8 * r.randint(4, 14)
    layers, writers = [], []
    for i in range(r.randint(1, 6)):
        pick = r.random()
        if pick < 0.2:
            mlp = None
        elif pick < 0.55:
            mlp = _dense(r.choice([8, 4, 1]) * r.randint(2, 30))
        else:
            experts, identity = r.randint(1, 9), r.choice([0, 0, 1, 3, 6])
            mlp = _moe(8 * r.randint(2, 10), experts, identity, r.randint(1, experts + identity))
        if r.random() < 0.55:
            if writers and r.random() < 0.45:
                j = r.choice(writers)
                o = layers[j]["mixer"]
                mixer = _conv(o["heads"], o["kv_heads"], o["dim"], o["vdim"], r.choice([0.1, 0.3]), r.randint(1, 6), kv_from=j)
            else:
                kv = r.randint(1, 3)
                mixer = _conv(kv * r.randint(1, 3), kv, r.choice([7, 12, 16, 24, 40, 64]), r.choice([5, 8, 16, 36, 64, 80]),
                              r.choice([0.1, 0.3, 0.5]), r.randint(1, 8))
                writers.append(i)
            layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
        else:
            kv, dim = r.randint(1, 3), even(8, 72)
            mixer = _turned(kv * r.randint(1, 3), kv, dim, r.choice([2, 8, 16, 22, 40, 64, 80]), r.choice([0.1, dim ** -0.5, 0.4]),
                            r.choice([100.0, 1e4, 7e5]), r.choice([dim, even(2, dim), 0]), r.choice([1, 2, 7, 16, 17, 48, 500]),
                            r.choice([0, 0, 1, 4, 16, 21]))
            layers.append({"type": "attention_2", "mixer": mixer, "mlp": mlp})
    raw = {"architecture": "Gunulorn", "vocab": r.randint(50, 400), "width": width, "norm": {"eps": r.choice([1e-6, 1e-5, 1e-4])},
           "logit_scale": r.choice([1.0, 0.25, 3.0]), "layers": layers}
    if r.random() < 0.7:
        raw["logit_softcap"] = r.choice([5.0, 12.0, 30.0])
    return raw
