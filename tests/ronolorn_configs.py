"""Tiny Ronolorn configurations for the tests; they differ from one another in every size, in the number of
streams, in the order of the layers and in which options are there at all."""
from __future__ import annotations


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def _window(heads, kv_heads, dim, vdim, scale, base, dims, size, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "mask": {"size": size}}


def _tied(heads, kv_heads, dim, scale, base, dims, size, scaling=None):
    return _window(heads, kv_heads, dim, dim, scale, base, dims, size, scaling)


RONOLORN_TINY = {
    # three streams; a window first; keys wider than values in the memory, values wider than keys in the window
    # layer; a stretched rotation whose ramp lies inside the pairs
    "P": {
        "vocab": 180, "width": 64, "streams": 3, "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0},
        "layers": [
            {"type": "attention", "mlp": _dense(72), "mixer": _window(4, 2, 16, 32, 0.4, 1e4, 8, 20)},
            {"type": "delta", "mlp": _dense(40), "mixer": _delta(4, 2, 20, 12, 3)},
            {"type": "attention_2", "mlp": _dense(56), "mixer": _tied(6, 2, 24, 0.5, 50.0, 24, 9, (3.0, 64, 8.0, 0.5))},
            {"type": "delta", "mlp": None, "mixer": _delta(3, 3, 12, 40, 5)},
        ]},
    # one stream; one tap; a window of one key; no rotation at all, and no stretching; sizes that are no power of two
    "Q": {
        "vocab": 301, "width": 96, "streams": 1, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
        "layers": [
            {"type": "delta", "mlp": _dense(104), "mixer": _delta(6, 2, 36, 10, 1)},
            {"type": "attention_2", "mlp": None, "mixer": _tied(3, 1, 48, 0.3, 3e3, 20, 33)},
            {"type": "attention", "mlp": _dense(44), "mixer": _window(5, 5, 20, 12, 0.45, 3e3, 0, 1)},
            {"type": "attention", "mlp": _dense(40), "mixer": _window(2, 1, 36, 36, 0.2, 700.0, 36, 50, (2.0, 128, 32.0, 1.0))},
        ]},
    # five streams (more than the vector kernel keeps in registers); head sizes the tensor-core kernels take; a memory whose
    # heads are spread over several blocks; one query/key head for all
    "R": {
        "vocab": 384, "width": 128, "streams": 5, "norm": {"eps": 1e-5}, "embedding": {"scale": 11.0},
        "layers": [
            {"type": "attention_2", "mlp": _dense(192), "mixer": _tied(8, 2, 64, 0.2, 1e4, 32, 40, (4.0, 256, 16.0, 2.0))},
            {"type": "delta", "mlp": _dense(64), "mixer": _delta(4, 1, 32, 48, 4)},
            {"type": "attention", "mlp": _dense(96), "mixer": _window(6, 3, 64, 64, 0.15, 2.5e5, 64, 64)},
            {"type": "delta", "mlp": _dense(128), "mixer": _delta(2, 2, 64, 80, 2)},
        ]},
}


def ronolorn_config_dict(name: str) -> dict:
    import copy
    return dict(copy.deepcopy(RONOLORN_TINY[name]), architecture="Ronolorn")


def ronolorn_config(name: str):
    from tinyserve_b200.config import config_from_dict
    return config_from_dict(ronolorn_config_dict(name))


def decisive(folder: str, seed: int = 0, sharp: float = 6.0) -> str:
    """A random model made to show its parts.  With weights of 0.02 every head looks at all keys alike and a memory
    forgets within two tokens; here queries and keys are ``sharp`` times as large (the normed ones by their norm's
    weights), biases are large, the memories fade slowly and write in shares far from one half, and the streams'
    coefficients differ from stream to stream (a mix that is transposed, or a stream left out, shows)."""
    import os
    import torch
    from safetensors.torch import load_file, save_file
    path = os.path.join(folder, "model.safetensors")
    weights = load_file(path)
    g = torch.Generator().manual_seed(1000 + seed)
    uniform = lambda shape, lo, hi: lo + (hi - lo) * torch.rand(shape, generator=g)
    for name in list(weights):
        w = weights[name]
        if name.endswith((".mix.q", ".mix.k")) and name + ".conv" not in weights:
            w = w.float() * sharp
        elif name.endswith((".q.norm", ".k.norm")):
            w = w.float() * (sharp / 4) ** 0.5
        elif name.endswith((".q.b", ".k.b", ".v.b", ".o.b")):
            w = w.float() * 10.0
        elif name.endswith((".mix.v", ".mix.o", ".mlp.up", ".mlp.down", ".mix.g")):
            w = w.float() * 3.0
        elif name.endswith((".mix.a", ".mix.b")):
            w = w.float() * 8.0
        elif name.endswith(".A_log"):
            w = uniform(w.shape, -5.0, -1.5)
        elif name.endswith((".hc1.in", ".hc2.in", ".hc1.out", ".hc2.out")):
            w = uniform(w.shape, -0.4, 1.2)
        elif name.endswith((".hc1.mix", ".hc2.mix")):
            n = w.shape[0]
            w = 0.8 * torch.eye(n) + uniform(w.shape, -0.5, 0.5) / n ** 0.5
        else:
            continue
        weights[name] = w.to(weights[name].dtype)
    save_file(weights, path)
    return folder


def make_ronolorn_dir(folder, name: str, seed: int = 0, sharp: float = 6.0) -> str:
    from tinyserve_b200.weights import write_random_model
    return decisive(write_random_model(ronolorn_config(name), str(folder), seed=seed), seed, sharp)


def random_ronolorn_config_dict(seed: int) -> dict:
    """A configuration drawn from a seed: sizes that are no power of two and no multiple of 16 among them, any order
    of layer kinds, layers without feed-forward, windows of one key and wider than the prompts, rotation over all, a
    part or none of a head, stretched or not."""
    import random
    r = random.Random(seed)
    even = lambda lo, hi: 2 * r.randint(lo // 2, hi // 2)
    layers = []
    for i in range(r.randint(1, 6)):
        mlp = None if r.random() < 0.2 else _dense(r.choice([8, 4, 1]) * r.randint(2, 30))
        kind = r.choice(["delta", "delta", "attention", "attention_2"])
        kv = r.randint(1, 3)
        heads = kv * r.randint(1, 3)
        if kind == "delta":
            mixer = _delta(heads, kv, r.choice([4, 7, 12, 20, 32, 36, 64]), r.choice([1, 5, 8, 18, 33, 64, 80]), r.randint(1, 8))
        else:
            dim = even(8, 72)
            dims = r.choice([dim, even(2, dim), 0])
            scaling = (r.choice([2.0, 5.0, 1.5]), r.choice([32, 300, 4096]), r.choice([32.0, 6.0]), r.choice([1.0, 0.25])) if r.random() < 0.5 else None
            size, scale, base = r.choice([1, 2, 7, 16, 17, 48, 500]), r.choice([0.1, dim ** -0.5, 0.4]), r.choice([100.0, 1e4, 7e5])
            if kind == "attention":
                mixer = _window(heads, kv, dim, r.choice([2, 7, 16, 22, 40, 64, 80]), scale, base, dims, size, scaling)
            else:
                mixer = _tied(heads, kv, dim, scale, base, dims, size, scaling)
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Ronolorn", "vocab": r.randint(50, 400), "width": r.choice([8, 8, 1]) * r.randint(8, 14) + 40,
            "streams": r.choice([1, 2, 3, 4, 6]), "norm": {"eps": r.choice([1e-6, 1e-5, 1e-4])},
            "embedding": {"scale": r.choice([1.0, 0.5, 8.0])}, "layers": layers}
