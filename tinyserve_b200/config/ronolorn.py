"""Ronolorn: a pre-norm decoder (layer norms with a weight and no bias) on several parallel residual streams joined
by hyper-connections, with scaled embeddings, three kinds of mixer in any order, a dense feed-forward per layer
(or none), and logits from the embedding table.

Mixers: *delta* (a matrix memory per head under the gated delta rule: q, k and v pass a short causal convolution
and silu, q and k are unit vectors shared by groups of heads, one decay and one write strength per head and token, the
output RMS-normed per head and gated by silu); *attention* (grouped-query attention over a window, biases on q, k, v
and the output, values of a head size of their own, the first rot.dims columns of q and k turned in neighbouring
pairs); *attention_2* (grouped-query attention over a window without a value projection: the values are the keys
as projected; q and k RMS-normed over all their heads at once, then turned in neighbouring pairs with frequencies
that may be stretched by the ramp rule; one added to every softmax sum).

Feed-forward: W_down relu(W_up h)^2.

config.json: ``architecture`` "Ronolorn"; ``vocab``, ``width``, ``streams``; ``norm.eps``; ``embedding.scale``; ``layers``: a
list of {"type": "delta" | "attention" | "attention_2", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}.  delta
gives heads, kv_heads, dim, vdim, conv (taps); the attentions heads, kv_heads, dim, vdim, scale, mask {size}, rot {base,
dims, scaling {factor, original, fast, slow} or none}.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1``, ``norm2``, ``l<i>.hc1.{in,mix,out}``,
``hc2.{in,mix,out}``, ``l<i>.mix.*``, ``l<i>.mlp.{up,down}``: the tensor itself carries the name (no ".weight"), a bias
is ".b"."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import ClassVar

from .babadra import _rot
from .dudatar import _need, _number, _positive_int
from .model_config import ConfigError, LayerCall, LayerSpec, ModelConfig, ModelSpec, PartSpec

LAYER_TYPES = ("delta", "attention", "attention_2")


@dataclass(frozen=True)
class RonolornConfig(ModelConfig):
    architecture: ClassVar[str] = "Ronolorn"

    vocab: int = 0
    width: int = 0
    streams: int = 1
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    layers: tuple = ()               # the config's layer entries, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "RonolornConfig":
        layers = copy.deepcopy(_need(raw, "layers", "the model"))
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not one of {LAYER_TYPES}")
            mixer = _need(layer, "mixer", where)
            at = where + ".mixer"
            for key in ("heads", "dim"):
                _positive_int(mixer, key, at)
            mixer.setdefault("kv_heads", mixer["heads"])        # (left out: every query head has its own)
            if mixer["heads"] % _positive_int(mixer, "kv_heads", at):
                raise ConfigError(f"config.json: {at}: heads is no multiple of kv_heads")
            if kind == "attention_2":
                mixer.setdefault("vdim", mixer["dim"])
            _positive_int(mixer, "vdim", at)
            if kind == "delta":
                _positive_int(mixer, "conv", at)
            else:
                _number(mixer, "scale", at)
                _rot(mixer, at, mixer["dim"], exact=False)
                if mixer.get("mask") is not None:
                    _positive_int(mixer["mask"], "size", at + ".mask")
                if kind == "attention_2" and mixer["vdim"] != mixer["dim"]:
                    raise ConfigError(f"config.json: {at}.vdim {mixer['vdim']} must equal dim {mixer['dim']}: the values are the keys")
            mlp = layer.get("mlp")
            if mlp is not None:
                if _need(mlp, "kind", where + ".mlp") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not 'dense'")
                _positive_int(mlp, "ff", where + ".mlp")
        eps = _number(_need(raw, "norm", "the model"), "eps", "norm")
        if not eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        embedding = raw.get("embedding") or {}
        scale = _number(embedding, "scale", "embedding") if embedding.get("scale") is not None else 1.0
        return cls(vocab=_positive_int(raw, "vocab", "the model"), width=_positive_int(raw, "width", "the model"),
                   streams=_positive_int(raw, "streams", "the model"), norm_eps=eps, embedding_scale=scale, layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "layers": copy.deepcopy(list(self.layers))}

    # ------------------------------------------------------------------ parts
    def _mixer(self, layer: dict) -> PartSpec:
        m, w, eps = layer["mixer"], self.width, self.norm_eps
        names = {"q": "q", "k": "k", "v": "v", "o": "o"}
        if layer["type"] == "delta":
            return PartSpec("gated_delta_rule", {
                "hidden_size": w, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
                "conv_taps": m["conv"], "eps": eps, "names": dict(names, g="g", a="a", b="b")})
        rot, mask = m.get("rot"), m.get("mask") or {}
        position = None
        if rot and rot["dims"]:
            position = PartSpec("rotary", {"rotary_dim": rot["dims"], "theta": float(rot["base"]), "pairing": "interleaved",
                                           "scaling": dict(rot["scaling"]) if rot.get("scaling") else None})
        params = {"hidden_size": w, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                  "scale": float(m["scale"]), "position": position, "window": mask.get("size", 0), "bias": True}
        if layer["type"] == "attention":
            return PartSpec("attention", dict(params, out_bias=True, names=names))
        return PartSpec("attention", dict(params, tied_values=True, joint_norm=True, norm_eps=eps, sink_score=0.0,
                                          names=dict(names, q_norm="q.norm", k_norm="k.norm")))

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("layernorm", {"eps": self.norm_eps})
        names = {"mixer": "mix", "ffn": "mlp", "input_norm": "norm1", "ffn_norm": "norm2", "mixer_streams": "hc1", "ffn_streams": "hc2"}
        layers = []
        for layer in self.layers:
            ffn = None
            if layer.get("mlp") is not None:
                ffn = PartSpec("plain_mlp", {"hidden_size": self.width, "intermediate_size": layer["mlp"]["ff"],
                                             "activation": "relu_squared", "names": {"up": "up", "down": "down"}})
            layers.append(LayerSpec(self._mixer(layer), ffn, norm, arrangement="hyper_connections", names=names,
                                    options={"streams": self.streams}))
        order = tuple(LayerCall(i, i) for i in range(len(layers)))
        # a layer without a feed-forward has no use for its norm and its coefficients, should a checkpoint hold them
        unread = tuple(rf"l{i}\.(norm2|hc2\.(in|mix|out))" for i, layer in enumerate(self.layers) if layer.get("mlp") is None)
        return ModelSpec(
            self.vocab, self.width, tuple(layers), order, norm, tie_word_embeddings=True, weight_prefix="",
            names={"embed": "embed", "layers": "l{i}", "final_norm": "final.norm"}, embedding_scale=self.embedding_scale,
            streams=self.streams, name_rules=((r"\.weight$", ""), (r"\.bias$", ".b")), unread_names=unread)
