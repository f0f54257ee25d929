"""Gunulorn: a decoder whose blocks run their mixer and their feed-forward side by side, each on an RMS
norm of its own of the same stream, with two kinds of grouped-query attention in any order and a dense
or a mixture-of-experts feed-forward per layer (or none), and logits that are scaled, then soft-capped.

Mixers: *attention* (q, k and v pass a short causal convolution over time; no positions; a learned factor
per head on the scores and a learned sink per head; a layer may read an earlier layer's keys and values
with queries of its own) and *attention_2* (rotary positions in neighbouring pairs on q, k and on the
values, whose weighted sum is turned back by the query's position; a window beside the first tokens of
the sequence; one added to every softmax sum).

Feed-forward: dense, W_down act(W_up h + b) + b' with act a polynomial of normed powers (four learned
numbers); or silu-gated experts chosen by softmax score plus a correction, weighted by the chosen scores
over their sum, the last ``identity`` of which give back their input.

config.json: ``architecture`` "Gunulorn"; ``vocab``, ``width``; ``norm.eps``; ``logit_scale``;
``logit_softcap``; ``layers``: a list of {"type": "attention" | "attention_2", "mixer": {...}, "mlp":
{...} | null}.  attention gives heads, kv_heads, dim, vdim, scale, conv (taps) and optionally kv_from (the
layer whose keys and values it reads); attention_2 heads, kv_heads, dim, vdim, scale, rot {base, dims}
and mask {size, keep_first}; mlp is {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"},
"router": {"experts", "identity", "top"}}.

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.norm1``, ``norm2``,
``l<i>.mix.{q,k,v,o}``, ``l<i>.mix.{q,k,v}.conv``, ``temp``, ``sink``, ``l<i>.mlp.{up,down}``, ``up.b``,
``down.b``, ``act`` or ``l<i>.mlp.router``, ``correction``, ``e<k>.{gate,up,down}``: the tensor itself
carries the name (no ".weight")."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import ClassVar

from .dudatar import _need, _number, _positive_int
from .model_config import ConfigError, LayerCall, LayerSpec, ModelConfig, ModelSpec, PartSpec

LAYER_TYPES = ("attention", "attention_2")


def _count(d: dict, key: str, where: str, default: int = 0) -> int:
    """A whole number that may be zero, or absent."""
    value = d.get(key)
    if value is None:
        return default
    if isinstance(value, bool) or not isinstance(value, int) or value < 0:
        raise ConfigError(f"config.json: {where}.{key} {value!r} must be a whole number, zero or more")
    return value


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        _positive_int(mlp, "ff", where)
    elif kind == "moe":
        _positive_int(_need(mlp, "expert", where), "ff", where + ".expert")
        router = _need(mlp, "router", where)
        experts = _positive_int(router, "experts", where + ".router")
        router["identity"] = _count(router, "identity", where + ".router")
        if _positive_int(router, "top", where + ".router") > experts + router["identity"]:
            raise ConfigError(f"config.json: {where}.router: top exceeds experts and identity experts together")
    else:
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not 'dense' or 'moe'")


def _check_turns(mixer: dict, where: str) -> None:
    """Rotation and mask of attention_2."""
    rot = _need(mixer, "rot", where)
    dims = _need(rot, "dims", where + ".rot")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > mixer["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims {dims!r} must be even and at most {mixer['dim']}")
    if not _number(rot, "base", where + ".rot") > 0:
        raise ConfigError(f"config.json: {where}.rot.base must be positive")
    if mixer["vdim"] % 2:
        raise ConfigError(f"config.json: {where}.vdim {mixer['vdim']} must be even: values turn in pairs")
    mask = mixer.get("mask")
    if mask is not None:
        _positive_int(mask, "size", where + ".mask")
        mask["keep_first"] = _count(mask, "keep_first", where + ".mask")


@dataclass(frozen=True)
class GunulornConfig(ModelConfig):
    architecture: ClassVar[str] = "Gunulorn"

    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0
    layers: tuple = ()               # the config's layer entries, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "GunulornConfig":
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
            for key in ("heads", "dim", "vdim"):
                _positive_int(mixer, key, at)
            mixer.setdefault("kv_heads", mixer["heads"])        # (left out: every query head has its own)
            if mixer["heads"] % _positive_int(mixer, "kv_heads", at):
                raise ConfigError(f"config.json: {at}: heads is no multiple of kv_heads")
            _number(mixer, "scale", at)
            if kind == "attention_2":
                _check_turns(mixer, at)
            else:
                _count(mixer, "conv", at)
                j = mixer.get("kv_from")
                if j is not None:
                    if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
                        raise ConfigError(f"config.json: {at}.kv_from {j!r} must name an earlier layer")
                    other = layers[j]["mixer"]
                    if layers[j]["type"] != kind or other.get("kv_from") is not None:
                        raise ConfigError(f"config.json: {at}.kv_from: layer {j} has no keys and values of its own of this kind")
                    if any(other[key] != mixer[key] for key in ("heads", "kv_heads", "dim", "vdim")):
                        raise ConfigError(f"config.json: {at}.kv_from: layer {j} differs in heads or head sizes")
            _check_mlp(layer.get("mlp"), where + ".mlp")
        eps = _number(_need(raw, "norm", "the model"), "eps", "norm")
        if not eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        cap = raw.get("logit_softcap")
        if cap is not None and not _number(raw, "logit_softcap", "the model") >= 0:
            raise ConfigError("config.json: logit_softcap must not be negative")
        scale = _number(raw, "logit_scale", "the model") if raw.get("logit_scale") is not None else 1.0
        return cls(vocab=_positive_int(raw, "vocab", "the model"), width=_positive_int(raw, "width", "the model"), norm_eps=eps,
                   logit_scale=scale, logit_softcap=float(cap) if cap else 0.0, layers=tuple(layers))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out

    # ------------------------------------------------------------------ parts
    def _mixer(self, layer: dict) -> PartSpec:
        m = layer["mixer"]
        params = {"hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                  "value_dim": m["vdim"], "scale": float(m["scale"])}
        names = {"q": "q", "k": "k", "v": "v", "o": "o"}
        if layer["type"] == "attention":
            return PartSpec("attention", dict(params, conv_taps=m.get("conv") or 0, query_factor=True, sinks=True,
                                              borrows_kv=m.get("kv_from") is not None,
                                              names=dict(names, query_factor="temp", sinks="sink")))
        rot, mask = m["rot"], m.get("mask") or {}

        def turn(dims):
            return PartSpec("rotary", {"rotary_dim": dims, "theta": float(rot["base"]), "pairing": "interleaved"})

        return PartSpec("attention", dict(params, position=turn(rot["dims"]) if rot["dims"] else None, value_rotation=turn(m["vdim"]),
                                          window=mask.get("size", 0), keep_first=mask.get("keep_first", 0), sink_score=0.0,
                                          names=names))

    def _ffn(self, mlp):
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("poly_norm_mlp", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "eps": self.norm_eps,
                                              "names": {"up": "up", "down": "down", "act": "act"}})
        r = mlp["router"]
        return PartSpec("moe", {"hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "num_experts": r["experts"],
                                "identity": r["identity"], "top": r["top"], "activation": "silu_gated",
                                "router": "softmax_corrected"})

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm", {"eps": self.norm_eps})
        names = {"mixer": "mix", "ffn": "mlp", "input_norm": "norm1", "ffn_norm": "norm2"}
        layers = [LayerSpec(self._mixer(layer), self._ffn(layer.get("mlp")), norm, arrangement="parallel_two_norms", names=names)
                  for layer in self.layers]
        # a layer with kv_from reads the cache entry of the layer it names and writes none
        order = []
        for i, layer in enumerate(self.layers):
            j = layer["mixer"].get("kv_from") if layer["type"] == "attention" else None
            order.append(LayerCall(i, i if j is None else j, j is None))
        unread = tuple(rf"l{i}\.norm2" for i, layer in enumerate(self.layers) if layer.get("mlp") is None)
        return ModelSpec(
            self.vocab, self.width, tuple(layers), tuple(order), norm, tie_word_embeddings=False, weight_prefix="",
            names={"embed": "embed", "layers": "l{i}", "final_norm": "final.norm", "lm_head": "head"},
            logit_scale=self.logit_scale, logit_softcap=self.logit_softcap,
            name_rules=((r"\.weight$", ""), (r"\.bias$", ".b")), unread_names=unread)
