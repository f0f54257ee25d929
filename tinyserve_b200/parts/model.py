"""The decoder stack: embedding, blocks in a run order that is data, final norm, logits.

tinyserve's ``Model`` (serve.py:1195-1263): x = embed_tokens[ids]; the layers; the last
residual add with the final norm; logits = hidden @ W.T with W the embedding table when
``tie_word_embeddings`` else ``lm_head``.  Here only the rows whose logits are wanted go
through the final norm and the vocabulary projection, and logits are returned in 32-bit."""
from __future__ import annotations

from dataclasses import dataclass

from ..config.model_config import ModelConfig, ModelSpec
from ..kernels import ops
from .base import CacheSpec, ParamSpec, Part, StateSpec, build_norm, build_position_encoding, build_stream_op
from .block import add_and_norm, build_block


class Embedding(Part):
    capturable = True

    def __init__(self, vocab_size, hidden_size):
        super().__init__()
        self.vocab_size, self.hidden_size = vocab_size, hidden_size

    def param_specs(self):
        return {"weight": ParamSpec((self.vocab_size, self.hidden_size))}


class LMHead(Part):
    capturable = True

    def __init__(self, vocab_size, hidden_size):
        super().__init__()
        self.vocab_size, self.hidden_size = vocab_size, hidden_size

    def param_specs(self):
        return {"weight": ParamSpec((self.vocab_size, self.hidden_size))}


@dataclass(frozen=True)
class BoundCall:
    """A run-order entry resolved against the model: which block runs, which cache
    entry and which state entry (-1: none) its mixer uses."""

    layer: int
    cache: int
    state: int
    writes_cache: bool
    before: tuple = ()      # (stream operation, argument) pairs that run right before the block
    # every state entry of the call, by name: ((name, index), ...).  A mixer's one state has the name
    # ""; a mixer made of branches names a branch's states "<branch>" and "<branch>.<name>"; a block's
    # own states (those of its ``state_specs``) start with "block."
    states: tuple = ()

    def state_of(self, name: str) -> int:
        for key, index in self.states:
            if key == name:
                return index
        raise KeyError(f"the call has no state {name!r}; it has {[k for k, _ in self.states]}")

    def scoped(self, prefix: str) -> "BoundCall":
        """The call as the part that lives under ``prefix`` sees it: its states without the prefix."""
        states = tuple((key[len(prefix) + 1:] if key != prefix else "", index) for key, index in self.states
                       if key == prefix or key.startswith(prefix + "."))
        return BoundCall(self.layer, self.cache, _one_state(states), self.writes_cache, self.before, states)


def _one_state(states) -> int:
    """``BoundCall.state``: the mixer's state named "", or its only state, else -1."""
    own = [(key, index) for key, index in states if not key.startswith("block.")]
    return dict(own).get("", own[0][1] if len(own) == 1 else -1)


@dataclass(frozen=True)
class CacheEntryInfo:
    spec: CacheSpec
    group: int           # index into DecoderModel.cache_groups
    index_in_group: int


class DecoderModel(Part):
    def __init__(self, spec: ModelSpec):
        super().__init__()
        self.spec = spec
        self.vocab_size, self.hidden_size = spec.vocab_size, spec.hidden_size
        self.embed_tokens = Embedding(spec.vocab_size, spec.hidden_size)
        self.blocks = [build_block(layer, spec.hidden_size) for layer in spec.layers]
        self.norm = build_norm(spec.final_norm, spec.hidden_size)
        self.lm_head = None if spec.tie_word_embeddings else LMHead(spec.vocab_size, spec.hidden_size)
        self.embed_position = (build_position_encoding(spec.embedding_position)
                               if spec.embedding_position is not None else None)
        self.stream_ops = {name: build_stream_op(op) for name, op in spec.stream_ops}
        for name, op in self.stream_ops.items():
            op.set_path(f"{spec.weight_prefix}{name}")
        # checkpoint names are data of the specification
        self.embed_tokens.set_path(spec.name_of("embed"))
        for i, block in enumerate(self.blocks):
            block.set_path(spec.name_of("layers", i=i))
        self.norm.set_path(spec.name_of("final_norm"))
        if self.lm_head is not None:
            self.lm_head.set_path(spec.name_of("lm_head"))
        if self.embed_position is not None:
            self.embed_position.set_path(spec.name_of("embed_position"))
        if any(layer.options.get("streams", 0) != spec.streams for layer in spec.layers) or (spec.streams and self.stream_ops):
            raise ValueError(f"{spec.streams} residual streams: every layer keeps as many, and nothing runs between layers")
        self._resolve_order()
        #: every part allows a captured graph of its forward pass to be replayed
        self.capturable = all(part.capturable for part in self.named_parts())

    # ------------------------------------------------------------------ structure
    def _resolve_order(self):
        spec = self.spec
        cache_ids, self.cache_entries, self.cache_groups = {}, [], []
        self.state_entries, self.calls = [], []
        group_sizes = []
        # first pass: a cache entry takes its geometry from the call that writes it
        writers = {}
        for call in spec.order:
            if not 0 <= call.layer < len(self.blocks):
                raise ValueError(f"run order names layer {call.layer}, model has {len(self.blocks)}")
            if call.writes_cache:
                if call.cache in writers:
                    raise ValueError(f"cache entry {call.cache} is written by two calls")
                writers[call.cache] = call
        for call in spec.order:
            mixer = self.blocks[call.layer].mixer
            cspec = mixer.cache_spec()
            cache_index = -1
            if cspec is not None:
                if call.cache not in writers:
                    raise ValueError(f"cache entry {call.cache} is read but never written")
                wspec = self.blocks[writers[call.cache].layer].mixer.cache_spec()
                if wspec.tensors != cspec.tensors:
                    raise ValueError(f"cache entry {call.cache}: reader and writer differ in geometry")
                if call.cache not in cache_ids:
                    if wspec not in self.cache_groups:
                        self.cache_groups.append(wspec)
                        group_sizes.append(0)
                    g = self.cache_groups.index(wspec)
                    cache_ids[call.cache] = len(self.cache_entries)
                    self.cache_entries.append(CacheEntryInfo(wspec, g, group_sizes[g]))
                    group_sizes[g] += 1
                cache_index = cache_ids[call.cache]
            named = dict(mixer.state_specs())
            block_states = getattr(self.blocks[call.layer], "state_specs", None)
            if block_states is not None:
                named.update({f"block.{name}": sspec for name, sspec in block_states().items()})
            states = []
            for name, sspec in named.items():
                states.append((name, len(self.state_entries)))
                self.state_entries.append(sspec)
            before = tuple((self.stream_ops[name], arg) for name, arg in call.before)
            self.calls.append(BoundCall(call.layer, cache_index, _one_state(states), call.writes_cache, before,
                                        tuple(states)))
        self.group_sizes = group_sizes

    def named_parts(self):
        yield self.embed_tokens
        if self.embed_position is not None:
            yield from self.embed_position.named_parts()
        for op in self.stream_ops.values():
            yield from op.named_parts()
        for block in self.blocks:
            yield from block.named_parts()
        yield self.norm
        if self.lm_head is not None:
            yield self.lm_head

    def prepare(self, runtime):
        for part in self.named_parts():
            part.prepare(runtime)

    # ------------------------------------------------------------------ forward
    def forward(self, ctx):
        """Run this step's tokens; returns 32-bit logits [len(ctx.logit_rows), vocab]."""
        residual = ops.embed_lookup(self.embed_tokens.w["weight"], ctx.token_ids, ctx.slot_tokens,
                                    scale=self.spec.embedding_scale)
        if self.embed_position is not None:
            self.embed_position.add_to_embeddings(residual, ctx)
        first = residual.clone() if any(op.needs_first for op in self.stream_ops.values()) else None
        if self.spec.streams:
            residual = ops.Streams(residual, self.spec.streams)
        x = None
        for call in self.calls:
            for op, arg in call.before:
                residual, x = op.forward(residual, x, first, ctx, arg)
            x = self.blocks[call.layer].forward(x, residual, ctx, call)
        if ctx.num_logit_rows == 0:
            return None
        hidden = add_and_norm(self.norm, x, residual, rows=ctx.logit_rows, compute_dtype=ctx.dtype)
        head = self.lm_head.w["weight"] if self.lm_head is not None else self.embed_tokens.w["weight"]
        logits = ops.linear(hidden, head, out_float32=True)
        if self.spec.logit_softcap > 0 or self.spec.logit_scale != 1.0:
            ops.softcap_(logits, self.spec.logit_softcap, self.spec.logit_scale)
        return logits


def build_model(config: ModelConfig) -> DecoderModel:
    """From an architecture's configuration to a model made of parts: the configuration names
    the parts, layer by layer, and the run order; nothing else of it reaches the parts."""
    return DecoderModel(config.model_spec())
