"""A decoder as data (``ModelSpec``) and the object built from it (``Model``).

``ModelSpec.order`` is the list of layer calls of one forward pass.  A call names the layer to run
and the cache entry it uses; by default call i runs layer i with a cache entry of its own.  A
layer may be named by several calls (each call then has its own cache entry unless told
otherwise), and a call may name an earlier call's cache entry with ``cache_of``: it then reads
that entry and writes nothing.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..csrc import ops
from .base import PartSpec, RunContext, TensorSpec, resolve_branch
from .block import LayerSpec, build_layer
from .linear import linear
from .registry import build_part
from .streams import StreamUpdate, read_streams


@dataclass
class LayerCall:
    layer: int
    cache_of: Optional[int] = None     # index of an earlier call whose cache entry this call reads
    pass_index: Optional[int] = None   # the call opens this pass over a stretch of layers (see ModelSpec.pass_input)


@dataclass
class ModelSpec:
    vocab_size: int
    hidden_size: int
    layers: list                        # list[LayerSpec]
    final_norm: PartSpec
    tie_word_embeddings: bool
    order: Optional[list] = None        # list[LayerCall]; None = every layer once, in order
    embed_name: str = "model.embed_tokens.weight"
    layer_prefix: str = "model.layers.{}."
    final_norm_prefix: str = "model.norm."
    lm_head_name: str = "lm_head.weight"
    init_std: float = 0.02
    norm_init_std: float = 0.0          # random-weights mode: norm weights are 1 + N(0, this)
    layer_ids: Optional[list] = None    # what stands in layer_prefix for each layer; None = its index in ``layers``
    streams: int = 1                    # copies of the residual stream (see parts.streams)
    logit_scale: float = 1.0            # logits = head(x) * logit_scale, then, with a cap,
    logit_softcap: float = 0.0          # logits = cap * tanh(logits / cap)
    embed_scale: float = 1.0            # the stream starts as embed[token] * embed_scale
    pass_input: Optional[PartSpec] = None   # what the stream goes through before a call that opens a pass (parts.passes)
    pass_input_prefix: str = "loop."

    def calls(self):
        if self.order is None:
            return [LayerCall(i) for i in range(len(self.layers))]
        return list(self.order)


def _full_name(prefix: str, name: str) -> str:
    """A part's tensor name as the model knows it: behind the part's prefix, or, if it starts with ``/``, a name
    of the whole model (a tensor that several layers read)."""
    return name[1:] if name.startswith("/") else prefix + name


class _Fetch:
    """Fetches a part's tensors by local name from the model-wide source.  A tensor of the whole model (``/name``)
    is fetched once and handed to every part that asks for it."""

    def __init__(self, source, prefix, shared: dict):
        self.source, self.prefix, self.shared = source, prefix, shared

    def __call__(self, name):
        full = _full_name(self.prefix, name)
        if name.startswith("/"):
            if full not in self.shared:
                self.shared[full] = self.source.get(full)
            return self.shared[full]
        return self.source.get(full)

    def has(self, name):
        return self.source.has(_full_name(self.prefix, name))


class Model:
    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.layers = [build_layer(ls) for ls in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm)
        self.pass_input = build_part("pass_input", spec.pass_input) if spec.pass_input is not None else None
        if self.pass_input is not None and spec.streams > 1:
            raise ValueError("passes over a stretch of layers go with one copy of the residual stream")
        self.calls = spec.calls()
        self.after_call = None      # a hook (call index, stream, pending) for whoever wants to look at the stream layer by layer
        if spec.layer_ids is not None and len(spec.layer_ids) != len(spec.layers):
            raise ValueError("layer_ids: one entry per layer")
        for i, c in enumerate(self.calls):
            if not (0 <= c.layer < len(self.layers)):
                raise ValueError(f"call {i} names layer {c.layer}, which does not exist")
            if c.pass_index is not None and self.pass_input is None:
                raise ValueError(f"call {i} opens a pass, but the model has no pass input")
            if c.cache_of is not None and not (0 <= c.cache_of < i and self.calls[c.cache_of].cache_of is None):
                raise ValueError(f"call {i}: cache_of must name an earlier call that owns its cache entry")

    @property
    def graph_safe(self) -> bool:
        return all(part.graph_safe for _, part in self._named_parts())

    # ------------------------------------------------------------------ tensors
    def _named_parts(self):
        for i, layer in enumerate(self.layers):
            lp = self.spec.layer_prefix.format(i if self.spec.layer_ids is None else self.spec.layer_ids[i])
            for sub, part in layer.parts():
                yield lp + sub, part
        yield self.spec.final_norm_prefix, self.final_norm
        if self.pass_input is not None:
            yield self.spec.pass_input_prefix, self.pass_input

    def tensor_specs(self, has=None) -> dict:
        """Every tensor the model needs, by full name."""
        s = self.spec
        out = {s.embed_name: TensorSpec((s.vocab_size, s.hidden_size))}
        for prefix, part in self._named_parts():
            part_has = (lambda n, p=prefix: has(_full_name(p, n))) if has is not None else None
            for name, ts in part.tensor_specs(part_has).items():
                full = _full_name(prefix, name)
                if full in out and tuple(out[full].shape) != tuple(ts.shape):
                    raise ValueError(f"tensor {full!r} is wanted with the shapes {out[full].shape} and {ts.shape}")
                out[full] = ts
        if not s.tie_word_embeddings:
            out[s.lm_head_name] = TensorSpec((s.vocab_size, s.hidden_size))
        return out

    def cache_specs(self) -> list:
        """One entry per call: the cache spec of its layer, or None, or ('shared', j); a call that reads an earlier
        call's entry and keeps a state of its own beside it has a composite with a ``SharedCacheSpec``."""
        out = []
        for c in self.calls:
            if c.cache_of is not None:
                out.append(self.layers[c.layer].borrowing_cache_spec(c.cache_of))
            else:
                out.append(self.layers[c.layer].cache_spec())
        return out

    def load(self, source, ctx: RunContext) -> None:
        """``source.get(name)`` returns the device tensor of a full name; ``source.has(name)``."""
        self.ctx = ctx
        s = self.spec
        self.embed = source.get(s.embed_name)
        shared: dict = {}
        for prefix, part in self._named_parts():
            part.load(_Fetch(source, prefix, shared), ctx)
        self.lm_head = self.embed if s.tie_word_embeddings else source.get(s.lm_head_name)

    # ------------------------------------------------------------------ forward
    def forward(self, batch, cache) -> torch.Tensor:
        """Runs the rows of ``batch`` through every call; returns float32 logits ``[wanted, vocab]``."""
        ctx = self.ctx
        ops.mark_step()
        s = self.spec
        x = torch.empty((batch.T, s.streams * s.hidden_size), dtype=torch.float32, device=ctx.device)
        ops.embedding(batch.input_ids, self.embed, x, ctx.err, feed=ctx.feed, copies=s.streams, scale=s.embed_scale)
        pending = None
        recalled = self.pass_input.recall(x) if self.pass_input is not None else None
        for i, c in enumerate(self.calls):
            if c.pass_index is not None:
                x, pending = self.pass_input.forward(x, pending, recalled, c.pass_index)
            pending = self.layers[c.layer].forward(x, pending, batch, cache.view(i))
            if self.after_call is not None:
                self.after_call(i, x, pending)
        if s.streams > 1 or isinstance(pending, StreamUpdate):
            h, _ = read_streams(self.final_norm, x, s.streams, pending, None)       # the copies are summed
        else:
            h, _ = self.final_norm.forward(x, resolve_branch(self.final_norm, pending))
        n_want = batch.want_rows.numel()
        if n_want == 0:
            return torch.empty((0, s.vocab_size), dtype=torch.float32, device=ctx.device)
        logits = linear(ctx, h, self.lm_head, torch.float32, a_rows=batch.want_rows)
        if s.logit_scale != 1.0 or s.logit_softcap > 0:
            ops.scale_softcap(logits, s.logit_scale, s.logit_softcap)
        return logits
