"""Dubarax described as parts, layer by layer.

A pre-norm decoder, ``x += mixer(n1(x)); x += ff(n2(x))``, with RMS norms whose stored weights lie around zero (the multiplier
is one plus the weight) and no positions but those that masks and biases give.  A stretch of its layers runs several times
in a row with the same weights, every pass with a cache of its own and behind a projection of the stream and the embedding
rows (``parts.passes``).  Three mixers:

* ``parallel``: softmax attention inside chunks of the sequence, a score losing a fixed slope times the distance, beside
  lightning attention (a matrix memory with a fixed decay per head, silu on q, k and v, one norm over all heads and a sigmoid
  gate); the two are added with a constant each;
* ``attention``: sliding-window attention with capped scores and a learned bias by distance, on a logarithmic scale;
* ``mamba2``: the state-space dual form with a short convolution.

The feed-forward is a mixture of SwiGLU experts: softmax scores over all experts, the choice limited to the best groups of
neighbouring experts, weights as they are, and a shared expert without a gate.  Tensor names: ``embed``, ``loop.in|step``,
``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.dubarax_config import (ARCHITECTURE, DubaraxConfig, ParallelConfig, StateSpaceConfig, WindowAttentionConfig)
from ..parts import PartSpec, LayerSpec, LayerCall, ModelSpec

ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
                   "rel": "rel"}


def _norm(cfg: DubaraxConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", dict(size=cfg.hidden_size, eps=cfg.eps, weight_offset=1.0, weight_name=name))


def _attention(cfg: DubaraxConfig, m, **options) -> PartSpec:
    return PartSpec("paged_attention", dict(
        hidden_size=cfg.hidden_size, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, bias=True,
        out_bias=True, position=PartSpec("none"), scale=m.scale, round_weights=True, names=ATTENTION_NAMES, **options))


def linear_slopes(heads: int) -> list:
    """What a distance of one takes off the scores of head h: ``2^(-8 (h + 1) / heads)``."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def _mixer(cfg: DubaraxConfig, m) -> PartSpec:
    W, eps = cfg.hidden_size, cfg.eps
    if isinstance(m, ParallelConfig):
        left = _attention(cfg, m.left, chunk=m.left.chunk, distance_slopes=linear_slopes(m.left.heads))
        right = PartSpec("lightning_attention", dict(hidden_size=W, heads=m.right.heads, dim=m.right.dim, vdim=m.right.vdim,
                                                     decay=m.right.decay, eps=eps))
        return PartSpec("side_by_side", dict(hidden_size=W, members=[left, right], names=["left.", "right."], eps=eps,
                                             member_scales=[m.left_scale, m.right_scale]))
    if isinstance(m, WindowAttentionConfig):
        return _attention(cfg, m, window=m.window, score_softcap=m.softcap, distance_far=m.bias_max)
    if isinstance(m, StateSpaceConfig):
        return PartSpec("state_space_dual", dict(hidden_size=W, heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups,
                                                 conv=m.conv, norm_groups=m.norm_groups, eps=eps))
    raise TypeError(type(m))


def _feed_forward(cfg: DubaraxConfig, f) -> PartSpec:
    names = {"router": "router", "expert_gate": "e{}.gate", "expert_up": "e{}.up", "expert_down": "e{}.down",
             "shared_gate_proj": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down"}
    return PartSpec("sparse_moe_swiglu", dict(
        hidden_size=cfg.hidden_size, num_experts=f.experts, top_k=f.top, intermediate_size=f.ff,
        shared_intermediate_size=f.shared_ff, shared_gate=False, groups=f.groups, names=names))


def layer_order(count: int, loop) -> list:
    """The calls of a forward pass: the looped stretch once per pass, its first layer opening the pass."""
    if loop is None:
        return [LayerCall(i) for i in range(count)]
    order = [LayerCall(i) for i in range(loop.start)]
    for t in range(loop.times):
        order += [LayerCall(i, pass_index=t if i == loop.start else None) for i in range(loop.start, loop.stop)]
    return order + [LayerCall(i) for i in range(loop.stop, count)]


def build_spec(cfg: DubaraxConfig) -> ModelSpec:
    layers = []
    for L in cfg.layers:
        parts = {"norm1": _norm(cfg, "norm1"), "mixer": _mixer(cfg, L.mixer)}
        if L.mlp is not None:
            parts.update(norm2=_norm(cfg, "norm2"), feed_forward=_feed_forward(cfg, L.mlp))
        layers.append(LayerSpec(parts=parts, names={"norm1": "", "mixer": "mix.", "norm2": "", "feed_forward": "mlp."}))
    passes = None
    if cfg.loop is not None:
        passes = PartSpec("recall", dict(size=cfg.hidden_size, passes=cfg.loop.times))
    return ModelSpec(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, layers=layers,
                     order=layer_order(len(layers), cfg.loop), final_norm=_norm(cfg, "final.norm"), tie_word_embeddings=False,
                     embed_scale=cfg.embed_scale, pass_input=passes, embed_name="embed", layer_prefix="l{}.",
                     final_norm_prefix="", lm_head_name="head")


register_architecture(ARCHITECTURE, DubaraxConfig.from_dict, build_spec)
