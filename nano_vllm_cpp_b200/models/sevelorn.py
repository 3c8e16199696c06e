"""Sevelorn described as parts, layer by layer.

A decoder that keeps ``streams`` copies of its residual stream, wired to every sublayer through a learned link (``hc1`` for
the mixer, ``hc2`` for the feed-forward: hyper-connections, ``parts.streams``), with RMS norms whose stored weights lie
around zero (the multiplier is one plus the weight).  What a mixer reads is the normed row plus a short causal convolution
of the normed rows (``canon1``, ``parts.convolution``).  Two mixers:

* ``retention``: linear attention with a fixed decay per head, q and k turned in the halves pairing, heads divided by their
  root mean square, a silu gate on the concatenated heads;
* ``attention``: grouped-query softmax attention without positions, q and k each normed over all their heads at once, a
  sigmoid gate per head on the heads' outputs; with ``kv_from`` it has no keys and values of its own and reads the pages
  of the layer named.

Two feed-forwards: a dense one with the tanh form of gelu on its gate, and a mixture of SwiGLU experts whose router has a
bias and weighs the chosen experts by the softmax over their logits.  The stream starts as the embedding row times a
constant.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.hc1|hc2.in|out|mix``, ``l<i>.canon1``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sevelorn_config import ARCHITECTURE, SevelornConfig, RetentionConfig, GatedAttentionConfig
from ..parts import PartSpec, LayerSpec, LayerCall, ModelSpec


def _norm(cfg: SevelornConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", dict(size=cfg.hidden_size, eps=cfg.eps, weight_offset=1.0, weight_name=name))


def _mixer(cfg: SevelornConfig, m) -> PartSpec:
    W, eps = cfg.hidden_size, cfg.eps
    if isinstance(m, RetentionConfig):
        position = PartSpec("rotary_neox", dict(rotary_dim=m.rot_dims, theta=m.rot_base)) if m.rot_dims else PartSpec("none")
        return PartSpec("retention", dict(hidden_size=W, heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, eps=eps,
                                          position=position))
    if isinstance(m, GatedAttentionConfig):
        names = {"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_norm": "q.norm", "k_norm": "k.norm"}
        return PartSpec("paged_attention", dict(
            hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, bias=False,
            position=PartSpec("none"), scale=m.scale, qk_norm_eps=eps, qk_norm_whole=True, output_gate=True,
            own_kv=m.kv_from is None, round_weights=True, names=names))
    raise TypeError(type(m))


def _feed_forward(cfg: SevelornConfig, f) -> PartSpec:
    W = cfg.hidden_size
    if f.kind == "dense":
        return PartSpec("dense_swiglu", dict(hidden_size=W, intermediate_size=f.ff, activation="gelu_tanh",
                                             names={"gate": "gate", "up": "up", "down": "down"}))
    return PartSpec("sparse_moe_swiglu", dict(
        hidden_size=W, num_experts=f.experts, top_k=f.top, intermediate_size=f.ff, renormalize=True, router_bias=True,
        names={"router": "router", "router_bias": "router.b", "expert_gate": "e{}.gate", "expert_up": "e{}.up",
               "expert_down": "e{}.down"}))


def build_spec(cfg: SevelornConfig) -> ModelSpec:
    layers, order = [], []
    link = PartSpec("stream_link", dict(streams=cfg.streams))
    for i, L in enumerate(cfg.layers):
        parts = {"norm1": _norm(cfg, "norm1"), "mixer": _mixer(cfg, L.mixer), "link1": link}
        if cfg.taps:
            parts["input_filter"] = PartSpec("causal_convolution", dict(size=cfg.hidden_size, taps=cfg.taps, name="canon1"))
        if L.mlp is not None:
            parts.update(norm2=_norm(cfg, "norm2"), feed_forward=_feed_forward(cfg, L.mlp), link2=link)
        layers.append(LayerSpec(arrangement="hyper_connected", parts=parts, params={"streams": cfg.streams},
                                names={"norm1": "", "input_filter": "", "mixer": "mix.", "link1": "hc1.", "norm2": "",
                                       "feed_forward": "mlp.", "link2": "hc2."}))
        order.append(LayerCall(i, cache_of=getattr(L.mixer, "kv_from", None)))
    return ModelSpec(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, layers=layers, order=order,
                     final_norm=_norm(cfg, "final.norm"), tie_word_embeddings=False, streams=cfg.streams,
                     embed_scale=cfg.embed_scale, embed_name="embed", layer_prefix="l{}.", final_norm_prefix="",
                     lm_head_name="head")


register_architecture(ARCHITECTURE, SevelornConfig.from_dict, build_spec)
