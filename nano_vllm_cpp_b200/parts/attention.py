"""Causal self-attention over paged keys and values, with grouped query heads, an optional
window and a position encoding applied to q and k before the cache write."""
from __future__ import annotations

import math

import torch

from ..csrc import ops
from .base import Mixer, KVCacheSpec, TensorSpec, PartSpec
from .linear import linear
from .registry import register_part, build_part


class PagedAttention(Mixer):
    """Per row t at position p (src/model.cpp:764-786):

    ``q,k,v = h Wq^T + bq, h Wk^T + bk, h Wv^T + bv``; rotate q and k; write k and v to the page
    slot of p; ``out = softmax(q K^T * scale) V`` over keys ``[max(0, p+1-window), p]`` of the same
    request read from the cache (so rows of this step see one another through it); ``out Wo^T``.
    Query head h reads kv head ``h // (Hq / Hkv)`` (src/hip_ops.hip:484).  ``scale`` defaults to
    ``1/sqrt(head_dim)`` (src/model.cpp:710).

    Options beyond that, each off by default: values with a head size of their own (``v_head_dim``); an RMS norm
    over every q and k head before the rotation, with one weight vector per side shared by the heads (``qk_norm_eps``);
    a bias on the output projection (``out_bias``); a *sink* in every softmax, a key with the score ``sink_score``
    and no value, so that ``p_j = exp(s_j) / (exp(sink_score) + sum_i exp(s_i))``; a position encoding that pairs
    neighbouring elements or scales its cosines and sines; no value projection at all (``values_from_keys``: a key
    head as projected, before its norm and rotation, is also the value head, and there is no v tensor); softmax
    weights that stay float32 in the product with the values (``exact_weights``; the tensor-core kernels of the
    default path round them to bfloat16).  ``names`` gives the tensors' names where they are not
    the usual ones (keys: q, k, v, o, q_bias, k_bias, v_bias, o_bias, q_norm, k_norm, head_mix, sink).  A layer that
    uses one of these options runs the general kernels (``ops.qk_prepare_store``, ``ops.paged_attention_general``).

    Four more, which also run the general kernels.  ``keep_first``: with a window, the sequence's first so many
    positions stay visible behind it (row i reads j if ``j <= i`` and ``i - j < window or j < keep_first``), at their
    true positions; their pages are held to the request's end.  ``learned_sink``: the sink's score is a learned
    number per query head (tensor ``sink`` [heads]).  ``head_mix``: the heads' scaled scores are mixed before mask
    and softmax, ``s'_h = sum_g M[h, g] s_g`` with the learned ``M`` (tensor ``head_mix`` [heads, heads]); since a
    score is linear in its query, the rows' queries are mixed instead, once per row (``ops.mix_query_heads``), and a
    score becomes one product with all kv heads' keys side by side.  ``value_position`` (a position encoding over
    the whole value head): the value of position j is turned by j before it is stored, and a head's output at
    position i, the weighted sum of such values, is turned back by i, so that a value enters the output turned by
    ``j - i``.

    Three more of the plain general path.  ``qk_norm_weight`` False: the head norm of q and k has no weight
    tensors (a head is divided by its root mean square and nothing else).  ``qk_norm_after_rotation``: that norm
    follows the turn instead of preceding it (with a position encoding whose cosines and sines carry an amplitude,
    or that turns part of a head, the two orders differ).  ``score_softcap`` > 0: a scaled score s becomes
    ``score_softcap * tanh(s / score_softcap)`` before mask and softmax.  ``round_weights``: a bfloat16 run of
    this path rounds the softmax weights (computed in float32) to bfloat16 for their product with the values, as it
    rounds every other operand of a product, instead of taking them in as three bfloat16 terms.

    Three more, of the same path.  ``qk_norm_whole``: q's norm is taken over all its heads at once, k's over all of its
    heads (weights of that size), instead of head by head.  ``output_gate``: head h's output is multiplied by
    ``sigmoid(Wg h)_h``, one number per head and row (tensor ``g`` [heads, hidden]), where the attention kernel writes
    it.  ``own_kv`` False: the layer has no k and v tensors; its call reads the pages of an earlier call (whose kv heads
    and head sizes are the same) with its own queries, and writes none.

    Three more, of the same path.  ``chunk`` > 0 instead of a window: row i sees the positions of its own chunk of so many,
    counted from the sequence's start (``j <= i`` and ``j // chunk == i // chunk``).  ``distance_slopes`` (one number per
    query head): a score loses ``slope * (i - j)``, behind the cap.  ``distance_far``: a score gains a learned number that
    depends on head and distance, also behind the cap: row ``bucket(i - j)`` of the tensor ``rel`` [rows, heads], where
    distances below half of the rows have a row each and the others share the rest on a logarithmic scale that ends at
    ``distance_far`` (``distance_buckets``); the number of rows is the file's (``distance_rows`` for random weights).

    A layer of this path without head norms, positions, gates and borrowed keys skips the float32 projection in bfloat16
    runs: its projection makes bfloat16 rows that the attention kernels read in place, heads padded to one size in the
    weights.
    """

    _NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight",
              "q_bias": "q_proj.bias", "k_bias": "k_proj.bias", "v_bias": "v_proj.bias", "o_bias": "o_proj.bias", "g": "g_proj.weight",
              "q_norm": "q_norm.weight", "k_norm": "k_norm.weight", "head_mix": "head_mix", "sink": "sink", "rel": "rel"}

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, bias: bool,
                 position: PartSpec, window: int = 0, scale: float | None = None, v_head_dim: int | None = None,
                 qk_norm_eps: float | None = None, out_bias: bool = False, sink_score: float | None = None,
                 names: dict | None = None, values_from_keys: bool = False, exact_weights: bool = False,
                 keep_first: int = 0, learned_sink: bool = False, head_mix: bool = False,
                 value_position: PartSpec | None = None, qk_norm_weight: bool = True,
                 qk_norm_after_rotation: bool = False, score_softcap: float = 0.0, round_weights: bool = False,
                 qk_norm_whole: bool = False, output_gate: bool = False, own_kv: bool = True, chunk: int = 0,
                 distance_slopes: list | None = None, distance_far: int | None = None, distance_rows: int = 32):
        if num_heads % num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        self.hidden, self.Hq, self.Hkv, self.D = hidden_size, num_heads, num_kv_heads, head_dim
        self.Dv = int(v_head_dim) if v_head_dim else head_dim
        self.bias, self.window, self.out_bias = bias, int(window), bool(out_bias)
        self.qk_norm_eps = None if qk_norm_eps is None else float(qk_norm_eps)
        self.sink_score = None if sink_score is None else float(sink_score)
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(float(head_dim))
        self.position = build_part("position", position) if isinstance(position, PartSpec) else position
        self.names = dict(self._NAMES, **(names or {}))
        self.values_from_keys = bool(values_from_keys)
        self.qk_norm_weight, self.qk_norm_after = bool(qk_norm_weight), bool(qk_norm_after_rotation)
        self.softcap = float(score_softcap)
        self.weight_terms = 1 if round_weights else 3
        if self.softcap < 0:
            raise ValueError("score_softcap must not be negative")
        if self.values_from_keys and self.Dv != self.D:
            raise ValueError("values that are the keys have the keys' head size")
        if self.values_from_keys and bias:
            raise ValueError("values that are the keys: biased projections are not supported")
        self.keep_first = int(keep_first) if self.window > 0 else 0
        self.learned_sink, self.head_mix = bool(learned_sink), bool(head_mix)
        self.value_position = (build_part("position", value_position) if isinstance(value_position, PartSpec)
                               else value_position)
        if self.keep_first < 0:
            raise ValueError("keep_first must not be negative")
        if self.learned_sink and self.sink_score is not None:
            raise ValueError("a sink has a fixed score or a learned one, not both")
        if self.value_position is not None:
            vp = self.value_position
            if self.values_from_keys or vp.pairing != "halves" or vp.amplitude != 1.0 or vp.rotary_dim > self.Dv:
                raise ValueError("turned values: pairs (i, i + dims / 2) over at most the value head, no amplitude, and "
                                 "values of their own")
        self.qk_norm_whole, self.output_gate, self.own_kv = bool(qk_norm_whole), bool(output_gate), bool(own_kv)
        if self.qk_norm_whole and (self.qk_norm_eps is None or self.qk_norm_after):
            raise ValueError("a norm over all heads comes with its eps and precedes the turn")
        if not self.own_kv and (bias or self.values_from_keys):
            raise ValueError("a layer without keys and values of its own has no biases of theirs")
        self.chunk = int(chunk)
        self.distance_slopes = None if distance_slopes is None else [float(s) for s in distance_slopes]
        self.distance_far = None if distance_far is None else int(distance_far)
        self.distance_rows = int(distance_rows)
        if self.chunk < 0 or (self.chunk and self.window):
            raise ValueError("a layer sees a window or its own chunk, not both")
        if self.distance_slopes is not None and len(self.distance_slopes) != num_heads:
            raise ValueError("distance_slopes: one number per query head")
        if self.distance_far is not None and self.distance_far < 1:
            raise ValueError("distance_far must be positive")
        scored = bool(self.chunk or self.distance_slopes is not None or self.distance_far is not None)
        # the options that only the general kernels know, whatever the dtype
        self.extended = bool(self.keep_first or self.learned_sink or self.head_mix or self.value_position is not None)
        if self.extended and self.softcap > 0:
            raise ValueError("capped scores are not supported together with kept positions, learned sinks, mixed heads or turned values")
        if self.extended and (self.qk_norm_whole or self.output_gate or not self.own_kv):
            raise ValueError("a norm over all heads, an output gate and borrowed keys are not supported together with kept "
                             "positions, learned sinks, mixed heads or turned values")
        if self.extended and scored:
            raise ValueError("chunks and biases by distance are not supported together with kept positions, learned sinks, "
                             "mixed heads or turned values")
        self.general = (scored or self.extended or self.output_gate or not self.own_kv or self.softcap > 0 or self.values_from_keys or bool(exact_weights) or self.Dv != self.D or self.qk_norm_eps is not None or self.sink_score is not None
                        or self.position.pairing != "halves" or self.position.amplitude != 1.0)
        if self.general:
            if self.extended:
                if head_dim < 1 or self.Dv < 1 or self.Dv > 512:
                    raise ValueError(f"value heads of {self.Dv} elements are not supported: at most 512")
            elif head_dim < 1 or head_dim > 256 or self.Dv < 1 or self.Dv > 256:
                raise ValueError(f"head sizes {head_dim} / {self.Dv} are not supported: the general attention kernels "
                                 "take up to 256 elements per head")
        elif head_dim % 16 or head_dim > 256:
            raise ValueError(f"head_dim {head_dim} is not supported: the attention kernels take multiples "
                             "of 16 up to 256")

    # ------------------------------------------------------------------ weights
    def tensor_specs(self, available=None):
        H, q, kv, vv, n = self.hidden, self.Hq * self.D, self.Hkv * self.D, self.Hkv * self.Dv, self.names
        s = {n["q"]: TensorSpec((q, H)), n["k"]: TensorSpec((kv, H)),
             n["v"]: TensorSpec((vv, H)), n["o"]: TensorSpec((H, self.Hq * self.Dv))}
        if self.values_from_keys:
            del s[n["v"]]
        if not self.own_kv:
            del s[n["k"]], s[n["v"]]
        if self.output_gate:
            s[n["g"]] = TensorSpec((self.Hq, H))
        if self.bias:
            s.update({n["q_bias"]: TensorSpec((q,), kind="vector"), n["k_bias"]: TensorSpec((kv,), kind="vector"),
                      n["v_bias"]: TensorSpec((vv,), kind="vector")})
        if self.out_bias:
            s[n["o_bias"]] = TensorSpec((H,), kind="vector")
        if self.qk_norm_eps is not None and self.qk_norm_weight:
            whole = self.qk_norm_whole
            s[n["q_norm"]] = TensorSpec((q if whole else self.D,), init="ones", kind="vector")
            if self.own_kv:
                s[n["k_norm"]] = TensorSpec((kv if whole else self.D,), init="ones", kind="vector")
        if self.head_mix:
            s[n["head_mix"]] = TensorSpec((self.Hq, self.Hq), init="identity", kind="vector")
        if self.learned_sink:
            s[n["sink"]] = TensorSpec((self.Hq,), init="zeros", kind="vector")
        if self.distance_far is not None:       # the number of rows is the file's
            s[n["rel"]] = TensorSpec((None if available is not None else self.distance_rows, self.Hq), kind="vector")
        s.update(self.position.tensor_specs(available))      # a position encoding may have tensors of its own
        return s

    def load(self, fetch, ctx):
        self.ctx = ctx
        n = self.names
        self.position.load(fetch, ctx)
        self.slopes = self.bias_table = None
        if self.distance_slopes is not None:
            self.slopes = torch.tensor(self.distance_slopes, dtype=torch.float32, device=ctx.device)
        if self.distance_far is not None:       # spread out: one number per head and distance
            rel = fetch(n["rel"]).float()
            rows = torch.tensor(distance_buckets(rel.shape[0], self.distance_far), device=rel.device)
            self.bias_table = ops.bias_table_of(rel[rows].t())
        # q, k and v rows are stacked so that one product makes all three (src/model.cpp:508-513)
        rows = [fetch(n["q"])]
        if self.own_kv:
            rows += [fetch(n["k"])] + ([] if self.values_from_keys else [fetch(n["v"])])
        self.gate_col = sum(t.shape[0] for t in rows)                    # the output gates' rows come last
        if self.output_gate:
            rows.append(fetch(n["g"]))
        self.qkv_weight = _cat(rows)
        self.qkv_bias = None
        if self.bias:
            self.qkv_bias = _cat([fetch(n["q_bias"]), fetch(n["k_bias"]), fetch(n["v_bias"])])
        self.o_weight = fetch(n["o"])
        self.o_bias = fetch(n["o_bias"]) if self.out_bias else None
        # The tensor-core kernel wants one head size for q, k and v, a multiple of 16: a bfloat16 run of the general
        # path pads the three with zeros up to it (the scores and the sums are the same), and the output
        # projection gets zero columns for the padding.
        self.pad, self.direct = 0, False
        self.mix_weight = fetch(n["head_mix"]).float().contiguous() if self.head_mix else None
        self.sinks = fetch(n["sink"]).float().contiguous() if self.learned_sink else None
        if self.value_position is not None:
            self.value_position.load(fetch, ctx)
        if (self.general and not self.extended and ctx.fast_kernels and ctx.act_dtype == torch.bfloat16
                and self.o_weight.dtype == torch.bfloat16):
            self.pad = (max(self.D, self.Dv) + 15) // 16 * 16
            self.direct = (self.qkv_weight.dtype == torch.bfloat16 and self.position.rotary_dim == 0 and self.own_kv
                           and self.qk_norm_eps is None and not self.values_from_keys and not self.output_gate)
            if self.direct:
                self.pad = max(self.pad, 32)
                sizes = [(self.Hq, self.D), (self.Hkv, self.D), (self.Hkv, self.Dv)]
                self.qkv_weight = _pad_heads(self.qkv_weight, sizes, self.pad)
                if self.qkv_bias is not None:
                    self.qkv_bias = _pad_heads(self.qkv_bias, sizes, self.pad)
            if self.pad != self.Dv:
                w = torch.zeros((self.hidden, self.Hq, self.pad), dtype=self.o_weight.dtype, device=self.o_weight.device)
                w[:, :, :self.Dv] = self.o_weight.view(self.hidden, self.Hq, self.Dv)
                self.o_weight = w.view(self.hidden, self.Hq * self.pad)
        self.q_norm = self.k_norm = None
        if self.qk_norm_eps is not None and self.qk_norm_weight:
            self.q_norm, self.k_norm = fetch(n["q_norm"]), fetch(n["k_norm"]) if self.own_kv else None

    def cache_spec(self):
        if getattr(self, "pad", 0):
            return KVCacheSpec(self.Hkv, self.pad, self.window, chunk=self.chunk)
        return KVCacheSpec(self.Hkv, self.D, self.window, 0 if self.Dv == self.D else self.Dv, self.keep_first, chunk=self.chunk)

    # ------------------------------------------------------------------ forward
    def forward(self, h, batch, cache):
        ctx = self.ctx
        T = h.shape[0]
        if self.general:
            return self._forward_general(h, batch, cache)
        qkv = linear(ctx, h, self.qkv_weight, ctx.act_dtype, bias=self.qkv_bias)
        bt = batch.block_tables[cache.group]
        ops.rope_store(qkv, batch.positions, self.position.inv_freq(), self.position.rotary_dim, cache.k, cache.v,
                       bt, batch.row_entry, self.Hq, self.Hkv, self.D, cache.write, ctx.err,
                       rot_positions=self.position.rotation_positions(batch), pair_axis=self.position.pair_axis())
        att = torch.empty((T, self.Hq * self.D), dtype=ctx.act_dtype, device=h.device)
        self._attend(qkv, cache, bt, batch, att)
        return linear(ctx, att, self.o_weight, torch.float32, bias=self.o_bias)

    def _forward_general(self, h, batch, cache):
        """The projections come out in float32 (the head norms read them); q after norm and rotation, and the keys
        and values in their pages, are in the activation dtype; scores, weights and sums are float32."""
        ctx, T = self.ctx, h.shape[0]
        Hq, Hkv, D, Dv = self.Hq, self.Hkv, self.D, self.Dv
        if self.direct:
            return self._forward_direct(h, batch, cache)
        proj = linear(ctx, h, self.qkv_weight, torch.float32, bias=self.qkv_bias)
        bt = batch.block_tables[cache.group]
        if self.extended:
            return self._forward_extended(proj, bt, batch, cache)
        P = self.pad
        q = torch.empty((T, Hq * (P or D)), dtype=ctx.act_dtype, device=h.device)
        pos = self.position
        # (values that are the keys are read where the keys are, as projected: the kernel norms and turns its own copy)
        ops.qk_prepare_store(proj, 0, Hq * D, Hq * D if self.values_from_keys else (Hq + Hkv) * D, batch.positions, batch.row_entry, bt, self.q_norm,
                             self.k_norm, self.qk_norm_eps or 0.0, pos.inv_freq(), pos.rotary_dim,
                             pos.pairing == "interleaved", pos.amplitude, q, cache.k, cache.v, Hq,
                             Hkv if self.own_kv else 0, D, Dv, cache.write and self.own_kv, ctx.err,
                             norm_always=self.qk_norm_eps is not None, norm_after=self.qk_norm_after,
                             norm_whole=self.qk_norm_whole)
        gate = proj[:, self.gate_col:self.gate_col + Hq] if self.output_gate else None
        att = torch.empty((T, Hq * (P or Dv)), dtype=ctx.act_dtype, device=h.device)
        if P:
            self._attend_general(q, cache, bt, batch, att, P, gate)
        else:
            ops.paged_attention_general(q, cache.k, cache.v, bt, batch.row_entry, batch.positions, self.scale,
                                        self.window, att, Hq, Hkv, D, Dv, sink_score=self.sink_score,
                                        softcap=self.softcap, gate=gate, chunk=self.chunk, slopes=self.slopes,
                                        bias_table=self.bias_table)
        return linear(ctx, att, self.o_weight, torch.float32, bias=self.o_bias)

    def _forward_direct(self, h, batch, cache):
        """Heads that go from the projection to the scores as they are: one bfloat16 product makes q, k and v with all heads
        padded to one size, keys and values are copied to their pages, and the attention kernels read q where it is."""
        ctx, P = self.ctx, self.pad
        qkv = linear(ctx, h, self.qkv_weight, torch.bfloat16, bias=self.qkv_bias)
        bt = batch.block_tables[cache.group]
        ops.rope_store(qkv, batch.positions, self.position.inv_freq(), 0, cache.k, cache.v, bt, batch.row_entry, self.Hq,
                       self.Hkv, P, cache.write, ctx.err)
        att = torch.empty((h.shape[0], self.Hq * P), dtype=torch.bfloat16, device=h.device)
        self._attend_general(qkv, cache, bt, batch, att, P, None)
        return linear(ctx, att, self.o_weight, torch.float32, bias=self.o_bias)

    def _attend_general(self, q, cache, bt, batch, att, P, gate):
        """Entries of one row go to the split-key decode kernel (with weights that keep their float32 bits, or as one
        rounded term), the others to a tensor-core kernel (tcgen05, else mma.sync), where float32 weights enter the product
        with the values as three bfloat16 terms; the decode kernel and the mma.sync kernel add the sink to the softmax's
        denominator.  ``q``: rows whose first Hq * P elements are the query heads."""
        ctx, Hq, Hkv = self.ctx, self.Hq, self.Hkv
        scored = dict(softcap=self.softcap, gate=gate, chunk=self.chunk, slopes=self.slopes, bias_table=self.bias_table)
        single = batch.n_single if ops.attention_decode_usable(cache.k, P) else 0
        if single:
            ops.attention_decode(q, cache.k, cache.v, bt, batch.row_entry, batch.positions, self.scale, self.window,
                                 att, Hq, Hkv, P, batch.max_context if batch.decode_only else batch.max_single_context,
                                 rows=None if batch.decode_only else batch.single_rows, err=ctx.err,
                                 sink_score=self.sink_score, float_weights=self.weight_terms == 3, **scored)
        if single < batch.S:
            tiles = (batch.T - single) // ops.attention_prefill_tile_rows() + (batch.S - single)
            ops.attention_prefill(q, cache.k, cache.v, bt, batch.cu_rows, batch.entry_pos0, tiles, self.scale,
                                  self.window, att, Hq, Hkv, P, err=ctx.err, min_rows=2 if single else 1,
                                  kernel="mma" if self.sink_score is not None and self.weight_terms == 3 else "auto",
                                  sink_score=self.sink_score, weight_terms=self.weight_terms, **scored)

    def _forward_extended(self, proj, bt, batch, cache):
        """Kept first positions, learned sinks, mixed heads, turned values.  The queries stay float32 from the
        projection to the scores (rotation and mixing included); scores, weights and sums are float32; keys and
        values are in their pages in the activation dtype."""
        ctx, T, dev = self.ctx, proj.shape[0], proj.device
        Hq, Hkv, D, Dv = self.Hq, self.Hkv, self.D, self.Dv
        pos, vp = self.position, self.value_position
        span = Hkv if self.head_mix else 1
        # A bfloat16 run whose sizes the tensor-core kernel takes goes there with all its entries, single rows too:
        # the queries are rounded to bfloat16 once, after rotation and mixing.  Else the general kernel, float32
        # queries against the pages.
        fast = (ctx.fast_kernels and ctx.act_dtype == torch.bfloat16 and cache.k.dtype == torch.bfloat16
                and self.sink_score is None and self.scale > 0 and ops.attention_prefill_wide_usable(D, span, Dv))
        q = torch.empty((T, Hq * D), dtype=torch.bfloat16 if fast and not self.head_mix else torch.float32, device=dev)
        ops.qk_prepare_store(proj, 0, Hq * D, (Hq + Hkv) * D, batch.positions, batch.row_entry, bt, self.q_norm,
                             self.k_norm, self.qk_norm_eps or 0.0, pos.inv_freq(), pos.rotary_dim,
                             pos.pairing == "interleaved", pos.amplitude, q, cache.k, cache.v, Hq, Hkv, D, Dv,
                             cache.write, ctx.err, v_inv_freq=vp.inv_freq() if vp is not None else None,
                             v_rot_dim=vp.rotary_dim if vp is not None else 0)
        if self.head_mix:
            mixed = torch.empty((T, Hq * Hkv * D), dtype=torch.bfloat16 if fast else torch.float32, device=dev)
            ops.mix_query_heads(q, self.mix_weight, mixed, Hq, Hkv, D)
            q = mixed
        turned = vp is not None and vp.rotary_dim > 0
        att = torch.empty((T, Hq * Dv), dtype=torch.float32 if turned else ctx.act_dtype, device=dev)
        if fast:
            # A step that holds entries of one row sends them to a form of their own: where all query heads read the
            # same keys (mixed heads, or one kv head) and are at most 16, a CTA takes all heads of a row and reads
            # its keys once; else the narrow form, which also takes the step's other short entries (up to 16 rows)
            # and in which a CTA's warps share out the keys of one entry and head.  The longer entries go to the form
            # that gives a warp 16 rows of a tile, in the same step if it holds both kinds.
            short = 0
            if batch.n_single:
                by_heads = ops.attention_wide_heads_usable(D, span, Dv, Hq, Hkv, cache.v.shape[1])
                short = 1 if by_heads else ops.attention_wide_narrow_rows()
                context = batch.max_context if batch.decode_only else max(batch.max_single_context, short)
                keys = min(context, self.window + self.keep_first + short) if self.window > 0 else context
                ops.attention_prefill_wide(q, cache.k, cache.v, bt, batch.cu_rows, batch.entry_pos0, batch.S, self.scale,
                                           self.window, att, Hq, Hkv, D, Dv, keep_first=self.keep_first,
                                           sinks=self.sinks, key_span=span, narrow=True, heads=by_heads, max_keys=keys)
            if batch.n_single < batch.S:
                tiles = batch.T // ops.attention_prefill_wide_tile_rows() + batch.S
                ops.attention_prefill_wide(q, cache.k, cache.v, bt, batch.cu_rows, batch.entry_pos0, tiles, self.scale,
                                           self.window, att, Hq, Hkv, D, Dv, keep_first=self.keep_first,
                                           sinks=self.sinks, key_span=span, min_rows=short + 1)
        else:
            ops.paged_attention_general(q, cache.k, cache.v, bt, batch.row_entry, batch.positions, self.scale,
                                        self.window, att, Hq, Hkv, D, Dv, sink_score=self.sink_score, sinks=self.sinks,
                                        keep_first=self.keep_first, key_span=span)
        if turned:
            back = torch.empty((T, Hq * Dv), dtype=ctx.act_dtype, device=dev)
            ops.rotate_heads(att, batch.positions, vp.inv_freq(), vp.rotary_dim, -1.0, back, Hq, Dv)
            att = back
        return linear(ctx, att, self.o_weight, torch.float32, bias=self.o_bias)

    def _attend(self, qkv, cache, bt, batch, att):
        """Which kernel runs which rows.  float32 runs keep the plain kernel for every row, so that their sums have
        one order however the work is cut.  bfloat16 runs send entries of one row to the split-key decode kernel and
        the other entries to the prefill kernel, in the same step if it holds both kinds."""
        ctx = self.ctx
        if not (ctx.fast_kernels and ctx.act_dtype == torch.bfloat16 and cache.k.dtype == torch.bfloat16):
            ops.paged_attention_plain(qkv, cache.k, cache.v, bt, batch.row_entry, batch.positions, self.scale,
                                      self.window, att, self.Hq, self.Hkv, self.D)
            return
        single = batch.n_single if ops.attention_decode_usable(cache.k, self.D) else 0
        if single:
            ops.attention_decode(qkv, cache.k, cache.v, bt, batch.row_entry, batch.positions, self.scale, self.window,
                                 att, self.Hq, self.Hkv, self.D,
                                 batch.max_context if batch.decode_only else batch.max_single_context,
                                 rows=None if batch.decode_only else batch.single_rows, err=ctx.err)
        if single < batch.S:
            tm = ops.attention_prefill_tile_rows()
            min_rows = 2 if single else 1
            # an upper bound of the entries' tiles that depends on the step's totals only (CTAs without a tile leave
            # at once): a captured step serves every step with the same totals, however its rows are cut
            tiles = (batch.T - single) // tm + (batch.S - single)
            ops.attention_prefill(qkv, cache.k, cache.v, bt, batch.cu_rows, batch.entry_pos0, tiles, self.scale,
                                  self.window, att, self.Hq, self.Hkv, self.D, err=ctx.err, min_rows=min_rows)


def distance_buckets(rows: int, far: int) -> list:
    """For the distances 0, 1, ... up to the first that all farther ones share a row with: the row of a learned table of
    ``rows`` rows.  Below ``half = rows // 2`` every distance has its own; distance n beyond has ``half + floor(ln(n / half) /
    ln(far / half) * (rows - half))``, at most the last one.  Worked out in double."""
    half = rows // 2
    out = list(range(half))
    while not out or out[-1] < rows - 1:
        n = len(out)
        if half == 0 or far <= half:            # (no room for a logarithmic part)
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))
    return out


def _pad_heads(w, sizes, P: int):
    """Rows (or entries) of stacked heads, ``sizes`` = [(heads, elements per head)], with zeros behind every head up to P."""
    parts, at = [], 0
    for heads, d in sizes:
        block = w[at:at + heads * d].view(heads, d, *w.shape[1:])
        at += heads * d
        full = torch.zeros((heads, P, *w.shape[1:]), dtype=w.dtype, device=w.device)
        full[:, :d] = block
        parts.append(full.view(heads * P, *w.shape[1:]))
    return torch.cat(parts, dim=0).contiguous()


def _cat(ts):
    if len({t.dtype for t in ts}) > 1:
        ts = [t.float() for t in ts]
    return torch.cat(ts, dim=0).contiguous()


register_part("mixer", "paged_attention", PagedAttention)
