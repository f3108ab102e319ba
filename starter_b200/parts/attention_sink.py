"""Grouped-query attention whose positions enter through the scores and the mask: a logarithmic distance
penalty per head, chunks of the sequence, a window (which may keep the first keys), a sink in the softmax (learnt per
head, or a fixed number), a cap on the scores, a sigmoid gate per head (each optional, see ``SinkAttentionSpec``);
optionally with rotary positions on the leading entries of queries and keys, with the keys as projected standing in
for values, with biases and short convolutions behind the projections, and with queries and keys normed over their
whole rows and values over their heads.

One step of it: one stacked product gives ``[q | k | v | g]``; ``ops.sink_prepare`` files keys and values
at each token's own position and forms the gates; the attention kernel reads the queries from the stacked
rows, the keys and values from the cache, and applies the gate; the output projection follows.  A whole
prompt, a later portion and a single token are the same code: every query is told its absolute position,
and chunks are counted from the sequence's start.  With a convolution the last inputs of every channel are a
per-sequence state: ``state_at`` says where in the slot's floats they lie (another mixer may share the slot).
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache.layout import KVNeed, StateNeed
from .base import ParamSpec, Part, bytes_of


class SinkAttention(Part):
    def __init__(self, spec, dtype, position=None):
        super().__init__(spec, dtype)
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"{spec.num_heads} query heads cannot share {spec.num_kv_heads} key/value heads")
        if (position is None) != (spec.position is None):
            raise ValueError("the attention's spec and the position part it is handed do not agree")
        if spec.window is None and spec.chunk is None and spec.keep_first:
            raise ValueError("first keys are kept by a window or a chunk; this attention sees all keys")
        #: which kernel follows the projections: the one with norms (either rotation; the half-split one always), the
        #: one with the interleaved rotation alone, or the one without a rotation
        self.normed = getattr(spec.position, "kind", None) == "rope_partial" or spec.row_norm or spec.unit_values
        if (position is not None or spec.values_from_keys or self.normed) and spec.head_gate:
            raise ValueError("head gates are formed by the kernel that files keys and values without a rotation")
        if self.normed and spec.values_from_keys:
            raise ValueError("values taken from the keys go with interleaved rotary positions and no norms")
        if (spec.conv is not None or spec.bias) and spec.head_gate:
            raise ValueError("head gates have no bias and no convolution")
        if not spec.own_kv and (spec.conv is not None or spec.bias or spec.values_from_keys):
            raise ValueError("an attention without keys and values of its own has plain query projections")
        if spec.values_from_keys and spec.value_dim != spec.head_dim:
            raise ValueError(f"values taken from the keys have their size: {spec.head_dim}, not {spec.value_dim}")
        if spec.fixed_sink is not None and spec.sink:
            raise ValueError("a sink is either learnt per head or a fixed number")
        self.position = position
        if max(spec.head_dim, spec.value_dim) > 256:
            raise ValueError(f"head sizes {spec.head_dim} / {spec.value_dim} exceed the 256 entries the kernels take")
        self.q_size = spec.num_heads * spec.head_dim
        self.kv_size = spec.num_kv_heads * (spec.head_dim + (0 if spec.values_from_keys else spec.value_dim))
        self.penalty = self.sink = self.taps = self.biases = self.row_norm = None
        #: what a short convolution runs over: every channel of q, k and v, and the stacked product's padding
        self.convolved = -(-(self.q_size + self.kv_size) // 8) * 8
        self.state_at = 0

    def kv_need(self):
        s = self.spec
        if not s.own_kv:
            return None
        # every key stays: a later query of the same chunk may still read it (chunks bound what is read)
        return KVNeed(s.num_kv_heads, s.head_dim, s.window, s.value_dim)

    def state_need(self):
        taps = self.spec.conv or 1
        return StateNeed(((taps - 1) * self.convolved,), "float32") if taps > 1 else None

    def param_specs(self):
        s = self.spec
        if not s.own_kv:
            out = {"q": ParamSpec((self.q_size, s.hidden_size)), "o": ParamSpec((s.hidden_size, s.num_heads * s.value_dim))}
            return {**out, **self._extra_specs()}
        out = {
            "q": ParamSpec((self.q_size, s.hidden_size)),
            "k": ParamSpec((s.num_kv_heads * s.head_dim, s.hidden_size)),
            "v": ParamSpec((s.num_kv_heads * s.value_dim, s.hidden_size)),
            "o": ParamSpec((s.hidden_size, s.num_heads * s.value_dim)),
        }
        if s.values_from_keys:
            del out["v"]
        return {**out, **self._extra_specs()}

    def _projected(self):
        """``{name: channels}`` of the projections this layer has."""
        s = self.spec
        out = {"q": self.q_size}
        if s.own_kv:
            out["k"] = s.num_kv_heads * s.head_dim
            if not s.values_from_keys:
                out["v"] = s.num_kv_heads * s.value_dim
        return out

    def _extra_specs(self):
        s, out = self.spec, {}
        for name, channels in self._projected().items():
            if s.bias:
                out[f"{name}_bias"] = ParamSpec((channels,), "bias32")
            if s.conv is not None:
                out[f"{name}_conv"] = ParamSpec((channels, s.conv), "vector32")
            if s.row_norm and name != "v":
                out[f"{name}_norm"] = ParamSpec((channels,), "gain32")
        if s.distance_penalty:
            out["r1"] = ParamSpec((s.num_heads,), "vector32")
            out["r2"] = ParamSpec((s.num_heads,), "slope")
        if s.sink:
            out["sink"] = ParamSpec((s.num_heads,), "vector32")
        if s.head_gate:
            out["g"] = ParamSpec((s.num_heads, s.hidden_size))
        return out

    def set_params(self, params):
        s = self.spec
        def stacked(rows):
            # rows of zeros bring the product's width to a multiple of 8, so that every token's queries
            # start on a 16-byte boundary for the kernels that copy them in 16-byte pieces
            pad = -sum(r.shape[0] for r in rows) % 8
            if pad:
                rows = rows + [torch.zeros((pad, s.hidden_size), dtype=rows[0].dtype, device=rows[0].device)]
            return torch.cat(rows, dim=0).contiguous()

        projected = self._projected()
        self.qkvg = None
        if s.own_kv:
            self.qkvg = stacked([params[n] for n in projected] + ([params["g"]] if s.head_gate else []))
        def channels(name):
            rows = torch.cat([params[f"{n}_{name}"].float() for n in projected], dim=0)
            padding = rows.new_zeros((self.convolved - rows.shape[0], *rows.shape[1:]))
            return torch.cat([rows, padding], dim=0).contiguous()

        if s.bias:
            self.biases = channels("bias")
        if s.conv is not None:
            self.taps = channels("conv")
        elif s.bias:
            # the bias alone: one tap that passes the current token through
            self.taps = torch.ones((self.convolved, 1), dtype=torch.float32, device=self.biases.device)
        if s.row_norm:
            self.row_norm = (params["q_norm"].float().contiguous(),
                             params["k_norm"].float().contiguous() if s.own_kv else None)
        # the rows a layer that only reads another layer's cache needs: queries and gates
        self.qg = stacked([params["q"]] + ([params["g"]] if s.head_gate else []))
        self.o = params["o"].contiguous()
        if s.distance_penalty:
            self.penalty = (params["r1"].float().contiguous(), params["r2"].float().contiguous())
        if s.sink:
            self.sink = params["sink"].float().contiguous()
        elif s.fixed_sink is not None:
            self.sink = torch.full((s.num_heads,), float(s.fixed_sink), dtype=torch.float32, device=self.o.device)

    def prepare(self, max_position: int) -> bool:
        """Host-side growth before a step; True if device tables were reallocated."""
        if self.position is not None:
            return bool(self.position.ensure(max_position + 1))
        return False

    def __call__(self, x, ctx, entry, writes_cache=True):
        s = self.spec
        cache = ctx.cache
        keys, values = cache.entry_pages(entry)
        if writes_cache and not s.own_kv:
            raise ValueError("this attention has no keys and values to write; the run order must name it a reader")
        if not writes_cache and self.taps is not None:
            raise ValueError("this attention's biases and convolutions cover keys and values; it cannot only read")
        weight = self.qkvg if writes_cache else self.qg
        proj = ops.linear(x, weight, status=ctx.status)
        if self.taps is not None:
            proj = ops.short_conv(proj, 0, self.convolved, self.taps, None, self.biases, cache.entry_state(entry),
                                  self.state_at, ctx.seq_slot, ctx.seq_q_start, ctx.seq_q_len, ctx.max_q_len)
        if self.normed:
            # queries normed and turned in place; keys normed and turned, values normed on their way into the cache
            ops.sink_prepare_norm(proj, s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim, ctx.tok_pos, ctx.tok_slot,
                                  cache.block_table, keys, values,
                                  self.position.rotation() if self.position is not None else None, self.row_norm,
                                  s.unit_values, s.norm_eps, write_cache=writes_cache)
            a = ops.sink_attention_step(proj, keys, values, cache.block_table, ctx, s.num_heads, s.num_kv_heads,
                                        s.head_dim, s.value_dim, s.scale, self.penalty, self.sink, None, s.chunk, s.window,
                                        s.keep_first, s.softcap)
            return ops.linear(a, self.o, status=ctx.status)
        if self.position is not None or s.values_from_keys:
            # queries turned in place, keys turned on their way into the cache, values as projected
            cos, sin, dims = ops.sink_tables(self.position.rotation() if self.position is not None else None, s.head_dim)
            ops.sink_prepare_rot(proj, s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim, ctx.tok_pos, ctx.tok_slot,
                                 cache.block_table, keys, values, cos, sin, dims, values_from_keys=s.values_from_keys,
                                 write_cache=writes_cache)
            a = ops.sink_attention_step(proj, keys, values, cache.block_table, ctx, s.num_heads, s.num_kv_heads,
                                        s.head_dim, s.value_dim, s.scale, self.penalty, self.sink, None, s.chunk, s.window,
                                        s.keep_first, s.softcap)
            return ops.linear(a, self.o, status=ctx.status)
        gate = ops.sink_prepare(proj, s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim, ctx.tok_pos, ctx.tok_slot,
                                cache.block_table, keys, values, gated=s.head_gate, write_cache=writes_cache)
        a = ops.sink_attention_step(proj, keys, values, cache.block_table, ctx, s.num_heads, s.num_kv_heads,
                                    s.head_dim, s.value_dim, s.scale, self.penalty, self.sink, gate, s.chunk, s.window,
                                    s.keep_first, s.softcap)
        return ops.linear(a, self.o, status=ctx.status)

    def weight_bytes(self):
        return bytes_of(self.qkvg if self.qkvg is not None else self.qg, self.o, self.sink, self.taps, self.biases,
                        *(self.penalty or ()), *(self.row_norm or ()))
