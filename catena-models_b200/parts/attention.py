"""Grouped-query attention mixer with head RMSNorm on q and k, a position encoding, a full or
sliding causal mask and an optional per-head sigmoid gate on the output.

Order of operations (src/lfm3.rs:390-464): one matrix product over the packed rows
[Wq; Wk; Wv; Wgate] (src/lfm3.rs:1159-1262); head norm and rotation of q and k, k and the raw v
written to the cache (src/catena/lfm3.hex:622-781); scores scaled by 1/sqrt(head_dim), keys
hidden when k > p or, with a window W, when k + W <= p (src/catena/lfm3.hex:48-57); softmax and
the value sum in float; context times sigmoid(gate) per head (src/catena/lfm3.hex:25-46);
output projection.

A prompt step attends over the step's own keys and values (every sequence of such a step
starts at position 0); a decode step attends over the cache; an append step (several tokens on
top of started sequences) reads the keys below each sequence's first new position from the cache
and the rest from the step, and writes the step's keys and values to the cache afterwards, so
that a ring still holds what the step's windows reach back to.  All sizes and switches are
constructor parameters; the part knows neither its layer index nor its model.

Further switches, all off by default: `scale` (the factor on q . k instead of 1/sqrt(head_dim)); `sink_name`
(a learned logit per query head that joins the softmax's denominator and has neither key nor value);
`q_temp` = (coef, every), a factor 1 + coef * ln(floor((p + 1) / every) + 1) on the queries at position p;
`value_dim`, the size of a value head when it differs from the size of a query or key head.  The kernels
and the cache work with one head size, so heads of unequal or odd sizes are padded with zero rows of the
projections up to a common multiple of 16 (zero channels change no score and give zero outputs, which meet
zero columns of the output projection); `out_dtype` = "float32" leaves the output projection's result in float.

`chunk` = C > 0 (instead of a window): position p sees the earlier positions of its own chunk of C, chunks counted from the
sequence's start; the cache is a ring that holds the last C positions, as for a window of C.  `sink_value`: a constant logit
for every query head in place of the learned ones.  With a head norm, padded heads are normed over their real channels.

`softcap` = c > 0 bounds every score before the mask and the softmax: s <- c * tanh(s / c), s = (q . k) * scale.

`taps` = K >= 1 puts a short causal filter behind the query and key projections, one set of K taps per channel
(`q_taps`, `k_taps` name the tensors, [channels, K]): y_t = sum_j w[:, j] u_(t - K + 1 + j), zeros before the sequence's
start, before the rotation (K = 1 is a factor per channel; 0: no filter and no tensors).  For K > 1 the last K projected
rows of a sequence are part of the layer's state (float32, a ring beside the key/value pages).  `value_from_key`: the layer has no value projection; a position's value is its key
as the filter leaves it, before the rotation.  Filter, rotation and the cache write are one kernel
(`kernels.tap_rotate_store`), which leaves the step's rows as [q | turned k | v] for the attention kernels.

`bias`: q, k, v and the output projection have biases (`q_bias`, `k_bias`, `v_bias`, `out_bias` name the tensors).
`gate_channels` (with `output_gate`): the gate has a logit per channel of the concatenated heads instead of one per head.
`value_mix` = (role, name): values are mixed with those of another layer of the same step, v <- (1 - a) v + a v_first, before
they are cached; `name` is the tensor of the one number a, role "source" marks the layer whose own values (with their bias) are
v_first (its number is not used), "mix" the layers that mix.  With a bias, a mix or a position encoding that turns part of a
head (`position.dims`), everything between the projection and the attention is one kernel (`kernels.head_prepare`).
"""
from __future__ import annotations


import torch

from .. import kernels
from ..cache.spec import CompositeStateSpec, FixedStateSpec, KVStateSpec
from ..csrc.limits import ATTN_DECODE_CHUNK
from ..weights.loader import TensorSpec
from .base import Mixer, register_part
from .linear import Linear


class GQAttention(Mixer):
    prompt_capturable = True
    fused_decode_ok = True
    supports_append = True

    def __init__(self, prefix, hidden, heads, kv_heads, head_dim, window, position, qk_norm_eps,
                 output_gate, names=None, shares_kv=False, scale=None, sink_name=None, q_temp=None, value_dim=None,
                 out_dtype=None, softcap=0.0, taps=0, value_from_key=False, chunk=0, sink_value=None, bias=False,
                 gate_channels=False, value_mix=None):
        names = names or {}
        n = lambda key, default: prefix + names.get(key, default)
        qk_dim, v_dim = head_dim, value_dim or head_dim
        self.bias, self.value_mix = bool(bias), value_mix
        self.gate_channels = bool(gate_channels) and bool(output_gate)
        filtered = bool(taps) or bool(value_from_key)
        self.one_prepare = not filtered and (self.bias or value_mix is not None or bool(getattr(position, "dims", 0)))
        if value_mix is not None and value_mix[0] not in ("source", "mix"):
            raise ValueError("GQAttention: value_mix ('source' | 'mix', tensor name)")
        if (self.one_prepare or self.gate_channels) and (shares_kv or q_temp or filtered):
            raise ValueError("GQAttention: biases, mixed values, partial rotation and gates per channel go with neither shared keys, "
                             "filters nor a query temperature")
        if self.bias and out_dtype != "float32":
            raise ValueError("GQAttention: the output bias joins a float32 residual sum")
        if v_dim != qk_dim or ((scale is not None or self.one_prepare) and qk_dim % 16):
            head_dim = -(-max(qk_dim, v_dim) // 16) * 16       # one padded head size for q, k and v
        pad_qk = (heads, qk_dim, head_dim) if head_dim != qk_dim else None
        pad_k = (kv_heads, qk_dim, head_dim) if head_dim != qk_dim else None
        pad_v = (kv_heads, v_dim, head_dim) if head_dim != v_dim else None
        self.qk_dim, self.v_dim = qk_dim, v_dim
        self.softcap, self.taps, self.value_from_key = float(softcap or 0.0), int(taps or 0), bool(value_from_key)
        if self.softcap < 0.0 or self.taps < 0:
            raise ValueError("GQAttention: softcap >= 0 and taps >= 0")
        if self.value_from_key and (v_dim != qk_dim or shares_kv):
            raise ValueError("GQAttention: values that are the keys have the keys' size, and a layer of its own keys")
        if (self.taps > 0 or self.value_from_key) and (shares_kv or qk_norm_eps is not None or q_temp or output_gate):
            raise ValueError("GQAttention: the filtered form has neither head norm, query temperature, gate nor shared keys")
        self.filtered = self.taps > 0 or self.value_from_key
        if self.filtered or self.one_prepare:
            self.fused_decode_ok = False       # its decode step runs a kernel of its own between the products
        self.sink_name, self.sink = (prefix + sink_name if sink_name else None), None
        self.q_temp = (float(q_temp[0]), int(q_temp[1])) if q_temp else None
        self.out_dtype = {None: None, "float32": torch.float32}[out_dtype]
        self.hidden, self.heads, self.kv_heads, self.head_dim = hidden, heads, kv_heads, head_dim
        if chunk and window:
            raise ValueError("GQAttention: a window or chunks, not both")
        if sink_name and sink_value is not None:
            raise ValueError("GQAttention: learned sinks or a constant one")
        self.sink_value = sink_value
        self.window = int(window or 0)
        self.reach = self.window or int(chunk or 0)          # how many positions the cache keeps (0: all)
        self.mask = -int(chunk) if chunk else self.window    # the mask as the attention kernels take it
        self.position = position
        self.qk_norm_eps = qk_norm_eps           # None: no head norm
        self.output_gate = bool(output_gate)
        self.q_size, self.kv_size = heads * head_dim, kv_heads * head_dim
        # shares_kv: this layer has no key/value projections of its own; it attends over the keys
        # and values of the layer that owns the state unit the plan gives it
        self.shares_kv = bool(shares_kv)
        mats, rows, pads = [n("q", "attn_q.weight")], [heads * qk_dim], [pad_qk]
        if not self.shares_kv:
            mats.append(n("k", "attn_k.weight"))
            rows.append(kv_heads * qk_dim)
            pads.append(pad_k)
            if not self.value_from_key:
                mats.append(n("v", "attn_v.weight"))
                rows.append(kv_heads * v_dim)
                pads.append(pad_v)
        if self.output_gate:
            mats.append(n("gate", "attn_gate.weight"))
            rows.append(heads * v_dim if self.gate_channels else heads)
            pads.append(None)
        self.qkvg = Linear(mats, rows, hidden, head_rows=pads, row_multiple=8 if self.one_prepare or self.gate_channels else 1)
        # channels of a head that the attention leaves: all, or with a gate per channel those that are no padding
        self.ctx_dim = v_dim if self.gate_channels else head_dim
        self.bias_names = [n("q_bias", "attn_q.bias"), n("k_bias", "attn_k.bias"), n("v_bias", "attn_v.bias")] if self.bias else []
        self.out_bias_name = n("out_bias", "attn_output.bias") if self.bias else None
        self.qkv_bias = self.out_bias = self.mix_share = None
        self.out = Linear(n("out", "attn_output.weight"), hidden, heads * v_dim,
                          head_cols=(heads, v_dim, head_dim) if head_dim != v_dim and not self.gate_channels else None)
        self.q_norm_name, self.k_norm_name = n("q_norm", "attn_q_norm.weight"), n("k_norm", "attn_k_norm.weight")
        self.q_norm_w = self.k_norm_w = None
        self.tap_names = (n("q_taps", "attn_q.conv"), n("k_taps", "attn_k.conv")) if self.taps > 0 else ()
        self.tap_w = None
        # 1/sqrt(head_dim) in float32, as the reference bakes it (src/catena/qwen35_wmma_attention.hex:3-22)
        self.scale = float(torch.tensor(1.0, dtype=torch.float32) / torch.sqrt(torch.tensor(float(qk_dim), dtype=torch.float32)))
        if scale is not None:
            self.scale = float(scale)

    def children(self):
        return [self.qkvg, self.out, self.position]

    def tensor_specs(self):
        specs = [TensorSpec(self.sink_name, (self.heads,), "vector")] if self.sink_name else []
        if self.taps > 0:
            specs += [TensorSpec(self.tap_names[0], (self.heads * self.qk_dim, self.taps), "conv"),
                      TensorSpec(self.tap_names[1], (self.kv_heads * self.qk_dim, self.taps), "conv")]
        if self.bias:
            sizes = [self.heads * self.qk_dim, self.kv_heads * self.qk_dim, self.kv_heads * self.v_dim, self.hidden]
            specs += [TensorSpec(name, (size,), "vector") for name, size in zip(self.bias_names + [self.out_bias_name], sizes)]
        if self.value_mix is not None:
            specs.append(TensorSpec(self.value_mix[1], (), "vector"))
        if self.qk_norm_eps is None:
            return specs
        specs.append(TensorSpec(self.q_norm_name, (self.qk_dim,), "norm"))
        if not self.shares_kv:
            specs.append(TensorSpec(self.k_norm_name, (self.qk_dim,), "norm"))
        return specs

    def bind(self, tensors, rt):
        self._bound = []
        if self.filtered:
            if self.taps > 0:
                # heads padded with zero channels get taps of zero
                padded = []
                for t in self.tap_names:
                    w = tensors[t].to(torch.float32).view(-1, self.qk_dim, self.taps)
                    full = torch.zeros((w.shape[0], self.head_dim, self.taps), dtype=torch.float32, device=w.device)
                    full[:, :self.qk_dim] = w
                    padded.append(full.view(-1, self.taps))
                self.tap_w = torch.cat(padded).contiguous()
            else:
                self.tap_w = torch.ones((self.q_size + self.kv_size, 1), dtype=torch.float32, device=rt.device)
            self._bound.append(self.tap_w)
        if self.bias:
            parts = []
            for name, size in zip(self.bias_names, (self.qk_dim, self.qk_dim, self.v_dim)):
                parts.append(torch.nn.functional.pad(tensors[name].to(torch.float32).view(-1, size), (0, self.head_dim - size)).reshape(-1))
            self.qkv_bias = torch.cat(parts).contiguous()
            self.out_bias = tensors[self.out_bias_name].to(torch.float32).contiguous()
            self._bound += [self.qkv_bias, self.out_bias]
        if self.value_mix is not None and self.value_mix[0] == "mix":
            self.mix_share = tensors[self.value_mix[1]].to(torch.float32).reshape(1).contiguous()
            self._bound.append(self.mix_share)
        if self.sink_name:
            self.sink = tensors[self.sink_name].to(torch.float32).contiguous()
            self._bound.append(self.sink)
        elif self.sink_value is not None:
            self.sink = torch.full((self.heads,), float(self.sink_value), dtype=torch.float32, device=rt.device)
            self._bound.append(self.sink)
        if self.qk_norm_eps is not None:
            padded = lambda w: torch.nn.functional.pad(w.to(torch.float32), (0, self.head_dim - self.qk_dim)).contiguous()
            self.q_norm_w = padded(tensors[self.q_norm_name])
            self._bound.append(self.q_norm_w)
            if not self.shares_kv:
                self.k_norm_w = padded(tensors[self.k_norm_name])
                self._bound.append(self.k_norm_w)

    def state_spec(self):
        kv = KVStateSpec(self.kv_heads, self.head_dim, self.reach)
        if self.taps > 1:
            # a ring of `taps` projected rows [q | k] per sequence, the row of position s in row s % taps
            return CompositeStateSpec((kv, FixedStateSpec((self.taps * (self.q_size + self.kv_size),), "float32")))
        return kv

    def _forward_filtered(self, rt, batch, x, state):
        """q and k behind the taps, v = k before the rotation: one kernel leaves [q | turned k | v] side by side
        and, except in an append step (whose attention reads what is older from the cache first), in the cache."""
        QS, KVS, QH, KVH, HD = self.q_size, self.kv_size, self.heads, self.kv_heads, self.head_dim
        kv, own = state.views if self.taps > 1 else (state, None)
        proj = self.qkvg.apply(rt, x)                                    # [T, QS + KVS]
        decode = batch.kind == "decode"
        # a decode step needs the queries only: its keys and values go straight to the cache
        packed = torch.empty((batch.T, QS if decode else QS + 2 * KVS), dtype=x.dtype, device=x.device)
        rate = self.position.rate_table()
        kernels.tap_rotate_store(proj, None, self.tap_w, None if own is None else own.tensor, packed, batch, QS, HD, rate,
                                 getattr(self.position, "magnitude", 1.0),
                                 kv=(kv.pool, kv.pages, kv.ptab, KVH, HD, 0), one_token_each=decode,
                                 interleaved=self.position.pairing == "interleaved", value_from_key=True, ring=kv.ring,
                                 store=not batch.append, rows_out=not decode, from_zero=batch.prefill)
        q = packed[:, :QS]
        ctx = torch.empty((batch.T, QS), dtype=x.dtype, device=x.device)
        if decode:
            entries = kv.spec.entries(kv.spec.length_class(batch.max_end))
            n_chunks = max(1, -(-entries // ATTN_DECODE_CHUNK))
            part_o, part_ml = rt.scratch_attn_decode(batch.B, QH, HD, n_chunks)
            kernels.attn_decode(ctx, q, None, batch.seq_pos0, batch.seq_slot, kv.pool, kv.pages, kv.ptab, kv.ring,
                                self.mask, QH, KVH, HD, n_chunks, self.scale, part_o, part_ml, sink=self.sink,
                                softcap=self.softcap)
        else:
            k, v = packed[:, QS:QS + KVS], packed[:, QS + KVS:]
            if batch.append:
                rt.attention_append(ctx, q, k, v, None, batch, kv, QH, KVH, HD, self.mask, self.scale, sink=self.sink,
                                    softcap=self.softcap)
                kernels.kv_store(packed[:, QS:], batch.tok_pos, batch.tok_seq, batch.seq_slot, batch.seq_end, kv.pool,
                                 kv.pages, kv.ptab, kv.ring, KVH, HD)
            else:
                rt.attention_prefill(ctx, q, k, v, None, batch, QH, KVH, HD, self.mask, self.scale, sink=self.sink,
                                     softcap=self.softcap)
        return self.out.apply(rt, ctx, out_dtype=self.out_dtype)

    def _prepare(self, batch, proj, state):
        """Biases, head norms, rotation, mixed values and (except in an append step) the cache write, in place."""
        QS, KVS, HD = self.q_size, self.kv_size, self.head_dim
        mix = None
        if self.mix_share is not None:
            if "v_first" not in batch.shared:
                raise ValueError("GQAttention: mixed values need an earlier layer of the step with value_mix ('source', ...)")
            mix = (*batch.shared["v_first"], self.mix_share)
        kv = None if batch.append else (state.pool, state.pages, state.ptab, state.ring)
        kernels.head_prepare(proj, batch, self.heads, self.kv_heads, HD, bias=self.qkv_bias, wq=self.q_norm_w, wk=self.k_norm_w,
                             norm_dim=self.qk_dim, eps=self.qk_norm_eps or 0.0, rate=self.position.rate_table(),
                             interleaved=self.position.pairing == "interleaved", mag=getattr(self.position, "magnitude", 1.0),
                             value_dim=self.v_dim, mix=mix, kv=kv)
        if self.value_mix is not None and self.value_mix[0] == "source":
            batch.shared["v_first"] = (proj[:, QS + KVS:QS + 2 * KVS], self.v_dim, HD)

    def forward(self, rt, batch, x, state):
        QS, KVS, QH, KVH, HD = self.q_size, self.kv_size, self.heads, self.kv_heads, self.head_dim
        if self.filtered:
            return self._forward_filtered(rt, batch, x, state)
        if self.shares_kv != (not state.owned):
            raise ValueError("a layer that shares keys and values must be given another layer's state unit "
                             "by the plan (owns_state=False), and only such a layer")
        proj = self.qkvg.apply(rt, x)                  # [T, QS + 2 KVS (+ QH)], or [T, QS (+ QH)] when sharing
        interleaved = self.position.pairing == "interleaved"
        if self.one_prepare:
            self._prepare(batch, proj, state)
            gate = proj[:, QS + 2 * KVS:] if self.output_gate else None
        elif self.shares_kv:
            # q only: head norm and rotation over the q heads, nothing written to the cache
            kernels.qk_prepare(proj, self.q_norm_w, None, self.position.rate_table(), batch.tok_pos, batch.tok_seq,
                               batch.seq_slot, batch.seq_end, None, 0, None, 0, QH, 0, HD, self.qk_norm_eps or 0.0,
                               interleaved=interleaved, q_temp=self.q_temp, norm_dim=self.qk_dim)
            gate = proj[:, QS:] if self.output_gate else None
        else:
            # an append step keeps the cache as it is until its attention has run
            pool = None if batch.append else state.pool
            kernels.qk_prepare(proj, self.q_norm_w, self.k_norm_w, self.position.rate_table(), batch.tok_pos,
                               batch.tok_seq, batch.seq_slot, batch.seq_end, pool, state.pages, state.ptab,
                               state.ring, QH, KVH, HD, self.qk_norm_eps or 0.0, interleaved=interleaved, q_temp=self.q_temp,
                               norm_dim=self.qk_dim)
            gate = proj[:, QS + 2 * KVS:] if self.output_gate else None
        q = proj[:, :QS]
        ctx = torch.empty((batch.T, QH * self.ctx_dim), dtype=x.dtype, device=x.device)
        stored = {"value_dim": self.ctx_dim, "gate_channels": self.gate_channels}
        if batch.prefill or batch.append:
            if self.shares_kv and batch.append and state.ring:
                raise NotImplementedError("an append step of a layer that shares the keys and values of a sliding "
                                          "layer: the owner's ring no longer holds what this layer's windows need")
            if self.shares_kv:
                # the owner left this step's keys and values for its readers; bring them beside q so
                # that the attention kernel sees one packed buffer
                k_own, v_own = batch.shared[("kv", state.unit)]
                packed = torch.empty((batch.T, QS + 2 * KVS), dtype=x.dtype, device=x.device)
                packed[:, :QS].copy_(q)
                packed[:, QS:QS + KVS].copy_(k_own)
                packed[:, QS + KVS:].copy_(v_own)
                q, k, v = packed[:, :QS], packed[:, QS:QS + KVS], packed[:, QS + KVS:]
            else:
                k, v = proj[:, QS:QS + KVS], proj[:, QS + KVS:QS + 2 * KVS]
                batch.shared[("kv", state.unit)] = (k, v)
            if batch.append:
                rt.attention_append(ctx, q, k, v, gate, batch, state, QH, KVH, HD, self.mask, self.scale, sink=self.sink,
                                    softcap=self.softcap, **stored)
                if not self.shares_kv:
                    kernels.kv_store(proj[:, QS:QS + 2 * KVS], batch.tok_pos, batch.tok_seq, batch.seq_slot,
                                     batch.seq_end, state.pool, state.pages, state.ptab, state.ring, KVH, HD)
            else:
                rt.attention_prefill(ctx, q, k, v, gate, batch, QH, KVH, HD, self.mask, self.scale, sink=self.sink,
                                     softcap=self.softcap, **stored)
        else:
            # launched for the longest sequence that this step's length class allows, so that a
            # recording of the step serves every step of the class
            entries = state.spec.entries(state.spec.length_class(batch.max_end))
            n_chunks = max(1, -(-entries // ATTN_DECODE_CHUNK))
            part_o, part_ml = rt.scratch_attn_decode(batch.B, QH, HD, n_chunks)
            kernels.attn_decode(ctx, q, gate, batch.seq_pos0, batch.seq_slot, state.pool, state.pages, state.ptab,
                                state.ring, self.mask, QH, KVH, HD, n_chunks, self.scale, part_o, part_ml, sink=self.sink,
                                softcap=self.softcap, **stored)
        if self.bias:
            return kernels.Terms([(self.out.apply(rt, ctx, out_dtype=self.out_dtype), 1.0, 1), (self.out_bias, 1.0, 0)])
        return self.out.apply(rt, ctx, out_dtype=self.out_dtype, partial_ok=batch.partial_sums_ok and self.out_dtype is None)


register_part("mixer", "gqa_attention", GQAttention)
