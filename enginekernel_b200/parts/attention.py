"""Grouped-query attention over the paged cache.

Per token: q/k/v projections without bias (one fused product), optional RMSNorm of each
query and key head over the head dimension, position encoding of queries and keys, keys
and values stored in the cache entry, softmax(scale * q.K^T) V over the keys the token may
see (all earlier ones, or the last ``window``), output projection
(engine/ek_model.py:298-325 for prompts, 380-403 for decode; formula 475-488).
Query head h reads KV head h // (num_heads // num_kv_heads).

Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``scale``,
``qk_norm_eps`` (None: no q/k norm), ``window`` (None: all keys), ``position`` (a
position PartSpec or None).  Tensors: ``q`` [NH*D, H], ``k``, ``v`` [NKV*D, H], ``o``
[H, NH*D], and with q/k norm ``q_norm``, ``k_norm`` [D].  q, k and v are concatenated at
load as the reference does (engine/ek_model.py:140-144).

Optional parameters, all off by default, for designs that differ there:

``bias``               which of ``"q"``, ``"k"``, ``"v"`` carry a bias (tensors ``q_bias`` ...
                       [heads * D]); it is added in 32-bit before the head norm.  ``"o"``: the output projection
                       has one (``o_bias`` [H]), added behind its product or, with ``leave_bias=True``, left to the
                       reader of the result.
``values``             ``"keys"``: there is no value projection - a token's value is its key as
                       projected (with bias, before the key's norm and rotation).
``query_temperature``  ``(coef, every)``: the query of the token at position p is multiplied by
                       1 + coef * ln(floor((p + 1) / every) + 1).
``sink``               the score of one more key without a value that every query sees: its
                       exponential is one more term of the softmax denominator (0.0: "+ 1").
``value_dim``          size of a value head when it differs from ``head_dim`` (``v`` is then [NKV * E, H]
                       and ``o`` [H, NH * E]); the cache and the kernels see heads of the larger of the
                       two sizes (rounded up to 8 values), the shorter ones padded with zeros.
``unit_norm_after_rotation``  an eps: queries and keys are rotated first and then divided by their root
                       mean square over the head (no gain), instead of the gained norm before rotation.
``keep_first``         with a window: the first ``keep_first`` positions of a sequence stay visible to every
                       later token, at their true positions.  The cache then keeps all keys.
``head_gate``          every head's output is multiplied by the sigmoid of one number per token and head,
                       a projection of the mixer's input (tensor ``gate`` [NH, H]), before ``o``.
``kv_projection``      False: the layer has no ``k`` and ``v``; it reads the keys and values another run
                       stored in the cache entry it shares (a run with ``writes_cache=False``).
``keep_all_keys``      the cache keeps every key although this layer sees a window (layers that share an
                       entry may see different windows).
``chunk``              position p sees only its own chunk of positions, floor(p / chunk), counted from the
                       sequence's first position.
``cache_window``       how many of a sequence's last keys the cache entry has to keep (default: the window or
                       the chunk); layers that share an entry name the largest of theirs.
``softcap``            a score s becomes softcap * tanh(s / softcap) before the softmax.
``pairing``            ``"neighbours"``: the rotation turns values (2i, 2i + 1) of a head instead of (i, i + rot/2);
                       the rows of the query and key projections are reordered once at load.
``qk_norm_over``       ``"projection"``: the gained norm takes one mean over all query heads of a token and one over
                       all its key heads (``q_norm`` [NH*D], ``k_norm`` [NKV*D]) instead of one per head.
``sinks``              True: a learned sink score per query head (tensor ``sink`` [NH]) instead of one constant.
``value_dim``, ``unit_norm_after_rotation``, ``keep_first`` and ``head_gate`` send the layer down one path: a single
product for everything that reads the input, a prepare kernel that knows padded heads, and the ``mma.sync`` or the
general attention kernel.  The others ride on the ordinary path.
"""

from __future__ import annotations

import torch

from ..ops import kernels
from ..ops.linear import linear, pair_product_wins, row_scale_of, tc_takes
from ..registry import lookup_part, register_part
from .base import DeferredNorm, Mixer
from .rope import neighbours_to_halves
from .spec import CacheSpec, TensorSpec

FUSE_ROPE_ROWS = 64       # the q/k/v product does norm, rotation and cache write itself up to here
WIDE_CLUSTER_PAGES = 64     # clusters of more than 8 key splits only from this many pages of context


@register_part("mixer", "attention")
class Attention(Mixer):
    @classmethod
    def tensors(cls, spec):
        p, w = spec.params, spec.weights
        h, nh, nkv, d = p["hidden_size"], p["num_heads"], p["num_kv_heads"], p["head_dim"]
        e = int(p.get("value_dim") or d)
        out = [TensorSpec(w["q"], (nh * d, h))]
        if p.get("kv_projection", True):
            out.append(TensorSpec(w["k"], (nkv * d, h)))
            if p.get("values", "projection") != "keys":
                out.append(TensorSpec(w["v"], (nkv * e, h)))
        if p.get("head_gate"):
            out.append(TensorSpec(w["gate"], (nh, h)))
        out.append(TensorSpec(w["o"], (h, nh * e)))
        if p.get("qk_norm_eps") is not None:
            whole = p.get("qk_norm_over", "head") == "projection"
            out.append(TensorSpec(w["q_norm"], (nh * d if whole else d,), "gain"))
            if p.get("kv_projection", True):     # (else the keys it reads were normed by the run that stored them)
                out.append(TensorSpec(w["k_norm"], (nkv * d if whole else d,), "gain"))
        if p.get("sinks"):
            out.append(TensorSpec(w["sink"], (nh,)))
        sizes = {"q": nh * d, "k": nkv * d, "v": nkv * e, "o": h}
        for which in p.get("bias") or ():
            if p.get("kv_projection", True) or which in ("q", "o"):
                out.append(TensorSpec(w[which + "_bias"], (sizes[which],)))
        return out

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        self.hidden = int(self.param("hidden_size"))
        self.num_heads = int(self.param("num_heads"))
        self.num_kv_heads = int(self.param("num_kv_heads"))
        self.head_dim = int(self.param("head_dim"))
        self.scale = float(self.param("scale"))
        self.qk_norm_eps = spec.params.get("qk_norm_eps")
        self.window = spec.params.get("window")
        self.kv_projection = bool(spec.params.get("kv_projection", True))
        bias = tuple(spec.params.get("bias") or ())
        self.output_biased = "o" in bias
        self.biased = tuple(b for b in bias if b != "o" and (self.kv_projection or b == "q"))
        self.chunk = spec.params.get("chunk")
        self.softcap = spec.params.get("softcap")
        self.neighbours = spec.params.get("pairing", "halves") == "neighbours"
        if spec.params.get("pairing", "halves") not in ("halves", "neighbours"):
            raise ValueError("attention: pairing is 'halves' or 'neighbours'")
        if self.chunk is not None and (self.chunk < 1 or self.window or spec.params.get("keep_first")):
            raise ValueError("attention: a chunk is at least 1 and takes the place of a window")
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError("attention: the soft cap must be positive")
        self.values_from_keys = spec.params.get("values", "projection") == "keys"
        self.query_temperature = spec.params.get("query_temperature")
        self.sink = spec.params.get("sink")
        self.has_sinks = bool(spec.params.get("sinks"))
        if self.has_sinks and self.sink is not None:
            raise ValueError("attention: one sink score for all heads or one per head, not both")
        if spec.params.get("qk_norm_over", "head") not in ("head", "projection"):
            raise ValueError("attention: the norm of queries and keys is over a 'head' or the 'projection'")
        self.whole_norm = spec.params.get("qk_norm_over", "head") == "projection"
        if spec.params.get("values", "projection") not in ("projection", "keys"):
            raise ValueError("attention: values are 'projection' or 'keys'")
        if any(b not in ("q", "k", "v") for b in self.biased) or (self.values_from_keys and "v" in self.biased):
            raise ValueError("attention: bias names q, k, v (v only with a value projection)")
        if self.query_temperature is not None and int(self.query_temperature[1]) < 1:
            raise ValueError("attention: the query temperature steps every >= 1 positions")
        if self.whole_norm and (self.qk_norm_eps is None or self.biased or self.values_from_keys
                                or self.query_temperature is not None):
            raise ValueError("attention: a norm over the projection needs qk_norm_eps and does not combine with biases, "
                             "values from keys or a query temperature")
        self.bias = {"q": None, "k": None, "v": None}
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        kernels.check_head_dim(self.head_dim)
        self.value_dim = int(spec.params.get("value_dim") or self.head_dim)
        self.unit_norm_eps = spec.params.get("unit_norm_after_rotation")
        self.keep_first = int(spec.params.get("keep_first") or 0)
        self.head_gate = bool(spec.params.get("head_gate"))
        self.keep_all_keys = bool(spec.params.get("keep_all_keys")) or self.keep_first > 0
        self.general = (self.value_dim != self.head_dim or self.unit_norm_eps is not None or self.keep_first > 0
                        or self.head_gate)
        if not self.kv_projection and self.values_from_keys:
            raise ValueError("attention: values from keys need a key projection")
        #: the head size the cache and the kernels see
        self.padded_dim = self.head_dim
        if self.general:
            if self.values_from_keys or self.query_temperature is not None or self.sink is not None:
                raise ValueError("attention: value_dim, unit_norm_after_rotation, keep_first and head_gate do not "
                                 "combine with values from keys, a query temperature or a sink")
            if self.unit_norm_eps is not None and (self.biased or self.qk_norm_eps is not None):
                raise ValueError("attention: unit_norm_after_rotation does not combine with biases or the gained norm")
            if self.keep_first and not self.window:
                raise ValueError("attention: keep_first needs a window")
            # (a multiple of 32 where the 16-bit attention kernels can take it: at most a quarter more)
            widest = max(self.head_dim, self.value_dim)
            self.padded_dim = -(-widest // 32) * 32 if dtype == torch.bfloat16 and widest >= 64 else -(-widest // 8) * 8
            if self.padded_dim > kernels.MAX_HEAD_DIM:
                self.padded_dim = -(-widest // 8) * 8
            kernels.check_head_dim(self.padded_dim)
            # (this path takes normalised activations and returns a plain tensor)
            self.takes_deferred_norm = self.defers_norm = False
        if self.output_biased:                   # (the product alone is not the result yet)
            self.defers_norm = False
        pos = spec.params.get("position")
        self.position = lookup_part("position", pos.kind)(pos, dtype, device) if pos else None
        if self.neighbours and self.position is not None and \
                int(getattr(self.position, "rotary_dim", 0)) > self.head_dim:
            raise ValueError("attention: the rotation covers more values than a head has")
        self.w_qkv = self.w_o = self.q_gain = self.k_gain = self.sinks = None

    def cache_spec(self):
        window = self.spec.params.get("cache_window") or self.window or self.chunk
        return CacheSpec("kv", heads=self.num_kv_heads, head_dim=self.padded_dim,
                         window=None if self.keep_all_keys else window)

    def prepare(self, max_positions):
        if self.position is not None:
            self.position.prepare(max_positions)

    def _tiles_key(self):
        return ("prefill_tc_tiles", self.num_heads // self.num_kv_heads, self.num_kv_heads * self.head_dim)

    def begin_step(self, ctx):
        """The table of tiles of the tcgen05 prompt attention, once per step and shape of the heads."""
        if self.general or ctx.is_decode or ctx.n_seqs > kernels.PREFILL_TC_MAX_SEQS or not self.scale > 0 or \
                not kernels.attention_prefill_tc_supported(self.dtype, self.head_dim, self.num_heads,
                                                           self.num_kv_heads):
            return
        key = self._tiles_key()
        if key in ctx.shared:
            return
        per_tile = kernels.PREFILL_TC_ROWS // (self.num_heads // self.num_kv_heads)
        rows = -(-ctx.n_tokens // per_tile) + ctx.n_seqs
        tiles = ctx.workspace.get(f"prefill_tc_tiles_{key[1]}_{key[2]}", (rows, 4), torch.int32)
        n = kernels.attention_prefill_tiles(tiles, ctx.n_tokens, ctx.positions, ctx.token_slot, ctx.cu_seqlens,
                                            ctx.n_seqs, self.num_heads, self.num_kv_heads, self.head_dim)
        ctx.shared[key] = (tiles, n)

    def _by_head(self, t, n, reorder):
        """[n * size, ...] -> [n * padded_dim, ...]: a head's values in the kernels' order (``reorder``: they turn
        with the rotation), zeros behind them."""
        size = t.shape[0] // n
        t = t.reshape(n, size, *t.shape[1:])
        if reorder and self.neighbours and self.position is not None:
            t = t.index_select(1, neighbours_to_halves(size, int(self.position.rotary_dim)).to(t.device))
        if size != self.padded_dim:
            out = torch.zeros((n, self.padded_dim) + tuple(t.shape[2:]), dtype=t.dtype, device=t.device)
            out[:, :size] = t
            t = out
        return t.reshape(n * self.padded_dim, *t.shape[2:])

    def _load_vectors(self, tensors):
        """Biases of the projections and gains of the head norms, in 32-bit and in the kernels' order."""
        w, f32 = self.spec.weights, torch.float32
        for which in self.biased:
            n = self.num_heads if which == "q" else self.num_kv_heads
            self.bias[which] = self._by_head(tensors[w[which + "_bias"]].to(f32), n, which != "v").contiguous()
        if self.qk_norm_eps is not None:
            heads = (self.num_heads, self.num_kv_heads) if self.whole_norm else (1, 1)
            self.q_gain = self._by_head(tensors[w["q_norm"]].to(f32), heads[0], True).contiguous()
            if self.kv_projection:
                self.k_gain = self._by_head(tensors[w["k_norm"]].to(f32), heads[1], True).contiguous()
        if self.has_sinks:
            self.sinks = tensors[w["sink"]].to(f32).contiguous()
        if self.output_biased:
            self.output_bias = tensors[w["o_bias"]].to(f32).contiguous()

    def _load_general(self, tensors):
        """[q | k | v | gate] as one weight, every head padded with zero rows to ``padded_dim``, zero rows
        up to a multiple of 64; ``o`` with zero columns where the value heads are padded."""
        w, big = self.spec.weights, self.padded_dim
        self._load_vectors(tensors)
        rows = [self._by_head(tensors[w["q"]], self.num_heads, True)]
        if self.kv_projection:
            rows += [self._by_head(tensors[w["k"]], self.num_kv_heads, True),
                     self._by_head(tensors[w["v"]], self.num_kv_heads, False)]
        if self.head_gate:
            rows.append(tensors[w["gate"]])
        n = sum(r.shape[0] for r in rows)
        if n % 64:
            rows.append(torch.zeros((-n % 64, self.hidden), dtype=rows[0].dtype, device=rows[0].device))
        self.w_qkv = torch.cat(rows, dim=0).to(self.dtype).contiguous()
        o = tensors[w["o"]].view(self.hidden, self.num_heads, self.value_dim)
        if self.value_dim != big:
            wide = torch.zeros((self.hidden, self.num_heads, big), dtype=o.dtype, device=o.device)
            wide[:, :, :self.value_dim] = o
            o = wide
        self.w_o = o.reshape(self.hidden, self.num_heads * big).to(self.dtype).contiguous()

    def _forward_general(self, x, ctx, entry, writes_cache, leave_bias=False):
        t, big, nh, nkv = ctx.n_tokens, self.padded_dim, self.num_heads, self.num_kv_heads
        pos = self.position
        rows = linear(x, self.w_qkv, ctx, "qkv", n_rows=t)
        k_col = nh * big
        gate_col = k_col + (2 * nkv * big if self.kv_projection else 0)
        if self.whole_norm:
            self._whole_norm_kv(rows, ctx, entry, writes_cache and self.kv_projection)
        elif self.qk_norm_eps is not None or self.biased:
            kernels.qk_prepare_padded_kv(
                rows, t, self.q_gain, self.k_gain, pos.cos if pos else _no_table(self.device),
                pos.sin if pos else _no_table(self.device), pos.rotary_dim if pos else 0, ctx.positions,
                ctx.token_slot, entry.k_pages, entry.v_pages, entry.block_table, nh, nkv, big,
                self.qk_norm_eps if self.qk_norm_eps is not None else 0.0, self.head_dim,
                write_kv=writes_cache and self.kv_projection, q_bias=self.bias["q"], k_bias=self.bias["k"],
                v_bias=self.bias["v"])
        else:
            kernels.qk_rope_unit_kv(
                rows, t, k_col, k_col + nkv * big, pos.cos if pos else _no_table(self.device),
                pos.sin if pos else _no_table(self.device), pos.rotary_dim if pos else 0, ctx.positions,
                ctx.token_slot, entry.k_pages, entry.v_pages, entry.block_table, nh, nkv, big, self.head_dim,
                self.unit_norm_eps or 0.0, unit=self.unit_norm_eps is not None,
                write_kv=writes_cache and self.kv_projection)
        out = ctx.workspace.get("attn_out", (t, nh * big), self.dtype)
        visible = self._visible(ctx)
        gate = rows[:, gate_col:] if self.head_gate else None
        mask = {"chunk": self.chunk, "softcap": self.softcap, "sinks": self.sinks}
        if not ctx.is_decode and kernels.attention_prefill_supported(self.dtype, big, nh, nkv):
            kernels.attention_prefill_bf16(out, rows, t, ctx.positions, ctx.token_slot, ctx.cu_seqlens, ctx.n_seqs,
                                           entry.k_pages, entry.v_pages, entry.block_table, nh, nkv, big, self.scale,
                                           self.window, keep_first=self.keep_first, gate=gate, **mask)
            return self._project(out, ctx, None, leave_bias)
        if ctx.is_decode and kernels.attention_decode_supported(self.dtype, big):
            # blocks = tokens x KV heads (x 16-row blocks of the group), three fit an SM: every token's own
            # window is cut so that the blocks about fill the machine, never finer than two pages a split
            blocks = t * nkv * -(-(nh // nkv) // 16)
            splits = max(1, min(3 * kernels.sm_count(self.device) // blocks, -(-visible // 128)))
            acc = ml = None
            if splits > 1:
                acc = ctx.workspace.get("attn_part_acc", (t, nh, splits, big), torch.float32)
                ml = ctx.workspace.get("attn_part_ml", (t, nh, splits, 2), torch.float32)
            kernels.attention_decode_bf16(out, rows, t, ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages,
                                          entry.block_table, nh, nkv, big, self.scale, self.window, splits, 0, acc, ml,
                                          keep_first=self.keep_first, gate=gate, **mask)
            return self._project(out, ctx, None, leave_bias)
        splits, per_split, acc, ml = 1, 0, None, None
        blocks = t * nh
        if blocks < 2 * kernels.sm_count(self.device) and visible > 512:
            splits = max(1, min(-(-visible // 256), -(-4 * kernels.sm_count(self.device) // blocks), 64))
        if splits > 1:
            per_split = -(-(-(-ctx.max_context // splits)) // 128) * 128
            splits = -(-ctx.max_context // per_split)
        if splits > 1:
            acc = ctx.workspace.get("attn_part_acc", (t, nh, splits, big), torch.float32)
            ml = ctx.workspace.get("attn_part_ml", (t, nh, splits, 2), torch.float32)
        kernels.attention_generic(out, rows, t, ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages,
                                  entry.block_table, nh, nkv, big, self.scale, self.window, splits, per_split,
                                  acc, ml, keep_first=self.keep_first, gate=gate, **mask)
        return self._project(out, ctx, None, leave_bias)

    def _whole_norm_kv(self, rows, ctx, entry, write_kv):
        pos = self.position
        kernels.qk_whole_norm_kv(
            rows, ctx.n_tokens, self.q_gain, self.k_gain, pos.cos if pos else _no_table(self.device),
            pos.sin if pos else _no_table(self.device), pos.rotary_dim if pos else 0, ctx.positions, ctx.token_slot,
            entry.k_pages, entry.v_pages, entry.block_table, self.num_heads, self.num_kv_heads, self.padded_dim,
            self.qk_norm_eps, norm_dim=self.head_dim, write_kv=write_kv)

    def load(self, tensors):
        if self.general:
            return self._load_general(tensors)
        w = self.spec.weights
        self._load_vectors(tensors)
        rows = [self._by_head(tensors[w["q"]], self.num_heads, True)]
        if self.kv_projection:
            rows.append(self._by_head(tensors[w["k"]], self.num_kv_heads, True))
            if not self.values_from_keys:
                rows.append(tensors[w["v"]])
        self.w_qkv = torch.cat(rows, dim=0).to(self.dtype).contiguous()
        self.w_o = tensors[w["o"]].to(self.dtype).contiguous()

    def bytes_read_per_step(self, n_tokens):
        return sum(t.numel() * t.element_size() for t in (self.w_qkv, self.w_o, self.q_gain, self.k_gain,
                                                          self.sinks, self.output_bias, *self.bias.values()) if t is not None)

    # ------------------------------------------------------------------
    takes_deferred_norm = True
    defers_norm = True

    def _visible(self, ctx):
        """Keys a token of this step sees at most."""
        if self.chunk:
            return min(ctx.max_context, self.chunk)
        return min(ctx.max_context, self.window + self.keep_first) if self.window else ctx.max_context

    def _project(self, out, ctx, defer, leave_bias):
        y = linear(out, self.w_o, ctx, "attn_proj", n_rows=ctx.n_tokens, defer=None if self.output_biased else defer,
                   image=self.product_image())
        if self.output_bias is None or leave_bias:
            return y
        biased = ctx.workspace.get("attn_proj_biased", (ctx.n_tokens, self.hidden), self.dtype)
        kernels.bias_act(biased, y, self.output_bias, None, n_rows=ctx.n_tokens)
        return biased

    def forward(self, x, ctx, entry, writes_cache=True, defer=None, leave_bias=False):
        t = ctx.n_tokens
        pos = self.position
        if self.general:
            if isinstance(x, DeferredNorm):
                raise kernels.KernelError("this attention layer takes normalised activations, not a deferred norm")
            return self._forward_general(x, ctx, entry, writes_cache, leave_bias)
        writes_cache = writes_cache and self.kv_projection
        if self._fuses_rope(x, ctx):
            # few rows, heads of 128: norm, rotation and cache write ride on the product's epilogue
            row_scale, xin = (row_scale_of(x), x.scaled) if isinstance(x, DeferredNorm) else (None, x)
            qkv = ctx.workspace.get("qkv", (t, self.w_qkv.shape[0]), self.dtype)
            kernels.gemm_tc_qkv_rope(
                qkv, xin, self.w_qkv, t, self.q_gain, self.k_gain,
                self.qk_norm_eps if self.qk_norm_eps is not None else 0.0, pos.cos, pos.sin,
                ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages, entry.block_table,
                self.num_heads, self.num_kv_heads, write_kv=writes_cache, row_scale=row_scale)
            out = ctx.workspace.get("attn_out", (t, self.num_heads * self.head_dim), self.dtype)
            self._attend(out, qkv, ctx, entry)
            return self._project(out, ctx, defer, leave_bias)
        if self._fuses_prepare(x, ctx):
            # the same for designs with biases, a query temperature, values taken from the keys,
            # or no rotation at all
            row_scale, xin = (row_scale_of(x), x.scaled) if isinstance(x, DeferredNorm) else (None, x)
            qkv = ctx.workspace.get("qkv", (t, self.w_qkv.shape[0]), self.dtype)
            kernels.gemm_tc_qkv_prepare(
                qkv, xin, self.w_qkv, t, self.q_gain, self.k_gain,
                self.qk_norm_eps if self.qk_norm_eps is not None else 0.0,
                pos.cos if pos else None, pos.sin if pos else None,
                ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages, entry.block_table,
                self.num_heads, self.num_kv_heads, write_kv=writes_cache, row_scale=row_scale,
                q_bias=self.bias["q"], k_bias=self.bias["k"], v_bias=self.bias["v"],
                q_temperature=self.query_temperature, values_from_keys=self.values_from_keys)
            out = ctx.workspace.get("attn_out", (t, self.num_heads * self.head_dim), self.dtype)
            self._attend(out, qkv, ctx, entry)
            return self._project(out, ctx, defer, leave_bias)
        if self._fuses_rope_of_many_rows(x, ctx):
            # many rows, heads of 128: the same on the epilogue of the product on pairs of SMs
            qkv = ctx.workspace.get("qkv", (t, self.w_qkv.shape[0]), self.dtype)
            kernels.gemm_pair_qkv_rope(
                qkv, x, self.w_qkv, t, self.q_gain, self.k_gain,
                self.qk_norm_eps if self.qk_norm_eps is not None else 0.0, pos.cos, pos.sin,
                ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages, entry.block_table,
                self.num_heads, self.num_kv_heads, write_kv=writes_cache)
            out = ctx.workspace.get("attn_out", (t, self.num_heads * self.head_dim), self.dtype)
            self._attend(out, qkv, ctx, entry)
            return self._project(out, ctx, defer, leave_bias)
        qkv = linear(x, self.w_qkv, ctx, "qkv", n_rows=t)
        prepare = (qkv, t, self.q_gain, self.k_gain,
                   pos.cos if pos else _no_table(self.device), pos.sin if pos else _no_table(self.device),
                   pos.rotary_dim if pos else 0, ctx.positions, ctx.token_slot, entry.k_pages,
                   entry.v_pages, entry.block_table, self.num_heads, self.num_kv_heads, self.head_dim,
                   self.qk_norm_eps if self.qk_norm_eps is not None else 0.0)
        if self.whole_norm:
            self._whole_norm_kv(qkv, ctx, entry, writes_cache)
        elif self._plain:
            kernels.qk_norm_rope_kv(*prepare, write_kv=writes_cache)
        else:
            kernels.qk_prepare_kv(*prepare, write_kv=writes_cache, q_bias=self.bias["q"],
                                  k_bias=self.bias["k"], v_bias=self.bias["v"],
                                  q_temperature=self.query_temperature,
                                  values_from_keys=self.values_from_keys)
        out = ctx.workspace.get("attn_out", (t, self.num_heads * self.head_dim), self.dtype)
        self._attend(out, qkv, ctx, entry)
        return self._project(out, ctx, defer, leave_bias)

    @property
    def _plain(self):
        """None of the optional parameters that change what happens between the projection and
        the cache is on (sinks only change the softmax)."""
        return not self.biased and not self.values_from_keys and self.query_temperature is None and not self.whole_norm

    def _fuses_rope(self, x, ctx):
        xin = x.scaled if isinstance(x, DeferredNorm) else x
        pos = self.position
        return (self._plain and self.kv_projection and self.dtype == torch.bfloat16 and ctx.n_tokens <= FUSE_ROPE_ROWS
                and self.head_dim == kernels.QKV_ROPE_HEAD_DIM and pos is not None
                and getattr(pos, "rotary_dim", 0) == self.head_dim and tc_takes(xin, self.w_qkv))

    def product_image(self):
        """``"extended"`` when this layer's q/k/v product of few rows runs the extended epilogue."""
        pos = self.position
        if ((not self._plain or pos is None) and not self.whole_norm and self.dtype == torch.bfloat16
                and self.head_dim == kernels.QKV_ROPE_HEAD_DIM
                and (pos is None or getattr(pos, "rotary_dim", 0) == self.head_dim)):
            return "extended"
        return None

    def _fuses_prepare(self, x, ctx):
        xin = x.scaled if isinstance(x, DeferredNorm) else x
        return (self.product_image() == "extended" and self.kv_projection and ctx.n_tokens <= FUSE_ROPE_ROWS
                and tc_takes(xin, self.w_qkv))

    def _fuses_rope_of_many_rows(self, x, ctx):
        pos = self.position
        if (not self._plain or not self.kv_projection or isinstance(x, DeferredNorm) or self.dtype != torch.bfloat16
                or self.head_dim != kernels.QKV_ROPE_HEAD_DIM or pos is None
                or getattr(pos, "rotary_dim", 0) != self.head_dim):
            return False
        qkv = ctx.workspace.get("qkv", (ctx.n_tokens, self.w_qkv.shape[0]), self.dtype)
        return pair_product_wins(qkv, x, self.w_qkv, ctx.n_tokens, kernels.PAIR_EPI_BF16)

    def _attend(self, out, qkv, ctx, entry):
        t = ctx.n_tokens
        visible = self._visible(ctx)
        mask = {"chunk": self.chunk, "softcap": self.softcap, "sinks": self.sinks}
        fast_decode = ctx.is_decode and kernels.attention_decode_supported(self.dtype, self.head_dim)
        if not ctx.is_decode and kernels.attention_prefill_supported(
                self.dtype, self.head_dim, self.num_heads, self.num_kv_heads):
            prefill = kernels.attention_prefill_bf16
            if ctx.n_seqs <= kernels.PREFILL_TC_MAX_SEQS and self.scale > 0 and \
                    kernels.attention_prefill_tc_supported(self.dtype, self.head_dim, self.num_heads,
                                                           self.num_kv_heads):
                prefill = kernels.attention_prefill_tc      # tcgen05: head sizes 64 and 128
            extra = {}
            if prefill is kernels.attention_prefill_tc:
                made = ctx.shared.get(self._tiles_key())
                if made is not None:                 # (made in begin_step; a part driven alone has none)
                    extra = dict(tiles=made[0], n_tiles=made[1])
            prefill(
                out, qkv, t, ctx.positions, ctx.token_slot, ctx.cu_seqlens, ctx.n_seqs,
                entry.k_pages, entry.v_pages, entry.block_table, self.num_heads, self.num_kv_heads,
                self.head_dim, self.scale, self.window, sink=self.sink, **mask, **extra)
            return
        if ctx.is_decode and t <= 65535 and kernels.attention_decode_tma_supported(
                self.dtype, self.head_dim, self.num_heads, self.num_kv_heads):
            # blocks = tokens x KV heads x splits, two fit an SM; a split takes whole pages and the
            # splits of a token are one cluster
            blocks = t * self.num_kv_heads
            pages = -(-visible // kernels.PAGE)
            # (more than 8 blocks a token only pay with many pages each: long contexts, few sequences)
            limit = kernels.decode_tma_max_splits(self.head_dim, self.device) if pages >= WIDE_CLUSTER_PAGES else \
                kernels.DECODE_TMA_PORTABLE_SPLITS
            splits = max(1, min(2 * kernels.sm_count(self.device) // blocks, pages, limit))
            splits = 1 << (splits.bit_length() - 1)      # clusters of 3, 5, 6, 7 pack the GPCs badly
            kernels.attention_decode_tma(
                out, qkv, t, ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages,
                entry.block_table, self.num_heads, self.num_kv_heads, self.head_dim, self.scale,
                self.window, splits, sink=self.sink, **mask)
            return
        if fast_decode:
            # blocks = tokens x KV heads (x 16-row blocks of the group); three fit an SM.  Split
            # the keys so that the blocks just fill the machine once, or about twice when one
            # filling cannot be approached; never finer than two pages a split.
            blocks = t * self.num_kv_heads * -(-(self.num_heads // self.num_kv_heads) // 16)
            resident = 3 * kernels.sm_count(self.device)
            splits = resident // blocks
            if blocks * splits < 0.7 * resident:
                splits = int(1.8 * resident / blocks + 0.5)
            splits = max(1, min(splits, -(-visible // 128)))
            unit = 64
        else:
            blocks = t * self.num_heads
            splits = 1
            if blocks < 2 * kernels.sm_count(self.device) and visible > 512:
                splits = max(1, min(-(-visible // 256), -(-4 * kernels.sm_count(self.device) // blocks), 64))
            unit = 128
        per_split, acc, ml = 0, None, None
        if splits > 1 and not fast_decode:      # the decode kernel cuts each token's own range
            per_split = -(-(-(-ctx.max_context // splits)) // unit) * unit
            splits = -(-ctx.max_context // per_split)
        if splits > 1:
            acc = ctx.workspace.get("attn_part_acc", (t, self.num_heads, splits, self.head_dim),
                                    torch.float32)
            ml = ctx.workspace.get("attn_part_ml", (t, self.num_heads, splits, 2), torch.float32)
        args = (out, qkv, t, ctx.positions, ctx.token_slot, entry.k_pages, entry.v_pages,
                entry.block_table, self.num_heads, self.num_kv_heads, self.head_dim, self.scale,
                self.window, splits, per_split, acc, ml)
        fn = kernels.attention_decode_bf16 if fast_decode else kernels.attention_generic
        fn(*args, sink=self.sink, **mask)


_EMPTY = {}


def _no_table(device):
    key = str(device)
    if key not in _EMPTY:
        _EMPTY[key] = torch.zeros((1, 0), dtype=torch.float32, device=device)
    return _EMPTY[key]
