"""Python faces of the CUDA kernels: argument checks, then one launch each.

Every function takes CUDA tensors and launches on torch's current stream.  There is
no CPU or torch fallback: a tensor that is not on a CUDA device, or a kernel library
that cannot be built or loaded, raises.  The reference pairs every Triton kernel with
a torch fallback chosen at call time (engine/ek_kernels.py:1025-1559); here the plain
counterparts live only in the tests.
"""

from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_longlong, c_ulonglong, c_void_p

import torch

from . import lib
from .lib import Function, KernelError, count_extra_launches

PAGE = 64                 # tokens per cache page; must equal EK_PAGE in csrc/common.cuh
MAX_HEAD_DIM = 256        # of the 16-bit attention kernels
PREPARE_MAX_HEAD_DIM = 512      # of the kernels that norm, rotate and store heads; equals EK_MAX_HEAD_DIM in csrc/common.cuh
WHOLE_NORM_MAX_VALUES = 50 * 1024     # query and key values of a token that qk_whole_norm_kv keeps in shared memory
GENERIC_MAX_HEAD_DIM = 1024     # the general attention kernel alone takes head sizes up to here

_SUFFIX = {torch.float32: "f32", torch.bfloat16: "bf16"}
_P = c_void_p


def _suffix(dtype) -> str:
    try:
        return _SUFFIX[dtype]
    except KeyError:
        raise KernelError(f"kernels exist for float32 and bfloat16, not {dtype}") from None


def _ptr(t):
    return None if t is None else t.data_ptr()


def _slow_stream():
    return torch.cuda.current_stream().cuda_stream


# The handle of torch's current stream on the current device.  The public way costs the host 3 us
# a launch (a Stream object is built each time); torch's own raw accessors, where this build of
# torch has them, a tenth of that.
_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_raw_device = getattr(torch._C, "_cuda_getDevice", None)


def _stream():
    if _raw_stream is None or _raw_device is None:
        return _slow_stream()
    return _raw_stream(_raw_device())


def _need_cuda(*tensors):
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise KernelError("enginekernel_b200 kernels run on CUDA tensors only; got a tensor on "
                              f"{t.device} (there is no CPU path)")


def _need(cond, msg):
    if not cond:
        raise KernelError(msg)


def _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, new_keys_only, chunk=None):
    """While a launch record is active: what an attention launch has to read and compute.  Reads
    the positions back (a synchronisation, which is why it is done only then).  Keys and values:
    for single tokens every visible key of every token; for prompts (``new_keys_only``) each
    token's own key and value once, as the work is bound by its flops anyway."""
    if not lib.recording():
        return
    pos = positions[:n_tokens].to(torch.int64)
    visible = torch.clamp(pos + 1, min=0)
    if window:
        visible = torch.clamp(visible, max=int(window))
    if chunk:
        visible = torch.where(pos >= 0, pos % int(chunk) + 1, visible)
    keys = int(visible.sum().item())
    live = int((pos >= 0).sum().item())
    size = q.element_size()
    kv_tokens = live if new_keys_only else keys
    lib.annotate(bytes=size * (2 * kv_tokens * n_kv_heads * head_dim + 2 * live * n_q_heads * head_dim),
                 flops=4 * keys * n_q_heads * head_dim)


def _per_dtype(module, name, argtypes):
    return {dt: Function(module, f"{name}_{sfx}", argtypes) for dt, sfx in _SUFFIX.items()}


# ------------------------------------------------------------------ elementwise
_embed = _per_dtype("elementwise", "ek_embed", [_P, _P, _P, c_int, c_int, c_int, c_float, _P, _P, c_int, c_int, _P])
_scale_f32 = Function("elementwise", "ek_scale_f32", [_P, c_longlong, c_float, _P])
_scale_cap_f32 = Function("elementwise", "ek_scale_cap_f32", [_P, c_longlong, c_float, c_float, _P])
_rmsnorm = _per_dtype("elementwise", "ek_rmsnorm",
                      [_P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, _P])
_add_residual = _per_dtype("elementwise", "ek_add_residual", [_P, _P, c_longlong, _P])
_act_mul = _per_dtype("elementwise", "ek_act_mul", [_P, _P, c_int, c_int, c_int, c_float, _P])
# "clamped": min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, -limit, limit) + 1)
GATE_ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "clamped": 2}


def embed(resid, table, ids, n_tokens, scale=1.0, pos_table=None, positions=None, accumulate=False):
    """resid[t, :] = table[ids[t], :] * scale as 32-bit, for the first ``n_tokens`` ids; with
    ``pos_table`` [positions, hidden] also + pos_table[positions[t], :] (rows whose position is
    negative get none).  A plain launch: the first kernel of a step.  ``accumulate``: the same
    values are added to what ``resid`` holds instead (the embedding output fed in again)."""
    _need_cuda(resid, table, ids, pos_table, positions)
    _need(resid.dtype == torch.float32 and ids.dtype == torch.int32, "embed: resid f32, ids int32")
    _need(table.is_contiguous() and resid.is_contiguous(), "embed: contiguous tensors")
    vocab, hidden = table.shape
    _need(resid.shape[-1] == hidden and resid.shape[0] >= n_tokens, "embed: resid shape")
    max_positions = 0
    if pos_table is not None:
        _need(pos_table.dtype == table.dtype and pos_table.is_contiguous() and pos_table.shape[-1] == hidden
              and positions is not None and positions.dtype == torch.int32,
              "embed: position table [positions, hidden] in the embedding's dtype, int32 positions")
        max_positions = pos_table.shape[0]
    if lib.recording():
        lib.annotate(bytes=n_tokens * hidden * (table.element_size() * (2 if pos_table is not None else 1)
                                                + (8 if accumulate else 4)))
    _embed[table.dtype](_ptr(resid), _ptr(table), _ptr(ids), n_tokens, hidden, vocab, float(scale),
                        _ptr(pos_table), _ptr(positions), max_positions, 1 if accumulate else 0, _stream())


def scale_(x, scale, n=None):
    """x *= scale in place (32-bit values; the first ``n`` of them)."""
    _need_cuda(x)
    _need(x.dtype == torch.float32 and x.is_contiguous(), "scale_: contiguous 32-bit values")
    count = x.numel() if n is None else n
    if lib.recording():
        lib.annotate(bytes=8 * count)
    _scale_f32(_ptr(x), count, float(scale), _stream())


def scale_cap_(x, scale, cap, n=None):
    """x <- cap tanh(scale x / cap) in place (32-bit values; the first ``n`` of them)."""
    _need_cuda(x)
    _need(x.dtype == torch.float32 and x.is_contiguous() and cap > 0, "scale_cap_: contiguous 32-bit values, a positive cap")
    count = x.numel() if n is None else n
    if lib.recording():
        lib.annotate(bytes=8 * count)
    _scale_cap_f32(_ptr(x), count, float(scale), float(cap), _stream())


def rmsnorm(y, resid, gain, eps, add=None, rows=None, n_rows=None, write_back=True):
    """y = gain * n(resid [+ add]); with ``add`` the stream is updated in place when
    ``write_back``.  ``rows`` (int32) picks stream rows; y then has one row per entry."""
    _need_cuda(y, resid, gain, add, rows)
    hidden = resid.shape[-1]
    _need(resid.dtype == torch.float32 and gain.dtype == torch.float32, "rmsnorm: 32-bit stream and gain")
    _need(gain.numel() == hidden and y.shape[-1] == hidden, "rmsnorm: sizes disagree")
    _need(add is None or (add.dtype == y.dtype and add.shape[-1] == hidden and add.is_contiguous()),
          "rmsnorm: add must have y's dtype and the stream's width")
    _need(y.is_contiguous() and resid.is_contiguous(), "rmsnorm: contiguous tensors")
    if n_rows is None:
        n_rows = rows.numel() if rows is not None else resid.shape[0]
    _need(y.shape[0] >= n_rows, "rmsnorm: y has too few rows")
    if lib.recording():
        per_value = 4 + y.element_size() + ((y.element_size() + (4 if write_back else 0)) if add is not None else 0)
        lib.annotate(bytes=n_rows * hidden * per_value)
    _rmsnorm[y.dtype](_ptr(y), _ptr(resid), _ptr(add), _ptr(gain), _ptr(rows), float(eps),
                      n_rows, hidden, 1 if write_back else 0, _stream())


_rmsnorm_scaled_sum = _per_dtype("elementwise", "ek_rmsnorm_scaled_sum",
                                 [_P, _P, _P, _P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, _P])


def rmsnorm_scaled_sum(y, resid, a, gain, eps, scale_a=None, b=None, scale_b=None, rows=None, n_rows=None,
                       write_back=True):
    """stream += a * scale_a + b * scale_b (element by element; the scales are 32-bit vectors of the
    stream's width, absent: ones; ``b`` may be absent), then y = gain * n(stream).  ``rows`` (int32)
    picks stream rows (and the same rows of ``a`` and ``b``); y then has one row per entry."""
    _need_cuda(y, resid, a, gain, scale_a, b, scale_b, rows)
    hidden = resid.shape[-1]
    _need(resid.dtype == torch.float32 and gain.dtype == torch.float32 and gain.numel() == hidden
          and y.shape[-1] == hidden and y.is_contiguous() and resid.is_contiguous(),
          "rmsnorm_scaled_sum: 32-bit stream and gain of one width")
    for t in (a, b):
        _need(t is None or (t.dtype == y.dtype and t.shape[-1] == hidden and t.is_contiguous()),
              "rmsnorm_scaled_sum: the summands have y's dtype and the stream's width")
    for t in (scale_a, scale_b):
        _need(t is None or (t.dtype == torch.float32 and t.numel() == hidden and t.is_contiguous()),
              "rmsnorm_scaled_sum: 32-bit scales of the stream's width")
    _need(a is not None and (b is not None or scale_b is None), "rmsnorm_scaled_sum: a scale without its summand")
    if n_rows is None:
        n_rows = rows.numel() if rows is not None else resid.shape[0]
    _need(y.shape[0] >= n_rows, "rmsnorm_scaled_sum: y has too few rows")
    if lib.recording():
        lib.annotate(bytes=n_rows * hidden * (4 + (4 if write_back else 0)
                                              + y.element_size() * (2 if b is None else 3)))
    _rmsnorm_scaled_sum[y.dtype](_ptr(y), _ptr(resid), _ptr(a), _ptr(scale_a), _ptr(b), _ptr(scale_b), _ptr(gain),
                                 _ptr(rows), float(eps), n_rows, hidden, 1 if write_back else 0, _stream())


_add_scaled = _per_dtype("elementwise", "ek_add_scaled", [_P, _P, _P, _P, _P, c_longlong, c_int, _P])


def add_scaled(resid, a, scale_a=None, b=None, scale_b=None, n_rows=None):
    """stream += a * scale_a + b * scale_b, element by element, without a norm (scales: 32-bit vectors of
    the stream's width, absent: ones; ``b`` may be absent)."""
    _need_cuda(resid, a, scale_a, b, scale_b)
    hidden = resid.shape[-1]
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and a.is_contiguous() and a.shape[-1] == hidden
          and (b is None or (b.dtype == a.dtype and b.is_contiguous() and b.shape[-1] == hidden)),
          "add_scaled: 32-bit stream, summands of its width")
    for t in (scale_a, scale_b):
        _need(t is None or (t.dtype == torch.float32 and t.numel() == hidden and t.is_contiguous()),
              "add_scaled: 32-bit scales of the stream's width")
    n = (n_rows if n_rows is not None else resid.shape[0]) * hidden
    if lib.recording():
        lib.annotate(bytes=n * (8 + a.element_size() * (1 if b is None else 2)))
    _add_scaled[a.dtype](_ptr(resid), _ptr(a), _ptr(scale_a), _ptr(b), _ptr(scale_b), n, hidden, _stream())


def add_residual(resid, x, n_rows=None):
    _need_cuda(resid, x)
    n = (n_rows if n_rows is not None else resid.shape[0]) * resid.shape[-1]
    _need(resid.dtype == torch.float32 and x.shape[-1] == resid.shape[-1], "add_residual: shapes")
    _add_residual[x.dtype](_ptr(resid), _ptr(x), n, _stream())


def silu_mul(out, gu, n_rows=None):
    """out[r, i] = silu(gu[r, i]) * gu[r, I + i] for gu of width 2I."""
    act_mul(out, gu, "silu", n_rows)


def act_mul(out, gu, activation="silu", n_rows=None, limit=0.0):
    """out[r, i] = act(gu[r, i]) * gu[r, I + i] for gu of width 2I; ``activation`` is ``"silu"`` or
    ``"gelu_tanh"`` (0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))); ``"clamped"`` with a positive
    ``limit``: with g' = min(g, limit), u' = clamp(u, -limit, limit), g' sigmoid(1.702 g') (u' + 1)."""
    _need_cuda(out, gu)
    _need(activation != "clamped" or limit > 0, "act_mul: the clamped gate needs a positive limit")
    _need(activation in GATE_ACTIVATIONS, f"act_mul: no activation {activation!r}")
    inter = gu.shape[-1] // 2
    _need(gu.shape[-1] == 2 * inter and out.shape[-1] == inter and out.dtype == gu.dtype,
          "act_mul: out must be [rows, I] for gu [rows, 2I]")
    _need(out.is_contiguous() and gu.is_contiguous(), "act_mul: contiguous tensors")
    rows = n_rows if n_rows is not None else gu.shape[0]
    if lib.recording():
        lib.annotate(bytes=3 * rows * inter * gu.element_size())
    for r0 in range(0, rows, 65535):
        r1 = min(rows, r0 + 65535)
        _act_mul[gu.dtype](_ptr(out[r0:]), _ptr(gu[r0:]), r1 - r0, inter, GATE_ACTIVATIONS[activation],
                           float(limit), _stream())


_embed_pair = _per_dtype("elementwise", "ek_embed_pair",
                         [_P, _P, _P, _P, _P, _P, c_longlong, c_int, c_int, c_int, c_longlong, c_longlong, _P])
_keep_last_token = Function("elementwise", "ek_keep_last_token", [_P, c_longlong, _P, _P, _P, c_int, _P])
_cast_columns = _per_dtype("elementwise", "ek_cast_columns", [_P, c_int, c_int, _P, c_int, c_int, _P])
_rmsnorm_post_add = _per_dtype("elementwise", "ek_rmsnorm_post_add",
                               [_P, _P, _P, c_float, _P, c_float, _P, _P, c_float, _P, c_float, c_int, c_int, _P])
_bias_act = _per_dtype("elementwise", "ek_bias_act", [_P, _P, c_int, c_int, c_int, _P, c_int, c_int, c_int, _P])
ROW_ACTIVATIONS = {None: 0, "none": 0, "gelu_tanh": 1, "silu": 2}


def embed_pair(resid, table, ids, positions, token_slot, before, n_tokens, buckets, mul_prev, mul_cur):
    """resid[t] += table[(previous * mul_prev + ids[t] * mul_cur) mod buckets], and table[buckets] for a
    sequence's first token (position 0).  The token before t is the step's token t - 1 when that continues
    the same sequence, else ``before[slot]`` (int32, one per slot).  Rows with a negative position are skipped."""
    _need_cuda(resid, table, ids, positions, token_slot, before)
    hidden = resid.shape[-1]
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and table.is_contiguous()
          and tuple(table.shape) == (buckets + 1, hidden), "embed_pair: 32-bit stream, table [buckets + 1, hidden]")
    _need(before.dtype == torch.int32 and ids.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "embed_pair: int32 indices and previous tokens")
    if lib.recording():
        lib.annotate(bytes=n_tokens * hidden * (table.element_size() + 8))
    _embed_pair[table.dtype](_ptr(resid), _ptr(table), _ptr(ids), _ptr(positions), _ptr(token_slot), _ptr(before),
                             before.stride(0), n_tokens, hidden, int(buckets), int(mul_prev), int(mul_cur), _stream())


def keep_last_token(before, ids, positions, token_slot, n_tokens):
    """before[slot] = the last token each sequence of the step brought."""
    _need_cuda(before, ids, positions, token_slot)
    _need(before.dtype == torch.int32, "keep_last_token: int32 state")
    _keep_last_token(_ptr(before), before.stride(0), _ptr(ids), _ptr(positions), _ptr(token_slot), n_tokens, _stream())


def cast_columns(dst, col0, src, n_rows):
    """dst[r, col0 : col0 + W] = src[r, :] (32-bit, [rows, W]) rounded to dst's type."""
    _need_cuda(dst, src)
    width = src.shape[-1]
    _need(src.dtype == torch.float32 and src.is_contiguous() and dst.stride(-1) == 1
          and col0 + width <= dst.shape[-1], "cast_columns: 32-bit source rows that fit the destination's")
    if lib.recording():
        lib.annotate(bytes=n_rows * width * (4 + dst.element_size()))
    _cast_columns[dst.dtype](_ptr(dst), dst.stride(0), col0, _ptr(src), width, n_rows, _stream())


def rmsnorm_post_add(y, resid, a, gain_post, eps_post, gain=None, eps=0.0, weight_a=1.0, b=None, weight_b=1.0,
                     bias=None, n_rows=None):
    """stream += gain_post * n(u), u = a * weight_a + b * weight_b + bias (``b``, ``bias`` optional; the
    weights are plain numbers), and then, when ``y`` is given, y = gain * n(stream): a sublayer's result
    normed on its way into the stream and the next reader's norm, one pass over the row."""
    _need_cuda(y, resid, a, gain_post, gain, b, bias)
    hidden = resid.shape[-1]
    _need(resid.dtype == torch.float32 and resid.is_contiguous() and gain_post.dtype == torch.float32
          and gain_post.numel() == hidden, "rmsnorm_post_add: 32-bit stream and gains of its width")
    _need(a.is_contiguous() and a.shape[-1] == hidden and (b is None or (b.dtype == a.dtype and b.is_contiguous()
          and b.shape[-1] == hidden)), "rmsnorm_post_add: results of the stream's width")
    _need(y is None or (y.dtype == a.dtype and y.is_contiguous() and y.shape[-1] == hidden and gain is not None
                        and gain.dtype == torch.float32 and gain.numel() == hidden),
          "rmsnorm_post_add: y in the results' type with a 32-bit gain")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == hidden), "rmsnorm_post_add: 32-bit bias")
    n = n_rows if n_rows is not None else resid.shape[0]
    if lib.recording():
        lib.annotate(bytes=n * hidden * (8 + a.element_size() * ((1 if b is None else 2) + (0 if y is None else 1))))
    _rmsnorm_post_add[a.dtype](_ptr(y), _ptr(resid), _ptr(a), float(weight_a), _ptr(b), float(weight_b), _ptr(bias),
                               _ptr(gain_post), float(eps_post), _ptr(gain), float(eps), n, hidden, _stream())


def bias_act(out, x, bias=None, activation=None, col0=0, n_rows=None):
    """out[r, i] = act(x[r, col0 + i] + bias[i]) over out's width; ``x`` is 32-bit or of out's type;
    ``activation`` None, ``"gelu_tanh"`` or ``"silu"``."""
    _need_cuda(out, x, bias)
    _need(activation in ROW_ACTIVATIONS, f"bias_act: no activation {activation!r}")
    width = out.shape[-1]
    _need(out.is_contiguous() and x.stride(-1) == 1 and x.dtype in (torch.float32, out.dtype)
          and col0 + width <= x.shape[-1], "bias_act: rows of out's width inside x's rows")
    _need(bias is None or (bias.dtype == torch.float32 and bias.numel() == width), "bias_act: a 32-bit bias of out's width")
    n = n_rows if n_rows is not None else out.shape[0]
    if lib.recording():
        lib.annotate(bytes=n * width * (x.element_size() + out.element_size()))
    _bias_act[out.dtype](_ptr(out), _ptr(x), 1 if x.dtype == torch.float32 else 0, x.stride(0), col0, _ptr(bias),
                         width, n, ROW_ACTIVATIONS[activation], _stream())


# ------------------------------------------------------------------ dynamic tanh, averages over the depth
_dynamic_tanh = _per_dtype("depth", "ek_dynamic_tanh",
                           [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P])
_depth_join = _per_dtype("depth", "ek_depth_join",
                         [_P, _P, _P, _P, c_longlong, _P, c_int, c_int, c_float, _P, _P, _P, _P, _P, c_float, c_float,
                          _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, _P])


def _tanh_norm_args(y, norm, hidden, name):
    """(y, alpha, w, b) pointers of one reader; ``norm`` is (alpha [1], w [hidden], b [hidden]) in 32-bit."""
    if y is None:
        return [None] * 4
    alpha, w, b = norm
    _need_cuda(y, alpha, w, b)
    _need(y.is_contiguous() and y.shape[-1] == hidden, f"{name}: packed rows of the stream's width")
    for t, n in ((alpha, 1), (w, hidden), (b, hidden)):
        _need(t.dtype == torch.float32 and t.is_contiguous() and t.numel() == n,
              f"{name}: 32-bit alpha [1], weight and shift of the stream's width")
    return [_ptr(t) for t in (y, alpha, w, b)]


def dynamic_tanh(y, stream, norm, second=None, second_norm=None, add=None, rows=None, n_rows=None, write_back=True):
    """y = tanh(alpha x) w + b with ``norm`` = (alpha, w, b) in 32-bit, and the same of ``second_norm`` into
    ``second``; x = stream [+ add], the stream updated in place when ``write_back``.  ``rows`` (int32) picks
    stream rows (and the same rows of ``add``)."""
    _need_cuda(y, stream, second, add, rows)
    hidden = stream.shape[-1]
    _need(stream.dtype == torch.float32 and stream.is_contiguous(), "dynamic_tanh: a 32-bit stream")
    _need(add is None or (add.dtype == y.dtype and add.is_contiguous() and add.shape[-1] == hidden),
          "dynamic_tanh: add has y's type and the stream's width")
    _need(second is None or second.dtype == y.dtype, "dynamic_tanh: both readers have one type")
    n = n_rows if n_rows is not None else (rows.numel() if rows is not None else stream.shape[0])
    if lib.recording():
        lib.annotate(bytes=n * hidden * (4 + y.element_size() * ((1 if second is None else 2) + (0 if add is None else 1))
                                         + (4 if add is not None and write_back else 0)))
    _dynamic_tanh[y.dtype](*_tanh_norm_args(y, norm, hidden, "dynamic_tanh"),
                           *_tanh_norm_args(second, second_norm, hidden, "dynamic_tanh"), _ptr(stream), _ptr(add),
                           _ptr(rows), n, hidden, 1 if write_back else 0, _stream())


def depth_join(x_next, x, first, kept, n, depth, mult, a, gate_a, f=None, gate_f=None, bias_a=None, pair=None,
               keep=True, y1=None, norm1=None, y2=None, norm2=None, n_rows=None):
    """What stands between two layers.  r = x + mult (sigmoid(z_a + b_a) a + sigmoid(z_f + b_f) f), kept as entry
    n - 1 of ``kept`` [entries, rows, hidden] when ``keep``; x_next = sum_(j < n) depth[j] X_j + depth[n] r with
    X_0 = ``first`` and X_j = kept[j - 1]; y1, y2 = tanh norms of x_next (``norm1``, ``norm2`` as in
    :func:`dynamic_tanh`, absent: not wanted).  ``gate_a`` = (z_a [rows, hidden], b_a [hidden] 32-bit), ``gate_f`` alike;
    ``f`` absent: no second sublayer.  ``bias_a`` (32-bit) is added to ``a``; ``pair`` = (b, gain_a, gain_b, eps,
    weight) instead: the first result is weight (a / rms(a) gain_a + b / rms(b) gain_b)."""
    _need_cuda(x_next, x, first, kept, depth, a, f, bias_a, y1, y2)
    hidden = x.shape[-1]
    rows = n_rows if n_rows is not None else x.shape[0]
    for t in (x_next, x, first):
        _need(t.dtype == torch.float32 and t.is_contiguous() and t.shape[-1] == hidden and t.shape[0] >= rows,
              "depth_join: 32-bit streams [rows, hidden]")
    _need(depth.dtype == torch.float32 and depth.is_contiguous() and depth.numel() == n + 1,
          "depth_join: one 32-bit weight per earlier result and one for this one")
    entries = n if keep else n - 1
    _need(entries == 0 or (kept is not None and kept.dtype == torch.float32 and kept.is_contiguous() and kept.dim() == 3
                           and kept.shape[0] >= entries and kept.shape[1] >= rows and kept.shape[2] == hidden),
          "depth_join: room for the kept results [entries, rows, hidden]")
    (za, ba), (zf, bf) = gate_a, gate_f if f is not None else (None, None)
    b = gain_a = gain_b = None
    eps = weight = 0.0
    if pair is not None:
        b, gain_a, gain_b, eps, weight = pair
    for t in (a, b, za, f, zf, y1, y2):
        _need(t is None or (t.is_cuda and t.dtype == a.dtype and t.is_contiguous() and t.shape[-1] == hidden),
              "depth_join: results and gate products of one type and the stream's width")
    for t in (ba, bf, bias_a, gain_a, gain_b):
        _need(t is None or (t.is_cuda and t.dtype == torch.float32 and t.is_contiguous() and t.numel() == hidden),
              "depth_join: 32-bit vectors of the stream's width")
    if lib.recording():
        # x, X_0 .. X_(n-1), x' and r; the results and gate products; the readers' rows (X_0 is x itself in the first layer)
        streams = (0 if x.data_ptr() == first.data_ptr() else 1) + n + 1 + (1 if keep else 0)
        narrow = sum(1 for t in (a, b, za, f, zf, y1, y2) if t is not None)
        lib.annotate(bytes=rows * hidden * (4 * streams + a.element_size() * narrow))
    _depth_join[a.dtype](_ptr(x), _ptr(x_next), _ptr(first), _ptr(kept),
                         kept.stride(0) if kept is not None else 0, _ptr(depth), n, 1 if keep else 0, float(mult), _ptr(a),
                         _ptr(bias_a), _ptr(b), _ptr(gain_a), _ptr(gain_b), float(eps), float(weight), _ptr(za), _ptr(ba),
                         _ptr(f), _ptr(zf), _ptr(bf), *_tanh_norm_args(y1, norm1, hidden, "depth_join"),
                         *_tanh_norm_args(y2, norm2, hidden, "depth_join"), rows, hidden, _stream())


# ------------------------------------------------------------------ rope + cache write
_rope_kv = _per_dtype("rope_kv", "ek_qk_norm_rope_kv",
                      [_P, c_int, _P, _P, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int,
                       c_int, c_int, c_float, c_int, _P])


def check_head_dim(head_dim):
    if not 1 <= head_dim <= PREPARE_MAX_HEAD_DIM:
        raise KernelError(f"head size {head_dim} is not supported: the kernels that prepare heads take "
                          f"sizes up to {PREPARE_MAX_HEAD_DIM}")


_qk_prepare = _per_dtype("rope_kv", "ek_qk_prepare_kv",
                         [_P, c_int, _P, _P, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int,
                          c_int, c_int, c_float, c_int, _P, _P, _P, c_float, c_int, c_int, _P])


def qk_prepare_kv(qkv, n_tokens, q_gain, k_gain, cos, sin, rot_dim, positions, token_slot,
                  k_pages, v_pages, block_table, n_q_heads, n_kv_heads, head_dim, eps,
                  write_kv=True, q_bias=None, k_bias=None, v_bias=None, q_temperature=None,
                  values_from_keys=False):
    """:func:`qk_norm_rope_kv` with what some designs put around it.  ``q_bias``, ``k_bias``,
    ``v_bias`` (32-bit, [heads * D]) are added to the projections first; ``q_temperature=(coef,
    every)`` multiplies the finished query by 1 + coef * ln(floor((position + 1) / every) + 1);
    ``values_from_keys``: ``qkv`` is [T, (NQ + NKV) D] without value heads, and the value stored
    for a token is its key as projected (bias added, before the key norm and rotation)."""
    _need_cuda(qkv, cos, sin, positions, token_slot, k_pages, v_pages, block_table, q_bias, k_bias, v_bias)
    check_head_dim(head_dim)
    heads = n_q_heads + (1 if values_from_keys else 2) * n_kv_heads
    _need(qkv.stride(-1) == 1 and (qkv.shape[-1] == heads * head_dim
                                   or (not write_kv and qkv.shape[-1] == n_q_heads * head_dim)), "qk_prepare_kv: qkv width")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and cos.shape[-1] * 2 == rot_dim, "qk_prepare_kv: 32-bit tables of rot_dim/2 columns")
    _need(k_pages.dtype == qkv.dtype and v_pages.dtype == qkv.dtype, "qk_prepare_kv: cache dtype")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "qk_prepare_kv: int32 indices")
    for g in (q_gain, k_gain):
        _need(g is None or (g.dtype == torch.float32 and g.numel() == head_dim), "qk gains: 32-bit [D]")
    for b, n in ((q_bias, n_q_heads), (k_bias, n_kv_heads), (v_bias, n_kv_heads)):
        _need(b is None or (b.dtype == torch.float32 and b.is_contiguous() and b.numel() == n * head_dim),
              "qk_prepare_kv: biases are 32-bit [heads * D]")
    _need(not (values_from_keys and v_bias is not None), "qk_prepare_kv: values taken from keys have no bias")
    coef, every = (0.0, 1) if q_temperature is None else (float(q_temperature[0]), int(q_temperature[1]))
    _need(every >= 1, "qk_prepare_kv: the temperature's step must be at least one position")
    if lib.recording():
        lib.annotate(bytes=n_tokens * head_dim * qkv.element_size() * (2 * n_q_heads + 3 * n_kv_heads))
    _qk_prepare[qkv.dtype](_ptr(qkv), qkv.stride(0), _ptr(q_gain), _ptr(k_gain), _ptr(cos), _ptr(sin),
                           rot_dim, _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages),
                           _ptr(block_table), block_table.stride(0), n_tokens, n_q_heads, n_kv_heads,
                           head_dim, float(eps), 1 if write_kv else 0, _ptr(q_bias), _ptr(k_bias),
                           _ptr(v_bias), coef, every, 1 if values_from_keys else 0, _stream())


_qk_prepare_padded = _per_dtype("rope_kv", "ek_qk_prepare_padded_kv",
                                [_P, c_int, _P, _P, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int,
                                 c_int, c_int, c_float, c_int, _P, _P, _P, c_int, c_int, c_int, c_float, _P])


def qk_prepare_padded_kv(qkv, n_tokens, q_gain, k_gain, cos, sin, rot_dim, positions, token_slot,
                         k_pages, v_pages, block_table, n_q_heads, n_kv_heads, head_dim, eps, norm_dim,
                         write_kv=True, q_bias=None, k_bias=None, v_bias=None, value_unit_eps=None,
                         value_dim=None):
    """:func:`qk_prepare_kv` for heads padded with zeros to ``head_dim`` (the cache's head size): the
    gained norm of queries and keys takes its mean over ``norm_dim`` values; with ``value_unit_eps`` every
    value head is divided by its root mean square over ``value_dim`` values before it is stored."""
    _need_cuda(qkv, cos, sin, positions, token_slot, k_pages, v_pages, block_table, q_bias, k_bias, v_bias)
    check_head_dim(head_dim)
    heads = n_q_heads + (2 * n_kv_heads if write_kv else 0)      # (keys and values are read only to be stored)
    _need(qkv.stride(-1) == 1 and qkv.shape[-1] >= heads * head_dim, "qk_prepare_padded_kv: row width")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and cos.shape[-1] * 2 == rot_dim, "qk_prepare_padded_kv: 32-bit tables of rot_dim/2 columns")
    _need(k_pages.dtype == qkv.dtype and v_pages.dtype == qkv.dtype, "qk_prepare_padded_kv: cache dtype")
    for g in (q_gain, k_gain):
        _need(g is None or (g.dtype == torch.float32 and g.numel() == head_dim), "qk gains: 32-bit [D]")
    for b, n in ((q_bias, n_q_heads), (k_bias, n_kv_heads), (v_bias, n_kv_heads)):
        _need(b is None or (b.dtype == torch.float32 and b.is_contiguous() and b.numel() == n * head_dim),
              "qk_prepare_padded_kv: biases are 32-bit [heads * D]")
    if lib.recording():
        lib.annotate(bytes=n_tokens * head_dim * qkv.element_size() * (2 * n_q_heads + 3 * n_kv_heads))
    _qk_prepare_padded[qkv.dtype](_ptr(qkv), qkv.stride(0), _ptr(q_gain), _ptr(k_gain), _ptr(cos), _ptr(sin),
                                  rot_dim, _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages),
                                  _ptr(block_table), block_table.stride(0), n_tokens, n_q_heads, n_kv_heads,
                                  head_dim, float(eps), 1 if write_kv else 0, _ptr(q_bias), _ptr(k_bias),
                                  _ptr(v_bias), int(norm_dim), 1 if value_unit_eps is not None else 0,
                                  int(value_dim or head_dim), float(value_unit_eps or 0.0), _stream())


def qk_norm_rope_kv(qkv, n_tokens, q_gain, k_gain, cos, sin, rot_dim, positions, token_slot,
                    k_pages, v_pages, block_table, n_q_heads, n_kv_heads, head_dim, eps,
                    write_kv=True):
    """In place on the q part of ``qkv`` [T, (NQ + 2 NKV) D]; keys and values go to the pages."""
    _need_cuda(qkv, cos, sin, positions, token_slot, k_pages, v_pages, block_table)
    check_head_dim(head_dim)
    _need(qkv.stride(-1) == 1 and (qkv.shape[-1] == (n_q_heads + 2 * n_kv_heads) * head_dim
                                   or (not write_kv and qkv.shape[-1] == n_q_heads * head_dim)),
          "qk_norm_rope_kv: qkv width")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and cos.shape[-1] * 2 == rot_dim, "qk_norm_rope_kv: 32-bit tables of rot_dim/2 columns")
    _need(k_pages.dtype == qkv.dtype and v_pages.dtype == qkv.dtype, "qk_norm_rope_kv: cache dtype")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "qk_norm_rope_kv: int32 indices")
    for g in (q_gain, k_gain):
        _need(g is None or (g.dtype == torch.float32 and g.numel() == head_dim), "qk gains: 32-bit [D]")
    if lib.recording():
        lib.annotate(bytes=n_tokens * head_dim * qkv.element_size() * (2 * n_q_heads + 3 * n_kv_heads))
    _rope_kv[qkv.dtype](_ptr(qkv), qkv.stride(0), _ptr(q_gain), _ptr(k_gain), _ptr(cos), _ptr(sin),
                        rot_dim, _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages),
                        _ptr(block_table), block_table.stride(0), n_tokens, n_q_heads, n_kv_heads,
                        head_dim, float(eps), 1 if write_kv else 0, _stream())


_whole_norm_kv = _per_dtype("rope_kv", "ek_qk_whole_norm_kv",
                            [_P, c_int, _P, _P, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                             c_int, c_float, c_int, _P])


def qk_whole_norm_kv(rows, n_tokens, q_gain, k_gain, cos, sin, rot_dim, positions, token_slot, k_pages, v_pages,
                     block_table, n_q_heads, n_kv_heads, head_dim, eps, norm_dim=None, write_kv=True):
    """Queries and keys normed over the whole projection before they are cut into heads: all query heads of a
    token share one root mean square, all its key heads another (gains [heads * D], 32-bit); then the rotation.
    ``rows`` [T, .] holds query, key and value heads ``head_dim`` apart (keys and values are read only when
    ``write_kv``); queries stay in place, keys and values go to the pages.  ``norm_dim``: values a head really has,
    when heads are padded with zeros."""
    _need_cuda(rows, q_gain, k_gain, cos, sin, positions, token_slot, k_pages, v_pages, block_table)
    check_head_dim(head_dim)
    heads = n_q_heads + (2 * n_kv_heads if write_kv else 0)
    _need((n_q_heads + n_kv_heads) * head_dim <= WHOLE_NORM_MAX_VALUES,
          f"qk_whole_norm_kv: query and key heads of a token hold at most {WHOLE_NORM_MAX_VALUES} values together")
    _need(rows.stride(-1) == 1 and rows.shape[-1] >= heads * head_dim, "qk_whole_norm_kv: row width")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous() and sin.is_contiguous()
          and cos.shape[-1] * 2 == rot_dim, "qk_whole_norm_kv: 32-bit tables of rot_dim/2 columns")
    _need(k_pages.dtype == rows.dtype and v_pages.dtype == rows.dtype, "qk_whole_norm_kv: cache dtype")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "qk_whole_norm_kv: int32 indices")
    for g, n in ((q_gain, n_q_heads),) + (((k_gain, n_kv_heads),) if write_kv else ()):
        _need(g is not None and g.dtype == torch.float32 and g.is_contiguous() and g.numel() == n * head_dim,
              "qk_whole_norm_kv: gains are 32-bit [heads * D]")
    if lib.recording():
        lib.annotate(bytes=n_tokens * head_dim * rows.element_size() * (2 * n_q_heads + (4 * n_kv_heads if write_kv else 0)))
    _whole_norm_kv[rows.dtype](_ptr(rows), rows.stride(0), _ptr(q_gain), _ptr(k_gain), _ptr(cos), _ptr(sin), rot_dim,
                               _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages), _ptr(block_table),
                               block_table.stride(0), n_tokens, n_q_heads, n_kv_heads, head_dim,
                               int(norm_dim or head_dim), float(eps), 1 if write_kv else 0, _stream())


_rope_unit_kv = _per_dtype("rope_kv", "ek_qk_rope_unit_kv",
                           [_P, c_int, c_int, c_int, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int,
                            c_int, c_int, c_int, c_int, c_float, c_int, c_int, _P])


def qk_rope_unit_kv(rows, n_tokens, k_col, v_col, cos, sin, rot_dim, positions, token_slot, k_pages, v_pages,
                    block_table, n_q_heads, n_kv_heads, head_dim, norm_dim, eps, unit=True, write_kv=True):
    """Rotation first, then every query and key head divided by its root mean square over its first
    ``norm_dim`` values (no gain; ``unit`` False: rotation alone).  ``rows`` [T, .] holds a token's
    query heads from column 0 (in place), and - read only when ``write_kv`` - its key heads from
    ``k_col`` and value heads from ``v_col``, each ``head_dim`` apart; keys and values go to the pages."""
    _need_cuda(rows, cos, sin, positions, token_slot, k_pages, v_pages, block_table)
    check_head_dim(head_dim)
    _need(rows.stride(-1) == 1 and rows.shape[-1] >= n_q_heads * head_dim, "qk_rope_unit_kv: row width")
    _need(not write_kv or (k_col + n_kv_heads * head_dim <= rows.shape[-1]
                           and v_col + n_kv_heads * head_dim <= rows.shape[-1]),
          "qk_rope_unit_kv: key and value columns lie within the row")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and sin.is_contiguous() and cos.shape[-1] * 2 == rot_dim, "qk_rope_unit_kv: 32-bit tables of rot_dim/2 columns")
    _need(k_pages.dtype == rows.dtype and v_pages.dtype == rows.dtype, "qk_rope_unit_kv: cache dtype")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "qk_rope_unit_kv: int32 indices")
    if lib.recording():
        lib.annotate(bytes=n_tokens * head_dim * rows.element_size() * (2 * n_q_heads + (4 * n_kv_heads if write_kv else 0)))
    _rope_unit_kv[rows.dtype](_ptr(rows), rows.stride(0), k_col, v_col, _ptr(cos), _ptr(sin), rot_dim,
                              _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages), _ptr(block_table),
                              block_table.stride(0), n_tokens, n_q_heads, n_kv_heads, head_dim, norm_dim,
                              float(eps), 1 if unit else 0, 1 if write_kv else 0, _stream())


# ------------------------------------------------------------------ attention
_attn_generic = _per_dtype("attention_generic", "ek_attention_generic",
                           [_P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                            c_float, c_int, c_int, c_int, _P, _P, c_float, _P, c_int, _P, c_int, c_int, c_float, _P])
_NO_SINK = float("-inf")


def _sink(sink) -> float:
    """The kernels' encoding of an attention sink: its score, or -inf for none."""
    return _NO_SINK if sink is None else float(sink)


def _sinks(sinks, n_q_heads):
    """One sink score per query head (32-bit, on the device), or None."""
    if sinks is None:
        return None
    _need_cuda(sinks)
    _need(sinks.dtype == torch.float32 and sinks.is_contiguous() and sinks.numel() == n_q_heads,
          "attention: per-head sinks are 32-bit, one per query head")
    return sinks.data_ptr()


def attention_generic(out, q, n_tokens, positions, token_slot, k_pages, v_pages, block_table,
                      n_q_heads, n_kv_heads, head_dim, scale, window=None, n_splits=1,
                      keys_per_split=0, part_acc=None, part_ml=None, sink=None, sinks=None, keep_first=0,
                      gate=None, chunk=None, softcap=None):
    """out[t, h*D:(h+1)*D] = softmax(scale q.K^T) V over the keys token t may see.  ``sink``: the
    score of one more key without a value that every query sees - exp(sink) is added to the
    softmax denominator (the same in every attention kernel below).  ``sinks`` [NQ] (32-bit):
    one such score per query head instead (in every attention kernel).

    ``q`` is any tensor whose row t starts with the NQ*D query values (the fused q/k/v
    rows qualify).  With ``n_splits`` > 1 the keys are cut every ``keys_per_split`` and
    merged from ``part_acc`` [T, NQ, splits, D] / ``part_ml`` [T, NQ, splits, 2] (32-bit).
    ``keep_first`` (with a window): the first ``keep_first`` positions of a sequence stay visible to
    every later token beside its window.  ``gate`` [T, >= NQ] (rows may be a view into wider rows):
    head h's output at token t is multiplied by sigmoid(gate[t, h]).  ``chunk`` (instead of a window):
    position p sees only positions of its own chunk, floor(p / chunk).  ``softcap``: a score s becomes
    softcap * tanh(s / softcap) before the softmax.
    """
    _need_cuda(out, q, positions, token_slot, k_pages, v_pages, block_table, part_acc, part_ml, gate)
    _need(gate is None or (gate.dtype == q.dtype and gate.stride(-1) == 1 and gate.shape[-1] >= n_q_heads),
          "attention: the gate holds one value per token and query head, in q's dtype")
    _need(1 <= head_dim <= GENERIC_MAX_HEAD_DIM, f"attention_generic: head sizes up to {GENERIC_MAX_HEAD_DIM}")
    _need(out.dtype == q.dtype == k_pages.dtype, "attention: one dtype for q, cache and out")
    _need(out.is_contiguous() and out.shape[-1] == n_q_heads * head_dim, "attention: out [T, NQ*D]")
    _need(q.stride(-1) == 1, "attention: q rows must be dense")
    if n_splits > 1:
        _need(part_acc is not None and part_ml is not None
              and part_acc.numel() >= n_tokens * n_q_heads * n_splits * head_dim
              and part_ml.numel() >= n_tokens * n_q_heads * n_splits * 2, "attention: split buffers")
    _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, False, chunk)
    _attn_generic[q.dtype](_ptr(out), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot),
                           _ptr(k_pages), _ptr(v_pages), _ptr(block_table), block_table.stride(0),
                           n_tokens, n_q_heads, n_kv_heads, head_dim, float(scale),
                           int(window or 0), n_splits, keys_per_split, _ptr(part_acc),
                           _ptr(part_ml), _sink(sink), _sinks(sinks, n_q_heads), int(keep_first or 0),
                           _ptr(gate), gate.stride(0) if gate is not None else 0, int(chunk or 0),
                           float(softcap or 0.0), _stream())
    if n_splits > 1:
        count_extra_launches()               # the merge kernel


_attn_generic_cross = _per_dtype("attention_generic", "ek_attention_generic_cross",
                                 [_P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                                  c_float, c_int, c_int, c_int, _P, _P, c_int, _P])
_mix_heads = _per_dtype("attention_generic", "ek_mix_heads",
                        [_P, _P, _P, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, _P])


def attention_generic_cross(parts, q, n_tokens, positions, token_slot, k_pages, v_pages, block_table, n_q_heads,
                            n_kv_heads, head_dim, scale, window=None, n_splits=1, keys_per_split=0, part_acc=None,
                            part_ml=None, keep_first=0):
    """parts[t, g, c, :] = softmax_g(scale q_g.K^T) V_c: every query head's weights (against its own key
    head) applied to the values of EVERY key/value head c, in 32-bit ([T, NQ, NKV, D]) - what designs need
    that mix the heads' weights behind the softmax (:func:`mix_heads`).  Split buffers as in
    :func:`attention_generic`, with NQ * NKV rows a token."""
    _need_cuda(parts, q, positions, token_slot, k_pages, v_pages, block_table, part_acc, part_ml)
    _need(1 <= head_dim <= GENERIC_MAX_HEAD_DIM, f"attention_generic_cross: head sizes up to {GENERIC_MAX_HEAD_DIM}")
    _need(q.dtype == k_pages.dtype and parts.dtype == torch.float32 and parts.is_contiguous()
          and parts.numel() >= n_tokens * n_q_heads * n_kv_heads * head_dim and q.stride(-1) == 1,
          "attention_generic_cross: parts [T, NQ, NKV, D] in 32-bit")
    if n_splits > 1:
        _need(part_acc is not None and part_ml is not None
              and part_acc.numel() >= n_tokens * n_q_heads * n_kv_heads * n_splits * head_dim
              and part_ml.numel() >= n_tokens * n_q_heads * n_kv_heads * n_splits * 2, "attention: split buffers")
    _attention_cost(q, n_tokens, positions, n_q_heads * n_kv_heads, n_kv_heads, head_dim, window, False)
    _attn_generic_cross[q.dtype](_ptr(parts), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot),
                                 _ptr(k_pages), _ptr(v_pages), _ptr(block_table), block_table.stride(0),
                                 n_tokens, n_q_heads, n_kv_heads, head_dim, float(scale), int(window or 0),
                                 n_splits, keys_per_split, _ptr(part_acc), _ptr(part_ml), int(keep_first or 0),
                                 _stream())
    if n_splits > 1:
        count_extra_launches()


def mix_heads(out, parts, mix, positions, n_tokens, n_q_heads, n_kv_heads, head_dim, value_dim, gate=None):
    """out[t, h, :] = sigmoid(gate[t, h, :]) * sum_g mix[h, g] parts[t, g, h // (NQ / NKV), :value_dim]
    (``gate`` optional, rows of at least NQ * value_dim values in out's type; ``mix`` [NQ, NQ] 32-bit)."""
    _need_cuda(out, parts, mix, positions, gate)
    _need(parts.dtype == torch.float32 and mix.dtype == torch.float32 and mix.is_contiguous()
          and mix.numel() == n_q_heads * n_q_heads and out.is_contiguous()
          and out.shape[-1] == n_q_heads * value_dim, "mix_heads: out [T, NQ * value_dim], mix [NQ, NQ]")
    _need(gate is None or (gate.dtype == out.dtype and gate.stride(-1) == 1
                           and gate.shape[-1] >= n_q_heads * value_dim), "mix_heads: gate rows in out's type")
    if lib.recording():
        lib.annotate(bytes=n_tokens * n_q_heads * (4 * n_kv_heads * head_dim + 2 * value_dim * out.element_size()),
                     flops=2 * n_tokens * n_q_heads * n_q_heads * value_dim)
    _mix_heads[out.dtype](_ptr(out), _ptr(parts), _ptr(mix), _ptr(gate), gate.stride(0) if gate is not None else 0,
                          _ptr(positions), n_tokens, n_q_heads, n_kv_heads, head_dim, value_dim, _stream())


_attn_decode_bf16 = Function("attention_decode_bf16", "ek_attention_decode_bf16",
                             [_P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                              c_float, c_int, c_int, c_int, _P, _P, c_float, _P, c_int, _P, c_int, c_int, c_float, _P])


_attn_decode_cross = Function("attention_decode_bf16", "ek_attention_decode_cross_bf16",
                              [_P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                               c_float, c_int, c_int, c_int, _P, _P, c_int, _P])


def attention_decode_cross_bf16(parts, q, n_tokens, positions, token_slot, k_pages, v_pages, block_table, n_q_heads,
                                n_kv_heads, head_dim, scale, window=None, n_splits=1, keys_per_split=0, part_acc=None,
                                part_ml=None, keep_first=0):
    """:func:`attention_generic_cross` for single tokens in bfloat16 on the register-streaming decode kernel:
    a block takes a token, a key head's group and ONE value head, for every pair of the two; split buffers
    hold NQ * NKV rows a token."""
    _need_cuda(parts, q, positions, token_slot, k_pages, v_pages, block_table, part_acc, part_ml)
    _need(attention_decode_supported(q.dtype, head_dim), "attention_decode_cross_bf16: head sizes in steps of 32")
    _need(q.dtype == k_pages.dtype == torch.bfloat16 and parts.dtype == torch.float32 and parts.is_contiguous()
          and parts.numel() >= n_tokens * n_q_heads * n_kv_heads * head_dim and q.stride(-1) == 1
          and q.stride(0) % 8 == 0, "attention_decode_cross_bf16: parts [T, NQ, NKV, D] in 32-bit")
    if n_splits > 1:
        _need(part_acc is not None and part_ml is not None
              and part_acc.numel() >= n_tokens * n_q_heads * n_kv_heads * n_splits * head_dim
              and part_ml.numel() >= n_tokens * n_q_heads * n_kv_heads * n_splits * 2, "attention: split buffers")
    _attention_cost(q, n_tokens, positions, n_q_heads * n_kv_heads, n_kv_heads, head_dim, window, False)
    _attn_decode_cross(_ptr(parts), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot), _ptr(k_pages),
                       _ptr(v_pages), _ptr(block_table), block_table.stride(0), n_tokens, n_q_heads, n_kv_heads,
                       head_dim, float(scale), int(window or 0), n_splits, keys_per_split, _ptr(part_acc),
                       _ptr(part_ml), int(keep_first or 0), _stream())
    if n_splits > 1:
        count_extra_launches()


def _gate_args(gate, q, n_q_heads):
    """(pointer, row stride) of the optional per-head gate, checked."""
    _need(gate is None or (gate.is_cuda and gate.dtype == q.dtype and gate.stride(-1) == 1
                           and gate.shape[-1] >= n_q_heads),
          "attention: the gate holds one value per token and query head, in q's dtype")
    return _ptr(gate), (gate.stride(0) if gate is not None else 0)


def attention_decode_supported(dtype, head_dim):
    return dtype == torch.bfloat16 and head_dim % 32 == 0 and 32 <= head_dim <= MAX_HEAD_DIM


def attention_decode_bf16(out, q, n_tokens, positions, token_slot, k_pages, v_pages, block_table,
                          n_q_heads, n_kv_heads, head_dim, scale, window=None, n_splits=1,
                          keys_per_split=0, part_acc=None, part_ml=None, sink=None, sinks=None, keep_first=0,
                          gate=None, chunk=None, softcap=None):
    """One query token per row of ``q`` (bfloat16, head_dim a multiple of 32): same contract
    as :func:`attention_generic` (its options included); ``keys_per_split`` must be a
    multiple of 16, or 0 to cut every token's own window into ``n_splits`` equal parts."""
    _need_cuda(out, q, positions, token_slot, k_pages, v_pages, block_table, part_acc, part_ml)
    _need(attention_decode_supported(q.dtype, head_dim),
          "attention_decode_bf16: bfloat16 and a head size that is a multiple of 32")
    _need(out.dtype == q.dtype == k_pages.dtype, "attention: one dtype for q, cache and out")
    _need(out.is_contiguous() and out.shape[-1] == n_q_heads * head_dim, "attention: out [T, NQ*D]")
    _need(q.stride(-1) == 1 and q.stride(0) % 8 == 0, "attention: dense, 16-byte aligned q rows")
    if n_splits > 1:
        _need(keys_per_split % 16 == 0, "attention_decode_bf16: keys_per_split multiple of 16")
        _need(part_acc is not None and part_ml is not None
              and part_acc.numel() >= n_tokens * n_q_heads * n_splits * head_dim
              and part_ml.numel() >= n_tokens * n_q_heads * n_splits * 2, "attention: split buffers")
    _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, False, chunk)
    _attn_decode_bf16(_ptr(out), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot),
                      _ptr(k_pages), _ptr(v_pages), _ptr(block_table), block_table.stride(0),
                      n_tokens, n_q_heads, n_kv_heads, head_dim, float(scale), int(window or 0),
                      n_splits, keys_per_split, _ptr(part_acc), _ptr(part_ml), _sink(sink),
                      _sinks(sinks, n_q_heads), int(keep_first or 0), *_gate_args(gate, q, n_q_heads),
                      int(chunk or 0), float(softcap or 0.0), _stream())
    if n_splits > 1:
        count_extra_launches()               # the merge kernel


_attn_decode_tma = Function("attention_decode_tma", "ek_attention_decode_tma",
                            [_P, _P, c_int, _P, _P, _P, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int,
                             c_float, c_int, c_int, _P, c_float, _P, c_int, c_float, _P])
_attn_decode_tma_max = Function("attention_decode_tma", "ek_attention_decode_tma_max_splits", [c_int],
                                check_status=False)
DECODE_TMA_PORTABLE_SPLITS = 8
_decode_tma_max_splits = {}


def decode_tma_max_splits(head_dim, device=None):
    """Blocks that may share one token's pages in :func:`attention_decode_tma`: 16 where the device
    schedules thread-block clusters of that size for this head size, else the portable 8."""
    key = (head_dim, torch.cuda.current_device() if device is None else torch.device(device).index)
    if key not in _decode_tma_max_splits:
        with torch.cuda.device(key[1] if key[1] is not None else torch.cuda.current_device()):
            n = int(_attn_decode_tma_max(head_dim))
        _decode_tma_max_splits[key] = n if n in (8, 16) else DECODE_TMA_PORTABLE_SPLITS
    return _decode_tma_max_splits[key]


def attention_decode_tma_supported(dtype, head_dim, n_q_heads, n_kv_heads):
    return dtype == torch.bfloat16 and head_dim in (64, 128) and n_q_heads // n_kv_heads <= 16


def attention_decode_tma(out, q, n_tokens, positions, token_slot, k_pages, v_pages, block_table,
                         n_q_heads, n_kv_heads, head_dim, scale, window=None, n_splits=1, sink=None, chunk=None,
                         softcap=None, sinks=None):
    """One new token per sequence (bfloat16, head size 64 or 128, at most 16 heads a group): the
    cache pages come by TMA, started before the kernel ahead has finished; ``n_splits`` (1 to 8)
    blocks (16 where :func:`decode_tma_max_splits` says so) share a token's pages and merge inside
    a thread-block cluster.

    Precondition: ``positions``, ``token_slot`` and ``block_table`` are read before the kernel
    waits for the one ahead of it, so whatever wrote them (an upload, the state advance of the
    step before) must be separated from this launch by a launch that is not programmatic:
    :func:`embed`, the first kernel of every step, is one."""
    _need_cuda(out, q, positions, token_slot, k_pages, v_pages, block_table)
    _need(attention_decode_tma_supported(q.dtype, head_dim, n_q_heads, n_kv_heads),
          "attention_decode_tma: bfloat16, head size 64 or 128, at most 16 query heads a KV head")
    _need(out.dtype == q.dtype == k_pages.dtype, "attention: one dtype for q, cache and out")
    _need(out.is_contiguous() and out.shape[-1] == n_q_heads * head_dim, "attention: out [T, NQ*D]")
    _need(q.stride(-1) == 1 and q.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0,
          "attention: dense, 4-byte aligned q rows")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.dim() == 4
          and k_pages.shape[1:] == (n_kv_heads, PAGE, head_dim), "attention: pages [P, NKV, 64, D]")
    _need(1 <= n_splits <= decode_tma_max_splits(head_dim, q.device),
          f"attention_decode_tma: 1 to {decode_tma_max_splits(head_dim, q.device)} splits on this device")
    _need(n_tokens <= 65535, "attention_decode_tma: at most 65535 tokens a call")
    _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, False, chunk)
    _attn_decode_tma(_ptr(out), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot),
                     _ptr(k_pages), _ptr(v_pages), k_pages.shape[0], _ptr(block_table),
                     block_table.stride(0), n_tokens, n_q_heads, n_kv_heads, head_dim, float(scale),
                     int(window or 0), n_splits, _ptr(tc_status(q.device)), _sink(sink),
                     _sinks(sinks, n_q_heads), int(chunk or 0), float(softcap or 0.0), _stream())


_attn_prefill_bf16 = Function("attention_prefill_bf16", "ek_attention_prefill_bf16",
                              [_P, _P, c_int, _P, _P, _P, c_int, c_int, _P, _P, _P, c_int, c_int,
                               c_int, c_int, c_float, c_int, c_float, _P, c_int, _P, c_int, c_int, c_float, _P])


def attention_prefill_supported(dtype, head_dim, n_q_heads, n_kv_heads):
    return (dtype == torch.bfloat16 and head_dim % 16 == 0 and 16 <= head_dim <= MAX_HEAD_DIM
            and n_q_heads // n_kv_heads <= 128)


def attention_prefill_bf16(out, q, n_tokens, positions, token_slot, cu_seqlens, n_seqs, k_pages,
                           v_pages, block_table, n_q_heads, n_kv_heads, head_dim, scale,
                           window=None, sink=None, sinks=None, keep_first=0, gate=None, chunk=None,
                           softcap=None):
    """Several new tokens per sequence (bfloat16): sequence b owns rows cu_seqlens[b] ..
    cu_seqlens[b+1] of ``q``, which stand at consecutive positions; their keys and values
    are already in the pages.  ``keep_first``, ``gate``, ``chunk`` and ``softcap`` as in
    :func:`attention_generic`."""
    _need_cuda(out, q, positions, token_slot, cu_seqlens, k_pages, v_pages, block_table)
    _need(attention_prefill_supported(q.dtype, head_dim, n_q_heads, n_kv_heads),
          "attention_prefill_bf16: bfloat16, head size a multiple of 16, at most 128 heads a group")
    _need(out.dtype == q.dtype == k_pages.dtype, "attention: one dtype for q, cache and out")
    _need(out.is_contiguous() and out.shape[-1] == n_q_heads * head_dim, "attention: out [T, NQ*D]")
    _need(q.stride(-1) == 1 and q.stride(0) % 8 == 0, "attention: dense, 16-byte aligned q rows")
    _need(cu_seqlens.dtype == torch.int32 and cu_seqlens.numel() >= n_seqs + 1, "attention: cu_seqlens")
    _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, True, chunk)
    _attn_prefill_bf16(_ptr(out), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot),
                       _ptr(cu_seqlens), n_seqs, n_tokens, _ptr(k_pages), _ptr(v_pages),
                       _ptr(block_table), block_table.stride(0), n_q_heads, n_kv_heads, head_dim,
                       float(scale), int(window or 0), _sink(sink), _sinks(sinks, n_q_heads),
                       int(keep_first or 0), *_gate_args(gate, q, n_q_heads), int(chunk or 0),
                       float(softcap or 0.0), _stream())


_attn_prefill_tc = Function("attention_prefill_tc", "ek_attention_prefill_tc",
                            [_P, _P, c_int, _P, c_int, c_int, _P, _P, c_int, _P, c_int, c_int,
                             c_int, c_int, c_float, c_int, _P, c_float, _P, c_int, c_float, _P])
_attn_prefill_tiles = Function("attention_prefill_tc", "ek_attention_prefill_tiles",
                               [_P, c_int, _P, _P, _P, c_int, c_int, c_int, _P])
_attn_prefill_cross = Function("attention_prefill_bf16", "ek_attention_prefill_cross_bf16",
                               [_P, _P, c_int, _P, _P, _P, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int,
                                c_float, c_int, c_int, _P])


def attention_prefill_cross_bf16(parts, q, n_tokens, positions, token_slot, cu_seqlens, n_seqs, k_pages, v_pages,
                                 block_table, n_q_heads, n_kv_heads, head_dim, scale, window=None, keep_first=0):
    """:func:`attention_generic_cross` for prompts in bfloat16 on the ``mma.sync`` kernel: a block takes a
    tile of (token, head of the group) rows against one key head and ONE value head, for every pair of the two."""
    _need_cuda(parts, q, positions, token_slot, cu_seqlens, k_pages, v_pages, block_table)
    _need(attention_prefill_supported(q.dtype, head_dim, n_q_heads, n_kv_heads), "attention_prefill_cross_bf16: sizes")
    _need(q.dtype == k_pages.dtype == torch.bfloat16 and parts.dtype == torch.float32 and parts.is_contiguous()
          and parts.numel() >= n_tokens * n_q_heads * n_kv_heads * head_dim and q.stride(-1) == 1
          and q.stride(0) % 8 == 0, "attention_prefill_cross_bf16: parts [T, NQ, NKV, D] in 32-bit")
    _attention_cost(q, n_tokens, positions, n_q_heads * n_kv_heads, n_kv_heads, head_dim, window, True)
    _attn_prefill_cross(_ptr(parts), _ptr(q), q.stride(0), _ptr(positions), _ptr(token_slot), _ptr(cu_seqlens), n_seqs,
                        n_tokens, _ptr(k_pages), _ptr(v_pages), _ptr(block_table), block_table.stride(0), n_q_heads,
                        n_kv_heads, head_dim, float(scale), int(window or 0), int(keep_first or 0), _stream())


PREFILL_TC_ROWS = 128       # (token, query head of a group) rows a block of attention_prefill_tc owns
PREFILL_TC_MAX_SEQS = 1024


def attention_prefill_tc_supported(dtype, head_dim, n_q_heads, n_kv_heads):
    group = n_q_heads // n_kv_heads
    return dtype == torch.bfloat16 and head_dim in (64, 128) and 128 % group == 0


_l2_bytes = {}
PREFILL_BAND_L2_SHARE = 0.5


def prefill_band_tokens(n_kv_heads, head_dim, device=None) -> int:
    """Tokens of context whose 16-bit keys and values of one layer fill ``PREFILL_BAND_L2_SHARE`` of
    the device's L2: the sequences that the prompt attention works on together."""
    index = torch.cuda.current_device() if device is None or torch.device(device).index is None \
        else torch.device(device).index
    if index not in _l2_bytes:
        _l2_bytes[index] = int(torch.cuda.get_device_properties(index).L2_cache_size)
    return max(1, int(_l2_bytes[index] * PREFILL_BAND_L2_SHARE) // (4 * n_kv_heads * head_dim))


def attention_prefill_tiles(tiles, n_tokens, positions, token_slot, cu_seqlens, n_seqs, n_q_heads, n_kv_heads,
                            head_dim):
    """Fill ``tiles`` (int32 [>= tiles_needed, 4]) with the table of tiles that
    :func:`attention_prefill_tc` walks for this step's sequences and these head counts: (first token,
    tokens, position of the first, slot) per tile; the sequences in bands whose keys and values fit
    L2 together (longest context first), inside a band the longest key ranges first; padded with
    empty tiles.
    It is read by the attention kernels before they wait for the kernel ahead of them, so it has
    to be made before the step's first kernel (:func:`embed`, a plain launch), not just before the
    attention; returns the number of entries to pass on."""
    _need_cuda(tiles, positions, token_slot, cu_seqlens)
    tok_per_tile = PREFILL_TC_ROWS // (n_q_heads // n_kv_heads)
    need = -(-n_tokens // tok_per_tile) + n_seqs
    _need(tiles.dtype == torch.int32 and tiles.is_contiguous() and tiles.numel() >= 4 * need
          and tiles.data_ptr() % 16 == 0, "attention_prefill_tiles: int32 [tiles, 4], 16-byte aligned")
    _need(n_seqs <= PREFILL_TC_MAX_SEQS, f"attention_prefill_tc: at most {PREFILL_TC_MAX_SEQS} sequences a step")
    _need(cu_seqlens.dtype == torch.int32 and cu_seqlens.numel() >= n_seqs + 1, "attention: cu_seqlens")
    _attn_prefill_tiles(_ptr(tiles), need, _ptr(cu_seqlens), _ptr(positions), _ptr(token_slot), n_seqs,
                        tok_per_tile, prefill_band_tokens(n_kv_heads, head_dim, tiles.device), _stream())
    return need


def attention_prefill_tc(out, q, n_tokens, positions, token_slot, cu_seqlens, n_seqs, k_pages,
                         v_pages, block_table, n_q_heads, n_kv_heads, head_dim, scale, window=None,
                         tiles=None, n_tiles=0, sink=None, chunk=None, softcap=None, sinks=None):
    """:func:`attention_prefill_bf16` on tcgen05 tensor cores (head sizes 64 and 128, groups
    that divide 128): TMA-fed pages, scores and P.V in TMEM.  ``tiles`` / ``n_tiles``: the table
    :func:`attention_prefill_tiles` made for this step (made once, before the step's first
    kernel, and used by every layer); without it the table is made here and the stream is
    waited for, which suits a single call, not a model's step."""
    _need_cuda(out, q, positions, token_slot, cu_seqlens, k_pages, v_pages, block_table, tiles)
    _need(attention_prefill_tc_supported(q.dtype, head_dim, n_q_heads, n_kv_heads),
          "attention_prefill_tc: bfloat16, head size 64 or 128, a group size that divides 128")
    _need(out.dtype == q.dtype == k_pages.dtype, "attention: one dtype for q, cache and out")
    _need(out.is_contiguous() and out.shape[-1] == n_q_heads * head_dim, "attention: out [T, NQ*D]")
    _need(q.stride(-1) == 1 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0,
          "attention: dense, 16-byte aligned q rows")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.dim() == 4
          and k_pages.shape[1:] == (n_kv_heads, PAGE, head_dim), "attention: pages [P, NKV, 64, D]")
    if tiles is None:
        tok_per_tile = PREFILL_TC_ROWS // (n_q_heads // n_kv_heads)
        tiles = torch.empty((-(-n_tokens // tok_per_tile) + n_seqs, 4), dtype=torch.int32, device=q.device)
        n_tiles = attention_prefill_tiles(tiles, n_tokens, positions, token_slot, cu_seqlens, n_seqs,
                                          n_q_heads, n_kv_heads, head_dim)
        torch.cuda.current_stream().synchronize()
    _need(tiles.dtype == torch.int32 and tiles.numel() >= 4 * n_tiles and tiles.data_ptr() % 16 == 0,
          "attention_prefill_tc: the table of tiles")
    _attention_cost(q, n_tokens, positions, n_q_heads, n_kv_heads, head_dim, window, True, chunk)
    _attn_prefill_tc(_ptr(out), _ptr(q), q.stride(0), _ptr(tiles), n_tiles, n_tokens, _ptr(k_pages),
                     _ptr(v_pages), k_pages.shape[0], _ptr(block_table), block_table.stride(0), n_q_heads,
                     n_kv_heads, head_dim, float(scale), int(window or 0),
                     _ptr(tc_status(q.device)), _sink(sink), _sinks(sinks, n_q_heads), int(chunk or 0),
                     float(softcap or 0.0), _stream())


# ------------------------------------------------------------------ matrix products
_gemm_f32 = Function("gemm_f32", "ek_gemm_nt_f32",
                     [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P])
EPI_BF16, EPI_F32, EPI_SWIGLU, EPI_GEGLU = 0, 1, 2, 3      # GEGLU: the gate is the tanh form of GELU
# ("clamped" is EPI_SWIGLU with a gate_limit)
GATED_EPILOGUES = {"silu": EPI_SWIGLU, "gelu_tanh": EPI_GEGLU, "clamped": EPI_SWIGLU}
# EPI_BF16 computed by the compiled image that also holds the extended q/k/v epilogue (swapped form):
# for the other few-row products of a model whose q/k/v product runs there, so that one kernel's code
# serves them all (see Mixer.product_image)
EPI_BF16_EXTENDED = 4


def gemm_f32(out, x, w, n_rows=None):
    """out[M, N] = x[M, K] . w[N, K]^T in true 32-bit."""
    _need_cuda(out, x, w)
    _need(out.dtype == x.dtype == w.dtype == torch.float32, "gemm_f32: float32 tensors")
    _need(x.stride(-1) == 1 and w.stride(-1) == 1 and out.stride(-1) == 1, "gemm_f32: dense rows")
    m = n_rows if n_rows is not None else x.shape[0]
    n, k = w.shape
    _need(x.shape[-1] == k and out.shape[-1] == n and out.shape[0] >= m, "gemm_f32: shapes disagree")
    if lib.recording():
        lib.annotate(bytes=4 * (n * k + m * k + m * n), flops=2 * m * n * k)
    _gemm_f32(_ptr(out), _ptr(x), _ptr(w), m, n, k, x.stride(0), w.stride(0), out.stride(0), _stream())


B200_SM_COUNT = 148        # used only where no device can be asked (launch plans worked out on a CPU box)
_sm_counts = {}


def sm_count(device=None) -> int:
    """Streaming multiprocessors of ``device`` (the current one if None), asked once."""
    if not torch.cuda.is_available():
        return B200_SM_COUNT
    index = torch.cuda.current_device() if device is None or torch.device(device).index is None \
        else torch.device(device).index
    if index not in _sm_counts:
        _sm_counts[index] = int(torch.cuda.get_device_properties(index).multi_processor_count)
    return _sm_counts[index]


_SPLIT_PARTIAL_FLOATS = 4 * 1024 * 1024      # 16 MiB of split partials per device
_SPLIT_TICKETS = 16384
_split_scratch = {}


def split_scratch(device):
    """Per-device scratch of products whose K is split over more blocks than a cluster holds:
    partial tiles and zeroed tickets.  Created on first use; create it before capturing a graph
    (``ModelRunner`` does)."""
    key = str(torch.device(device))
    if key not in _split_scratch:
        _split_scratch[key] = (torch.empty(_SPLIT_PARTIAL_FLOATS, dtype=torch.float32, device=device),
                               torch.zeros(_SPLIT_TICKETS, dtype=torch.int32, device=device))
    return _split_scratch[key]


_gemm_tc = Function("gemm_tc_bf16", "ek_gemm_tc_bf16",
                    [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                     _P, _P, c_longlong, c_int, _P, c_int, c_int, c_float, _P, c_int, _P, _P, c_float, _P, _P])
_tc_status = {}
TC_SWAP_MAX_ROWS = 64


def tc_status(device):
    """One int per device that the tensor-core GEMM sets when a barrier wait times out."""
    key = str(torch.device(device))
    if key not in _tc_status:
        _tc_status[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _tc_status[key]


def check_tc_status(device):
    """Synchronises; raises if a kernel gave up a bounded barrier wait since the last check (products:
    1 producer, 2 MMA, 3 epilogue, 4 copies before exit; decode attention 41, 42; others by their
    kernel) and clears the word, so that the next check speaks of later launches only."""
    code = int(tc_status(device).item())
    if code:
        tc_status(device).zero_()
        raise KernelError(f"a bounded barrier wait ran out in a tensor-core kernel (code {code}); "
                          "results since the last check are invalid")


_wait_that_runs_out = Function("gemm_tc_bf16", "ek_tc_wait_that_runs_out", [_P, c_int, ctypes.c_uint, _P])


def wait_that_runs_out(device, code=77, limit=4096):
    """Launch one thread that waits ``limit`` rounds for a barrier nothing completes, gives up and
    records ``code`` in the device's status word - what a kernel does when a wait of its own runs
    out.  The kernel ends by itself; :func:`check_tc_status` then raises."""
    with torch.cuda.device(device):
        _wait_that_runs_out(_ptr(tc_status(device)), int(code), int(limit), _stream())


TC_MAX_CLUSTER = 8          # blocks of a thread-block cluster (the portable limit)


def swap_k_split(n_out, k, epilogue):
    """Blocks that share a tile's K in the swapped form: two blocks fit an SM - fill those 296
    places, keep at least 8 K blocks a block, stay within one cluster, and take a power of two
    (clusters of 3, 5, 6 or 7 blocks do not pack the GPCs evenly: 5 -> 4 was worth 0.6-1 % of a step)."""
    tiles = -(-n_out // (64 if epilogue in (EPI_SWIGLU, EPI_GEGLU) else 128))
    k_blocks = -(-k // 64)
    split = max(1, min(2 * sm_count() // tiles, k_blocks // 8, TC_MAX_CLUSTER))
    return 1 << (split.bit_length() - 1)


def gemm_tc_bf16(out, x, w, epilogue=EPI_BF16, n_rows=None, swap=None, k_split=None, cluster=True,
                 row_scale=None, residual=None, gate_limit=0.0):
    """out = x . w^T (or the SwiGLU of it) on tcgen05 tensor cores with TMA-staged operands.

    ``swap`` (default: at most 64 rows) puts the weights on the 128-row side of the MMA and
    splits K over ``k_split`` blocks; otherwise 128 x 128 tiles of the output.  Up to 8 splits
    add their partial tiles through the distributed shared memory of a thread-block cluster
    (``cluster``), more of them through scratch in global memory.

    Two options of the swapped form carry a norm that was moved out of its own kernel.
    ``row_scale=(ss, size, eps)``: row r of the 32-bit result is multiplied by
    rsqrt(sum(ss[r, :]) / size + eps) before the epilogue (``ss`` [rows, tiles], 32-bit).
    ``gate_limit`` > 0 (with ``EPI_SWIGLU``): the clamped gate of :func:`act_mul` in place of SiLU.
    ``residual=(stream, gain, ss_out)`` (bfloat16 result, N a multiple of 4): the result is added to
    the 32-bit ``stream`` [rows, N] in place, ``out`` gets stream * gain, and ``ss_out`` [rows,
    ceil(N / 128)] the sum of stream^2 over each 128-column tile.
    """
    _need_cuda(out, x, w)
    m = n_rows if n_rows is not None else x.shape[0]
    n, k = w.shape
    _need(x.dtype == w.dtype == torch.bfloat16, "gemm_tc_bf16: bfloat16 operands")
    _need(k % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0,
          f"gemm_tc_bf16: inner size {k} and row strides must be multiples of 8")
    _need(x.stride(-1) == 1 and w.stride(-1) == 1 and out.stride(-1) == 1 and x.shape[-1] == k,
          "gemm_tc_bf16: dense rows of matching inner size")
    _need(x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0, "gemm_tc_bf16: 16-byte aligned operands")
    n_out = n // 2 if epilogue in (EPI_SWIGLU, EPI_GEGLU) else n
    _need(out.shape[-1] == n_out and out.shape[0] >= m, "gemm_tc_bf16: out shape")
    _need(out.dtype == (torch.float32 if epilogue == EPI_F32 else torch.bfloat16), "gemm_tc_bf16: out dtype")
    if swap is None:
        swap = m <= TC_SWAP_MAX_ROWS
    _need(epilogue != EPI_BF16_EXTENDED or swap, "gemm_tc_bf16: the extended image is a swapped form")
    _need(not swap or m <= TC_SWAP_MAX_ROWS, "gemm_tc_bf16: the swapped form takes at most 64 rows")
    partials, tickets = split_scratch(x.device)
    if k_split is None:
        k_split = swap_k_split(n_out, k, epilogue) if swap else 1
    if row_scale is not None or residual is not None:
        cluster, k_split = True, min(k_split, TC_MAX_CLUSTER)     # these forms have no scratch path
    ss_in, ss_tiles, size, eps = None, 0, 0, 0.0
    if row_scale is not None:
        ss_in, size, eps = row_scale
        _need(swap and ss_in.dtype == torch.float32 and ss_in.is_contiguous() and ss_in.dim() == 2
              and ss_in.shape[0] >= m and ss_in.is_cuda, "gemm_tc_bf16: row_scale needs 32-bit sums [rows, tiles]")
        ss_tiles = ss_in.shape[1]
    stream, gain, ss_out, ld_stream = None, None, None, 0
    if residual is not None:
        stream, gain, ss_out = residual
        _need_cuda(stream, gain, ss_out)
        _need(swap and epilogue in (EPI_BF16, EPI_BF16_EXTENDED) and n % 4 == 0 and out.stride(0) % 4 == 0,
              "gemm_tc_bf16: residual needs the swapped form, a bfloat16 result and N a multiple of 4")
        _need(stream.dtype == torch.float32 and stream.stride(-1) == 1 and stream.stride(0) % 4 == 0
              and stream.shape[-1] == n and stream.shape[0] >= m and stream.data_ptr() % 16 == 0,
              "gemm_tc_bf16: residual stream [rows, N] in 32-bit, 16-byte aligned rows")
        _need(gain.dtype == torch.float32 and gain.numel() == n and gain.data_ptr() % 16 == 0,
              "gemm_tc_bf16: gain [N] in 32-bit")
        _need(ss_out.dtype == torch.float32 and ss_out.is_contiguous() and ss_out.shape[0] >= m
              and ss_out.shape[1] == -(-n // 128), "gemm_tc_bf16: ss_out [rows, ceil(N/128)] in 32-bit")
        ld_stream = stream.stride(0)
    if lib.recording():
        moved = 2 * (n * k + m * k) + m * n_out * out.element_size() + (8 * m * n if residual is not None else 0)
        lib.annotate(bytes=moved, flops=2 * m * n * k, label=f"{n}x{k}")
    _gemm_tc(_ptr(out), _ptr(x), _ptr(w), m, n, k, x.stride(0), w.stride(0), out.stride(0),
             epilogue, 1 if swap else 0, k_split, 1 if cluster else 0, _ptr(partials), _ptr(tickets),
             _SPLIT_PARTIAL_FLOATS, _SPLIT_TICKETS, _ptr(ss_in), ss_tiles, int(size), float(eps),
             _ptr(stream), ld_stream, _ptr(gain), _ptr(ss_out), float(gate_limit), _ptr(tc_status(x.device)),
             _stream())


_gemm_pair = Function("gemm_pair_bf16", "ek_gemm_pair_bf16",
                      [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P, _P])
PAIR_EPI_BF16, PAIR_EPI_ADD_F32, PAIR_EPI_SWIGLU, PAIR_EPI_GEGLU = 0, 1, 2, 4
PAIR_GATED_EPILOGUES = {"silu": PAIR_EPI_SWIGLU, "gelu_tanh": PAIR_EPI_GEGLU, "clamped": PAIR_EPI_SWIGLU}


def gemm_pair_takes(out, x, w, epilogue) -> bool:
    """Whether :func:`gemm_pair_bf16` can address these operands (16-byte aligned rows)."""
    return (x.dtype == w.dtype == torch.bfloat16 and w.shape[1] % 8 == 0 and x.stride(0) % 8 == 0
            and w.stride(0) % 8 == 0 and x.stride(-1) == 1 and w.stride(-1) == 1 and out.stride(-1) == 1
            and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0 and out.data_ptr() % 16 == 0
            and out.stride(0) % (4 if epilogue == PAIR_EPI_ADD_F32 else 8) == 0)


def gemm_pair_bf16(out, x, w, epilogue=PAIR_EPI_BF16, n_rows=None, gate_limit=0.0):
    """The product for many rows on pairs of SMs (``tcgen05.mma.cta_group::2``, 256 x 256 tiles, a
    persistent launch).  ``PAIR_EPI_BF16``: out [M, N] = x . w^T in bfloat16; ``PAIR_EPI_ADD_F32``:
    out [M, N] (32-bit) += x . w^T; ``PAIR_EPI_SWIGLU``: out [M, N / 2] = silu(x . wg^T) * (x . wu^T)
    with w = [gate rows; up rows]; ``PAIR_EPI_GEGLU``: the same with the tanh form of GELU;
    ``gate_limit`` > 0 with ``PAIR_EPI_SWIGLU``: the clamped gate of :func:`act_mul`."""
    _need_cuda(out, x, w)
    m = n_rows if n_rows is not None else x.shape[0]
    n, k = w.shape
    _need(gemm_pair_takes(out, x, w, epilogue) and x.shape[-1] == k,
          "gemm_pair_bf16: bfloat16 operands with dense, 16-byte aligned rows of matching inner size")
    _need(epilogue in (PAIR_EPI_BF16, PAIR_EPI_ADD_F32, PAIR_EPI_SWIGLU, PAIR_EPI_GEGLU), "gemm_pair_bf16: epilogue")
    gated = epilogue in (PAIR_EPI_SWIGLU, PAIR_EPI_GEGLU)
    _need(not gated or n % 2 == 0, "gemm_pair_bf16: a gated epilogue needs gate and up rows")
    n_out = n // 2 if gated else n
    _need(out.shape[-1] == n_out and out.shape[0] >= m and x.shape[0] >= m, "gemm_pair_bf16: out shape")
    _need(out.dtype == (torch.float32 if epilogue == PAIR_EPI_ADD_F32 else torch.bfloat16),
          "gemm_pair_bf16: out dtype")
    if lib.recording():
        moved = 2 * (n * k + m * k) + m * n_out * (8 if epilogue == PAIR_EPI_ADD_F32 else 2)
        lib.annotate(bytes=moved, flops=2 * m * n * k, label=f"{n}x{k}")
    _gemm_pair(_ptr(out), _ptr(x), _ptr(w), m, n, k, x.stride(0), w.stride(0), out.stride(0), epilogue,
               float(gate_limit), _ptr(tc_status(x.device)), _stream())


_gemm_tc_qkv = Function("gemm_tc_bf16", "ek_gemm_tc_qkv_rope",
                        [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float,
                         _P, _P, c_float, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, _P, _P])
QKV_ROPE_HEAD_DIM = 128


def gemm_tc_qkv_rope(qkv, x, w, n_rows, q_gain, k_gain, qk_eps, cos, sin, positions, token_slot, k_pages,
                     v_pages, block_table, n_q_heads, n_kv_heads, write_kv=True, row_scale=None,
                     k_split=None):
    """The q/k/v product of an attention layer with heads of 128, fully rotated, for at most 64
    rows, with :func:`qk_norm_rope_kv` done in its epilogue on the 32-bit sums: q (normalised,
    rotated) goes to the q part of ``qkv`` [rows, (NQ + 2 NKV) * 128], k and v to the pages.
    ``row_scale`` as in :func:`gemm_tc_bf16`."""
    _need_cuda(qkv, x, w, cos, sin, positions, token_slot, k_pages, v_pages, block_table)
    m, (n, k) = n_rows, w.shape
    _need(x.dtype == w.dtype == qkv.dtype == k_pages.dtype == v_pages.dtype == torch.bfloat16,
          "gemm_tc_qkv_rope: bfloat16 operands, result and cache")
    _need(m <= TC_SWAP_MAX_ROWS and n == (n_q_heads + 2 * n_kv_heads) * QKV_ROPE_HEAD_DIM,
          "gemm_tc_qkv_rope: at most 64 rows, heads of 128")
    _need(k % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0 and x.stride(-1) == 1
          and w.stride(-1) == 1 and x.shape[-1] == k and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0,
          "gemm_tc_qkv_rope: dense, 16-byte aligned operand rows")
    _need(qkv.stride(-1) == 1 and qkv.shape[-1] == n and qkv.stride(0) % 4 == 0 and qkv.shape[0] >= m,
          "gemm_tc_qkv_rope: qkv [rows, (NQ + 2 NKV) * 128]")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and sin.is_contiguous() and cos.shape[-1] == QKV_ROPE_HEAD_DIM // 2,
          "gemm_tc_qkv_rope: 32-bit tables of 64 columns")
    for g in (q_gain, k_gain):
        _need(g is None or (g.is_cuda and g.dtype == torch.float32 and g.numel() == QKV_ROPE_HEAD_DIM),
              "qk gains: 32-bit [128]")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.dim() == 4
          and k_pages.shape[1:] == (n_kv_heads, PAGE, QKV_ROPE_HEAD_DIM), "attention: pages [P, NKV, 64, 128]")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "gemm_tc_qkv_rope: int32 indices")
    ss_in, ss_tiles, size, eps = None, 0, 0, 0.0
    if row_scale is not None:
        ss_in, size, eps = row_scale
        _need(ss_in.is_cuda and ss_in.dtype == torch.float32 and ss_in.is_contiguous() and ss_in.dim() == 2
              and ss_in.shape[0] >= m, "gemm_tc_qkv_rope: row_scale needs 32-bit sums [rows, tiles]")
        ss_tiles = ss_in.shape[1]
    if k_split is None:
        k_split = swap_k_split(n, k, EPI_BF16)
    if lib.recording():
        lib.annotate(bytes=2 * (n * k + m * k + m * n), flops=2 * m * n * k)
    _gemm_tc_qkv(_ptr(qkv), _ptr(x), _ptr(w), m, k, x.stride(0), w.stride(0), qkv.stride(0), k_split,
                 _ptr(ss_in), ss_tiles, int(size), float(eps), _ptr(q_gain), _ptr(k_gain), float(qk_eps),
                 _ptr(cos), _ptr(sin), _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages),
                 _ptr(block_table), block_table.stride(0), n_q_heads, n_kv_heads, 1 if write_kv else 0,
                 _ptr(tc_status(x.device)), _stream())


_gemm_tc_qkv_prepare = Function("gemm_tc_bf16", "ek_gemm_tc_qkv_prepare",
                                [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float,
                                 _P, _P, c_float, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int,
                                 _P, _P, _P, c_float, c_int, c_int, _P, _P])


def gemm_tc_qkv_prepare(qkv, x, w, n_rows, q_gain, k_gain, qk_eps, cos, sin, positions, token_slot, k_pages,
                        v_pages, block_table, n_q_heads, n_kv_heads, write_kv=True, row_scale=None,
                        k_split=None, q_bias=None, k_bias=None, v_bias=None, q_temperature=None,
                        values_from_keys=False):
    """:func:`gemm_tc_qkv_rope` with the options of :func:`qk_prepare_kv` done in the product's
    epilogue on the 32-bit sums (heads of 128, at most 64 rows): biases, the query temperature,
    values taken from the keys as projected (``w`` and ``qkv`` then hold NQ + NKV heads).  ``cos`` and
    ``sin`` may be None: no rotation."""
    _need_cuda(qkv, x, w, cos, sin, positions, token_slot, k_pages, v_pages, block_table, q_bias, k_bias, v_bias)
    m, (n, k) = n_rows, w.shape
    heads = n_q_heads + (1 if values_from_keys else 2) * n_kv_heads
    _need(x.dtype == w.dtype == qkv.dtype == k_pages.dtype == v_pages.dtype == torch.bfloat16,
          "gemm_tc_qkv_prepare: bfloat16 operands, result and cache")
    _need(m <= TC_SWAP_MAX_ROWS and n == heads * QKV_ROPE_HEAD_DIM, "gemm_tc_qkv_prepare: at most 64 rows, heads of 128")
    _need(k % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0 and x.stride(-1) == 1
          and w.stride(-1) == 1 and x.shape[-1] == k and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0,
          "gemm_tc_qkv_prepare: dense, 16-byte aligned operand rows")
    _need(qkv.stride(-1) == 1 and qkv.shape[-1] == n and qkv.stride(0) % 4 == 0 and qkv.shape[0] >= m,
          "gemm_tc_qkv_prepare: qkv [rows, heads * 128]")
    _need((cos is None) == (sin is None), "gemm_tc_qkv_prepare: both tables or none")
    if cos is not None:
        _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
              and sin.is_contiguous() and cos.shape[-1] == QKV_ROPE_HEAD_DIM // 2,
              "gemm_tc_qkv_prepare: 32-bit tables of 64 columns")
    for g in (q_gain, k_gain):
        _need(g is None or (g.is_cuda and g.dtype == torch.float32 and g.numel() == QKV_ROPE_HEAD_DIM),
              "qk gains: 32-bit [128]")
    for b, nh in ((q_bias, n_q_heads), (k_bias, n_kv_heads), (v_bias, n_kv_heads)):
        _need(b is None or (b.dtype == torch.float32 and b.is_contiguous() and b.numel() == nh * QKV_ROPE_HEAD_DIM),
              "gemm_tc_qkv_prepare: biases are 32-bit [heads * 128]")
    _need(not (values_from_keys and v_bias is not None), "gemm_tc_qkv_prepare: values taken from keys have no bias")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.dim() == 4
          and k_pages.shape[1:] == (n_kv_heads, PAGE, QKV_ROPE_HEAD_DIM), "attention: pages [P, NKV, 64, 128]")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32, "gemm_tc_qkv_prepare: int32 indices")
    coef, every = (0.0, 1) if q_temperature is None else (float(q_temperature[0]), int(q_temperature[1]))
    _need(every >= 1, "gemm_tc_qkv_prepare: the temperature's step must be at least one position")
    ss_in, ss_tiles, size, eps = None, 0, 0, 0.0
    if row_scale is not None:
        ss_in, size, eps = row_scale
        _need(ss_in.is_cuda and ss_in.dtype == torch.float32 and ss_in.is_contiguous() and ss_in.dim() == 2
              and ss_in.shape[0] >= m, "gemm_tc_qkv_prepare: row_scale needs 32-bit sums [rows, tiles]")
        ss_tiles = ss_in.shape[1]
    if k_split is None:
        k_split = swap_k_split(n, k, EPI_BF16)
    if lib.recording():
        lib.annotate(bytes=2 * (n * k + m * k + m * n), flops=2 * m * n * k)
    _gemm_tc_qkv_prepare(_ptr(qkv), _ptr(x), _ptr(w), m, k, x.stride(0), w.stride(0), qkv.stride(0), k_split,
                         _ptr(ss_in), ss_tiles, int(size), float(eps), _ptr(q_gain), _ptr(k_gain), float(qk_eps),
                         _ptr(cos), _ptr(sin), _ptr(positions), _ptr(token_slot), _ptr(k_pages), _ptr(v_pages),
                         _ptr(block_table), block_table.stride(0), n_q_heads, n_kv_heads, 1 if write_kv else 0,
                         _ptr(q_bias), _ptr(k_bias), _ptr(v_bias), coef, every, 1 if values_from_keys else 0,
                         _ptr(tc_status(x.device)), _stream())


_gemm_pair_qkv = Function("gemm_pair_bf16", "ek_gemm_pair_qkv_rope",
                          [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P, _P, c_float, _P, _P, _P, _P, _P,
                           _P, _P, c_int, c_int, c_int, c_int, _P, _P])


def gemm_pair_qkv_rope(qkv, x, w, n_rows, q_gain, k_gain, qk_eps, cos, sin, positions, token_slot, k_pages,
                       v_pages, block_table, n_q_heads, n_kv_heads, write_kv=True):
    """The q/k/v product of many rows (the pair kernel) with the per-head RMSNorm of q and k, the rotation
    and the cache write in its epilogue (heads of 128, fully rotated).  Of ``qkv`` only the q columns are
    written; k and v go to the pages.  Rows with a negative position are skipped."""
    _need_cuda(qkv, x, w, cos, sin, positions, token_slot, k_pages, v_pages, block_table)
    m, (n, k) = n_rows, w.shape
    _need(x.dtype == w.dtype == qkv.dtype == k_pages.dtype == v_pages.dtype == torch.bfloat16,
          "gemm_pair_qkv_rope: bfloat16 operands, result and cache")
    _need(n == (n_q_heads + 2 * n_kv_heads) * QKV_ROPE_HEAD_DIM and gemm_pair_takes(qkv, x, w, PAIR_EPI_BF16)
          and x.shape[-1] == k and x.shape[0] >= m,
          "gemm_pair_qkv_rope: heads of 128, dense 16-byte aligned operand rows")
    _need(qkv.shape[-1] == n and qkv.shape[0] >= m, "gemm_pair_qkv_rope: qkv [rows, (NQ + 2 NKV) * 128]")
    _need(cos.dtype == torch.float32 and sin.dtype == torch.float32 and cos.is_contiguous()
          and sin.is_contiguous() and cos.shape[-1] == QKV_ROPE_HEAD_DIM // 2,
          "gemm_pair_qkv_rope: 32-bit tables of 64 columns")
    for g in (q_gain, k_gain):
        _need(g is None or (g.is_cuda and g.dtype == torch.float32 and g.numel() == QKV_ROPE_HEAD_DIM),
              "qk gains: 32-bit [128]")
    _need(k_pages.is_contiguous() and v_pages.is_contiguous() and k_pages.dim() == 4
          and k_pages.shape[1:] == (n_kv_heads, PAGE, QKV_ROPE_HEAD_DIM), "attention: pages [P, NKV, 64, 128]")
    _need(block_table.dtype == torch.int32 and positions.dtype == torch.int32
          and token_slot.dtype == torch.int32 and positions.numel() >= m and token_slot.numel() >= m,
          "gemm_pair_qkv_rope: int32 indices, one per row")
    if lib.recording():
        lib.annotate(bytes=2 * (n * k + m * k + m * n), flops=2 * m * n * k, label=f"{n}x{k}")
    _gemm_pair_qkv(_ptr(qkv), _ptr(x), _ptr(w), m, k, x.stride(0), w.stride(0), qkv.stride(0),
                   _ptr(q_gain), _ptr(k_gain), float(qk_eps), _ptr(cos), _ptr(sin), _ptr(positions),
                   _ptr(token_slot), _ptr(k_pages), _ptr(v_pages), _ptr(block_table), block_table.stride(0),
                   n_q_heads, n_kv_heads, 1 if write_kv else 0, _ptr(tc_status(x.device)), _stream())


# ------------------------------------------------------------------ sampling and decode state
_sample = Function("sampling", "ek_sample",
                   [_P, _P, c_longlong, c_int, c_int, c_float, c_int, c_ulonglong, _P, _P, _P, _P, _P])
_sample_wide = Function("sampling", "ek_sample_wide",
                        [_P, _P, c_longlong, c_int, c_int, c_float, c_ulonglong, _P, _P, _P, _P, _P,
                         _P, c_int, _P])
_decode_advance = Function("sampling", "ek_decode_advance",
                           [_P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P])


def sampling_settings(temperature, top_k, seed, device):
    """The 4-int device block ``sample(dyn=...)`` reads its settings from."""
    import struct
    seed = int(seed) & 0xFFFFFFFFFFFFFFFF
    bits = struct.unpack("<i", struct.pack("<f", float(temperature)))[0]
    lo, hi = seed & 0xFFFFFFFF, seed >> 32
    as_i32 = lambda v: v - (1 << 32) if v >= (1 << 31) else v
    return torch.tensor([bits, int(top_k), as_i32(lo), as_i32(hi)], dtype=torch.int32, device=device)


def sample(out_token, logits, temperature, top_k, seed, streams=None, draws=None, active=None,
           n_rows=None, dyn=None):
    """out_token[r] from logits[r, :] (32-bit): arg-max when temperature is 0, else
    Gumbel-max over the top_k largest (0: all).  ``dyn`` (see ``sampling_settings``)
    overrides temperature, top_k and seed from device memory."""
    _need_cuda(out_token, logits, streams, draws, active, dyn)
    _need(logits.dtype == torch.float32 and logits.stride(-1) == 1, "sample: dense 32-bit logits")
    _need(out_token.dtype == torch.int32, "sample: int32 out")
    rows = n_rows if n_rows is not None else logits.shape[0]
    if lib.recording():
        lib.annotate(bytes=4 * rows * logits.shape[-1])
    _sample(_ptr(out_token), _ptr(logits), logits.stride(0), rows, logits.shape[-1],
            float(temperature), int(top_k), int(seed) & 0xFFFFFFFFFFFFFFFF, _ptr(streams),
            _ptr(draws), _ptr(active), _ptr(dyn), _stream())


SAMPLE_SEGMENTS = 32


_sample_cluster = Function("sampling", "ek_sample_cluster",
                           [_P, _P, c_longlong, c_int, c_int, c_float, c_int, c_ulonglong, _P, _P, _P, _P, _P])


def sample_cluster(out_token, logits, temperature, top_k, seed, streams=None, draws=None, active=None,
                   n_rows=None, dyn=None):
    """:func:`sample` with each row spread over the 8 blocks of a thread-block cluster (wide
    vocabularies with top-k: the radix digits are counted by all 8 and read through distributed
    shared memory).  Same tokens as :func:`sample`."""
    _need_cuda(out_token, logits, streams, draws, active, dyn)
    _need(logits.dtype == torch.float32 and logits.stride(-1) == 1, "sample: dense 32-bit logits")
    _need(out_token.dtype == torch.int32, "sample: int32 out")
    rows = n_rows if n_rows is not None else logits.shape[0]
    if lib.recording():
        lib.annotate(bytes=4 * rows * logits.shape[-1])
    _sample_cluster(_ptr(out_token), _ptr(logits), logits.stride(0), rows, logits.shape[-1],
                    float(temperature), int(top_k), int(seed) & 0xFFFFFFFFFFFFFFFF, _ptr(streams),
                    _ptr(draws), _ptr(active), _ptr(dyn), _stream())


def sample_wide(out_token, logits, temperature, seed, part_score, part_index, streams=None,
                draws=None, active=None, n_rows=None, dyn=None):
    """:func:`sample` without top-k, spread over ``SAMPLE_SEGMENTS`` blocks a row (for wide
    vocabularies).  ``part_score`` float32 / ``part_index`` int32: rows * SAMPLE_SEGMENTS each."""
    _need_cuda(out_token, logits, streams, draws, active, dyn, part_score, part_index)
    _need(logits.dtype == torch.float32 and logits.stride(-1) == 1, "sample: dense 32-bit logits")
    rows = n_rows if n_rows is not None else logits.shape[0]
    _need(part_score.dtype == torch.float32 and part_index.dtype == torch.int32
          and part_score.numel() >= rows * SAMPLE_SEGMENTS
          and part_index.numel() >= rows * SAMPLE_SEGMENTS, "sample_wide: partial buffers")
    if lib.recording():
        lib.annotate(bytes=4 * rows * logits.shape[-1])
    _sample_wide(_ptr(out_token), _ptr(logits), logits.stride(0), rows, logits.shape[-1],
                 float(temperature), int(seed) & 0xFFFFFFFFFFFFFFFF, _ptr(streams), _ptr(draws),
                 _ptr(active), _ptr(dyn), _ptr(part_score), _ptr(part_index), SAMPLE_SEGMENTS,
                 _stream())
    count_extra_launches()                   # partial kernel + final kernel


def decode_advance(sampled, token_ids, positions, draws, remaining, out_tokens, step_index,
                   stop_ids, n_stop, batch):
    _need_cuda(sampled, token_ids, positions, draws, remaining, out_tokens, step_index, stop_ids)
    for t in (sampled, token_ids, positions, draws, remaining, out_tokens, step_index):
        _need(t.dtype == torch.int32, "decode_advance: int32 state")
    _need(out_tokens.shape[-1] == batch, "decode_advance: out_tokens [steps, batch]")
    _decode_advance(_ptr(sampled), _ptr(token_ids), _ptr(positions), _ptr(draws), _ptr(remaining),
                    _ptr(out_tokens), _ptr(step_index), _ptr(stop_ids), n_stop, batch,
                    out_tokens.shape[0], _stream())


# ------------------------------------------------------------------ several residual streams
_hc_broadcast = Function("hyper", "ek_hc_broadcast", [_P, _P, c_int, c_int, c_int, _P])
_hc_step = _per_dtype("hyper", "ek_hc_step", [_P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P, c_float, _P, _P])
MAX_RESIDUAL_STREAMS = 8


def hc_broadcast(streams, x, n_tokens):
    """streams[t, s, :] = x[t, :] for every stream s (32-bit)."""
    _need_cuda(streams, x)
    _need(streams.dtype == x.dtype == torch.float32 and streams.is_contiguous() and x.is_contiguous()
          and streams.dim() == 3 and streams.shape[-1] == x.shape[-1], "hc_broadcast: streams [T, n, W], x [T, W], 32-bit")
    n, width = streams.shape[1], streams.shape[2]
    if lib.recording():
        lib.annotate(bytes=4 * n_tokens * width * (n + 1))
    _hc_broadcast(_ptr(streams), _ptr(x), n_tokens, n, width, _stream())


def hc_step(streams, n_tokens, y=None, write_mix=None, write_out=None, read_in=None, u=None, norm=None):
    """With ``y`` [T, W]: x_t <- sum_s write_mix[s, t] x_s + write_out[t] y for all streams at once, in
    place.  Then, with ``u`` [T, W] (32-bit): u = sum_s read_in[s] x_s (``read_in`` None: the plain
    sum).  With ``norm=(gain, eps, normed)``: normed [T, W] (an activation type) = gain * u * rsqrt(mean(u^2)
    + eps), with or without ``u`` itself.  Coefficients and gain are 32-bit device tensors."""
    gain, eps, normed = norm if norm is not None else (None, 0.0, None)
    _need_cuda(streams, y, write_mix, write_out, read_in, u, gain, normed)
    _need(streams.dtype == torch.float32 and streams.is_contiguous() and streams.dim() == 3,
          "hc_step: streams [T, n, W] in 32-bit")
    n, width = streams.shape[1], streams.shape[2]
    _need(n <= MAX_RESIDUAL_STREAMS, f"hc_step: at most {MAX_RESIDUAL_STREAMS} residual streams")
    for c, size in ((write_mix, n * n), (write_out, n), (read_in, n)):
        _need(c is None or (c.dtype == torch.float32 and c.is_contiguous() and c.numel() == size),
              "hc_step: 32-bit coefficients [n], [n], [n, n]")
    _need(y is None or (y.is_contiguous() and y.shape[-1] == width and write_mix is not None
                        and write_out is not None), "hc_step: y [T, W] with its coefficients")
    _need(u is None or (u.dtype == torch.float32 and u.is_contiguous() and u.shape[-1] == width),
          "hc_step: u [T, W] in 32-bit")
    _need(normed is None or (normed.is_contiguous() and normed.shape[-1] == width and gain.dtype == torch.float32
                             and gain.numel() == width and (y is None or y.dtype == normed.dtype)),
          "hc_step: normed [T, W] in y's type, 32-bit gain [W]")
    dtype = y.dtype if y is not None else (normed.dtype if normed is not None else torch.float32)
    if lib.recording():
        lib.annotate(bytes=n_tokens * width * (4 * n * (2 if y is not None else 1)
                                               + (y.element_size() if y is not None else 0)
                                               + (4 if u is not None else 0)
                                               + (normed.element_size() if normed is not None else 0)))
    _hc_step[dtype](_ptr(streams), _ptr(y), _ptr(write_mix), _ptr(write_out), _ptr(read_in), _ptr(u),
                    n_tokens, n, width, _ptr(gain), float(eps), _ptr(normed), _stream())


# ------------------------------------------------------------------ latent attention
_latent_prepare = _per_dtype("latent", "ek_latent_prepare",
                             [_P, _P, c_int, _P, _P, c_float, _P, _P, c_int, _P, _P, _P, _P, c_int, c_int,
                              c_int, c_int, c_int, c_int, c_int, _P])
_head_linear = _per_dtype("latent", "ek_head_linear",
                          [_P, c_int, c_int, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                           _P, _P, _P, _P])


def latent_prepare(cq, proj, n_tokens, gain_q, gain_kv, eps, cos, sin, rot_dims, positions, token_slot,
                   pages, block_table, q_rank, kv_rank, rot_dim, write_cache=True):
    """``proj`` [T, >= q_rank + kv_rank + rot_dim] (32-bit): cq = gain_q * rms-normed first part (activation
    type); the token's cache row (``pages`` [page, 1, PAGE, D], D >= kv_rank + rot_dim) becomes
    [gain_kv * rms-normed latent | rotated key part | zeros].  ``gain_q`` None: the first ``q_rank`` values go
    to ``cq`` as they are (plain projections that shared the product); ``q_rank`` 0 and ``cq`` None: there are none."""
    _need_cuda(cq, proj, gain_q, gain_kv, cos, sin, positions, token_slot, pages, block_table)
    _need(proj.dtype == torch.float32 and proj.stride(-1) == 1, "latent_prepare: 32-bit projections")
    _need((cq is None and q_rank == 0 and gain_q is None)
          or (cq is not None and cq.dtype == pages.dtype and cq.is_contiguous() and cq.shape[-1] == q_rank),
          "latent_prepare: cq [T, q_rank]")
    _need(pages.is_contiguous() and pages.dim() == 4 and pages.shape[1] == 1 and pages.shape[2] == PAGE,
          "latent_prepare: pages [page, 1, PAGE, D]")
    _need((gain_q is None or (gain_q.dtype == torch.float32 and gain_q.numel() == q_rank))
          and gain_kv.dtype == torch.float32 and gain_kv.numel() == kv_rank, "latent_prepare: 32-bit gains")
    _need(rot_dims == 0 or (cos.dtype == torch.float32 and cos.shape[-1] == rot_dims // 2 and cos.is_contiguous()
                            and sin.is_contiguous()), "latent_prepare: cos/sin [positions, rot_dims / 2]")
    d = pages.shape[-1]
    if lib.recording():
        lib.annotate(bytes=n_tokens * (4 * (q_rank + kv_rank + rot_dim) + pages.element_size() * (q_rank + d)))
    _latent_prepare[pages.dtype](_ptr(cq), _ptr(proj), proj.stride(0), _ptr(gain_q), _ptr(gain_kv), float(eps),
                                 _ptr(cos), _ptr(sin), rot_dims, _ptr(positions), _ptr(token_slot), _ptr(pages),
                                 _ptr(block_table), block_table.stride(0), n_tokens, q_rank, kv_rank, rot_dim, d,
                                 1 if write_cache else 0, _stream())


HEAD_LINEAR_LIBRARY_ROWS = 64     # bfloat16 products per head of more rows than this go to the library


def head_linear(out, x, w, n_tokens, heads, n_in, n_out, rot=None):
    """out[t, h, :n_out] = w[h]^T-applied x[t, h, :n_in] for every head: ``w`` is [heads, n_in, n_out],
    ``x`` [T, heads, >= n_in] and ``out`` [T, heads, >= n_out] (any row and head strides, dense
    values).  ``rot=(rot_dim, rot_dims, cos, sin, positions)``: the ``rot_dim`` values behind the
    ``n_in`` of a head are rotated (the first ``rot_dims`` of them, NeoX pairing) and written behind the
    ``n_out`` results, zeros up to the head's stride.  Many bfloat16 rows (a prompt) go through the
    library's batched product, as the other products of a prompt may; the kernel then only writes the
    rotated tail."""
    _need_cuda(out, x, w)
    _need(out.dtype == x.dtype == w.dtype, "head_linear: one dtype")
    _need(out.dim() == 3 and x.dim() == 3 and out.stride(-1) == 1 and x.stride(-1) == 1 and w.is_contiguous()
          and tuple(w.shape) == (heads, n_in, n_out), "head_linear: x, out [T, heads, .], w [heads, n_in, n_out]")
    r, rot_dims, cos, sin, positions = 0, -1, None, None, None
    if rot is not None:
        r, rot_dims, cos, sin, positions = rot
        _need_cuda(cos, sin, positions)
        _need(x.shape[-1] >= n_in + r and out.stride(1) >= n_out + r, "head_linear: room for the rotated tail")
    by_library = x.dtype == torch.bfloat16 and n_tokens > HEAD_LINEAR_LIBRARY_ROWS
    if by_library:
        def product():
            torch.bmm(x[:n_tokens, :, :n_in].transpose(0, 1), w, out=out[:n_tokens, :, :n_out].transpose(0, 1))
        product()
        if lib.recording():
            lib.record_library_call(f"library_bmm[{heads}x{n_out}x{n_in}]", product,
                                    bytes=2 * (heads * n_in * n_out + n_tokens * heads * (n_in + n_out)),
                                    flops=2 * n_tokens * heads * n_in * n_out)
        if rot is None:
            return
    if lib.recording():
        lib.annotate(bytes=x.element_size() * ((0 if by_library else heads * n_in * n_out)
                                               + n_tokens * heads * (n_in + n_out + 2 * r)),
                     flops=0 if by_library else 2 * n_tokens * heads * n_in * n_out)
    _head_linear[x.dtype](_ptr(out), out.stride(0), out.stride(1), _ptr(x), x.stride(0), x.stride(1),
                          None if by_library else _ptr(w),
                          n_tokens, heads, n_in, n_out, r, rot_dims, _ptr(cos), _ptr(sin), _ptr(positions),
                          _stream())


# ------------------------------------------------------------------ delta rule with a decay per key channel
_delta_prepare = Function("delta", "ek_delta_prepare",
                          [_P, _P, _P, _P, _P, c_int, _P, _P, c_longlong, c_longlong, _P, _P,
                           c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P])
_delta_low_rank = Function("delta", "ek_delta_low_rank",
                           [_P, _P, c_int, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, _P])
_delta_conv_tail = Function("delta", "ek_delta_conv_tail",
                            [_P, c_longlong, c_longlong, _P, c_int, _P, _P, _P, c_int, c_int, c_int, _P])
_delta_scan = Function("delta", "ek_delta_scan",
                       [_P, _P, _P, _P, _P, _P, _P, c_longlong, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                        _P])
_delta_out_norm = _per_dtype("delta", "ek_delta_out_norm",
                             [_P, _P, _P, _P, c_float, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                              c_int, c_int, c_int, c_int, _P])
DELTA_MAX_KEY_DIM = 256


def delta_state_rows(dim: int) -> int:
    """Rows of S per column that the scan keeps for keys of ``dim`` values (``dim`` rounded up to 32,
    64, 128 or 256)."""
    if not 0 < dim <= DELTA_MAX_KEY_DIM:
        raise KernelError(f"the delta-rule scan takes key sizes up to {DELTA_MAX_KEY_DIM}, not {dim}")
    for rows in (32, 64, 128, 256):
        if dim <= rows:
            return rows


def delta_low_rank(out, proj, n_tokens, offset, w2t, bias=None, a_log=None, dim=1):
    """The second half of a low-rank pair for every token: out[t, c] = f(bias[c] + sum_r w2t[r, c] *
    proj[t, offset + r]), all 32-bit.  With ``a_log`` [heads] (a head is ``dim`` neighbouring channels) f is
    the decay exp(-exp(a_log) * softplus(.)); without, the sigmoid."""
    _need_cuda(out, proj, w2t, bias, a_log)
    for t in (out, proj, w2t, bias, a_log):
        _need(t is None or (t.dtype == torch.float32 and t.stride(-1) == 1), "delta_low_rank: 32-bit tensors")
    rank, channels = w2t.shape
    _need(w2t.is_contiguous() and out.is_contiguous() and out.shape[-1] == channels, "delta_low_rank: w2t [rank, channels]")
    if lib.recording():
        lib.annotate(bytes=4 * (n_tokens * (rank + channels) + rank * channels), flops=2 * n_tokens * rank * channels)
    _delta_low_rank(_ptr(out), _ptr(proj), proj.stride(0), offset, rank, _ptr(w2t), _ptr(bias), _ptr(a_log), dim,
                    channels, n_tokens, 0 if a_log is not None else 1, _stream())


def delta_prepare(qn, kn, vc, beta, proj, n_tokens, conv_w, state, tail_offset, positions, token_slot, shape):
    """``shape`` = (heads, kv_heads, dim, vdim, taps, rank_a, rank_g).  ``proj`` [T, q|k|v|beta|a1|g1] in
    32-bit; ``state`` [slots, values] 32-bit with the convolution's last inputs from ``tail_offset`` on.
    Writes the unit q and k, the convolved v and beta (all 32-bit)."""
    _need_cuda(qn, kn, vc, beta, proj, conv_w, state, positions, token_slot)
    for t in (qn, kn, vc, beta, proj, conv_w, state):
        _need(t.dtype == torch.float32 and t.stride(-1) == 1, "delta_prepare: 32-bit tensors")
    if lib.recording():
        lib.annotate(bytes=4 * n_tokens * (proj.shape[-1] + 2 * qn.shape[-1] + vc.shape[-1]))
    _delta_prepare(_ptr(qn), _ptr(kn), _ptr(vc), _ptr(beta), _ptr(proj), proj.stride(0),
                   _ptr(conv_w), _ptr(state), state.stride(0),
                   tail_offset, _ptr(positions), _ptr(token_slot), n_tokens, *[int(v) for v in shape], _stream())


def delta_conv_tail(state, tail_offset, proj, cu_seqlens, positions, token_slot, n_seqs, channels, taps):
    """The last ``taps - 1`` convolution inputs of every sequence of the step go to its state."""
    _need_cuda(state, proj, cu_seqlens, positions, token_slot)
    _delta_conv_tail(_ptr(state), state.stride(0), tail_offset, _ptr(proj), proj.stride(0), _ptr(cu_seqlens),
                     _ptr(positions), _ptr(token_slot), n_seqs, channels, taps, _stream())


def delta_scan(out, qn, kn, vc, beta, decay, state, cu_seqlens, positions, token_slot, n_seqs, heads,
               kv_heads, dim, vdim, n_tokens=0, decay_per_head=False):
    """The recurrence over every sequence's tokens; S [heads, vdim, rows] at the start of a slot's state
    is read and written back.  ``decay`` is [T, heads * dim] (one per key channel) or, with
    ``decay_per_head``, [T, heads]."""
    _need_cuda(out, qn, kn, vc, beta, decay, state, cu_seqlens, positions, token_slot)
    _need(decay.is_contiguous() and decay.shape[-1] == (heads if decay_per_head else heads * dim),
          "delta_scan: decays [T, heads * dim], or [T, heads] with decay_per_head")
    if lib.recording():
        lib.annotate(bytes=4 * (n_tokens * (2 * kv_heads * dim + heads * dim + 2 * heads * vdim + heads)
                                + 2 * n_seqs * heads * vdim * delta_state_rows(dim)),
                     flops=6 * n_tokens * heads * dim * vdim)
    _delta_scan(_ptr(out), _ptr(qn), _ptr(kn), _ptr(vc), _ptr(beta), _ptr(decay), _ptr(state), state.stride(0),
                _ptr(cu_seqlens), _ptr(positions), _ptr(token_slot), n_seqs, heads, kv_heads, dim, vdim,
                1 if decay_per_head else 0, _stream())


def delta_out_norm(y, o, gate, w, eps, positions, n_tokens, shape, gate_activation=None):
    """y = o / rms(o) per head * w * gate in the activation type (``o`` [T, heads * vdim], ``gate`` rows of at
    least as many values, 32-bit).  ``gate_activation="silu"``: the gate is a raw projection and its SiLU is taken here."""
    _need_cuda(y, o, gate, w, positions)
    _need(gate_activation in (None, "silu"), "delta_out_norm: the gate is finished or takes SiLU")
    _need(o.dtype == gate.dtype == w.dtype == torch.float32 and y.is_contiguous() and o.is_contiguous()
          and gate.stride(-1) == 1, "delta_out_norm: 32-bit inputs")
    if lib.recording():
        lib.annotate(bytes=n_tokens * o.shape[-1] * (8 + y.element_size()))
    _delta_out_norm[y.dtype](_ptr(y), _ptr(o), _ptr(gate), _ptr(w), float(eps),
                             _ptr(positions), n_tokens, *[int(v) for v in shape], gate.stride(0),
                             1 if gate_activation == "silu" else 0, _stream())


# ------------------------------------------------------------------ linear recurrences with a decay per head
_conv_silu = Function("recurrent", "ek_conv_silu",
                      [_P, c_int, _P, c_int, c_int, _P, _P, _P, c_longlong, c_longlong, _P, _P, c_int, c_int, c_int, _P])
_conv_tail = Function("recurrent", "ek_conv_tail",
                      [_P, c_longlong, c_longlong, _P, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, _P])
_ssm_gates = Function("recurrent", "ek_ssm_gates", [_P, _P, _P, c_int, c_int, _P, _P, c_int, c_int, _P])
_xgate_scan = Function("recurrent", "ek_xgate_scan",
                       [_P, _P, _P, _P, c_int, c_int, c_int, _P, _P, c_float, _P, c_longlong, c_longlong, _P, _P, _P,
                        c_int, c_int, c_int, _P])
_decay_scan = Function("recurrent", "ek_decay_scan",
                       [_P, c_int, _P, c_int, _P, c_int, _P, c_int, _P, _P, _P, c_longlong, _P, _P, _P,
                        c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, c_int, _P])
_ssm_out = _per_dtype("recurrent", "ek_ssm_out",
                      [_P, _P, _P, c_int, _P, c_int, c_int, _P, _P, c_float, _P, c_int, c_int, c_int, c_int, _P])
_xlstm_out = _per_dtype("recurrent", "ek_xlstm_out",
                        [_P, _P, _P, _P, c_int, c_int, _P, c_float, c_float, _P, c_int, c_int, c_int, _P])
_rotate_heads = Function("recurrent", "ek_rotate_heads",
                         [_P, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, _P])
_head_norm_gate_out = _per_dtype("recurrent", "ek_head_norm_gate_out",
                                 [_P, _P, _P, c_int, c_int, _P, c_float, c_int, _P, c_int, c_int, c_int, _P])
DECAY_SCAN_MAX_KEY_DIM = 256


def decay_scan_rows(dim: int) -> int:
    """Rows of S per column that the decay scan keeps for keys of ``dim`` values (``dim`` rounded up to
    32, 64, 128 or 256)."""
    if not 0 < dim <= DECAY_SCAN_MAX_KEY_DIM:
        raise KernelError(f"the decay scan takes key sizes up to {DECAY_SCAN_MAX_KEY_DIM}, not {dim}")
    for rows in (32, 64, 128, 256):
        if dim <= rows:
            return rows


def _need_f32(name, *tensors):
    for t in tensors:
        _need(t is None or (t.dtype == torch.float32 and t.stride(-1) == 1), f"{name}: 32-bit tensors")


def conv_silu(out, proj, col0, conv_w, conv_b, state, tail_offset, positions, token_slot, n_tokens, channels, taps):
    """out[t, c] = silu(b[c] + sum_j w[c, taps-1-j] x[t-j, c]) with x = proj[., col0 + c] (all 32-bit): a
    causal convolution per channel whose last column multiplies the current token.  Tokens before the
    step's first of a sequence come from the slot's state ([channels, taps-1] from ``tail_offset`` on,
    oldest first; zeros for a new sequence)."""
    _need_cuda(out, proj, conv_w, conv_b, state, positions, token_slot)
    _need_f32("conv_silu", out, proj, conv_w, conv_b, state)
    _need(conv_w.is_contiguous() and tuple(conv_w.shape) == (channels, taps) and out.shape[-1] >= channels
          and col0 + channels <= proj.shape[-1], "conv_silu: weights [channels, taps], columns within the rows")
    if lib.recording():
        lib.annotate(bytes=8 * n_tokens * channels)
    _conv_silu(_ptr(out), out.stride(0), _ptr(proj), proj.stride(0), col0, _ptr(conv_w), _ptr(conv_b), _ptr(state),
               state.stride(0), tail_offset, _ptr(positions), _ptr(token_slot), n_tokens, channels, taps, _stream())


_conv_act = Function("recurrent", "ek_conv_act",
                     [_P, c_int, _P, c_int, c_int, _P, _P, _P, c_int, _P, c_longlong, c_longlong, _P, _P, c_int, c_int,
                      c_int, _P])
_lru_gates = Function("recurrent", "ek_lru_gates",
                      [_P, _P, _P, c_int, _P, _P, _P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, _P])
_lru_scan = _per_dtype("recurrent", "ek_lru_scan",
                       [_P, _P, _P, _P, c_int, c_int, _P, _P, c_longlong, _P, _P, _P, c_int, c_int, c_int, c_int, _P])


def conv_act(out, proj, col0, conv_w, conv_b, state, tail_offset, positions, token_slot, n_tokens, channels, taps,
             in_bias=None, activation="silu"):
    """:func:`conv_silu` with two options: ``in_bias`` [channels] is a bias of the projection itself, added
    to every input that belongs to a token (what lies before a sequence's start stays zero; the state's
    tail keeps the inputs without it); ``activation`` None leaves the SiLU out."""
    _need_cuda(out, proj, conv_w, conv_b, in_bias, state, positions, token_slot)
    _need_f32("conv_act", out, proj, conv_w, conv_b, in_bias, state)
    _need(activation in (None, "silu"), "conv_act: SiLU or nothing")
    _need(conv_w.is_contiguous() and tuple(conv_w.shape) == (channels, taps) and out.shape[-1] >= channels
          and col0 + channels <= proj.shape[-1], "conv_act: weights [channels, taps], columns within the rows")
    if lib.recording():
        lib.annotate(bytes=8 * n_tokens * channels)
    _conv_act(_ptr(out), out.stride(0), _ptr(proj), proj.stride(0), col0, _ptr(conv_w), _ptr(conv_b), _ptr(in_bias),
              1 if activation == "silu" else 0, _ptr(state), state.stride(0), tail_offset, _ptr(positions),
              _ptr(token_slot), n_tokens, channels, taps, _stream())


def lru_gates(a, x, u, w_a, b_a, w_i, b_i, lam, rate, n_tokens, parts, size, w_a_rows=None, w_i_rows=None):
    """Gates of a gated linear recurrence over ``parts * size`` channels: r = sigmoid(W_a[p] u_p + b_a),
    i = sigmoid(W_i[p] u_p + b_i) per part p; a = exp(-rate * r * softplus(lam)), x = sqrt(1 - a^2) * i * u.
    ``w_a``, ``w_i`` [parts, in, out] (transposed), everything 32-bit.  ``w_a_rows``, ``w_i_rows``: the same
    matrices [parts, out, in]; with them steps of at most 192 tokens run a warp per output channel."""
    _need_cuda(a, x, u, w_a, b_a, w_i, b_i, lam, w_a_rows, w_i_rows)
    _need_f32("lru_gates", a, x, u, w_a, b_a, w_i, b_i, lam, w_a_rows, w_i_rows)
    for t in (w_a_rows, w_i_rows):
        _need(t is None or (t.is_contiguous() and tuple(t.shape) == (parts, size, size)), "lru_gates: rows [parts, size, size]")
    width = parts * size
    _need(a.is_contiguous() and x.is_contiguous() and a.shape[-1] == width == x.shape[-1] and u.shape[-1] >= width
          and w_a.is_contiguous() and w_i.is_contiguous() and tuple(w_a.shape) == (parts, size, size) == tuple(w_i.shape)
          and lam.numel() == width, "lru_gates: a, x [T, parts * size]; weights [parts, size, size]")
    if lib.recording():
        lib.annotate(bytes=4 * (3 * n_tokens * width + 2 * parts * size * size), flops=4 * n_tokens * width * size)
    _lru_gates(_ptr(a), _ptr(x), _ptr(u), u.stride(0), _ptr(w_a), _ptr(b_a), _ptr(w_i), _ptr(b_i), _ptr(w_a_rows),
               _ptr(w_i_rows), _ptr(lam), float(rate), n_tokens, parts, size, _stream())


def lru_scan(out, a, x, side, side_col, side_bias, state, cu_seqlens, positions, token_slot, n_seqs, channels,
             write_state=True, n_tokens=0, max_new=1):
    """S_t = a_t S_(t-1) + x_t per channel over every sequence's tokens, S (the first ``channels`` values of a
    slot's state) read and written back; out[t, c] = S_t * gelu_tanh(side[t, side_col + c] + side_bias[c]).
    ``max_new``: the longest run of tokens a sequence brings (above 16 the kernel cuts runs into stretches that
    eight warps take side by side)."""
    _need_cuda(out, a, x, side, side_bias, state, cu_seqlens, positions, token_slot)
    _need_f32("lru_scan", a, x, side, side_bias, state)
    _need(out.is_contiguous() and a.is_contiguous() and x.is_contiguous() and out.shape[-1] == channels
          and a.shape[-1] == channels and side_col + channels <= side.shape[-1] and state.shape[-1] >= channels,
          "lru_scan: out, a, x [T, channels]")
    if lib.recording():
        lib.annotate(bytes=n_tokens * channels * (12 + out.element_size()) + 8 * n_seqs * channels)
    _lru_scan[out.dtype](_ptr(out), _ptr(a), _ptr(x), _ptr(side), side.stride(0), side_col, _ptr(side_bias),
                         _ptr(state), state.stride(0), _ptr(cu_seqlens), _ptr(positions), _ptr(token_slot), n_seqs,
                         channels, 1 if write_state else 0, int(max_new), _stream())


def conv_tail(state, tail_offset, proj, col0, cu_seqlens, positions, token_slot, n_seqs, channels, taps):
    """The last ``taps - 1`` convolution inputs of every sequence of the step go to its state."""
    _need_cuda(state, proj, cu_seqlens, positions, token_slot)
    _need_f32("conv_tail", state, proj)
    _conv_tail(_ptr(state), state.stride(0), tail_offset, _ptr(proj), proj.stride(0), col0, _ptr(cu_seqlens),
               _ptr(positions), _ptr(token_slot), n_seqs, channels, taps, _stream())


def ssm_gates(a, b, proj, col0, dt_bias, a_log, n_tokens, heads):
    """dt = softplus(proj[t, col0 + h] + dt_bias[h]); a[t, h] = exp(-exp(a_log[h]) dt), b[t, h] = dt."""
    _need_cuda(a, b, proj, dt_bias, a_log)
    _need_f32("ssm_gates", a, b, proj, dt_bias, a_log)
    _need(a.is_contiguous() and b.is_contiguous() and a.shape[-1] == heads == b.shape[-1]
          and dt_bias.numel() == heads == a_log.numel(), "ssm_gates: one value per head")
    _ssm_gates(_ptr(a), _ptr(b), _ptr(proj), proj.stride(0), col0, _ptr(dt_bias), _ptr(a_log), n_tokens, heads,
               _stream())


def xgate_scan(a, b, m_run, proj, col_i, col_f, bias_i, bias_f, cap, state, m_offset, cu_seqlens, positions,
               token_slot, n_seqs, heads, write_state=True):
    """Exponential gates kept stable by a running maximum: i = cap tanh((x_i + b_i) / cap), f =
    logsigmoid(cap tanh((x_f + b_f) / cap)), m_t = max(f + m_(t-1), i) continued from the slot's state
    (``heads`` values from ``m_offset`` on); a = exp(f + m_(t-1) - m_t), b = exp(i - m_t), m_run = m_t."""
    _need_cuda(a, b, m_run, proj, bias_i, bias_f, state, cu_seqlens, positions, token_slot)
    _need_f32("xgate_scan", a, b, m_run, proj, bias_i, bias_f, state)
    _need(a.is_contiguous() and b.is_contiguous() and m_run.is_contiguous() and a.shape[-1] == heads,
          "xgate_scan: a, b, m [T, heads]")
    _xgate_scan(_ptr(a), _ptr(b), _ptr(m_run), _ptr(proj), proj.stride(0), col_i, col_f, _ptr(bias_i), _ptr(bias_f),
                float(cap), _ptr(state), state.stride(0), m_offset, _ptr(cu_seqlens), _ptr(positions),
                _ptr(token_slot), n_seqs, heads, 1 if write_state else 0, _stream())


SCAN_COLUMNS = 16           # columns of S a block of the decay scan takes, one a lane; twice as many with two
SCAN_WIDE_TOKENS = 64       # sequences of at least this many tokens take two columns a lane
SCAN_BLOCKS_PER_SM = 6      # what a cut of long prompts into segments aims at
SCAN_MIN_SEGMENT = 128      # tokens
SCAN_MIN_SEGMENTS = 4       # (the walk of the states costs two thirds of a walk: two or three segments gain nothing)


def decay_scan_wide(columns, max_new) -> bool:
    """Whether a lane of :func:`decay_scan` takes two columns (long walks of enough columns)."""
    return max_new >= SCAN_WIDE_TOKENS and columns > SCAN_COLUMNS


def decay_scan_segments(n_seqs, heads, columns, max_new, device=None):
    """(segments of the longest sequence, tokens a segment) that :func:`decay_scan` cuts a step's sequences into; one
    segment where the sequences, heads and columns fill the machine, or the sequences are short."""
    tile = SCAN_COLUMNS * (2 if decay_scan_wide(columns, max_new) else 1)
    blocks = n_seqs * heads * -(-columns // tile)
    want = min(SCAN_BLOCKS_PER_SM * sm_count(device) // blocks, max_new // SCAN_MIN_SEGMENT)
    if want < SCAN_MIN_SEGMENTS:
        return 1, max_new
    length = -(-(-(-max_new // want)) // 64) * 64
    return -(-max_new // length), length


def decay_scan(out, q, k, v, a, b, state, cu_seqlens, positions, token_slot, n_seqs, heads, kv_heads, dim, vdim,
               ones_column=False, write_state=True, n_tokens=0, max_new=0, workspace=None, segments=None):
    """S_t = a_t S_(t-1) + b_t k_t v_t^T, out_t = S_t^T q_t per head over every sequence's tokens, S
    ([heads, columns, rows] at the start of a slot's state, 32-bit) read and written back.  ``q``, ``k``
    [T, >= kv_heads * dim] (head h reads key head h // (heads / kv_heads)), ``v`` [T, >= heads * vdim],
    ``a``, ``b`` [T, heads], or [heads] where they are the same for every token.  ``ones_column``: one more column whose v is 1 (it carries a n + b k and
    gives n . q); out is [T, heads * columns].  With ``workspace`` and ``max_new`` (tokens of the longest sequence) long
    sequences are cut into segments that run side by side (:func:`decay_scan_segments`, or ``segments`` as given)."""
    _need_cuda(out, q, k, v, a, b, state, cu_seqlens, positions, token_slot)
    _need_f32("decay_scan", out, q, k, v, a, b, state)
    cols = vdim + (1 if ones_column else 0)
    _need(out.shape[-1] == heads * cols and a.is_contiguous() and b.is_contiguous() and a.shape[-1] == heads
          and a.dim() == b.dim(), "decay_scan: out [T, heads * columns], a and b [T, heads] or [heads]")
    _need(state.stride(0) % 4 == 0 and state.shape[-1] >= heads * cols * decay_scan_rows(dim),
          "decay_scan: the state holds S and every slot starts on a 16-byte boundary")
    if lib.recording():
        lib.annotate(bytes=4 * (n_tokens * (2 * kv_heads * dim + 2 * heads * vdim + 2 * heads)
                                + 2 * n_seqs * heads * cols * decay_scan_rows(dim)),
                     flops=4 * n_tokens * heads * dim * cols)
    parts, length, carry, prods = 1, 0, None, None
    if workspace is not None and max_new > 1:
        parts, length = segments or decay_scan_segments(n_seqs, heads, cols, max_new, out.device)
        _need(length >= 1 and parts * length >= max_new, "decay_scan: the segments cover the longest sequence")
        if parts > 1:
            carry = workspace.get("scan_carry", (n_seqs, parts, heads * cols * decay_scan_rows(dim)), torch.float32)
            prods = workspace.get("scan_prods", (n_seqs, parts, heads), torch.float32)
    _decay_scan(_ptr(out), out.stride(0), _ptr(q), q.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0),
                _ptr(a), _ptr(b), _ptr(state), state.stride(0), _ptr(cu_seqlens), _ptr(positions), _ptr(token_slot),
                n_seqs, heads, kv_heads, dim, vdim, 1 if ones_column else 0, 1 if write_state else 0,
                heads if a.dim() > 1 else 0, _ptr(carry), _ptr(prods), parts, length,
                1 if decay_scan_wide(cols, max_new) else 0, _stream())
    if parts > 1:
        count_extra_launches()


def ssm_out(y, o, x, proj, col_z, d_skip, w, eps, positions, n_tokens, inner, vdim, parts):
    """y = n((o + D[head] x) silu(z)) w in the activation type, the norm over each of ``parts`` equal parts
    of the ``inner`` channels; z = proj[., col_z + c], x [T, >= inner] the convolved inputs."""
    _need_cuda(y, o, x, proj, d_skip, w, positions)
    _need_f32("ssm_out", o, x, proj, d_skip, w)
    _need(y.is_contiguous() and o.is_contiguous() and o.shape[-1] == inner == y.shape[-1] and w.numel() == inner,
          "ssm_out: y, o [T, inner]")
    if lib.recording():
        lib.annotate(bytes=n_tokens * inner * (12 + y.element_size()))
    _ssm_out[y.dtype](_ptr(y), _ptr(o), _ptr(x), x.stride(0), _ptr(proj), proj.stride(0), col_z, _ptr(d_skip),
                      _ptr(w), float(eps), _ptr(positions), n_tokens, inner, vdim, parts, _stream())


_norm_gate_out = _per_dtype("recurrent", "ek_norm_gate_out",
                            [_P, _P, _P, c_int, c_int, _P, c_float, _P, c_int, c_int, _P])


def norm_gate_out(y, o, proj, col_g, w, eps, positions, n_tokens):
    """y = o / rms(o) * w * sigmoid(proj[., col_g + c]) in the activation type, the root mean square taken over
    the whole row (all heads together)."""
    _need_cuda(y, o, proj, w, positions)
    _need_f32("norm_gate_out", o, proj, w)
    inner = y.shape[-1]
    _need(y.is_contiguous() and o.is_contiguous() and o.shape[-1] == inner == w.numel()
          and col_g + inner <= proj.shape[-1], "norm_gate_out: y, o, w of one width, the gate within the rows")
    if lib.recording():
        lib.annotate(bytes=n_tokens * inner * (8 + y.element_size()))
    _norm_gate_out[y.dtype](_ptr(y), _ptr(o), _ptr(proj), proj.stride(0), col_g, _ptr(w), float(eps), _ptr(positions),
                            n_tokens, inner, _stream())


def rotate_heads(x, col0, heads, dim, rot_dims, cos, sin, positions, n_tokens):
    """In place on ``x`` [T, .] (32-bit): ``heads`` heads of ``dim`` values from column ``col0``, the first
    ``rot_dims`` of each turned (value i with value i + rot_dims / 2) by the token's angles."""
    _need_cuda(x, cos, sin, positions)
    _need_f32("rotate_heads", x, cos, sin)
    _need(col0 + heads * dim <= x.shape[-1] and positions.dtype == torch.int32, "rotate_heads: heads within the rows")
    _need(rot_dims == 0 or (cos.is_contiguous() and sin.is_contiguous() and cos.shape[-1] * 2 == rot_dims),
          "rotate_heads: cos/sin [positions, rot_dims / 2]")
    if rot_dims == 0:
        return
    if lib.recording():
        lib.annotate(bytes=8 * n_tokens * heads * rot_dims)
    _rotate_heads(_ptr(x), x.stride(0), col0, heads, dim, rot_dims, _ptr(cos), _ptr(sin), _ptr(positions), n_tokens,
                  _stream())


def head_norm_gate_out(y, o, proj, col_g, w, eps, positions, n_tokens, heads, vdim, gate_activation="sigmoid"):
    """y = o / rms(o) per head * w * act(proj[., col_g + c]) in the activation type; ``w`` [heads * vdim] or None (no
    weight), act ``"sigmoid"`` or ``"silu"``."""
    _need_cuda(y, o, proj, w, positions)
    _need_f32("head_norm_gate_out", o, proj, w)
    _need(gate_activation in ("sigmoid", "silu"), "head_norm_gate_out: the gate takes a sigmoid or SiLU")
    _need(y.is_contiguous() and o.is_contiguous() and y.shape[-1] == o.shape[-1] == heads * vdim
          and (w is None or w.numel() == heads * vdim) and col_g + heads * vdim <= proj.shape[-1],
          "head_norm_gate_out: y, o, w of one width, the gate within the rows")
    if lib.recording():
        lib.annotate(bytes=n_tokens * heads * vdim * (8 + y.element_size()))
    _head_norm_gate_out[y.dtype](_ptr(y), _ptr(o), _ptr(proj), proj.stride(0), col_g, _ptr(w), float(eps),
                                 1 if gate_activation == "silu" else 0, _ptr(positions), n_tokens, heads, vdim,
                                 _stream())


def xlstm_out(y, o, m_run, proj, col_g, w, eps, q_scale, positions, n_tokens, heads, vdim):
    """``o`` [T, heads * (vdim + 1)] from the scan with n . q in each head's last column, both still to
    be multiplied by ``q_scale``: u = o q_scale / (max(|n . q| q_scale, exp(-m)) + 1e-6); y = u / rms(u)
    per head * w * sigmoid(proj[., col_g + c]) in the activation type."""
    _need_cuda(y, o, m_run, proj, w, positions)
    _need_f32("xlstm_out", o, m_run, proj, w)
    _need(y.is_contiguous() and o.is_contiguous() and m_run.is_contiguous() and y.shape[-1] == heads * vdim
          and o.shape[-1] == heads * (vdim + 1) and w.numel() == heads * vdim, "xlstm_out: shapes")
    if lib.recording():
        lib.annotate(bytes=n_tokens * heads * vdim * (8 + y.element_size()))
    _xlstm_out[y.dtype](_ptr(y), _ptr(o), _ptr(m_run), _ptr(proj), proj.stride(0), col_g, _ptr(w), float(eps),
                        float(q_scale), _ptr(positions), n_tokens, heads, vdim, _stream())


# ------------------------------------------------------------------ routed experts
_moe_route = Function("moe", "ek_moe_route", [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, _P, _P])
_moe_plan = Function("moe", "ek_moe_plan", [_P, _P, _P, _P, c_int, c_int, _P])
_moe_up = _per_dtype("moe", "ek_moe_expert_up",
                     [_P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P, _P])
_moe_down = _per_dtype("moe", "ek_moe_expert_down", [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P])
_moe_combine = _per_dtype("moe", "ek_moe_combine", [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P, c_int, _P])
_moe_up_tc = Function("moe", "ek_moe_expert_up_tc",
                      [_P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P, _P])
_moe_down_tc = Function("moe", "ek_moe_expert_down_tc", [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P])


def _moe_on_tensor_cores(a, w) -> bool:
    """bfloat16 rows that can be read 16 bytes at a time go to the mma.sync form of the expert products."""
    return (a.dtype == torch.bfloat16 and w.shape[-1] % 8 == 0 and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)
MOE_TILE_ROWS = 64          # must equal kTileRows in csrc/moe.cu
EXPERT_ACTIVATIONS = {"none": 0, "relu2": 1, "silu": 2, "gelu_tanh": 3, "clamped": 4}
ROUTE_WEIGHTS = {"scores_of_chosen": 0, "softmax_of_chosen": 1, "sigmoid": 2, "softmax": 3}


def moe_max_tiles(n_pairs: int, n_experts: int) -> int:
    """Most row tiles a plan of ``n_pairs`` (token, choice) pairs can have."""
    return -(-n_pairs // MOE_TILE_ROWS) + min(n_experts, n_pairs)


def moe_route(sel_expert, sel_weight, logits, n_tokens, n_groups, keep, top, scale, weights="scores_of_chosen",
              correction=None):
    """Router: ``logits`` [T, E] 32-bit -> the ``top`` chosen experts and their weights per token, times ``scale``.
    ``weights``: ``"scores_of_chosen"``, the chosen scores of the softmax over all experts, divided by their sum;
    ``"softmax_of_chosen"``, the softmax over the chosen logits alone; ``"sigmoid"``, the chosen logits' sigmoids
    as they are (all groups kept); ``"softmax"``, the chosen scores of the softmax over all experts as they are (all
    groups kept), where ``correction`` [E] (32-bit) joins the scores for the choice only."""
    _need_cuda(sel_expert, sel_weight, logits, correction)
    _need(correction is None or (weights == "softmax" and correction.dtype == torch.float32 and correction.is_contiguous()
                                 and correction.numel() == logits.shape[-1]),
          "moe_route: a 32-bit correction per expert goes with the weights 'softmax'")
    _need(weights in ROUTE_WEIGHTS, f"moe_route: no weights {weights!r}")
    _need(logits.dtype == torch.float32 and logits.stride(-1) == 1 and sel_expert.dtype == torch.int32
          and sel_weight.dtype == torch.float32, "moe_route: 32-bit logits and weights, int32 choices")
    _moe_route(_ptr(sel_expert), _ptr(sel_weight), _ptr(logits), logits.stride(0), n_tokens, logits.shape[-1], n_groups, keep,
               top, float(scale), ROUTE_WEIGHTS[weights], _ptr(correction), _stream())


def moe_plan(sorted_pair, tiles, n_tiles, sel_expert, n_pairs, n_experts):
    _need_cuda(sorted_pair, tiles, n_tiles, sel_expert)
    _moe_plan(_ptr(sorted_pair), _ptr(tiles), _ptr(n_tiles), _ptr(sel_expert), n_pairs, n_experts, _stream())


def moe_expert_up(out, x, w, tiles, n_tiles, sorted_pair, n_pairs, top, activation, gated=False, limit=0.0,
                  input_weight=None):
    """out[sorted row] = act(x[token of the pair] . w[expert]^T); ``w`` [E, N, K].  ``gated``: the
    rows of an expert's ``w`` alternate gate, up, gate, up ...; out [pairs, N / 2] holds
    act(gate) * up, taken from the 32-bit sums (``"clamped"`` as in :func:`act_mul`, with ``limit``).
    ``input_weight`` [pairs] (32-bit): a pair's input is multiplied by its weight (in the 32-bit sums)."""
    _need_cuda(out, x, w, tiles, n_tiles, sorted_pair, input_weight)
    _need(activation != "clamped" or (gated and limit > 0), "moe_expert_up: the clamped gate needs gate rows and a limit")
    _need(input_weight is None or (input_weight.dtype == torch.float32 and input_weight.is_contiguous()
                                   and input_weight.numel() >= n_pairs), "moe_expert_up: one 32-bit weight per pair")
    _need(out.dtype == x.dtype == w.dtype and x.is_contiguous() and w.is_contiguous() and out.is_contiguous(),
          "moe_expert_up: one dtype, contiguous")
    e, n, k = w.shape
    if lib.recording():
        lib.annotate(bytes=x.element_size() * (min(e, n_pairs) * n * k + n_pairs * (n + k)), flops=2 * n_pairs * n * k)
    fn = _moe_up_tc if _moe_on_tensor_cores(x, w) else _moe_up[x.dtype]
    fn(_ptr(out), _ptr(x), _ptr(w), _ptr(tiles), _ptr(n_tiles), _ptr(sorted_pair),
       moe_max_tiles(n_pairs, e), top, n, k, EXPERT_ACTIVATIONS[activation], 1 if gated else 0, float(limit),
       _ptr(input_weight), _stream())


def moe_expert_down(pair_out, a, w, tiles, n_tiles, sorted_pair, pair_weight, n_pairs):
    """pair_out[pair] = weight[pair] * (a[sorted row] . w[expert]^T) in 32-bit; ``w`` [E, N, K];
    ``pair_weight`` None: ones."""
    _need_cuda(pair_out, a, w, tiles, n_tiles, sorted_pair, pair_weight)
    _need(a.dtype == w.dtype and pair_out.dtype == torch.float32 and a.is_contiguous() and w.is_contiguous(),
          "moe_expert_down: 32-bit output")
    e, n, k = w.shape
    if lib.recording():
        lib.annotate(bytes=a.element_size() * (min(e, n_pairs) * n * k + n_pairs * k) + 4 * n_pairs * n,
                     flops=2 * n_pairs * n * k)
    fn = _moe_down_tc if _moe_on_tensor_cores(a, w) else _moe_down[a.dtype]
    fn(_ptr(pair_out), _ptr(a), _ptr(w), _ptr(tiles), _ptr(n_tiles), _ptr(sorted_pair),
       _ptr(pair_weight), moe_max_tiles(n_pairs, e), n, k, _stream())


def moe_combine(out, pair_out, n_tokens, top, add=None, identity=None):
    """out[t] = sum over the token's ``top`` pairs (+ add[t], in out's type).  ``identity=(chosen, weight, x, E)``:
    a pair whose expert number is E or more has no row in ``pair_out``; weight * x[t] takes its place (``x`` rows in
    out's type)."""
    _need_cuda(out, pair_out, add)
    width = out.shape[-1]
    _need(add is None or (add.dtype == out.dtype and add.is_contiguous() and add.shape[-1] == width),
          "moe_combine: what is added has out's type and width")
    chosen, weight, x, e = identity if identity is not None else (None, None, None, 0)
    _need_cuda(chosen, weight, x)
    _need(identity is None or (x.dtype == out.dtype and x.is_contiguous() and x.shape[-1] == width
                               and chosen.dtype == torch.int32 and weight.dtype == torch.float32
                               and chosen.is_contiguous() and weight.is_contiguous()),
          "moe_combine: identity experts take the input's rows in out's type, choices and 32-bit weights")
    if lib.recording():
        lib.annotate(bytes=n_tokens * width * (4 * top + out.element_size() * (1 + (add is not None) + (x is not None))))
    _moe_combine[out.dtype](_ptr(out), _ptr(pair_out), n_tokens, top, width, _ptr(add), _ptr(chosen), _ptr(weight),
                            _ptr(x), e, _stream())


def build_all():
    """Compile every kernel library (used by the build check)."""
    from . import build
    return build.build_all()
