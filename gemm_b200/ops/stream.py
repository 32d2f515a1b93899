"""Token-wise ops of models with a 32-bit residual stream (csrc/kernels/stream_ops.cu) and their PyTorch references.

``embed``        embedding rows (times a factor) as an f32 stream
``norm``         stream += pending update (+ a vector), then RMSNorm or Dynamic Tanh -> rows for the next projection; the update may have a
                 norm of its own (``PostNormed``)
``join``         stream += a weighted sum of several pending results; a copy of the rows for a projection of the stream itself
``qk_rows``      Q and K normed over all their heads at once, K / V to the cache, Q scaled for the attention kernels
``conv_rotary``  short causal convolution of Q and K, rotation, the rotated K and the K before it (as V) to the cache
``sigmoid_gate`` the heads' outputs times sigmoid(gate)
``token_gate``   GELU(z) times a row of a table, by token
``qk_unit``      Q / K divided by their root mean square per head, K / V to the cache, Q scaled for the attention kernels
``gated_norm``   RMSNorm over all heads' outputs times sigmoid(gate)
``part_norm``    RMSNorm of equal parts of a row, after (or before) multiplying by SiLU(gate) if there is one
``act_mul``      act(gate) * up of f32 rows
``gelu_rows``    the exact GELU of f32 rows

The rows that feed a projection have the width ``row_width(n, dtype)``: bf16 rows are padded with zeros to a multiple of 8 elements
(the 16-byte row pitch of a TMA tile); f32 rows are not padded.  A projection's result comes in as a tensor (bf16 or f32) or as
``ops.gemm.PendingPartials`` (K-split fp32 partial sums, added here in split order); the stream's update may also be ``ops.moe.PendingCombine``
(expert outputs whose weighted sum is formed here).  ``Update`` is a sum of results with factors, some times a number per token, and may end in an average
over the stream at earlier places (``Depth``).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from .. import _native
from .gemm import GATE_ACT_CODE, gated_act_ref

_c, _i, _f, _l = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_long


def _p(t):
    return _c(t.data_ptr()) if t is not None else _c(0)


def _s():
    return _c(torch.cuda.current_stream().cuda_stream)


def row_width(n: int, dtype: torch.dtype) -> int:
    return n if dtype == torch.float32 else (n + 7) // 8 * 8


def split_rows(y):
    """(base tensor, is_f32, number of partial slabs, slab stride, row stride) of a projection result."""
    if hasattr(y, "buf"):
        return y.buf, 1, y.n, y.rows * y.hidden, y.hidden
    assert y.stride(1) == 1 and y.dtype in (torch.float32, torch.bfloat16)
    return y, int(y.dtype == torch.float32), 1, 0, y.stride(0)


@dataclass
class DynTanh:
    """Dynamic Tanh in place of a norm: ``tanh(alpha x) weight + bias`` (f32 ``[W]``), no statistics of the row."""
    alpha: float
    weight: torch.Tensor
    bias: torch.Tensor

    def to(self, device) -> "DynTanh":
        return DynTanh(self.alpha, self.weight.to(device), self.bias.to(device))

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return torch.tanh(self.alpha * x) * self.weight + self.bias


@dataclass
class PostNormed:
    """A sublayer's result that passes ``post`` before it joins the stream."""
    delta: object
    post: DynTanh


@dataclass
class RmsPosted:
    """A result that is divided by its root mean square and multiplied by ``weight`` (f32 ``[W]``) before it joins the stream."""
    delta: object
    weight: torch.Tensor
    eps: float


@dataclass
class Depth:
    """Average behind an update: the stream with the update is kept as row block ``at`` of ``hist`` (f32 ``[places, T, W]``), and goes on as the sum of
    ``weights[j] * hist[j]`` over the places up to it (``weights`` f32 ``[at + 1]``).  ``base`` f32 ``[T, W]``: that sum over the places below ``first``."""
    hist: torch.Tensor
    at: int
    weights: torch.Tensor
    base: Optional[torch.Tensor] = None
    first: int = 0


DEPTH_BLOCK = 8


def depth_base(hist: torch.Tensor, places: int, weights: List[torch.Tensor]) -> torch.Tensor:
    """f32 ``[K, T, W]``: for each of the K (at most ``DEPTH_BLOCK``) coming averages the sum of ``weights[k][j] * hist[j]`` over the ``places`` kept so far."""
    if not hist.is_cuda:
        return torch.stack([sum(hist[j] * w[j] for j in range(places)) for w in weights])
    assert hist.is_contiguous() and len(weights) <= DEPTH_BLOCK and all(w.numel() >= places for w in weights)
    out = torch.empty(len(weights), *hist.shape[1:], dtype=torch.float32, device=hist.device)
    ptr = (ctypes.c_void_p * len(weights))(*(w.data_ptr() for w in weights))
    _native.check(_native.cuda().gb_depth_base(_p(hist), _l(hist.stride(0)), _i(places), ptr, _i(len(weights)), _p(out), _l(hist[0].numel()), _s()), "gb_depth_base")
    return out


@dataclass
class Update:
    """``parts``: (result, factor, number per token or None); at most three."""
    parts: List[Tuple[object, float, Optional[torch.Tensor]]]
    depth: Optional[Depth] = None


def settled(x: torch.Tensor, delta) -> torch.Tensor:
    """The stream with a pending update, as a new tensor (captured layers, CPU references)."""
    w = x.shape[1]
    if delta is None:
        return x.clone()
    if not isinstance(delta, Update):
        return x + whole(delta)[:, :w]
    y = x.clone()
    for d, f, g in delta.parts:
        y += whole(d)[:, :w] * (f if g is None else f * g.unsqueeze(1))
    if delta.depth is not None:
        d = delta.depth
        y = y * d.weights[d.at] + sum(d.hist[j] * d.weights[j] for j in range(d.first, d.at))
        if d.base is not None:
            y = y + d.base
    return y


def whole(y) -> torch.Tensor:
    """f32 copy of a projection result or of a pending update (CPU references, captured layers)."""
    if isinstance(y, PostNormed):
        return y.post(whole(y.delta)[:, : y.post.weight.numel()])
    if isinstance(y, RmsPosted):
        u = whole(y.delta)[:, : y.weight.numel()]
        return u / torch.sqrt(u.pow(2).mean(-1, keepdim=True) + y.eps) * y.weight
    if hasattr(y, "pair_row"):
        rows = y.pair_row.reshape(y.n_tok, y.k).long()
        g = y.y.float()[rows.clamp_min(0)] * (rows >= 0).unsqueeze(-1)
        return (g * y.weights.float().unsqueeze(-1)).sum(1)
    return (y.buf.sum(0) if hasattr(y, "buf") else y).float()


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    if not table.is_cuda:
        return table[ids.long()].float() * scale
    out = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    _native.check(_native.cuda().gb_embed_f32(_p(ids), _p(table), _i(int(table.dtype == torch.float32)), _p(out), _i(ids.numel()), _i(table.shape[1]),
                                              _i(table.shape[0]), _f(scale), _s()), "gb_embed_f32")
    return out


def _rms2_ref(x, weight, weight2, eps, delta, add, rows, out_dtype):
    w = x.shape[1]
    y = x
    if delta is not None:
        y = y + whole(delta)[:, :w]
    if add is not None:
        y = y + add
    if rows is None:
        x.copy_(y)
    else:
        y = y[rows]
    unit = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)
    outs = []
    for wt in (weight, weight2):
        if wt is not None:
            o = torch.zeros(y.shape[0], row_width(w, out_dtype), dtype=out_dtype)
            o[:, :w] = (unit * wt).to(out_dtype)
            outs.append(o)
    return outs


def norm2(x: torch.Tensor, weight: torch.Tensor, eps: float, delta: Optional[RmsPosted] = None, add: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
          weight2: Optional[torch.Tensor] = None, out_dtype=torch.bfloat16) -> List[torch.Tensor]:
    """``norm`` for an update with a norm of its own (``RmsPosted``), for ``add`` one row per token (f32 ``[T, W]``), and with the rows under a second weight as
    well: one list entry per weight."""
    t, w = x.shape
    n = t if rows is None else rows.numel()
    if not x.is_cuda:
        return _rms2_ref(x, weight, weight2, eps, delta, add, rows, out_dtype)
    d = delta.delta if delta is not None else None
    base, f32, parts, stride, ld = split_rows(d) if d is not None else (None, 1, 1, 0, w)
    outs = [torch.empty(n, row_width(w, out_dtype), dtype=out_dtype, device=x.device) for wt in (weight, weight2) if wt is not None]
    rc = _native.cuda().gb_stream_rms2(_p(x), _p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(delta.weight if delta is not None else None),
                                       _f(delta.eps if delta is not None else 0.0), _p(add), _p(weight), _p(weight2), _p(rows), _p(outs[0]),
                                       _p(outs[1] if weight2 is not None else None), _i(int(out_dtype == torch.float32)), _i(outs[0].shape[1]), _i(n), _i(w), _f(eps), _s())
    _native.check(rc, "gb_stream_rms2")
    return outs


class _JoinPart(ctypes.Structure):
    """``struct JoinPart`` of csrc/kernels/stream_ops.cu."""
    _fields_ = [("p", ctypes.c_void_p), ("pair_row", ctypes.c_void_p), ("weights", ctypes.c_void_p), ("stride", ctypes.c_long), ("f32", ctypes.c_int),
                ("n_part", ctypes.c_int), ("ld", ctypes.c_int), ("k", ctypes.c_int), ("scale", ctypes.c_float), ("row_scale", ctypes.c_void_p)]


def _join_parts(parts):
    arr = (_JoinPart * 3)()
    for a, (d, f, g) in zip(arr, parts):
        a.scale = f
        a.row_scale = g.data_ptr() if g is not None else None
        if hasattr(d, "pair_row"):
            a.p, a.f32, a.n_part, a.ld = d.y.data_ptr(), int(d.y.dtype == torch.float32), 1, d.y.stride(0)
            a.pair_row, a.weights, a.k = d.pair_row.data_ptr(), d.weights.data_ptr(), d.k
        else:
            base, a.f32, a.n_part, a.stride, a.ld = split_rows(d)
            a.p = base.data_ptr()
    return arr


def join(x: torch.Tensor, parts: List[Tuple], out_dtype=None) -> Optional[torch.Tensor]:
    """``x += sum of factor * result`` in place (at most three (result, factor) pairs, or (result, factor, f32 number per token or None): tensors, partial sums
    or pending expert sums); returns the new rows in ``out_dtype`` (None: nothing), of width ``row_width(W)``."""
    t, w = x.shape
    parts = [p if len(p) == 3 else (*p, None) for p in parts]
    if not x.is_cuda:
        x.copy_(settled(x, Update(parts)))
        if out_dtype is None:
            return None
        o = torch.zeros(t, row_width(w, out_dtype), dtype=out_dtype)
        o[:, :w] = x.to(out_dtype)
        return o
    arr = _join_parts(parts)
    out = torch.empty(t, row_width(w, out_dtype), dtype=out_dtype, device=x.device) if out_dtype is not None else None
    rc = _native.cuda().gb_stream_join(_p(x), ctypes.byref(arr), _i(len(parts)), _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1] if out is not None else 0), _i(t),
                                       _i(w), _s())
    _native.check(rc, "gb_stream_join")
    return out


def depth_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float, delta: Update, rows: Optional[torch.Tensor] = None, out_dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """``norm`` for an update that ends in an average (``Depth``): the stream with the update goes to its place in ``hist``, the average becomes the stream."""
    d = delta.depth
    t, w = x.shape
    n = t if rows is None else rows.numel()
    if not x.is_cuda:
        y = settled(x, delta)
        if rows is None:
            d.hist[d.at] = settled(x, Update(delta.parts))
            x.copy_(y)
        else:
            y = y[rows]
        if weight is None:
            return None
        o = torch.zeros(n, row_width(w, out_dtype), dtype=out_dtype)
        o[:, :w] = (y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * weight).to(out_dtype)
        return o
    assert d.hist.is_contiguous() and d.hist.shape[1:] == x.shape and d.at < d.hist.shape[0] + int(rows is not None) and d.weights.numel() == d.at + 1
    out = torch.empty(n, row_width(w, out_dtype), dtype=out_dtype, device=x.device) if weight is not None else None
    rc = _native.cuda().gb_stream_depth(_p(x), ctypes.byref(_join_parts(delta.parts)), _i(len(delta.parts)), _p(d.hist), _l(d.hist.stride(0)), _p(d.base), _i(d.first), _i(d.at), _p(d.weights), _p(weight),
                                        _p(rows), _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1] if out is not None else 0), _i(n), _i(w), _f(eps), _s())
    _native.check(rc, "gb_stream_depth")
    return out


def norm_gate(x: torch.Tensor, weight: torch.Tensor, eps: float, delta, dot: torch.Tensor, out_dtype=torch.bfloat16) -> Tuple[torch.Tensor, torch.Tensor]:
    """``norm``, and for every token the sigmoid of the product of its normalised row with one more row: ``dot`` f32 ``[W]`` is that row times ``weight``."""
    gate = torch.empty(x.shape[0], dtype=torch.float32, device=x.device)
    return norm(x, weight, eps, delta, out_dtype=out_dtype, dot=dot, gate=gate), gate


def norm(x: torch.Tensor, weight, eps: float, delta=None, add: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
         out_dtype=torch.bfloat16, dot: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """``x += delta + add`` in place (``x`` f32 ``[T, W]``; both optional), then ``x / rms(x) * weight`` (f32 ``[W]``), or ``weight(x)`` if it is a
    ``DynTanh``, as ``out_dtype`` rows of width ``row_width(W)``.  With ``rows`` (int64): only those stream rows are normalised, and the stream is left as it is.  ``weight``
    None: only the update."""
    if isinstance(delta, RmsPosted):
        return norm2(x, weight, eps, delta, add, rows, out_dtype=out_dtype)[0]
    factor = 1.0
    if isinstance(delta, Update):
        if delta.depth is not None:
            assert add is None and dot is None
            return depth_norm(x, weight, eps, delta, rows, out_dtype)
        (d, f, g), *more = delta.parts
        if more or g is not None or hasattr(d, "pair_row"):
            join(x, delta.parts)
            delta = None
        else:
            delta, factor = d, f
    t, w = x.shape
    n = t if rows is None else rows.numel()
    if not x.is_cuda:
        y = x
        if delta is not None:
            y = y + (whole(delta)[:, :w] * factor if factor != 1.0 else whole(delta)[:, :w])
        if add is not None:
            y = y + add
        if rows is None:
            x.copy_(y)
        else:
            y = y[rows]
        if weight is None:
            return None
        o = torch.zeros(n, row_width(w, out_dtype), dtype=out_dtype)
        o[:, :w] = (weight(y) if isinstance(weight, DynTanh) else y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * weight).to(out_dtype)
        if dot is not None:
            gate.copy_(torch.sigmoid((y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * dot).sum(-1)))
        return o
    out = torch.empty(n, row_width(w, out_dtype), dtype=out_dtype, device=x.device) if weight is not None else None
    if isinstance(weight, DynTanh) or isinstance(delta, PostNormed):
        assert add is None and dot is None and factor == 1.0 and (weight is None or isinstance(weight, DynTanh))
        post, d = (delta.post, delta.delta) if isinstance(delta, PostNormed) else (None, delta)
        moe = hasattr(d, "pair_row")
        base, f32, parts, stride, ld = (d.y, int(d.y.dtype == torch.float32), 1, 0, d.y.stride(0)) if moe else split_rows(d) if d is not None else (None, 0, 1, 0, w)
        wb = lambda m: (_f(m.alpha), _p(m.weight), _p(m.bias)) if m is not None else (_f(0.0), _c(0), _c(0))
        rc = _native.cuda().gb_stream_dyt(_p(x), _p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(d.pair_row) if moe else _c(0), _p(d.weights) if moe else _c(0),
                                          _i(d.k if moe else 0), *wb(post), *wb(weight), _p(rows), _p(out), _i(int(out_dtype == torch.float32)),
                                          _i(out.shape[1] if out is not None else 0), _i(n), _i(w), _s())
        _native.check(rc, "gb_stream_dyt")
        return out
    base, f32, parts, stride, ld = split_rows(delta) if delta is not None else (None, 0, 1, 0, w)
    rc = _native.cuda().gb_stream_norm(_p(x), _p(base), _i(f32), _i(parts), _l(stride), _i(ld), _f(factor), _p(add), _p(weight), _p(dot), _p(gate), _p(rows), _p(out),
                                       _i(int(out_dtype == torch.float32)), _i(out.shape[1] if out is not None else 0), _i(n), _i(w), _f(eps), _s())
    _native.check(rc, "gb_stream_norm")
    return out


def qk_unit(qkv, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, hq: int, hkv: int, dk: int, dv: int, eps: float, q_scale: float,
            unit: bool = True, positions: Optional[torch.Tensor] = None, temp: Tuple[float, float] = (0.0, 1.0)) -> torch.Tensor:
    """Rows ``[Q heads | K heads | V heads]`` -> ``q [T, hq, dkp]`` (times ``q_scale``) in the cache's dtype; K / V of token ``t`` go to cache slot
    ``slots[t]`` (-1: not stored).  ``k_cache [slots, hkv, dkp]`` and ``v_cache [slots, hkv, dvp]`` may be wider than the heads (zero padding).
    ``unit``: Q and K are divided by their root mean square over the head.  ``temp`` = (coef, every), with a coefficient: Q at position p is also multiplied by
    1 + coef ln(floor((p + 1) / every) + 1)."""
    base, f32, parts, stride, ld = split_rows(qkv)
    t = qkv.rows if hasattr(qkv, "buf") else qkv.shape[0]
    dkp, dvp = k_cache.shape[2], v_cache.shape[2]
    if not base.is_cuda:
        y = whole(qkv)
        q, k, v = y[:, : hq * dk].reshape(t, hq, dk), y[:, hq * dk: (hq + hkv) * dk].reshape(t, hkv, dk), y[:, (hq + hkv) * dk: (hq + hkv) * dk + hkv * dv].reshape(t, hkv, dv)
        if unit:
            q = q / torch.sqrt(q.pow(2).mean(-1, keepdim=True) + eps)
            k = k / torch.sqrt(k.pow(2).mean(-1, keepdim=True) + eps)
        if temp[0]:
            q = q * (1.0 + temp[0] * torch.log(torch.floor((positions.double() + 1) / temp[1]) + 1)).float().reshape(t, 1, 1)
        pad = torch.nn.functional.pad
        ok = slots >= 0
        k_cache[slots[ok].long()] = pad(k, (0, dkp - dk))[ok].to(k_cache.dtype)
        v_cache[slots[ok].long()] = pad(v, (0, dvp - dv))[ok].to(v_cache.dtype)
        return pad(q * q_scale, (0, dkp - dk)).to(k_cache.dtype)
    q = torch.empty(t, hq, dkp, dtype=k_cache.dtype, device=base.device)
    rc = _native.cuda().gb_qk_unit_store(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(slots), _p(q), _p(k_cache), _p(v_cache),
                                         _i(int(k_cache.dtype == torch.float32)), _l(k_cache.shape[0]), _i(t), _i(hq), _i(hkv), _i(dk), _i(dv), _i(dkp),
                                         _i(dvp), _f(eps), _f(q_scale), _i(int(unit)), _p(positions if temp[0] else None), _f(temp[0]), ctypes.c_double(temp[1]), _s())
    _native.check(rc, "gb_qk_unit_store")
    return q


def qk_rows(qkv, slots: torch.Tensor, q_norm: torch.Tensor, k_norm: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, hq: int, hkv: int, dk: int, dv: int,
            eps: float, q_scale: float) -> torch.Tensor:
    """As ``qk_unit``, with one RMS norm over all of Q and one over all of K (weights f32 ``[hq * dk]`` and ``[hkv * dk]``).  Columns behind V are not read."""
    base, f32, parts, stride, ld = split_rows(qkv)
    t = qkv.rows if hasattr(qkv, "buf") else qkv.shape[0]
    nq, nk, dkp, dvp = hq * dk, hkv * dk, k_cache.shape[2], v_cache.shape[2]
    if not base.is_cuda:
        y = whole(qkv)
        n = lambda z, w: z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w
        q, k, v = n(y[:, :nq], q_norm), n(y[:, nq: nq + nk], k_norm), y[:, nq + nk: nq + nk + hkv * dv]
        pad = torch.nn.functional.pad
        ok = slots >= 0
        k_cache[slots[ok].long()] = pad(k.reshape(t, hkv, dk), (0, dkp - dk))[ok].to(k_cache.dtype)
        v_cache[slots[ok].long()] = pad(v.reshape(t, hkv, dv), (0, dvp - dv))[ok].to(v_cache.dtype)
        return pad(q.reshape(t, hq, dk) * q_scale, (0, dkp - dk)).to(k_cache.dtype)
    q = torch.empty(t, hq, dkp, dtype=k_cache.dtype, device=base.device)
    rc = _native.cuda().gb_qk_rows_store(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(slots), _p(q_norm), _p(k_norm), _p(q), _p(k_cache), _p(v_cache),
                                         _i(int(k_cache.dtype == torch.float32)), _l(k_cache.shape[0]), _i(t), _i(hq), _i(hkv), _i(dk), _i(dv), _i(dkp), _i(dvp), _f(eps),
                                         _f(q_scale), _s())
    _native.check(rc, "gb_qk_rows_store")
    return q


def rotary_table(positions: torch.Tensor, freq: torch.Tensor, mag: float) -> torch.Tensor:
    """f32 ``[T, pairs, 2]``: cos and sin of position * freq (f64 ``[pairs]``), times ``mag``."""
    if not positions.is_cuda:
        a = positions.double().unsqueeze(1) * freq
        return torch.stack([torch.cos(a) * mag, torch.sin(a) * mag], dim=-1).float()
    out = torch.empty(positions.numel(), freq.numel(), 2, dtype=torch.float32, device=positions.device)
    _native.check(_native.cuda().gb_rotary_table(_p(positions), _p(freq), _f(mag), _p(out), _i(positions.numel()), _i(freq.numel()), _s()), "gb_rotary_table")
    return out


def conv_rotary(qk, table: torch.Tensor, slots: torch.Tensor, conv_w: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor,
                k_cache: torch.Tensor, v_cache: torch.Tensor, hq: int, hkv: int, d: int, q_scale: float, max_tokens: int) -> torch.Tensor:
    """Rows ``[Q heads | K heads]`` through a causal convolution over time (``conv_w`` f32 ``[channels, taps]``, the last tap meets the current token; the last
    ``taps - 1`` rows of a sequence are kept in ``state`` f32 ``[slots, taps - 1, channels]``), then neighbours (2i, 2i + 1) of each head turned by ``table``
    (``rotary_table``; dimensions behind its pairs pass).  Returns ``q [T, hq, dkp]`` times ``q_scale``; the rotated K and the K before the rotation (as V) go to
    cache slot ``slots[t]``.  ``max_tokens``: of the longest sequence."""
    base, f32, parts, stride, ld = split_rows(qk)
    t = qk.rows if hasattr(qk, "buf") else qk.shape[0]
    ch, taps = conv_w.shape
    dkp, dvp, dims = k_cache.shape[2], v_cache.shape[2], 2 * table.shape[1]
    if not base.is_cuda:
        x, y, cu = whole(qk)[:, :ch], torch.zeros(t, ch), cu_q.tolist()
        for s in range(len(cu) - 1):
            n = cu[s + 1] - cu[s]
            if n:
                rows = torch.cat([state[int(seq_slots[s])], x[cu[s]: cu[s + 1]]])
                y[cu[s]: cu[s + 1]] = sum(conv_w[:, j] * rows[j: j + n] for j in range(taps))
                state[int(seq_slots[s])] = rows[n:]
        h = y.reshape(t, hq + hkv, d)
        r = h.clone()
        c, sn = table[:, :, 0].unsqueeze(1), table[:, :, 1].unsqueeze(1)
        r[..., 0:dims:2], r[..., 1:dims:2] = h[..., 0:dims:2] * c - h[..., 1:dims:2] * sn, h[..., 1:dims:2] * c + h[..., 0:dims:2] * sn
        pad = torch.nn.functional.pad
        ok = slots >= 0
        k_cache[slots[ok].long()] = pad(r[:, hq:], (0, dkp - d))[ok].to(k_cache.dtype)
        v_cache[slots[ok].long()] = pad(h[:, hq:], (0, dvp - d))[ok].to(v_cache.dtype)
        return pad(r[:, :hq] * q_scale, (0, dkp - d)).to(k_cache.dtype)
    assert state.is_contiguous() and state.dtype == torch.float32
    q = torch.empty(t, hq, dkp, dtype=k_cache.dtype, device=base.device)
    rc = _native.cuda().gb_conv_rotary_store(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(table), _i(dims), _p(slots), _p(conv_w), _i(taps), _p(state),
                                             _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(q), _p(k_cache), _p(v_cache), _i(int(k_cache.dtype == torch.float32)),
                                             _l(k_cache.shape[0]), _i(hq), _i(hkv), _i(d), _i(dkp), _i(dvp), _f(q_scale), _i(max_tokens), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_conv_rotary_store")
    return q


def sigmoid_gate(a: torch.Tensor, proj, col: int, dv: int) -> torch.Tensor:
    """``a [T, H, dvp] *= sigmoid(gate)`` in place on the first ``dv`` columns of each head: the gate is columns ``col ...`` (head by head, ``dv`` each) of the
    projection result ``proj``."""
    t, hd, dvp = a.shape
    base, f32, parts, stride, ld = split_rows(proj)
    if not a.is_cuda:
        g = torch.sigmoid(whole(proj)[:, col: col + hd * dv]).reshape(t, hd, dv)
        a[:, :, :dv] = (a[:, :, :dv].float() * g).to(a.dtype)
        return a
    rc = _native.cuda().gb_sigmoid_gate(_p(a), _i(int(a.dtype == torch.float32)), _c(base.data_ptr() + col * base.element_size()), _i(f32), _i(parts), _l(stride), _i(ld),
                                        _i(t), _i(hd), _i(dv), _i(dvp), _s())
    _native.check(rc, "gb_sigmoid_gate")
    return a


def token_gate(z, ids: torch.Tensor, table: torch.Tensor, col: int, n: int, out_dtype=torch.bfloat16) -> torch.Tensor:
    """``gelu(z) * table[id, col : col + n]`` (the tanh form of GELU) -> rows ``[T, row_width(n)]``; ``z`` is a projection result of ``n`` columns."""
    base, f32, parts, stride, ld = split_rows(z)
    t = z.rows if hasattr(z, "buf") else z.shape[0]
    out = torch.empty(t, row_width(n, out_dtype), dtype=out_dtype, device=base.device)
    if not base.is_cuda:
        out.zero_()
        out[:, :n] = (torch.nn.functional.gelu(whole(z)[:, :n], approximate="tanh") * table[ids.long(), col: col + n].float()).to(out_dtype)
        return out
    rc = _native.cuda().gb_token_gate(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(ids), _p(table), _i(int(table.dtype == torch.float32)), _i(table.shape[1]), _i(col),
                                      _i(table.shape[0]), _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1]), _i(t), _i(n), _s())
    _native.check(rc, "gb_token_gate")
    return out


def gated_norm(o: torch.Tensor, proj, gate_col: int, weight: torch.Tensor, eps: float, out_dtype=torch.bfloat16) -> torch.Tensor:
    """``rms_norm(o) * weight * sigmoid(gate)``: ``o`` f32 ``[T, N]`` (all heads side by side), the gate is columns ``gate_col ...`` of the
    projection result ``proj``."""
    t, n = o.shape
    ldo = row_width(n, out_dtype)
    if not o.is_cuda:
        g = whole(proj)[:, gate_col: gate_col + n]
        out = torch.zeros(t, ldo, dtype=out_dtype)
        out[:, :n] = (o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * weight * torch.sigmoid(g)).to(out_dtype)
        return out
    base, f32, parts, stride, ld = split_rows(proj)
    out = torch.empty(t, ldo, dtype=out_dtype, device=o.device)
    gate = _c(base.data_ptr() + gate_col * base.element_size())
    rc = _native.cuda().gb_gated_norm(_p(o), _i(o.stride(0)), gate, _i(f32), _i(parts), _l(stride), _i(ld), _p(weight), _p(out),
                                      _i(int(out_dtype == torch.float32)), _i(ldo), _i(t), _i(n), _f(eps), _s())
    _native.check(rc, "gb_gated_norm")
    return out


def part_norm(o: torch.Tensor, weight: torch.Tensor, parts: int, eps: float, gate=None, gate_col: int = 0, out_dtype=torch.bfloat16,
              gate_after: bool = False) -> torch.Tensor:
    """``o`` f32 ``[T, N]`` times SiLU(gate) (columns ``gate_col ...`` of the projection result ``gate``, if given), then every one of ``parts`` equal
    parts divided by its root mean square and multiplied by ``weight`` (f32 ``[N]``, or shorter and repeated).  ``gate_after``: the gate multiplies the result."""
    t, n = o.shape
    ldo = row_width(n, out_dtype)
    if not o.is_cuda:
        g = torch.nn.functional.silu(whole(gate)[:, gate_col: gate_col + n]) if gate is not None else 1.0
        y = (o if gate_after else o * g).reshape(t, parts, n // parts)
        y = (y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)).reshape(t, n) * weight.repeat(n // weight.numel())
        if gate_after:
            y = y * g
        out = torch.zeros(t, ldo, dtype=out_dtype)
        out[:, :n] = y.to(out_dtype)
        return out
    base, f32, np_, stride, ld = split_rows(gate) if gate is not None else (None, 1, 1, 0, n)
    out = torch.empty(t, ldo, dtype=out_dtype, device=o.device)
    g = _c(base.data_ptr() + gate_col * base.element_size()) if gate is not None else _c(0)
    rc = _native.cuda().gb_part_norm(_p(o), _i(o.stride(0)), g, _i(f32), _i(np_), _l(stride), _i(ld), _p(weight), _i(weight.numel()), _p(out),
                                     _i(int(out_dtype == torch.float32)), _i(ldo), _i(t), _i(n), _i(parts), _f(eps), _i(int(gate_after)), _s())
    _native.check(rc, "gb_part_norm")
    return out


def gelu_rows(x: torch.Tensor) -> torch.Tensor:
    """The exact GELU, ``x (1 + erf(x / sqrt 2)) / 2``, of contiguous f32 rows."""
    if not x.is_cuda:
        return torch.nn.functional.gelu(x)
    assert x.is_contiguous() and x.dtype == torch.float32
    out = torch.empty_like(x)
    _native.check(_native.cuda().gb_gelu_f32(_p(x), _p(out), _l(x.numel()), _s()), "gb_gelu_f32")
    return out


def act_mul(gate_up: torch.Tensor, act: str, cap: float = 0.0) -> torch.Tensor:
    """``act(gate) * up`` of f32 rows ``[gate | up]`` (``ops.gemm.gated_act_ref``)."""
    rows, two_i = gate_up.shape
    inter = two_i // 2
    if not gate_up.is_cuda:
        return gated_act_ref(gate_up[:, :inter], gate_up[:, inter:], act, cap)
    out = torch.empty(rows, inter, dtype=torch.float32, device=gate_up.device)
    _native.check(_native.cuda().gb_act_mul_f32(_p(gate_up), _p(out), _l(rows), _i(inter), _i(gate_up.stride(0)), _i(GATE_ACT_CODE[act]), _f(cap), _s()),
                  "gb_act_mul_f32")
    return out
