"""Token-wise ops of models with a 32-bit residual stream (csrc/kernels/stream_ops.cu) and their PyTorch references.

``embed``        embedding rows (times a factor) as an f32 stream
``norm``         stream += pending update (+ a vector), then RMSNorm or Dynamic Tanh -> rows for the next projection; the update may have a
                 norm of its own (``PostNormed``)
``qk_unit``      Q / K divided by their root mean square per head, K / V to the cache, Q scaled for the attention kernels
``gated_norm``   RMSNorm over all heads' outputs times sigmoid(gate)
``part_norm``    RMSNorm of equal parts of a row, after multiplying by SiLU(gate) if there is one
``act_mul``      act(gate) * up of f32 rows

The rows that feed a projection have the width ``row_width(n, dtype)``: bf16 rows are padded with zeros to a multiple of 8 elements
(the 16-byte row pitch of a TMA tile); f32 rows are not padded.  A projection's result comes in as a tensor (bf16 or f32) or as
``ops.gemm.PendingPartials`` (K-split fp32 partial sums, added here in split order); the stream's update may also be ``ops.moe.PendingCombine``
(expert outputs whose weighted sum is formed here).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from .. import _native
from .gemm import gate_act_ref

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


def whole(y) -> torch.Tensor:
    """f32 copy of a projection result or of a pending update (CPU references, captured layers)."""
    if isinstance(y, PostNormed):
        return y.post(whole(y.delta)[:, : y.post.weight.numel()])
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


def norm(x: torch.Tensor, weight, eps: float, delta=None, add: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
         out_dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """``x += delta + add`` in place (``x`` f32 ``[T, W]``; both optional), then ``x / rms(x) * weight`` (f32 ``[W]``), or ``weight(x)`` if it is a
    ``DynTanh``, as ``out_dtype`` rows of width ``row_width(W)``.  With ``rows`` (int64): only those stream rows are normalised, and the stream is left as it is.  ``weight``
    None: only the update."""
    t, w = x.shape
    n = t if rows is None else rows.numel()
    if not x.is_cuda:
        y = x
        if delta is not None:
            y = y + whole(delta)[:, :w]
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
        return o
    out = torch.empty(n, row_width(w, out_dtype), dtype=out_dtype, device=x.device) if weight is not None else None
    if isinstance(weight, DynTanh) or isinstance(delta, PostNormed):
        assert add is None and (weight is None or isinstance(weight, DynTanh))
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
    rc = _native.cuda().gb_stream_norm(_p(x), _p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(add), _p(weight), _p(rows), _p(out),
                                       _i(int(out_dtype == torch.float32)), _i(out.shape[1] if out is not None else 0), _i(n), _i(w), _f(eps), _s())
    _native.check(rc, "gb_stream_norm")
    return out


def qk_unit(qkv, slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, hq: int, hkv: int, dk: int, dv: int, eps: float, q_scale: float,
            unit: bool = True) -> torch.Tensor:
    """Rows ``[Q heads | K heads | V heads]`` -> ``q [T, hq, dkp]`` (times ``q_scale``) in the cache's dtype; K / V of token ``t`` go to cache slot
    ``slots[t]`` (-1: not stored).  ``k_cache [slots, hkv, dkp]`` and ``v_cache [slots, hkv, dvp]`` may be wider than the heads (zero padding).
    ``unit``: Q and K are divided by their root mean square over the head."""
    base, f32, parts, stride, ld = split_rows(qkv)
    t = qkv.rows if hasattr(qkv, "buf") else qkv.shape[0]
    dkp, dvp = k_cache.shape[2], v_cache.shape[2]
    if not base.is_cuda:
        y = whole(qkv)
        q, k, v = y[:, : hq * dk].reshape(t, hq, dk), y[:, hq * dk: (hq + hkv) * dk].reshape(t, hkv, dk), y[:, (hq + hkv) * dk: (hq + hkv) * dk + hkv * dv].reshape(t, hkv, dv)
        if unit:
            q = q / torch.sqrt(q.pow(2).mean(-1, keepdim=True) + eps)
            k = k / torch.sqrt(k.pow(2).mean(-1, keepdim=True) + eps)
        pad = torch.nn.functional.pad
        ok = slots >= 0
        k_cache[slots[ok].long()] = pad(k, (0, dkp - dk))[ok].to(k_cache.dtype)
        v_cache[slots[ok].long()] = pad(v, (0, dvp - dv))[ok].to(v_cache.dtype)
        return pad(q * q_scale, (0, dkp - dk)).to(k_cache.dtype)
    q = torch.empty(t, hq, dkp, dtype=k_cache.dtype, device=base.device)
    rc = _native.cuda().gb_qk_unit_store(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(slots), _p(q), _p(k_cache), _p(v_cache),
                                         _i(int(k_cache.dtype == torch.float32)), _l(k_cache.shape[0]), _i(t), _i(hq), _i(hkv), _i(dk), _i(dv), _i(dkp),
                                         _i(dvp), _f(eps), _f(q_scale), _i(int(unit)), _s())
    _native.check(rc, "gb_qk_unit_store")
    return q


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


def part_norm(o: torch.Tensor, weight: torch.Tensor, parts: int, eps: float, gate=None, gate_col: int = 0, out_dtype=torch.bfloat16) -> torch.Tensor:
    """``o`` f32 ``[T, N]`` times SiLU(gate) (columns ``gate_col ...`` of the projection result ``gate``, if given), then every one of ``parts`` equal
    parts divided by its root mean square and multiplied by ``weight`` (f32 ``[N]``, or shorter and repeated)."""
    t, n = o.shape
    ldo = row_width(n, out_dtype)
    if not o.is_cuda:
        y = o
        if gate is not None:
            y = y * torch.nn.functional.silu(whole(gate)[:, gate_col: gate_col + n])
        y = y.reshape(t, parts, n // parts)
        y = (y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)).reshape(t, n) * weight.repeat(n // weight.numel())
        out = torch.zeros(t, ldo, dtype=out_dtype)
        out[:, :n] = y.to(out_dtype)
        return out
    base, f32, np_, stride, ld = split_rows(gate) if gate is not None else (None, 1, 1, 0, n)
    out = torch.empty(t, ldo, dtype=out_dtype, device=o.device)
    g = _c(base.data_ptr() + gate_col * base.element_size()) if gate is not None else _c(0)
    rc = _native.cuda().gb_part_norm(_p(o), _i(o.stride(0)), g, _i(f32), _i(np_), _l(stride), _i(ld), _p(weight), _i(weight.numel()), _p(out),
                                     _i(int(out_dtype == torch.float32)), _i(ldo), _i(t), _i(n), _i(parts), _f(eps), _s())
    _native.check(rc, "gb_part_norm")
    return out


def act_mul(gate_up: torch.Tensor, act: str) -> torch.Tensor:
    """``act(gate) * up`` of f32 rows ``[gate | up]``."""
    rows, two_i = gate_up.shape
    inter = two_i // 2
    if not gate_up.is_cuda:
        return gate_act_ref(gate_up[:, :inter], act) * gate_up[:, inter:]
    out = torch.empty(rows, inter, dtype=torch.float32, device=gate_up.device)
    _native.check(_native.cuda().gb_act_mul_f32(_p(gate_up), _p(out), _l(rows), _i(inter), _i(gate_up.stride(0)), _i(1 if act == "gelu_tanh" else 0), _s()),
                  "gb_act_mul_f32")
    return out
