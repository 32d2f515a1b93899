"""Recurrent mixers with input-dependent decay (csrc/kernels/recurrent.cu and its chunked forms) and their PyTorch references.

``causal_conv``  depthwise causal convolution + SiLU, the last inputs carried per sequence (Mamba-2)
``ssd``          Mamba-2:  S_t = exp(a dt_t) S_{t-1} + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t
``gla``          HGRN2:    S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,  o_t = S_t^T q_t
``rwkv``         RWKV:     o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,  S_t = diag(w_t) S_{t-1} + k_t v_t^T,  w = exp(-exp(z))
``mingru``       s_t = (1 - z_t) s_{t-1} + z_t c_t per channel, the gate z and the candidate c from the current token alone
``token_shift``  mixes of a token's row and the one before it, for the projections of ``rwkv``

State tensors: ``conv_state`` f32 ``[slots, taps - 1, channels]`` (oldest row first), ``state`` f32 ``[slots, heads, dim, vdim]``; one slot per
sequence, updated in place.
"""
from __future__ import annotations

import ctypes
import os
from typing import Optional

import torch

from .. import _native
from . import gemm
from .stream import row_width, split_rows, whole

_c, _i, _f, _l = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_long
F = torch.nn.functional


def _p(t):
    return _c(t.data_ptr()) if t is not None else _c(0)


def _s():
    return _c(torch.cuda.current_stream().cuda_stream)


# Launches whose longest sequence brings at least this many tokens take the chunked scans
CHUNKED = os.environ.get("GB_RECURRENT_CHUNKED", "1") != "0"
CHUNKED_MIN_TOKENS = 16


def can_chunk(rows: torch.Tensor, dim: int, vdim: int) -> bool:
    """Whether the chunked kernels take these rows: bf16 with a 16-byte pitch, key size up to 128."""
    return bool(rows.is_cuda and rows.dtype == torch.bfloat16 and dim <= 128 and dim % 8 == 0 and vdim % 8 == 0 and rows.stride(0) % 8 == 0 and rows.data_ptr() % 16 == 0)


def _n_rows(y) -> int:
    return y.rows if hasattr(y, "buf") else y.shape[0]


def _at(base: torch.Tensor, col: int):
    return _c(base.data_ptr() + col * base.element_size())


def causal_conv_ref(x, w, b, state, cu_q, seq_slots, out_dtype):
    t, ch = x.shape
    out = torch.zeros(t, row_width(ch, out_dtype), dtype=out_dtype)
    nh = w.shape[1] - 1
    cu = cu_q.tolist()
    for s in range(len(cu) - 1):
        if cu[s + 1] == cu[s]:
            continue
        rows = torch.cat([state[int(seq_slots[s])], x[cu[s]: cu[s + 1]]])
        y = sum(w[:, k] * rows[k: k + cu[s + 1] - cu[s]] for k in range(nh + 1)) + b
        out[cu[s]: cu[s + 1], :ch] = F.silu(y).to(out_dtype)
        state[int(seq_slots[s])] = rows[rows.shape[0] - nh:]
    return out


def causal_conv(proj, col: int, w: torch.Tensor, b: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, max_tokens: int,
                out_dtype=torch.bfloat16) -> torch.Tensor:
    """SiLU(conv + b) of the columns ``col ... col + channels - 1`` of the projection result ``proj`` -> rows ``[T, row_width(channels)]``."""
    ch, taps = w.shape
    base, f32, parts, stride, ld = split_rows(proj)
    if not base.is_cuda:
        return causal_conv_ref(whole(proj)[:, col: col + ch], w, b, state, cu_q, seq_slots, out_dtype)
    t = _n_rows(proj)
    assert state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty(t, row_width(ch, out_dtype), dtype=out_dtype, device=base.device)
    rc = _native.cuda().gb_causal_conv(_at(base, col), _i(f32), _i(parts), _l(stride), _i(ld), _p(w), _p(b), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots),
                                       _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1]), _i(ch), _i(taps), _i(max_tokens), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_causal_conv")
    return out


def ssd_ref(xbc, dt, dt_bias, a, d_skip, state, cu_q, seq_slots, heads, groups, dim, vdim):
    t, nv = xbc.shape[0], heads * vdim
    y = xbc.float()
    x = y[:, :nv].reshape(t, heads, vdim)
    bm = y[:, nv: nv + groups * dim].reshape(t, groups, dim).repeat_interleave(heads // groups, dim=1)
    cm = y[:, nv + groups * dim: nv + 2 * groups * dim].reshape(t, groups, dim).repeat_interleave(heads // groups, dim=1)
    dt = F.softplus(dt.float() + dt_bias, threshold=1e9)
    dec = torch.exp(a * dt)
    out = torch.zeros(t, nv)
    cu = cu_q.tolist()
    for s in range(len(cu) - 1):
        st = state[int(seq_slots[s])] if cu[s + 1] > cu[s] else None
        for i in range(cu[s], cu[s + 1]):
            st.mul_(dec[i].reshape(heads, 1, 1)).add_((dt[i].unsqueeze(-1) * bm[i]).unsqueeze(-1) * x[i].unsqueeze(1))
            out[i] = (torch.einsum("hde,hd->he", st, cm[i]) + d_skip.unsqueeze(-1) * x[i]).reshape(-1)
    return out


def ssd(xbc: torch.Tensor, dt, dt_col: int, dt_bias: torch.Tensor, a: torch.Tensor, d_skip: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor,
        seq_slots: torch.Tensor, heads: int, groups: int, dim: int, vdim: int, max_tokens: int = 1) -> torch.Tensor:
    """``xbc``: activated rows ``[x heads x vdim | B groups x dim | C groups x dim | ...]``; ``dt``: projection result (f32 or partial sums) whose
    columns ``dt_col ...`` are the step sizes before bias and softplus.  ``max_tokens``: of the longest sequence.  Returns f32 ``[T, heads * vdim]``."""
    base, f32, parts, stride, ld = split_rows(dt)
    if not base.is_cuda:
        return ssd_ref(xbc, whole(dt)[:, dt_col: dt_col + heads], dt_bias, a, d_skip, state, cu_q, seq_slots, heads, groups, dim, vdim)
    t = xbc.shape[0]
    assert f32 and state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty(t, heads * vdim, dtype=torch.float32, device=base.device)
    if CHUNKED and max_tokens >= CHUNKED_MIN_TOKENS and can_chunk(xbc, dim, vdim):
        rc = _native.cuda().gb_ssd_chunk(_p(xbc), _i(xbc.stride(0)), _i(t), _at(base, dt_col), _i(parts), _l(stride), _i(ld), _p(dt_bias), _p(a), _p(d_skip), _p(state),
                                         _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out), _i(heads * vdim), _i(heads), _i(groups), _i(dim), _i(vdim),
                                         _i(cu_q.numel() - 1), _c(_native.status_ptr()), _s())
        _native.check(rc, "gb_ssd_chunk")
        return out
    rc = _native.cuda().gb_recurrent_step(_i(0), _p(xbc), _i(int(xbc.dtype == torch.float32)), _i(1), _l(0), _i(xbc.stride(0)), _at(base, dt_col), _i(parts), _l(stride),
                                          _i(ld), _p(dt_bias), _p(a), _p(d_skip), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out), _i(heads * vdim),
                                          _i(heads), _i(groups), _i(dim), _i(vdim), _i(0), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_recurrent_step")
    return out


def gla_ref(q, v, z, lower, state, cu_q, seq_slots, heads, dim, vdim):
    t = q.shape[0]
    q, v = q.reshape(t, heads, dim), v.reshape(t, heads, vdim)
    f = (lower + (1 - lower) * torch.sigmoid(z)).reshape(t, heads, dim)
    k = ((1 - lower) * torch.sigmoid(-z)).reshape(t, heads, dim)
    out = torch.zeros(t, heads * vdim)
    cu = cu_q.tolist()
    for s in range(len(cu) - 1):
        st = state[int(seq_slots[s])] if cu[s + 1] > cu[s] else None
        for i in range(cu[s], cu[s + 1]):
            st.mul_(f[i].unsqueeze(-1)).add_(k[i].unsqueeze(-1) * v[i].unsqueeze(1))
            out[i] = torch.einsum("hde,hd->he", st, q[i]).reshape(-1)
    return out


def gla(qv, gate, gate_col: int, f_bias: torch.Tensor, lower: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, heads: int, dim: int,
        vdim: int, activated: bool = False, max_tokens: int = 1) -> torch.Tensor:
    """``qv``: projection result with columns ``[q heads x dim | v heads x vdim | ...]``, q before its SiLU or (``activated``) after it; ``gate``:
    projection result (f32 or partial sums) whose columns ``gate_col ...`` are the forget gates before bias and sigmoid.  Returns f32
    ``[T, heads * vdim]``."""
    gb, gf32, gparts, gstride, gld = split_rows(gate)
    nq, nv = heads * dim, heads * vdim
    if not gb.is_cuda:
        y = whole(qv)
        q = y[:, :nq] if activated else F.silu(y[:, :nq])
        return gla_ref(q, y[:, nq: nq + nv], whole(gate)[:, gate_col: gate_col + nq] + f_bias, lower, state, cu_q, seq_slots, heads, dim, vdim)
    base, f32, parts, stride, ld = split_rows(qv)
    t = _n_rows(qv)
    assert gf32 and state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty(t, nv, dtype=torch.float32, device=base.device)
    if CHUNKED and max_tokens >= CHUNKED_MIN_TOKENS and activated and not hasattr(qv, "buf") and can_chunk(base, dim, vdim):
        lib, n_seqs = _native.cuda(), cu_q.numel() - 1
        lib.gb_gla_chunk_workspace.restype = _l
        nb = int(lib.gb_gla_chunk_workspace(_l(t), _i(n_seqs), _i(heads), _i(dim)))
        ws = torch.empty(nb, dtype=torch.uint8, device=base.device)
        rc = lib.gb_gla_chunk(_p(base), _i(ld), _i(t), _at(gb, gate_col), _i(gparts), _l(gstride), _i(gld), _p(f_bias), _p(lower), _p(state), _i(state.shape[0]), _p(cu_q),
                              _p(seq_slots), _p(out), _i(nv), _i(heads), _i(dim), _i(vdim), _i(max_tokens), _i(n_seqs), _p(ws), _l(nb), _c(_native.status_ptr()), _s())
        _native.check(rc, "gb_gla_chunk", n=2)
        return out
    rc = _native.cuda().gb_recurrent_step(_i(1), _p(base), _i(f32), _i(parts), _l(stride), _i(ld), _at(gb, gate_col), _i(gparts), _l(gstride), _i(gld), _p(f_bias), _p(lower),
                                          _c(0), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out), _i(nv), _i(heads), _i(1), _i(dim), _i(vdim),
                                          _i(int(not activated)), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_recurrent_step")
    return out


def mingru_ref(x, g, z, x_bias, z_bias, state, cu_q, seq_slots, out_dtype):
    t, n = x.shape
    u, z = x + x_bias, z + z_bias
    keep, cand = torch.sigmoid(-z), torch.sigmoid(z) * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out, cu = torch.zeros(t, row_width(n, out_dtype), dtype=out_dtype), cu_q.tolist()
    for s in range(len(cu) - 1):
        st = state[int(seq_slots[s])].reshape(-1) if cu[s + 1] > cu[s] else None
        for i in range(cu[s], cu[s + 1]):
            st.mul_(keep[i]).add_(cand[i])
            out[i, :n] = (st * F.silu(g[i])).to(out_dtype)
    return out


def mingru(xg, z, z_col: int, x_bias: torch.Tensor, z_bias: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, n: int, max_tokens: int = 1,
           out_dtype=torch.bfloat16) -> torch.Tensor:
    """``xg``: projection result with columns ``[x | output gate]``, ``n`` each; ``z``: projection result (f32 or partial sums) whose columns ``z_col ...`` are the
    gate's logits.  With u = x + x_bias the candidate is u + 1/2 (u >= 0) or sigmoid(u); ``state`` f32 ``[slots, 1, 1, n]``.  Returns the rows
    ``s_t * silu(output gate)``, ``[T, row_width(n)]``."""
    zb, zf32, zparts, zstride, zld = split_rows(z)
    if not zb.is_cuda:
        y = whole(xg)
        return mingru_ref(y[:, :n], y[:, n: 2 * n], whole(z)[:, z_col: z_col + n], x_bias, z_bias, state, cu_q, seq_slots, out_dtype)
    base, f32, parts, stride, ld = split_rows(xg)
    t = _n_rows(xg)
    assert zf32 and state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty(t, row_width(n, out_dtype), dtype=out_dtype, device=base.device)
    rc = _native.cuda().gb_mingru(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _at(zb, z_col), _i(zparts), _l(zstride), _i(zld), _p(x_bias), _p(z_bias), _p(state),
                                  _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1]), _i(n), _i(max_tokens),
                                  _i(cu_q.numel() - 1), _i(int(CHUNKED and max_tokens >= CHUNKED_MIN_TOKENS)), _s())
    _native.check(rc, "gb_mingru")
    return out


def shift_pad(t: int) -> int:
    """Rows per mix of ``token_shift`` for ``t`` tokens: whole token tiles of the grouped product that follows."""
    tn = gemm.pick_tn(t) if t < 128 else 128
    return (t + tn - 1) // tn * tn


def shift_tile(pad: int) -> int:
    """Token tile of that product."""
    return 256 if pad >= 512 else min(pad, 128)


def token_shift(h: torch.Tensor, width: int, mu: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, pad: int, max_tokens: int) -> torch.Tensor:
    """Rows ``h [T, ld]`` -> ``[n, pad, ld]``: mix i of token t is ``h + (h' - h) * mu[i]`` with the row h' in front of it (``mu`` f32 ``[n, width]``).  The row in front
    of a sequence's first token comes from ``state`` f32 ``[slots, 1, width]``, its last one goes there.  Rows behind T are undefined."""
    t, ld = h.shape
    n = mu.shape[0]
    if not h.is_cuda:
        out, cu = torch.zeros(n, pad, ld, dtype=h.dtype), cu_q.tolist()
        x = h[:, :width].float()
        for s in range(len(cu) - 1):
            if cu[s + 1] > cu[s]:
                cur, slot = x[cu[s]: cu[s + 1]], int(seq_slots[s])
                prev = torch.cat([state[slot], cur[:-1]])
                out[:, cu[s]: cu[s + 1], :width] = (cur + (prev - cur) * mu.unsqueeze(1)).to(h.dtype)
                state[slot] = cur[-1:]
        return out
    assert h.stride(1) == 1 and state.is_contiguous() and state.dtype == torch.float32
    out = torch.empty(n, pad, ld, dtype=h.dtype, device=h.device)
    rc = _native.cuda().gb_token_shift(_p(h), _i(int(h.dtype == torch.float32)), _i(h.stride(0)), _i(width), _p(mu), _i(n), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots),
                                       _p(out), _l(pad * ld), _i(ld), _i(max_tokens), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_token_shift")
    return out


def tanh_rows(z, n: int, out_dtype=torch.bfloat16) -> torch.Tensor:
    """tanh of the first ``n`` columns of a projection result -> rows ``[T, row_width(n)]``."""
    base, f32, parts, stride, ld = split_rows(z)
    t = _n_rows(z)
    out = torch.empty(t, row_width(n, out_dtype), dtype=out_dtype, device=base.device)
    if not base.is_cuda:
        out.zero_()
        out[:, :n] = torch.tanh(whole(z)[:, :n]).to(out_dtype)
        return out
    rc = _native.cuda().gb_tanh_rows(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(out), _i(int(out_dtype == torch.float32)), _i(out.shape[1]), _i(t), _i(n), _s())
    _native.check(rc, "gb_tanh_rows")
    return out


def rwkv_ref(r, k, v, z, u, state, cu_q, seq_slots, heads, dim, vdim):
    t = r.shape[0]
    r, k, v = r.reshape(t, heads, dim), k.reshape(t, heads, dim), v.reshape(t, heads, vdim)
    w = torch.exp(-torch.exp(z)).reshape(t, heads, dim)
    bonus = (r * u.reshape(heads, dim) * k).sum(-1, keepdim=True)
    out = torch.zeros(t, heads * vdim)
    cu = cu_q.tolist()
    for s in range(len(cu) - 1):
        st = state[int(seq_slots[s])] if cu[s + 1] > cu[s] else None
        for i in range(cu[s], cu[s + 1]):
            out[i] = (torch.einsum("hde,hd->he", st, r[i]) + bonus[i] * v[i]).reshape(-1)
            st.mul_(w[i].unsqueeze(-1)).add_(k[i].unsqueeze(-1) * v[i].unsqueeze(1))
    return out


def can_fuse_decay(tokens: int, max_tokens: int, rank: int) -> bool:
    """Whether ``rwkv`` forms the decays from the middle of their low-rank projection: short portions of a few tokens (each sequence and
    head reads its part of the matrix), ranks up to 256."""
    return tokens <= 32 and max_tokens < CHUNKED_MIN_TOKENS and rank <= 256


def rwkv(rkv: torch.Tensor, z, w0: torch.Tensor, u: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, heads: int, dim: int, vdim: int,
         tokens: int, max_tokens: int = 1, w2: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``rkv [>= 3, pad, ld]``: receptances, keys and values of ``tokens`` tokens; ``z``: projection result (f32 or partial sums) whose columns, plus ``w0``, are the
    decay exponents (w = exp(-exp(z + w0))); ``u`` f32 ``[heads * dim]``.  ``w2`` (bf16 ``[heads * dim, rank]``, see ``can_fuse_decay``): ``z`` is the middle of a
    low-rank projection, and the exponents are ``w2 tanh(z) + w0``.  Returns f32 ``[tokens, heads * vdim]``."""
    gb, gf32, gparts, gstride, gld = split_rows(z)
    nq, nv = heads * dim, heads * vdim
    if not rkv.is_cuda:
        x, e = rkv[:, :tokens].float(), whole(z)
        if w2 is not None:
            e = torch.tanh(e[:, : w2.shape[1]]) @ w2.float().t()
        return rwkv_ref(x[0, :, :nq], x[1, :, :nq], x[2, :, :nv], e[:, :nq] + w0, u, state, cu_q, seq_slots, heads, dim, vdim)
    assert gf32 and state.is_contiguous() and state.dtype == torch.float32 and rkv.stride(2) == 1
    out = torch.empty(tokens, nv, dtype=torch.float32, device=rkv.device)
    ld, gs = rkv.stride(1), rkv.stride(0)
    if w2 is None and CHUNKED and max_tokens >= CHUNKED_MIN_TOKENS and can_chunk(rkv[0], dim, vdim) and gs % 8 == 0:
        lib, n_seqs = _native.cuda(), cu_q.numel() - 1
        lib.gb_gla_chunk_workspace.restype = _l
        nb = int(lib.gb_gla_chunk_workspace(_l(tokens), _i(n_seqs), _i(heads), _i(dim)))
        ws = torch.empty(nb, dtype=torch.uint8, device=rkv.device)
        rc = lib.gb_rwkv_chunk(_p(rkv), _l(gs), _i(ld), _i(tokens), _p(gb), _i(gparts), _l(gstride), _i(gld), _p(w0), _p(u), _p(state), _i(state.shape[0]), _p(cu_q),
                               _p(seq_slots), _p(out), _i(nv), _i(heads), _i(dim), _i(vdim), _i(max_tokens), _i(n_seqs), _p(ws), _l(nb), _c(_native.status_ptr()), _s())
        _native.check(rc, "gb_rwkv_chunk", n=2)
        return out
    rc = _native.cuda().gb_rwkv_step(_p(rkv), _i(int(rkv.dtype == torch.float32)), _l(gs), _i(ld), _p(gb), _i(gparts), _l(gstride), _i(gld), _p(w2),
                                     _i(w2.shape[1] if w2 is not None else 0), _p(w0), _p(u), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out), _i(nv), _i(heads),
                                     _i(dim), _i(vdim), _i(cu_q.numel() - 1), _s())
    _native.check(rc, "gb_rwkv_step")
    return out
