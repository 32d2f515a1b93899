"""Latent attention (csrc/kernels/latent.cu, latent_attn.cu) and its PyTorch references: keys and values are projections of a latent per token, which
is all that is cached, next to one rotated key part for all heads.

Two forms of the same attention:

* absorbed: the key projection is applied to the query instead (``q_lat = W_uk^T q``), the softmax weights sum the latents themselves, and the value
  projection is applied to the sum.  One "head" of keys for all query heads; every token is a row of its own with its own number of keys.  Decoding
  and short portions.
* expanded: keys and values of all heads are computed from the cached latents of a sequence, then attended to head by head.  Prompts.

``LatentPlan`` says which tokens of a step take which form.  Cache rows are ``[latent | rotated key part]``, padded to 8 elements in bf16.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass, field
from typing import Dict, Optional, Sequence, Tuple

import torch

from .. import _native
from . import gemm
from .stream import row_width, split_rows, whole

_c, _i, _f, _l = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_long

# Portions of at most this many tokens take the absorbed form: expanding a sequence's cache costs about as much as this many absorbed tokens
ABSORB_TOKENS = 16


def _p(t):
    return _c(t.data_ptr()) if t is not None else _c(0)


def _s():
    return _c(torch.cuda.current_stream().cuda_stream)


@dataclass
class LatentPlan:
    """Where each token of a step goes.  Absorbed tokens have rows ``0 .. n_abs - 1`` (``m`` rows per head in the group-major buffers); the expanded
    sequences' tokens have rows ``0 .. n_exp - 1`` and their cached rows ``0 .. n_kv - 1``."""
    n_abs: int
    m: int
    tile: int
    dst: Optional[torch.Tensor] = None           # int32 [T]: absorbed row, or -1 - expanded row; None: token t is absorbed row t
    abs_tok: Optional[torch.Tensor] = None       # int32 [n_abs] token of each absorbed row (None: itself)
    abs_seq: Optional[torch.Tensor] = None       # int32 [n_abs] row of the block table (None: itself)
    abs_kv: Optional[torch.Tensor] = None        # int32 [n_abs] number of keys (None: the batch's kv_len)
    splits: int = 1
    n_exp: int = 0
    n_kv: int = 0
    seqs: Optional[torch.Tensor] = None          # int32 [S] rows of the block table of the expanded sequences
    q0: Optional[torch.Tensor] = None            # int32 [S + 1] first expanded row of each
    kv0: Optional[torch.Tensor] = None           # int32 [S + 1] first cached row of each
    exp_tok: Optional[torch.Tensor] = None       # int32 [n_exp] token of each expanded row
    tiles: Optional[torch.Tensor] = None         # int32 [tiles, 2] {sequence, first token}: 256-token tiles, longest first
    by_heads: Dict[int, Tuple] = field(default_factory=dict)

    def groups(self, heads: int, device):
        """(segment starts, segment counts, output row of every absorbed row as token * heads + head) of a product with one group per head."""
        if heads not in self.by_heads:
            h = torch.arange(heads, dtype=torch.int32)
            rows = torch.full((heads, self.m), -1, dtype=torch.int32)
            tok = self.abs_tok.cpu() if self.abs_tok is not None else torch.arange(self.n_abs, dtype=torch.int32)
            rows[:, : self.n_abs] = tok.unsqueeze(0) * heads + h.unsqueeze(1)
            self.by_heads[heads] = ((h * self.m).to(device), torch.full((heads,), self.n_abs, dtype=torch.int32, device=device), rows.reshape(-1).to(device))
        return self.by_heads[heads]


def pick_latent_splits(n: int, max_kv: int, head_tiles: int, sm_count: int = 148) -> int:
    """Key ranges per token: enough work items to fill the GPU, at least two blocks of 128 keys each."""
    blocks = max(1, (max_kv + 127) // 128)
    return max(1, min(sm_count // max(1, n * head_tiles), blocks // 2 if blocks >= 2 else 1, 64))


def make_plan(q_lens: Sequence[int], kv_lens: Optional[Sequence[int]], max_kv: int, device, decode: bool, expand: bool, heads: Sequence[int]) -> LatentPlan:
    """``decode``: every sequence brings one token (nothing is read from the lists but their length, so that a captured step can go on).  ``expand``:
    whether longer portions may take the expanded form.  ``heads``: head counts to prepare for."""
    cuda = torch.device(device).type == "cuda"
    n = len(q_lens)
    i32 = dict(dtype=torch.int32, device=device)
    tiles_of = (max(heads) + 31) // 32 if heads else 1
    if decode:
        tile = gemm.pick_tn(n)
        p = LatentPlan(n, (n + tile - 1) // tile * tile, tile, splits=pick_latent_splits(n, max_kv, tiles_of) if cuda else 1)
    else:
        dst, at, asq, akv, et, seqs, q0, kv0, tiles = [], [], [], [], [], [], [0], [0], []
        t = 0
        for s, (q, kv) in enumerate(zip(q_lens, kv_lens)):
            if expand and q > ABSORB_TOKENS:
                for x in range(0, q, 256):
                    tiles.append((kv - q + min(x + 256, q), len(seqs), x))
                dst.extend(-1 - i for i in range(q0[-1], q0[-1] + q))
                et.extend(range(t, t + q))
                seqs.append(s); q0.append(q0[-1] + q); kv0.append(kv0[-1] + kv)
            else:
                dst.extend(range(len(at), len(at) + q))
                at.extend(range(t, t + q)); asq.extend([s] * q); akv.extend(range(kv - q + 1, kv + 1))
            t += q
        tile = gemm.pick_tn(max(1, len(at)))
        tiles.sort(reverse=True)
        ten = lambda x: torch.tensor(x, **i32)
        p = LatentPlan(len(at), (len(at) + tile - 1) // tile * tile, tile, ten(dst), ten(at), ten(asq), ten(akv),
                       pick_latent_splits(len(at), max(akv), tiles_of) if cuda and at else 1, q0[-1], kv0[-1], ten(seqs), ten(q0), ten(kv0), ten(et),
                       ten([x[1:] for x in tiles]).reshape(-1, 2))
    for h in heads:
        p.groups(h, device)
    return p


# ------------------------------------------------------------------------------------------ token-wise
def rotate_ref(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, mag: float) -> torch.Tensor:
    """Neighbours (2i, 2i + 1) of ``x [T, ..., 2 n]`` turned by position * freq[i], times ``mag``."""
    a = positions.double().reshape(-1, *([1] * (x.dim() - 1))) * freq
    c, s = (torch.cos(a) * mag).float(), (torch.sin(a) * mag).float()
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).reshape(x.shape)


def latent_store(rows, positions, slots, q_norm, kv_norm, freq, mag: float, cache: torch.Tensor, q_rank: int, rank: int, rot_dim: int, eps: float, dtype,
                 col: int = 0) -> Optional[torch.Tensor]:
    """Projection rows ``[q latent | kv latent | rotated key part]`` (from column ``col`` on) -> normalised q latents ``[T, row_width(q_rank)]``; the normalised kv
    latent and the rotated key part go to cache slot ``slots[t]``.  ``kv_norm`` None: the rows hold a q latent only; ``q_rank`` 0: they hold none."""
    base, f32, parts, stride, ld = split_rows(rows)
    t = rows.rows if hasattr(rows, "buf") else rows.shape[0]
    ldq = row_width(q_rank, dtype)
    if not base.is_cuda:
        y = whole(rows)[:, col:]
        n = lambda z: z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps)
        out = None
        if q_rank:
            out = torch.zeros(t, ldq, dtype=dtype)
            out[:, :q_rank] = (n(y[:, :q_rank]) * q_norm).to(dtype)
        if kv_norm is not None:
            c = n(y[:, q_rank: q_rank + rank]) * kv_norm
            r = rotate_ref(y[:, q_rank + rank: q_rank + rank + rot_dim], positions, freq, mag)
            ok = slots >= 0
            cache[slots[ok].long(), 0, : rank + rot_dim] = torch.cat([c, r], -1)[ok].to(cache.dtype)
        return out
    out = torch.empty(t, ldq, dtype=dtype, device=base.device) if q_rank else None
    rc = _native.cuda().gb_latent_store(_c(base.data_ptr() + col * base.element_size()), _i(f32), _i(parts), _l(stride), _i(ld), _p(positions), _p(slots), _p(q_norm), _p(kv_norm), _p(freq), _f(mag), _p(out),
                                        _i(ldq), _p(cache), _i(int(dtype == torch.float32)), _l(cache.shape[0]), _i(cache.shape[2]), _i(t), _i(q_rank), _i(rank),
                                        _i(rot_dim), _f(eps), _s())
    _native.check(rc, "gb_latent_store")
    return out


def latent_q(q, positions, freq, mag: float, scale: float, dst, absorbed, expanded, heads: int, dim: int, rot_dim: int) -> None:
    """Query rows (per head ``dim`` unrotated and ``rot_dim`` rotated columns), times ``scale``, rotated, to ``absorbed = (unrotated, rotated)`` or
    ``expanded = (unrotated, rotated)``: views ``[rows, heads, width]`` whose columns behind the data are zeroed; ``dst`` as in ``LatentPlan``."""
    base, f32, parts, stride, ld = split_rows(q)
    t = q.rows if hasattr(q, "buf") else q.shape[0]
    if not base.is_cuda:
        y = whole(q)[:, : heads * (dim + rot_dim)].reshape(t, heads, dim + rot_dim)
        n, r = y[..., :dim] * scale, rotate_ref(y[..., dim:], positions, freq, mag) * scale
        d = dst.long() if dst is not None else torch.arange(t)
        for view, sel, row in ((absorbed, d >= 0, d), (expanded, d < 0, -1 - d)):
            if view is None or not bool(sel.any()):
                continue
            for to, val in zip(view, (n, r)):
                z = torch.zeros(int(sel.sum()), heads, to.shape[2], dtype=to.dtype)
                z[..., : val.shape[2]] = val[sel].to(to.dtype)
                to[row[sel]] = z
        return
    args, f32_out = [], 0
    for view in (absorbed, expanded):
        for x in (view if view is not None else (None, None)):
            if x is not None:
                assert x.stride(2) == 1
                f32_out = int(x.dtype == torch.float32)
            args += [_p(x), _l(x.stride(0) if x is not None else 0), _l(x.stride(1) if x is not None else 0), _i(x.shape[2] if x is not None else 0)]
    rc = _native.cuda().gb_latent_q(_p(base), _i(f32), _i(parts), _l(stride), _i(ld), _p(positions), _p(freq), _f(mag), _f(scale), _p(dst), *args, _i(f32_out), _i(t), _i(heads),
                                    _i(dim), _i(rot_dim), _s())
    _native.check(rc, "gb_latent_q")


def gather_latents(cache: torch.Tensor, plan: LatentPlan, block_table: torch.Tensor, page_size: int) -> torch.Tensor:
    """The cached rows of the plan's expanded sequences, in order: ``[n_kv, width]``."""
    n, _, w = cache.shape
    if not cache.is_cuda:
        out = []
        kv0 = plan.kv0.tolist()
        for i, s in enumerate(plan.seqs.tolist()):
            pos = torch.arange(kv0[i + 1] - kv0[i])
            out.append(cache[block_table[s].long()[pos // page_size] * page_size + pos % page_size, 0])
        return torch.cat(out)
    out = torch.empty(plan.n_kv, w, dtype=cache.dtype, device=cache.device)
    rc = _native.cuda().gb_latent_gather(_p(cache), _l(n), _i(w * cache.element_size()), _p(plan.kv0), _p(plan.seqs), _i(plan.seqs.numel()), _p(block_table),
                                         _i(block_table.shape[1]), _i(page_size), _p(out), _i(plan.n_kv), _s())
    _native.check(rc, "gb_latent_gather")
    return out


# ------------------------------------------------------------------------------------------ absorbed form
def attend_latents_ref(q, cache, rank, width, plan, fb, page_size, sink):
    heads, m, _ = q.shape
    out = torch.zeros(heads, m, row_width(rank, cache.dtype), dtype=q.dtype)
    seq = plan.abs_seq.tolist() if plan.abs_seq is not None else list(range(plan.n_abs))
    kv = plan.abs_kv.tolist() if plan.abs_kv is not None else fb.kv_len.tolist()
    for i in range(plan.n_abs):
        pos = torch.arange(kv[i])
        c = cache[fb.block_table[seq[i]].long()[pos // page_size] * page_size + pos % page_size, 0, :width].float()
        s = q[:, i, :width].float() @ c.t() * math.log(2.0)
        if sink is not None:
            s = torch.cat([s, (sink * math.log(2.0)).unsqueeze(1)], dim=1)
        p = torch.softmax(s, dim=-1)[:, : kv[i]]
        out[:, i, :rank] = (p @ c[:, :rank]).to(q.dtype)
    return out


def attend_latents(q: torch.Tensor, cache: torch.Tensor, rank: int, width: int, plan: LatentPlan, fb, page_size: int, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """``q [heads, m, W]`` (rows 0 .. n_abs - 1 of each head live; times scale * log2 e) against the cached rows ``[slots, 1, W]``, whose first
    ``width`` columns are keys and first ``rank`` columns values -> summed latents ``[heads, m, row_width(rank)]``."""
    heads, m, _ = q.shape
    if not q.is_cuda:
        return attend_latents_ref(q, cache, rank, width, plan, fb, page_size, sink)
    wo = row_width(rank, cache.dtype)
    out = (torch.empty if wo == rank else torch.zeros)(heads, m, wo, dtype=q.dtype, device=q.device)      # the padding meets zero weights: finite
    lib = _native.cuda()
    if q.dtype == torch.bfloat16 and lib.gb_latent_decode_heads(_i(heads), _i(width), _i(rank), _i(page_size)):
        po = pl = None
        if plan.splits > 1:
            po = torch.empty(plan.splits, plan.n_abs, heads, rank, dtype=torch.float32, device=q.device)
            pl = torch.empty(plan.splits, plan.n_abs, heads, dtype=torch.float32, device=q.device)
        rc = lib.gb_latent_decode(_p(q), _p(cache), _i(cache.shape[2]), _l(cache.shape[0]), _p(plan.abs_seq), _p(plan.abs_kv), _p(fb.kv_len), _p(fb.block_table),
                                  _i(fb.block_table.shape[1]), _i(page_size), _i(plan.n_abs), _i(heads), _i(width), _i(rank), _i(plan.splits), _p(out), _i(m), _i(wo),
                                  _p(po), _p(pl), _p(sink), _c(_native.status_ptr()), _s())
        _native.check(rc, "gb_latent_decode", n=1 if plan.splits == 1 else 2)
        return out
    rc = lib.gb_attn_latent_any(_p(q), _l(q.stride(1)), _l(q.stride(0)), _p(cache), _i(cache.shape[2]), _p(out), _l(out.stride(1)), _l(out.stride(0)),
                                _i(int(q.dtype == torch.float32)), _p(fb.cu_q), _p(fb.kv_len), _p(plan.abs_seq), _p(plan.abs_kv), _p(fb.block_table),
                                _i(fb.block_table.shape[1]), _i(page_size), _i(fb.cu_q.numel() - 1), _l(cache.shape[0]), _i(plan.n_abs), _i(heads), _i(width),
                                _i(rank), _p(sink), _s())
    _native.check(rc, "gb_attn_latent_any")
    return out


# ------------------------------------------------------------------------------------------ expanded form
def can_expand(sp) -> bool:
    """Head sizes the expanded kernel is built for: at most 128 unrotated and 64 rotated key columns, at most 128 value columns."""
    return sp.head_dim <= 128 and 0 < sp.rot_dim <= 64 and sp.v_dim <= 128 and sp.kv_rank % 8 == 0


def attend_expanded(q_n: torch.Tensor, q_r: torch.Tensor, kv: torch.Tensor, cached: torch.Tensor, rank: int, plan: LatentPlan, sink, out: torch.Tensor) -> None:
    """Causal attention of the plan's expanded rows: ``q_n [n_exp, heads, dn]`` and ``q_r [n_exp, heads, dr]`` (times scale * log2 e) against ``kv [n_kv,
    heads x dn | heads x dv]`` and the rotated key parts (columns ``rank ...`` of the gathered cache rows ``cached``) -> ``out [T, heads, dv]`` at the
    rows' tokens."""
    n, heads, dn = q_n.shape
    dr, dv = q_r.shape[2], out.shape[2]
    if not q_n.is_cuda:
        for i in range(plan.seqs.numel()):
            a, b, k0, k1 = (int(x) for x in (plan.q0[i], plan.q0[i + 1], plan.kv0[i], plan.kv0[i + 1]))
            k = torch.cat([kv[k0:k1, : heads * dn].float().reshape(-1, heads, dn), cached[k0:k1, rank: rank + dr].float().unsqueeze(1).expand(-1, heads, dr)], -1)
            s = torch.einsum("qhd,khd->hqk", torch.cat([q_n[a:b], q_r[a:b]], -1).float(), k) * math.log(2.0)
            see = torch.arange(k1 - k0).unsqueeze(0) <= torch.arange(k1 - k0 - (b - a), k1 - k0).unsqueeze(1)
            s = s.masked_fill(~see, float("-inf"))
            if sink is not None:
                s = torch.cat([s, (sink * math.log(2.0)).reshape(heads, 1, 1).expand(heads, b - a, 1)], dim=2)
            p = torch.softmax(s, dim=-1)[:, :, : k1 - k0]
            out[plan.exp_tok[a:b].long()] = torch.einsum("hqk,khd->qhd", p, kv[k0:k1, heads * dn:].float().reshape(-1, heads, dv)).to(out.dtype)
        return
    e = kv.element_size()
    rc = _native.cuda().gb_latent_prefill(_p(q_n), _p(q_r), _p(kv), _c(cached.data_ptr() + rank * e), _c(kv.data_ptr() + heads * dn * e), _i(kv.stride(0)),
                                          _i(cached.stride(0)), _i(n), _i(kv.shape[0]), _p(plan.tiles), _i(plan.tiles.shape[0]), _p(plan.q0), _p(plan.kv0),
                                          _p(plan.exp_tok), _p(out), _i(heads), _i(dn), _i(dr), _i(dv), _p(sink), _c(_native.status_ptr()), _s())
    _native.check(rc, "gb_latent_prefill")
