"""Lightning attention (linear attention with a fixed decay per head; csrc/kernels/lightning.cu, lightning_chunk.cu) and its PyTorch reference.

``S_t = decay_h S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t`` with q, k, v = SiLU of the mixer's input projection.  ``state`` is f32
``[slots, heads, dim, vdim]``, one slot per sequence, updated in place.
"""
from __future__ import annotations

import ctypes
import os

import torch

from .. import _native
from .stream import split_rows, whole

_c, _i, _l = ctypes.c_void_p, ctypes.c_int, ctypes.c_long


def _p(t):
    return _c(t.data_ptr()) if t is not None else _c(0)


def _s():
    return _c(torch.cuda.current_stream().cuda_stream)


# Launches whose longest sequence brings at least this many tokens take the chunked scan (csrc/kernels/lightning_chunk.cu): its chain has
# one link per 128 tokens, that of the token-by-token kernel one per token
CHUNKED = os.environ.get("GB_LIGHTNING_CHUNKED", "1") != "0"
CHUNKED_MIN_TOKENS = 16


def can_chunk(proj, dim: int, vdim: int, activated: bool) -> bool:
    """Whether the chunked kernel takes this projection: activated bf16 rows with a 16-byte pitch, key size up to 128."""
    return bool(activated and not hasattr(proj, "buf") and proj.is_cuda and proj.dtype == torch.bfloat16 and dim <= 128 and dim % 8 == 0 and vdim % 8 == 0
                and proj.stride(0) % 8 == 0 and proj.data_ptr() % 16 == 0)


def lightning_ref(proj, decay, state, cu_q, seq_slots, heads, dim, vdim, activated=False) -> torch.Tensor:
    y = whole(proj)[:, : 2 * heads * dim + heads * vdim]
    if not activated:
        y = torch.nn.functional.silu(y)
    t = y.shape[0]
    q, k = y[:, : heads * dim].reshape(t, heads, dim), y[:, heads * dim: 2 * heads * dim].reshape(t, heads, dim)
    v = y[:, 2 * heads * dim:].reshape(t, heads, vdim)
    out = torch.zeros(t, heads * vdim, dtype=torch.float32)
    cu = cu_q.tolist()
    for s in range(len(cu) - 1):
        if cu[s + 1] == cu[s]:
            continue
        st = state[int(seq_slots[s])]
        for i in range(cu[s], cu[s + 1]):
            st.mul_(decay.reshape(heads, 1, 1)).add_(k[i].unsqueeze(-1) * v[i].unsqueeze(1))
            out[i] = torch.einsum("hde,hd->he", st, q[i]).reshape(-1)
    return out


def lightning(proj, decay: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_slots: torch.Tensor, heads: int, dim: int, vdim: int,
              activated: bool = False, max_tokens: int = 1) -> torch.Tensor:
    """``proj``: projection result with columns ``[q heads x dim | k heads x dim | v heads x vdim | ...]``, before the activation or
    (``activated``) after it.  ``max_tokens``: tokens of the longest sequence.  Returns the heads' outputs f32 ``[T, heads * vdim]``; ``state`` is
    advanced."""
    base, f32, parts, stride, ld = split_rows(proj)
    if not base.is_cuda:
        return lightning_ref(proj, decay, state, cu_q, seq_slots, heads, dim, vdim, activated)
    t = proj.rows if hasattr(proj, "buf") else proj.shape[0]
    n_seqs = cu_q.numel() - 1
    assert state.is_contiguous() and state.dtype == torch.float32 and decay.dtype == torch.float32
    out = torch.empty(t, heads * vdim, dtype=torch.float32, device=base.device)
    if CHUNKED and max_tokens >= CHUNKED_MIN_TOKENS and (heads * vdim) % 4 == 0 and can_chunk(proj, dim, vdim, activated):
        rc = _native.cuda().gb_lightning_chunk(_p(base), _i(ld), _i(t), _p(decay), _p(state), _i(state.shape[0]), _p(cu_q), _p(seq_slots), _p(out),
                                               _i(heads * vdim), _i(heads), _i(dim), _i(vdim), _i(n_seqs), _c(_native.status_ptr()), _s())
        _native.check(rc, "gb_lightning_chunk")
        return out
    rc = _native.cuda().gb_lightning_step(_p(base), _i(f32), _i(int(not activated)), _i(parts), _l(stride), _i(ld), _p(decay), _p(state), _i(state.shape[0]), _p(cu_q),
                                          _p(seq_slots), _p(out), _i(heads * vdim), _i(heads), _i(dim), _i(vdim), _i(n_seqs), _s())
    _native.check(rc, "gb_lightning_step")
    return out
