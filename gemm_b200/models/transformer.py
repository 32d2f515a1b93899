"""Decoder-only transformer (Qwen2 / Qwen3 dense and Qwen3-MoE) over a paged KV cache.

One ``forward`` serves prefill chunks, decode steps and mixed batches: tokens of all sequences are packed
into ``[T, hidden]`` rows, attention works from per-sequence metadata (``ForwardBatch``).  Every op is a
hand-written sm_100a kernel from ``gemm_b200.ops`` when the tensors are on a GPU; on CPU tensors the same
call sequence runs the PyTorch references, which is how the layer logic is tested without a GPU.

Layer recipe (reference: common/transformer.h:3550-4174):
  h = RMSNorm(x); qkv = h Wqkv^T (+bias); per-head QK-RMSNorm; NeoX RoPE; K/V -> paged cache;
  a = causal GQA attention; x += a Wo^T  [tensor-parallel: all-reduce]
  h = RMSNorm(x); dense: x += (SiLU(h Wg^T) * h Wu^T) Wd^T  [TP all-reduce]
                  MoE  : softmax router -> top-k -> renormalise; x += sum_k w_k FFN_k(h)  [EP dispatch / combine]
  logits = RMSNorm(x) Whead^T on the last token of every sequence.

Models described layer by layer (``ModelConfig.layer_specs``) run through the same loop: every layer names its mixer (attention with a window, kept
first tokens, a distance bias, capped scores or sinks, latent attention, lightning attention, HGRN2, Mamba-2, RWKV, minGRU, or two of them side by side)
and its feed-forward (dense or a mixture of experts) with sizes of its own, layers may be looped (every run has its own cache: ``KvCache`` is
indexed by run), and the residual stream is f32.  The feed-forward follows the mixer, or reads the same stream beside it (``parallel_ffn``).
A layer may hand on a weighted sum of all the streams so far (``depth_average``).
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass, field
from typing import List, Optional, Sequence

import torch

from .. import _native
from ..ops import attention as att
from ..ops import elementwise as ew
from ..ops import deltanet as dn
from ..ops import gemm, latent, lightning, moe, qlinear, recurrent, sampling, stream
from ..ops.mxfp8 import MxTensor
from .config import RECURRENT, LayerRun, LayerSpec, ModelConfig, MoeSpec
from .weights import LinearWeight, ModelWeights
from ..utils import profiler


@dataclass
class KvCache:
    """Paged KV storage: per layer ``k`` and ``v`` of shape ``[num_pages * page_size, Hkv_local, D]`` (bf16)."""
    k: List[torch.Tensor]
    v: List[torch.Tensor]
    page_size: int
    num_pages: int
    # Delta-Net layers of the hybrid models keep a fixed-size state per sequence slot instead of K/V pages:
    # conv[l] f32 [slots, conv_k - 1, qkv_dim], rec[l] f32 [slots, heads_v, d, d] (None for attention layers); shift[l] f32 [slots, 1, hidden]: the
    # row of the token in front (mixers that shift tokens)
    conv: Optional[List[Optional[torch.Tensor]]] = None
    rec: Optional[List[Optional[torch.Tensor]]] = None
    shift: Optional[List[Optional[torch.Tensor]]] = None
    # INT8 mode (``kv_dtype="int8"``): the pages live in ``kq`` / ``vq`` (int8 ``[slots, Hkv, D]``) with one f32 scale per slot and
    # head in ``ks`` / ``vs`` (the format of ops.attention.kv_store_q8), read directly by the INT8 decode attention kernel.  ``k`` /
    # ``v`` then name ONE bf16 staging buffer shared by all layers: the QK-norm + RoPE kernel writes a step's new rows there, the
    # prefill attention of a layer reads them there, and the store kernel quantises them into the layer's pages.
    kq: Optional[List[torch.Tensor]] = None
    vq: Optional[List[torch.Tensor]] = None
    ks: Optional[List[torch.Tensor]] = None
    vs: Optional[List[torch.Tensor]] = None

    @property
    def quantized(self) -> bool:
        return self.kq is not None

    @staticmethod
    def allocate(cfg: ModelConfig, num_pages: int, page_size: int, device, hkv_local: Optional[int] = None,
                 n_layers: Optional[int] = None, n_seq_slots: int = 64, first_layer: int = 0, kv_dtype: str = "bf16",
                 stage_pages: int = 0) -> "KvCache":
        """``kv_dtype="int8"`` keeps the pages as int8 + scales; ``stage_pages`` pages of bf16 staging (enough for the tokens of one
        forward pass, every sequence starting on a page boundary) are shared by all layers."""
        hkv = hkv_local if hkv_local is not None else cfg.n_kv_heads
        nl = n_layers if n_layers is not None else cfg.n_layers
        shape = (num_pages * page_size, hkv, cfg.head_dim)
        ssm = [cfg.is_ssm_layer(first_layer + i) for i in range(nl)]
        none = (0, hkv, cfg.head_dim)
        if cfg.is_layered:
            return KvCache._allocate_layered(cfg, num_pages, page_size, device, n_seq_slots, kv_dtype)
        if kv_dtype == "int8":
            if any(ssm) or cfg.head_dim != 128:
                raise ValueError("the INT8 KV cache is built for attention-only models with head_dim 128")
            stage = (max(stage_pages, 1) * page_size, hkv, cfg.head_dim)
            sk = torch.zeros(stage, dtype=torch.bfloat16, device=device)
            sv = torch.zeros(stage, dtype=torch.bfloat16, device=device)
            kv = KvCache([sk] * nl, [sv] * nl, page_size, num_pages)
            kv.kq = [torch.zeros(shape, dtype=torch.int8, device=device) for _ in range(nl)]
            kv.vq = [torch.zeros(shape, dtype=torch.int8, device=device) for _ in range(nl)]
            kv.ks = [torch.zeros(shape[:2], dtype=torch.float32, device=device) for _ in range(nl)]
            kv.vs = [torch.zeros(shape[:2], dtype=torch.float32, device=device) for _ in range(nl)]
            return kv
        if kv_dtype != "bf16":
            raise ValueError(f"unknown kv_dtype {kv_dtype!r}")
        kv = KvCache([torch.zeros(none if ssm[i] else shape, dtype=torch.bfloat16, device=device) for i in range(nl)],
                     [torch.zeros(none if ssm[i] else shape, dtype=torch.bfloat16, device=device) for i in range(nl)], page_size, num_pages)
        if any(ssm):
            kv.conv = [torch.zeros(n_seq_slots, cfg.ssm_d_conv - 1, cfg.ssm_qkv_dim, dtype=torch.float32, device=device) if ssm[i] else None
                       for i in range(nl)]
            kv.rec = [torch.zeros(n_seq_slots, cfg.ssm_n_heads_v, cfg.ssm_head_dim, cfg.ssm_head_dim, dtype=torch.float32, device=device)
                      if ssm[i] else None for i in range(nl)]
        return kv

    @staticmethod
    def _allocate_layered(cfg: ModelConfig, num_pages: int, page_size: int, device, n_seq_slots: int, kv_dtype: str) -> "KvCache":
        """One entry per layer RUN: K / V pages with the layer's own head sizes (attention); pages of latents and rotated key parts in ``k`` (latent
        attention; nothing for a layer that reads another's); ``rec`` f32 ``[slots, heads, dim, vdim]`` (recurrent mixers); ``conv`` f32 ``[slots, taps - 1,
        channels]`` (Mamba-2, attention behind a convolution); ``shift`` f32 ``[slots, 1, hidden]`` (RWKV)."""
        dtypes = {"bf16": torch.bfloat16, "f32": torch.float32}
        if kv_dtype not in dtypes:
            raise ValueError(f"models described layer by layer keep a bf16 or f32 KV cache, not {kv_dtype!r}")
        dt = dtypes[kv_dtype]
        kv = KvCache([], [], page_size, num_pages)
        kv.rec, kv.conv, kv.shift = [], [], []
        f32 = dict(dtype=torch.float32, device=device)
        for run in cfg.layer_runs():
            spec = cfg.layer_specs[run.layer]
            sp, rows, heads, dkp, dvp = spec.paged, 0, 1, 0, 0
            if sp is not None and sp.mixer == "latent":
                rows, dkp = (num_pages * page_size if sp.kv_from < 0 else 0), stream.row_width(sp.kv_rank + sp.rot_dim, dt)
            elif sp is not None:
                rows, heads, (dkp, dvp) = num_pages * page_size, sp.n_kv_heads, att.cache_head_dims(sp.head_dim, sp.v_dim, dt)
            kv.k.append(torch.zeros(rows, heads, dkp, dtype=dt, device=device))
            kv.v.append(torch.zeros(rows, heads, dvp, dtype=dt, device=device))
            rec = next((x for x in spec.mixers if x.mixer in RECURRENT), None)
            conv = next((x for x in spec.mixers if x.conv_taps), None)
            kv.rec.append(torch.zeros(n_seq_slots, rec.n_heads, rec.head_dim, rec.v_dim, **f32) if rec is not None else None)
            kv.conv.append(torch.zeros(n_seq_slots, conv.conv_taps - 1, conv.conv_channels, **f32) if conv is not None else None)
            kv.shift.append(torch.zeros(n_seq_slots, 1, cfg.hidden, **f32) if rec is not None and rec.mixer == "rwkv" else None)
        for name in ("rec", "conv", "shift"):
            if not any(t is not None for t in getattr(kv, name)):
                setattr(kv, name, None)
        return kv

    def recurrent(self, li: int) -> List[torch.Tensor]:
        """The per-slot state tensors of entry ``li`` (empty for attention layers)."""
        return [t[li] for t in (self.conv, self.rec, self.shift) if t is not None and t[li] is not None]

    def reset_slots(self, slots) -> None:
        """Zero the recurrent state of the given sequence slots (a new sequence starts from an empty state)."""
        if self.rec is None and self.conv is None:
            return
        idx = torch.as_tensor(list(slots), dtype=torch.long, device=self.k[0].device)
        for li in range(len(self.k)):
            for t in self.recurrent(li):
                t[idx] = 0

    def copy_pages(self, pairs) -> None:
        """``page dst <- page src`` for every ``(src, dst)`` of ``pairs`` in every layer's K and V: the copy-on-write step of a
        forked sequence (``serve.scheduler.KvBlockManager.fork`` names the tail page to copy)."""
        pairs = [p for p in pairs if p is not None]
        if not pairs:
            return
        dev = self.k[0].device
        src = torch.tensor([p[0] for p in pairs], dtype=torch.int32, device=dev)
        dst = torch.tensor([p[1] for p in pairs], dtype=torch.int32, device=dev)
        if self.quantized:
            for t in list(self.kq) + list(self.vq) + list(self.ks) + list(self.vs):
                pg = t.view(self.num_pages, self.page_size, *t.shape[1:])
                pg[dst.long()] = pg[src.long()]
            return
        for t in list(self.k) + list(self.v):
            if t.numel() == 0:
                continue
            if not t.is_cuda:
                pg = t.view(self.num_pages, self.page_size, *t.shape[1:])
                pg[dst.long()] = pg[src.long()]
                continue
            page_bytes = self.page_size * t.shape[1] * t.shape[2] * t.element_size()
            rc = _native.cuda().gb_kv_copy_pages(ctypes.c_void_p(t.data_ptr()), ctypes.c_void_p(src.data_ptr()), ctypes.c_void_p(dst.data_ptr()),
                                                 ctypes.c_int(len(pairs)), ctypes.c_int(self.num_pages), ctypes.c_long(page_bytes),
                                                 ctypes.c_void_p(torch.cuda.current_stream().cuda_stream))
            _native.check(rc, "gb_kv_copy_pages")

    def nbytes(self) -> int:
        if self.quantized:
            return sum(t.numel() * t.element_size() for t in list(self.kq) + list(self.vq) + list(self.ks) + list(self.vs)) + \
                2 * self.k[0].numel() * 2
        tot = sum(t.numel() * t.element_size() for t in list(self.k) + list(self.v))
        return tot + sum(t.numel() * 4 for li in range(len(self.k)) for t in self.recurrent(li))


@dataclass
class ForwardBatch:
    ids: torch.Tensor              # int32 [T]
    positions: torch.Tensor        # int32 [T]
    slots: torch.Tensor            # int32 [T] cache slot of every token (-1 = do not store)
    cu_q: torch.Tensor             # int32 [B+1]
    kv_len: torch.Tensor           # int32 [B] length including this step's tokens
    block_table: torch.Tensor      # int32 [B, max_pages]
    work: torch.Tensor             # int32 [n_work, 4] attention work list
    logit_rows: torch.Tensor       # int32/int64 [B'] rows of T whose logits are wanted
    num_splits: int = 1
    embeds: Optional[torch.Tensor] = None   # bf16 [T, H]: injected embeddings instead of ids (vision tokens)
    n_tokens: int = 0
    seq_slots: Optional[torch.Tensor] = None   # int32 [B] state slot of every sequence (Delta-Net layers); default 0..B-1
    positions3: Optional[torch.Tensor] = None  # int32 [3, T] (t, h, w) positions for M-RoPE; default: all three = positions
    is_decode: bool = False                    # every sequence contributes exactly one token (selects the decode attention kernel)
    deepstack: Optional[torch.Tensor] = None   # bf16 [n_deepstack, T, H] added to the stream after the first layers (Qwen3-VL)
    # INT8 KV cache: where a step's new K / V rows sit in the bf16 staging buffer, and (prefill) the block table of the staged sequences
    stage_slots: Optional[torch.Tensor] = None # int32 [T]
    stage_bt: Optional[torch.Tensor] = None    # int32 [B, pages]
    # attention work lists by head shape (models whose layers differ in it): (query heads, KV heads, span) -> (work, KV splits)
    plans: Optional[dict] = None
    q_lens: Optional[List[int]] = None             # host copies of the chunk and sequence lengths, from which a missing plan is made
    kv_lens: Optional[List[int]] = None
    # context-parallel prefill: the cache slots whose K / V rows this rank contributes to the per-layer all-gather (staging order)
    cp_send_slots: Optional[torch.Tensor] = None   # int64 [p_local * page_size]

    @staticmethod
    def build(q_lens: Sequence[int], ctx_lens: Sequence[int], ids, block_table: torch.Tensor, page_size: int, hq: int, hkv: int,
              device, num_splits: int = 1, all_logits: bool = False, seq_slots: Optional[Sequence[int]] = None,
              stage: bool = False) -> "ForwardBatch":
        """Host-side assembly from per-sequence chunk lengths and the lengths already cached.  ``stage`` (INT8 KV cache) also lays the
        step's tokens out in the staging buffer: a decode step row by row, a prefill step with every sequence on a page boundary."""
        b = len(q_lens)
        pos, slots, cu = [], [], [0]
        bt = block_table.cpu()
        for s in range(b):
            for i in range(q_lens[s]):
                p = ctx_lens[s] + i
                pos.append(p)
                slots.append(int(bt[s, p // page_size]) * page_size + p % page_size)
            cu.append(cu[-1] + q_lens[s])
        t = cu[-1]
        rows = list(range(t)) if all_logits else [cu[s + 1] - 1 for s in range(b) if q_lens[s] > 0]
        i32 = dict(dtype=torch.int32, device=device)
        ids_t = ids.to(device=device, dtype=torch.int32) if torch.is_tensor(ids) else torch.tensor(ids, **i32)
        st_slots = st_bt = None
        if stage:
            if all(q == 1 for q in q_lens):
                st_slots = torch.arange(t, **i32)
            else:
                if any(c != 0 for c in ctx_lens):
                    raise NotImplementedError("INT8 KV cache: a prefill chunk must start its sequence (the attention of a later chunk "
                                              "would have to read the quantised history; raise max_prefill_tokens or use the bf16 cache)")
                pages = [(q + page_size - 1) // page_size for q in q_lens]
                first, ss = [0], []
                for s in range(b):
                    ss.extend(first[s] * page_size + i for i in range(q_lens[s]))
                    first.append(first[s] + pages[s])
                st_slots = torch.tensor(ss, **i32)
                st_bt = torch.zeros(b, max(max(pages), 1), dtype=torch.int32)
                for s in range(b):
                    st_bt[s, : pages[s]] = torch.arange(first[s], first[s] + pages[s], dtype=torch.int32)
                st_bt = st_bt.to(device)
        return ForwardBatch(stage_slots=st_slots, stage_bt=st_bt, plans={}, q_lens=list(q_lens), kv_lens=[c + q for c, q in zip(ctx_lens, q_lens)],
                            ids=ids_t, positions=torch.tensor(pos, **i32), slots=torch.tensor(slots, **i32),
                            cu_q=torch.tensor(cu, **i32), kv_len=torch.tensor([c + q for c, q in zip(ctx_lens, q_lens)], **i32),
                            block_table=block_table.to(device=device, dtype=torch.int32),
                            work=att.build_work(q_lens, hq, hkv, num_splits).to(device),
                            logit_rows=torch.tensor(rows, dtype=torch.int64, device=device), num_splits=num_splits, n_tokens=t,
                            seq_slots=torch.tensor(list(seq_slots) if seq_slots is not None else list(range(b)), **i32),
                            is_decode=(b > 0 and all(q == 1 for q in q_lens)))


def attention_plan(q_lens: Sequence[int], max_kv: int, hq: int, hkv: int, span: int, device, decode: bool):
    """(work list on the device, KV splits) of the tcgen05 attention kernels for one head shape; ``span`` is the most keys a position
    sees (0 = no limit)."""
    splits = att.pick_splits(len(q_lens), hkv, min(max_kv, span + 128) if span else max_kv) if decode and torch.device(device).type == "cuda" else 1
    return att.build_work(q_lens, hq, hkv, splits).to(device), splits


# K-split partial sums for decode-sized row projections (GB_SPLIT_PROJ=0 switches them off)
SPLIT_PROJ = os.environ.get("GB_SPLIT_PROJ", "1") != "0"


FUSE_ATTN_QUANT = os.environ.get("GB_FUSE_ATTN_QUANT", "1") != "0"


# mixers and feed-forward that read the same stream as branches of a captured decode step (GB_BRANCHES=0: one after the other)
BRANCHES = os.environ.get("GB_BRANCHES", "1") != "0"


PAIR_DOWN = os.environ.get("GB_PAIR_DOWN", "1") != "0"


class SingleProcess:
    """Parallel context of an unsharded model: every collective is the identity."""
    tp_size = 1
    tp_rank = 0
    ep_size = 1
    ep_rank = 0

    def tp_all_reduce(self, x: torch.Tensor) -> torch.Tensor:
        return x

    def row_linear(self, lw: "LinearWeight", x: torch.Tensor, x_mx=None):
        """Row-parallel projection (o_proj / down_proj).  Returns the residual update: a tensor, or an object that
        ``add_norm`` / ``materialize`` know how to finish (a reduction still in flight)."""
        return apply_linear_split(lw, x, x_mx)

    def add_norm(self, delta, weight: torch.Tensor, eps: float, residual: Optional[torch.Tensor], **kw):
        """``residual += delta`` (if a residual is given) followed by RMSNorm; see ``ops.elementwise.rmsnorm``."""
        return ew.rmsnorm(delta, weight, eps, residual=residual, **kw)

    def materialize(self, delta) -> torch.Tensor:
        return delta.materialize() if hasattr(delta, "materialize") else delta

    def moe_ffn(self, model: "Transformer", lw, h: torch.Tensor, h_mx=None) -> Optional[torch.Tensor]:
        return None            # None -> the model runs its local MoE path


def apply_linear(lw: LinearWeight, x: torch.Tensor, x_mx: Optional[MxTensor] = None, out_dtype=torch.bfloat16) -> torch.Tensor:
    """``x W^T (+ bias)`` in the weight's format; ``x_mx`` is an already-quantised copy of ``x`` if the caller has one."""
    if lw.is_quant:                       # ggml blocks in HBM: fused dequant-GEMV (<= 4 tokens) or dequant-GEMM
        return qlinear.linear(x, lw.q, bias=lw.bias, out_dtype=out_dtype)
    if lw.fmt == "bf16":
        return gemm.linear(x, lw.w, bias=lw.bias, out_dtype=out_dtype, w_tiled=lw.tiled)
    xm = x_mx if x_mx is not None else ew.mx_quantize(x, sf_layout=32 if x.shape[0] <= 32 else 128)
    y = gemm.linear_mx(xm, lw.mx, out_dtype=out_dtype, bias=lw.bias)
    return y


def apply_linear_split(lw: LinearWeight, x: torch.Tensor, x_mx: Optional[MxTensor] = None):
    """``apply_linear`` for a projection whose result goes into the residual stream: a decode-sized MXFP8 projection with few
    output tiles (o_proj: 16 tiles of 128 rows, 32 k-steps each) is cut along K so that it fills the GPU, and the partial sums
    are left for the residual add + RMSNorm kernel that follows."""
    if lw.is_quant:
        if x.is_cuda and x.shape[0] <= qlinear.GEMV_MAX_TOKENS:
            return qlinear.gemv_partials(x, lw.q, bias=lw.bias)      # K-split partial sums, added by the consumer
        if x.is_cuda:
            sp = qlinear.pick_gemm_splits(lw.q.rows, lw.q.k, x.shape[0])
            if sp > 1:
                return qlinear.gemm_partials(x, lw.q, sp, bias=lw.bias)
        return apply_linear(lw, x, x_mx)
    if lw.fmt == "bf16" and SPLIT_PROJ and x is not None and x.is_cuda and lw.n % 128 == 0:
        sp = gemm.pick_partials(lw.n, x.shape[0], lw.k, False)
        if sp > 1:
            return gemm.linear_partials(x, lw.w, sp, bias=lw.bias, w_tiled=lw.tiled)
        return apply_linear(lw, x, x_mx)
    if lw.fmt != "bf16" and SPLIT_PROJ:
        xm = x_mx if x_mx is not None else (ew.mx_quantize(x, sf_layout=32 if x.shape[0] <= 32 else 128) if x.is_cuda else None)
        if xm is not None and xm.data.is_cuda:
            sp = gemm.pick_partials(lw.mx.rows, xm.rows, lw.mx.k, True)
            if sp > 1:
                return gemm.linear_mx_partials(xm, lw.mx, sp, bias=lw.bias)
            return gemm.linear_mx(xm, lw.mx, bias=lw.bias)
    return apply_linear(lw, x, x_mx)


def apply_linear_stream(lw: LinearWeight, x: torch.Tensor):
    """A projection whose result joins an f32 stream or an f32 computation: f32, or K-split partial sums for the consumer to add."""
    if lw.fmt == "f32":
        return gemm.linear_f32(x, lw.w, bias=lw.bias)
    sp = gemm.pick_partials(lw.n, x.shape[0], (lw.k + 63) // 64 * 64, False) if SPLIT_PROJ and x.is_cuda else 1
    if sp > 1:
        return gemm.linear_partials(x, lw.w, sp, bias=lw.bias, w_tiled=lw.tiled)
    return gemm.linear(x, lw.w, bias=lw.bias, out_dtype=torch.float32, w_tiled=lw.tiled)


def apply_linear_rows(lw: LinearWeight, x: torch.Tensor):
    """A projection for a token-wise kernel: f32 (or K-split partial sums) for decode-sized batches, bf16 rows for prefill-sized ones."""
    return apply_linear_mixer(lw, x)[0]


def apply_linear_mixer(lw: LinearWeight, x: torch.Tensor, silu_rows: int = 0):
    """The input projection of a mixer: as ``apply_linear_stream`` for decode-sized batches (the mixer's kernels add the partial sums), bf16
    rows for prefill-sized ones, with SiLU on the first ``silu_rows`` features.  Returns ``(result, whether SiLU was applied)``."""
    if lw.fmt == "f32" or x.shape[0] <= 64:
        return apply_linear_stream(lw, x), False
    return gemm.linear(x, lw.w, bias=lw.bias, w_tiled=lw.tiled, silu_rows=silu_rows), silu_rows > 0


def expert_gate_up_mx(x_q: torch.Tensor, x_sf: torch.Tensor, w13: LinearWeight, n_w_groups: int, seg_start: torch.Tensor,
                      seg_count: torch.Tensor, tn: int, hq: torch.Tensor, hsf: torch.Tensor, row_valid: Optional[torch.Tensor] = None,
                      extras=None, w_groups: Optional[int] = None, scratch: Optional[torch.Tensor] = None) -> None:
    """MXFP8 expert gate/up projection + SiLU(gate) * up + re-quantisation into ``hq`` / ``hsf`` (the down projection's input).

    Decode-sized batches (token tile 32) run the two-accumulator GEMM with the activation and the quantiser in its epilogue.
    Prefill-sized batches (token tile 128) run one plain GEMM over the stacked [gate; up] rows and a fused SiLU*up+quantise
    kernel: two 128-token accumulators cannot be double-buffered in TMEM, so the fused epilogue would serialise with the
    tensor-core work there (measured 2.1 ms against 0.8 ms for 16384 tokens x top-8)."""
    two_i, hid = w13.rows_per_group, w13.k
    wv = w13.mx.data.view(n_w_groups, two_i, hid)
    if tn == 32 or not x_q.is_cuda:
        gemm.grouped_linear(x_q, wv, seg_start, seg_count, tn, out=hq, dual=True, sfa=w13.mx.sf, sfb=x_sf, quant_out=True, out_sf=hsf,
                            extras=extras, w_groups=w_groups, w_tiled=w13.mx.tiled)
        return
    gu = scratch if scratch is not None else torch.empty(x_q.shape[0], two_i, dtype=torch.bfloat16, device=x_q.device)
    gemm.grouped_linear(x_q, wv, seg_start, seg_count, tn, out=gu, sfa=w13.mx.sf, sfb=x_sf, extras=extras, w_groups=w_groups,
                        w_tiled=w13.mx.tiled)
    ew.silu_mul_quant(gu, hq, hsf, row_valid, sf_layout=tn)


class Transformer:
    def __init__(self, weights: ModelWeights, kv: KvCache, par=None):
        self.w = weights
        self.cfg = weights.cfg
        self.kv = kv
        self.par = par if par is not None else SingleProcess()
        cfg = self.cfg
        self.hq_local = cfg.n_heads // weights.tp_size
        self.hkv_local = max(1, cfg.n_kv_heads // weights.tp_size)
        self.q_scale = ew.softmax_scale_log2(cfg.head_dim)
        self.mx = weights.fmt == "mxfp8"
        self.runs = cfg.layer_runs() if cfg.is_layered else [LayerRun(i) for i in range(len(weights.layers))]
        # models described layer by layer: f32 stream, activations in the weights' own width
        self.stream_f32 = cfg.is_layered
        self.act_dtype = torch.float32 if weights.fmt == "f32" else torch.bfloat16
        rd = cfg.rope_dim or cfg.head_dim
        if cfg.mrope_sections and sum(cfg.mrope_sections) > 0:
            rd = 2 * sum(cfg.mrope_sections)           # the rotary width under M-RoPE (common/transformer.h:1229-1232)
        self.rope_dim = rd
        self.rope_table = ew.rope_table(min(max(cfg.max_seq_len, 4096), 65536), rd, cfg.rope_theta, weights.embed.device) \
            if weights.embed.is_cuda and not cfg.is_layered else None
        self.mixer_blocks = {"attention": self.masked_attention_block, "lightning": self.lightning_block, "mamba2": self.mamba2_block, "hgrn2": self.hgrn2_block,
                             "latent": self.latent_block, "rwkv": self.rwkv_block, "mingru": self.mingru_block}
        self._branches: List = []      # streams of a captured step's branches
        self.snapshots = {}            # layer -> hidden rows captured after that layer (debug / DeepStack)
        self.snapshot_layers: Sequence[int] = ()

    # ------------------------------------------------------------------------------------------------
    def attention_block(self, li: int, lw, h: torch.Tensor, h_mx: Optional[MxTensor], fb: ForwardBatch) -> torch.Tensor:
        cfg = self.cfg
        # decode-sized batches: the projection is cut along K and the rope kernel sums the partials (not with an output gate,
        # whose columns are read again below)
        qkv = apply_linear(lw.wqkv, h, h_mx) if cfg.attn_output_gate else apply_linear_split(lw.wqkv, h, h_mx)
        if self.kv.quantized:
            return self._attention_q8(li, lw, qkv, fb)
        if getattr(self.par, "cp_world", 1) > 1:
            return self._attention_cp(li, lw, qkv, fb)
        q = ew.qk_norm_rope(qkv, fb.positions, fb.slots, lw.q_norm, lw.k_norm, self.kv.k[li], self.kv.v[li], self.hq_local,
                            self.hkv_local, cfg.head_dim, cfg.rope_theta, cfg.rms_eps, self.q_scale, self.rope_dim, table=self.rope_table,
                            positions3=fb.positions3, sections=cfg.mrope_sections)
        if (self.mx and lw.wo.fmt != "bf16" and not cfg.attn_output_gate and FUSE_ATTN_QUANT
                and att.can_decode_mx(q, self.hkv_local, fb.num_splits, fb.is_decode)):
            # decode: the attention kernel emits the MXFP8 operand of the output projection itself
            a_mx = att.attention_decode_mx(q, self.kv.k[li], self.kv.v[li], fb.cu_q, fb.kv_len, fb.block_table, self.kv.page_size, fb.work,
                                           window=cfg.sliding_window, sf_layout=32 if q.shape[0] <= 32 else 128, num_splits=fb.num_splits)
            return self.par.row_linear(lw.wo, None, a_mx)
        if self.mx and lw.wo.fmt != "bf16" and not cfg.attn_output_gate and FUSE_ATTN_QUANT and att.can_attention_mx(q, fb.num_splits):
            a_mx = att.attention_mx(q, self.kv.k[li], self.kv.v[li], fb.cu_q, fb.kv_len, fb.block_table, self.kv.page_size, fb.work,
                                    causal=True, window=cfg.sliding_window, sf_layout=32 if q.shape[0] <= 32 else 128)
            return self.par.row_linear(lw.wo, None, a_mx)
        a = att.attention(q, self.kv.k[li], self.kv.v[li], fb.cu_q, fb.kv_len, fb.block_table, self.kv.page_size, fb.work,
                          num_splits=fb.num_splits, causal=True, window=cfg.sliding_window, decode=fb.is_decode)
        a2 = a.reshape(a.shape[0], self.hq_local * cfg.head_dim)
        if cfg.attn_output_gate:
            g0 = (self.hq_local + 2 * self.hkv_local) * cfg.head_dim
            dn.gate_mul(a2, qkv[:, g0: g0 + self.hq_local * cfg.head_dim])
        return self.par.row_linear(lw.wo, a2)

    def _attention_cp(self, li: int, lw, qkv, fb: ForwardBatch) -> torch.Tensor:
        """Attention under context parallelism (``parallel.context.ContextParallel`` as the parallel context).  The cache holds
        this rank's pages only; ``fb.slots`` is -1 for a token another rank stores.  Decode: flash partials over the local shard,
        merged across the ranks.  Prefill: the rank's own tokens attend over the all-gathered K / V rows of the prompt."""
        cfg, kv = self.cfg, self.kv
        q = ew.qk_norm_rope(qkv, fb.positions, fb.slots, lw.q_norm, lw.k_norm, kv.k[li], kv.v[li], self.hq_local, self.hkv_local,
                            cfg.head_dim, cfg.rope_theta, cfg.rms_eps, self.q_scale, self.rope_dim, table=self.rope_table,
                            positions3=fb.positions3, sections=cfg.mrope_sections)
        if fb.is_decode:
            a = self.par.attention(q, kv.k[li], kv.v[li], fb.cu_q, fb.kv_len, fb.block_table, kv.page_size, fb.work,
                                   num_splits=fb.num_splits, decode=True)
        else:
            if fb.cp_send_slots is None:
                raise ValueError("a context-parallel prefill needs the forward batch of ContextParallel.build_prefill")
            kg, vg = self.par.gather_kv(kv.k[li], kv.v[li], fb.cp_send_slots)
            a = att.attention(q, kg, vg, fb.cu_q, fb.kv_len, fb.block_table, kv.page_size, fb.work, num_splits=1, causal=True)
        a2 = a.reshape(a.shape[0], self.hq_local * cfg.head_dim)
        if cfg.attn_output_gate:
            g0 = (self.hq_local + 2 * self.hkv_local) * cfg.head_dim
            dn.gate_mul(a2, qkv[:, g0: g0 + self.hq_local * cfg.head_dim])
        return self.par.row_linear(lw.wo, a2)

    def _attention_q8(self, li: int, lw, qkv, fb: ForwardBatch) -> torch.Tensor:
        """Attention with the INT8 KV cache: the new K / V rows go through the bf16 staging buffer (QK-norm + RoPE write them
        there), are quantised into the layer's pages, and a decode step reads the INT8 pages directly; a prefill step attends over
        the staged bf16 rows of its own tokens."""
        cfg, kv = self.cfg, self.kv
        if fb.stage_slots is None:
            raise ValueError("the INT8 KV cache needs a ForwardBatch built with stage=True")
        if fb.stage_slots.numel() > kv.k[li].shape[0] or (fb.stage_bt is not None and int(fb.stage_bt.shape[1]) * kv.page_size > kv.k[li].shape[0]):
            raise ValueError("the forward pass has more tokens than the KV staging buffer holds")
        q = ew.qk_norm_rope(qkv, fb.positions, fb.stage_slots, lw.q_norm, lw.k_norm, kv.k[li], kv.v[li], self.hq_local, self.hkv_local,
                            cfg.head_dim, cfg.rope_theta, cfg.rms_eps, self.q_scale, self.rope_dim, table=self.rope_table,
                            positions3=fb.positions3, sections=cfg.mrope_sections)
        att.kv_store_q8(kv.k[li], kv.v[li], fb.stage_slots, fb.slots, kv.kq[li], kv.vq[li], kv.ks[li], kv.vs[li])
        if fb.is_decode:
            a = att.attention_decode_q8(q, kv.kq[li], kv.vq[li], kv.ks[li], kv.vs[li], fb.kv_len, fb.block_table, kv.page_size,
                                        num_splits=fb.num_splits, window=cfg.sliding_window)
        else:
            if fb.stage_bt is None:
                raise NotImplementedError("INT8 KV cache: steps of several tokens per sequence on top of cached history (speculative "
                                          "verification, later prefill chunks) are not built")
            a = att.attention(q, kv.k[li], kv.v[li], fb.cu_q, fb.kv_len, fb.stage_bt, kv.page_size, fb.work, num_splits=1, causal=True,
                              window=cfg.sliding_window)
        a2 = a.reshape(a.shape[0], self.hq_local * cfg.head_dim)
        if cfg.attn_output_gate:
            g0 = (self.hq_local + 2 * self.hkv_local) * cfg.head_dim
            dn.gate_mul(a2, qkv[:, g0: g0 + self.hq_local * cfg.head_dim])
        return self.par.row_linear(lw.wo, a2)

    def ssm_block(self, li: int, lw, h: torch.Tensor, h_mx: Optional[MxTensor], fb: ForwardBatch) -> torch.Tensor:
        """Gated Delta-Net layer: projections -> causal conv + SiLU -> recurrence + gated norm -> output projection."""
        cfg, ssm = self.cfg, lw.ssm
        qd = cfg.ssm_qkv_dim
        proj = apply_linear(ssm.w_in, h, h_mx)                        # [T, qkv_dim + d_inner]
        ab = moe.router_logits(h, ssm.w_ab)                           # f32 [T, 2 * heads_v]
        slots = fb.seq_slots if fb.seq_slots is not None else torch.arange(fb.cu_q.numel() - 1, dtype=torch.int32, device=h.device)
        conv = dn.conv_silu(proj[:, :qd], ssm.conv_w, self.kv.conv[li], fb.cu_q, slots)
        out = dn.deltanet(conv, proj[:, qd:], ab, ssm.a, ssm.dt_bias, ssm.norm, self.kv.rec[li], fb.cu_q, slots, cfg.ssm_n_heads_k,
                          cfg.ssm_n_heads_v, cfg.ssm_head_dim, cfg.rms_eps)
        return self.par.row_linear(ssm.w_out, out)

    def attention_plans(self, q_lens: Sequence[int], max_kv: int, device, decode: bool) -> dict:
        """Work lists for every head shape of the model (made up front where nothing may be allocated later: a captured decode step)."""
        plans = {}
        if any(sp.mixer == "latent" for sp in (self.cfg.layer_specs or ())):
            plans["latent"] = self.latent_plan(q_lens, [max_kv] * len(q_lens), max_kv, device, decode)
        for sp in (x for spec in (self.cfg.layer_specs or ()) for x in spec.mixers):
            if sp.mixer == "attention" and (sp.n_heads, sp.n_kv_heads, sp.span) not in plans:
                plans[(sp.n_heads, sp.n_kv_heads, sp.span)] = attention_plan(q_lens, max_kv, sp.n_heads, sp.n_kv_heads, sp.span, device, decode)
            if sp.mixer == "rwkv" and "shift" not in plans:
                plans["shift"] = self.shift_plan(sum(q_lens), device)
        return plans

    @staticmethod
    def shift_plan(t: int, device):
        """(rows per mix, segment starts, segment counts) of the grouped product over four mixes of ``t`` tokens."""
        pad = recurrent.shift_pad(t)
        return pad, torch.arange(4, dtype=torch.int32, device=device) * pad, torch.full((4,), t, dtype=torch.int32, device=device)

    def masked_attention_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """Attention of a layer described by ``LayerSpec``: biased projection -> norm of Q and K (per head or over all of them) or convolution and rotation, cache
        store -> attention with a window, kept first tokens and distance bias, capped scores, a sink -> gate -> output projection.  ``li`` is the
        run, which has its own cache."""
        kc, vc, eps = self.kv.k[li], self.kv.v[li], self.cfg.rms_eps
        qkv, _ = apply_linear_mixer(lw.wqkv, h)
        hq, hkv, d, dv = sp.n_heads, sp.n_kv_heads, sp.head_dim, sp.v_dim
        # capped scores: the queries carry scale / cap, and the kernels multiply by cap * log2 e behind the tanh
        scale = (sp.scale or d ** -0.5) * (1.0 / sp.softcap if sp.softcap else att.LOG2E)
        if sp.rotary is not None:
            q = stream.conv_rotary(qkv, self.rotary_table(lw, sp, fb), fb.slots, lw.conv_w, self.kv.conv[li], fb.cu_q, fb.seq_slots, kc, vc, hq, hkv, d, scale, self.most_tokens(fb))
        elif sp.qk_norm_rows:
            q = stream.qk_rows(qkv, fb.slots, lw.q_norm, lw.k_norm, kc, vc, hq, hkv, d, dv, eps, scale)
        else:
            q = stream.qk_unit(qkv, fb.slots, kc, vc, hq, hkv, d, dv, eps, scale, unit=sp.qk_unit, positions=fb.positions, temp=(sp.temp_coef, sp.temp_every))
        key = (hq, hkv, sp.span)
        if fb.plans is None:
            fb.plans = {}
        if key not in fb.plans and q.is_cuda:
            fb.plans[key] = attention_plan(fb.q_lens, max(fb.kv_lens), *key, q.device, fb.is_decode)
        a = att.attention_masked(q, kc, vc, fb.cu_q, fb.kv_len, fb.block_table, self.kv.page_size, window=sp.window, keep_first=sp.keep_first,
                                 bias=lw.rel_bias, plan=fb.plans.get(key), decode=fb.is_decode, softcap=sp.softcap, sink=lw.sink, log_bias=lw.log_bias)
        if sp.out_gate:
            a = stream.sigmoid_gate(a, qkv, sp.q_dim + hkv * (d + dv), dv)
        return apply_linear_stream(lw.wo, a.reshape(a.shape[0], -1))

    @staticmethod
    def most_tokens(fb: ForwardBatch) -> int:
        """Tokens of the batch's longest sequence."""
        return max(fb.q_lens) if fb.q_lens else 1

    def rotary_table(self, lw, sp: LayerSpec, fb: ForwardBatch) -> torch.Tensor:
        """cos and sin of the step's positions, formed once per forward pass and kind of rotation."""
        key = tuple(vars(sp.rotary).values())
        if key not in self._rotary:
            self._rotary[key] = stream.rotary_table(fb.positions, lw.rot_freq, sp.rotary.magnitude)
        return self._rotary[key]

    def rwkv_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """RWKV-style time mixing: five mixes with the token in front -> four projections as one grouped product, low-rank decay (f32) -> recurrence with a bonus
        for the current token -> RMSNorm per head * SiLU(gate) -> output projection."""
        w, t, most, n = lw.rwkv, h.shape[0], self.most_tokens(fb), sp.q_dim
        if fb.plans is None:
            fb.plans = {}
        if "shift" not in fb.plans:
            fb.plans["shift"] = self.shift_plan(t, h.device)
        pad, seg, cnt = fb.plans["shift"]
        mix = recurrent.token_shift(h, self.cfg.hidden, w.mu, self.kv.shift[li], fb.cu_q, fb.seq_slots, pad, most)
        ld = stream.row_width(n, self.act_dtype)
        if w.w_in.fmt == "f32":
            rkvg = torch.empty(4, pad, ld, dtype=torch.float32, device=h.device)
            gemm.batched_linear_f32(mix[:4], w.w_in.w.view(4, n, -1), rkvg)
        else:
            # decode-sized batches keep the projections in f32
            rkvg = torch.empty(4, pad, ld, dtype=torch.float32 if t <= 64 else torch.bfloat16, device=h.device)
            gemm.grouped_linear(mix[:4].view(4 * pad, -1), w.w_in.w.view(4, w.w_in.rows_per_group, -1), seg, cnt, recurrent.shift_tile(pad), out=rkvg.view(4 * pad, ld),
                                n_out=n, w_tiled=w.w_in.tiled)
        z, w2 = apply_linear_stream(w.w1, mix[4, :t]), None
        if w.w2_rows is not None and recurrent.can_fuse_decay(t, most, sp.decay_rank):
            w2 = w.w2_rows
        else:
            z = apply_linear_stream(w.w2, recurrent.tanh_rows(z, sp.decay_rank, self.act_dtype))
        o = recurrent.rwkv(rkvg, z, w.w0, w.u, self.kv.rec[li], fb.cu_q, fb.seq_slots, sp.n_heads, sp.head_dim, sp.v_dim, t, most, w2)
        y = stream.part_norm(o, w.norm, sp.n_heads, self.cfg.rms_eps, rkvg[3, :t], 0, self.act_dtype, gate_after=True)
        return apply_linear_stream(w.w_out, y)

    def branch(self, i: int, x: torch.Tensor, fn):
        """``fn()`` as branch ``i`` of the graph while a decode step is captured, beside what the current stream does until ``join_branch(i)``; at once otherwise.
        What the branch reads must stay alive until then: memory is handed out again in the order of the stream that asked for it."""
        if not (BRANCHES and x.is_cuda and torch.cuda.is_current_stream_capturing()):
            return fn()
        while len(self._branches) <= i:
            self._branches.append(torch.cuda.Stream(x.device))
        side = self._branches[i]
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            return fn()

    def join_branch(self, i: int, x: torch.Tensor) -> None:
        if BRANCHES and x.is_cuda and torch.cuda.is_current_stream_capturing():
            torch.cuda.current_stream().wait_stream(self._branches[i])

    def mixer_parts(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """(result, factor) of the mixer, or of each of the two side by side."""
        if sp.mixer != "parallel":
            return [(self.mixer_blocks[sp.mixer](li, lw, sp, h, fb), 1.0)]
        right = self.branch(1, h, lambda: self.mixer_blocks[sp.right.mixer](li, lw, sp.right, h, fb))
        left = self.mixer_blocks[sp.left.mixer](li, lw, sp.left, h, fb)
        self.join_branch(1, h)
        return [(left, sp.left_scale), (right, sp.right_scale)]

    def parallel_layer(self, li: int, lw, sp: LayerSpec, x: torch.Tensor, delta, first: Optional[torch.Tensor], fb: ForwardBatch):
        """A layer whose mixer and feed-forward read the same stream, with the token input behind them; returns the pending update of the token input."""
        cfg, layer = self.cfg, self.runs[li].layer
        hs = stream.norm2(x, lw.attn_norm, cfg.rms_eps, delta, add=first if self.runs[li].again else None, weight2=lw.ffn_norm, out_dtype=self.act_dtype)
        ffn = None
        if sp.has_ffn:
            with profiler.region("ffn", "block", "ffn", li):
                ffn = self.branch(0, x, lambda: self.stream_ffn(lw, sp, hs[1]))
        with profiler.region(sp.mixer, "block", "attention", li):
            parts = self.mixer_parts(li, lw, sp, hs[0], fb)
        if sp.has_ffn:
            self.join_branch(0, x)
            parts.append((ffn, 1.0))
        rows = stream.join(x, parts, self.act_dtype if lw.side is not None else None)
        if lw.side is None:
            return None
        z = apply_linear_stream(lw.side.gate, rows)
        g = stream.token_gate(z, fb.ids, self.w.side_embed, layer * cfg.side_dim, cfg.side_dim, self.act_dtype)
        return stream.RmsPosted(apply_linear_stream(lw.side.proj, g), lw.side.norm, cfg.rms_eps)

    def weighted_tail(self, li: int, lw, sp: LayerSpec, x: torch.Tensor, delta: stream.Update, hist: Optional[torch.Tensor]) -> stream.Update:
        """The feed-forward of a layer whose results join the stream with a factor; returns the pending update with the average behind it, if there is one."""
        eps = self.cfg.rms_eps
        if sp.has_ffn:
            gate = None
            if lw.sh_dot is not None:
                h, gate = stream.norm_gate(x, lw.ffn_norm, eps, delta, lw.sh_dot, self.act_dtype)
            else:
                h = stream.norm(x, lw.ffn_norm, eps, delta, out_dtype=self.act_dtype)
            with profiler.region("ffn", "block", "ffn", li):
                delta = stream.Update(self.ffn_parts(lw, sp, h, gate))
        if hist is not None:
            # every DEPTH_BLOCK places, the sums over the places so far are formed for the layers until the next time: each place is read once for all of them
            at, n = li + 1, stream.DEPTH_BLOCK
            if at > 1 and (at - 1) % n == 0:
                self._depth = (at, stream.depth_base(hist, at, [self.w.layers[r.layer].depth_w for r in self.runs[li: li + n]]))
            first, base = self._depth if at > n else (0, None)
            delta.depth = stream.Depth(hist, at, lw.depth_w, base[at - first] if base is not None else None, first)
        return delta

    def lightning_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """Lightning attention: projection -> SiLU + decayed recurrence -> RMSNorm over all heads * sigmoid(gate) -> output projection."""
        proj, activated = apply_linear_mixer(lw.lin.w_in, h, silu_rows=2 * sp.q_dim + sp.n_heads * sp.v_dim)
        o = lightning.lightning(proj, lw.lin.decay, self.kv.rec[li], fb.cu_q, fb.seq_slots, sp.n_heads, sp.head_dim, sp.v_dim, activated,
                                max(fb.q_lens) if fb.q_lens else 1)
        y = stream.gated_norm(o, proj, 2 * sp.q_dim + sp.n_heads * sp.v_dim, lw.lin.norm, self.cfg.rms_eps, self.act_dtype)
        return apply_linear_stream(lw.lin.w_out, y)

    def mingru_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """minGRU: projection -> recurrence per channel (gates and candidates f32) * SiLU(output gate) -> output projection."""
        w = lw.gru
        xg, z, col = self._mixer_rows(w.w_in, h, w.z_row)
        y = recurrent.mingru(xg, z, col, w.x_bias, w.z_bias, self.kv.rec[li], fb.cu_q, fb.seq_slots, sp.v_dim, self.most_tokens(fb), self.act_dtype)
        return apply_linear_stream(w.w_out, y)

    def mamba2_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """Mamba-2: projection -> causal convolution + SiLU -> recurrence -> norm of y * SiLU(z) -> output projection.  The step sizes stay f32."""
        w, nv, most = lw.mamba, sp.n_heads * sp.v_dim, max(fb.q_lens) if fb.q_lens else 1
        proj, dt, dt_col = self._mixer_rows(w.w_in, h, w.dt_row)
        xbc = recurrent.causal_conv(proj, nv, w.conv_w, w.conv_b, self.kv.conv[li], fb.cu_q, fb.seq_slots, most, self.act_dtype)
        y = recurrent.ssd(xbc, dt, dt_col, w.dt_bias, w.a, w.d, self.kv.rec[li], fb.cu_q, fb.seq_slots, sp.n_heads, sp.state_groups, sp.head_dim, sp.v_dim, most)
        return apply_linear_stream(w.w_out, stream.part_norm(y, w.norm, sp.norm_parts, self.cfg.rms_eps, proj, 0, self.act_dtype))

    def hgrn2_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """HGRN2: projection -> SiLU(q), recurrence with a forget gate per key channel (f32) -> RMSNorm per head -> output projection."""
        w = lw.gla
        qv, gate, col = self._mixer_rows(w.w_in, h, w.f_row, silu_rows=sp.q_dim)
        o = recurrent.gla(qv, gate, col, w.f_bias, w.lower, self.kv.rec[li], fb.cu_q, fb.seq_slots, sp.n_heads, sp.head_dim, sp.v_dim, activated=qv is not gate,
                          max_tokens=max(fb.q_lens) if fb.q_lens else 1)
        return apply_linear_stream(w.w_out, stream.part_norm(o, w.norm, sp.n_heads, self.cfg.rms_eps, out_dtype=self.act_dtype))

    @staticmethod
    def _mixer_rows(w_in: LinearWeight, h: torch.Tensor, at: int, silu_rows: int = 0):
        """Input projection whose features from ``at`` on feed a recurrence's gates and stay f32: (rows, result that holds the gates, their column).
        One product for decode-sized batches; for prefill-sized ones bf16 rows (with SiLU on the first ``silu_rows``) and an f32 product."""
        if w_in.fmt == "f32" or h.shape[0] <= 64:
            proj = apply_linear_stream(w_in, h)
            return proj, proj, at
        main, gates = w_in.rows(0, at), w_in.rows(at, w_in.n)
        return gemm.linear(h, main.w, w_tiled=main.tiled, silu_rows=silu_rows), gemm.linear(h, gates.w, out_dtype=torch.float32, w_tiled=gates.tiled), 0

    def latent_plan(self, q_lens, kv_lens, max_kv: int, device, decode: bool) -> latent.LatentPlan:
        specs = [sp for sp in self.cfg.layer_specs if sp.mixer == "latent"]
        expand = torch.device(device).type == "cuda" and self.act_dtype == torch.bfloat16 and all(latent.can_expand(sp) for sp in specs)
        return latent.make_plan(q_lens, kv_lens, max_kv, device, decode, expand, sorted({sp.n_heads for sp in specs}))

    def latent_block(self, li: int, lw, sp: LayerSpec, h: torch.Tensor, fb: ForwardBatch):
        """Latent attention: q and kv latents -> norms, cache store -> query heads (without a q latent: part of the first projection) -> attention over the cached
        latents (absorbed) or over keys and values expanded from them -> gate -> output projection.  A layer with ``kv_from`` reads the cache of that layer."""
        w, dt, dev = lw.latent, self.act_dtype, h.device
        hd, d, rd, r = sp.n_heads, sp.head_dim, sp.rot_dim, sp.kv_rank
        cache = self.kv.k[li if sp.kv_from < 0 else sp.kv_from]
        if fb.plans is None:
            fb.plans = {}
        plan = fb.plans.get("latent")
        if plan is None:
            plan = fb.plans["latent"] = self.latent_plan(fb.q_lens, fb.kv_lens, max(fb.kv_lens), dev, fb.is_decode)
        mag = sp.rotary.magnitude
        rows_a = apply_linear_rows(w.w_a, h)
        cq = None
        if sp.q_rank or w.kv_norm is not None:
            cq = latent.latent_store(rows_a, fb.positions, fb.slots, w.q_norm, w.kv_norm, w.freq, mag, cache, sp.q_rank, r, rd, self.cfg.rms_eps, dt,
                                     0 if sp.q_rank else w.cols["kv"])
        q = apply_linear_rows(w.w_qb, cq) if sp.q_rank else rows_a
        dp, vp, rp = (stream.row_width(n, dt) for n in (d, sp.v_dim, rd))
        a = torch.empty(h.shape[0], hd * vp, dtype=dt, device=dev)
        qa = qn = en = er = None
        if plan.n_abs:
            qa, qn = torch.empty(hd, plan.m, cache.shape[2], dtype=dt, device=dev), torch.empty(hd, plan.m, dp, dtype=dt, device=dev)
        if plan.n_exp:
            en, er = torch.empty(plan.n_exp, hd, dp, dtype=dt, device=dev), torch.empty(plan.n_exp, hd, rp, dtype=dt, device=dev)
        latent.latent_q(q, fb.positions, w.freq, mag, sp.scale * att.LOG2E, plan.dst, (qn.transpose(0, 1), qa[:, :, r:].transpose(0, 1)) if qa is not None else None,
                        (en, er) if en is not None else None, hd, d, rd)
        if qa is not None:
            seg, cnt, rows = plan.groups(hd, dev)
            if dt == torch.float32:
                gemm.batched_linear_f32(qn, w.w_uk.w.view(hd, r, d), qa[:, :, :r])
            else:
                gemm.grouped_linear(qn.view(-1, dp), w.w_uk.w.view(hd, -1, dp), seg, cnt, plan.tile, out=qa.view(-1, cache.shape[2]), n_out=r, w_tiled=w.w_uk.tiled)
            o = latent.attend_latents(qa, cache, r, r + rd, plan, fb, self.kv.page_size, w.sink)
            if dt == torch.float32:
                # nothing is expanded in f32: the absorbed rows are the tokens in order
                gemm.batched_linear_f32(o[:, : plan.n_abs], w.w_uv.w.view(hd, vp, r), a.view(-1, hd, vp).transpose(0, 1))
            else:
                gemm.grouped_linear(o.view(-1, o.shape[2]), w.w_uv.w.view(hd, vp, -1), seg, cnt, plan.tile, out=a.view(-1, vp), row_map=rows, n_out=vp, w_tiled=w.w_uv.tiled)
        if en is not None:
            rows_kv = latent.gather_latents(cache, plan, fb.block_table, self.kv.page_size)
            kvx = gemm.linear(rows_kv[:, : w.w_kv.k], w.w_kv.w, w_tiled=w.w_kv.tiled)
            latent.attend_expanded(en, er, kvx, rows_kv, r, plan, w.sink, a.view(-1, hd, vp))
        if sp.out_gate:
            stream.sigmoid_gate(a.view(-1, hd, vp), rows_a, w.cols["gate"], sp.v_dim)
        return apply_linear_stream(lw.wo, a)

    def stream_moe(self, lw, m: MoeSpec, h: torch.Tensor):
        """Mixture of experts of a layer described by ``LayerSpec``; the weighted sum stays pending for the stream's norm."""
        rt = dict(mode=m.router, renorm=(2 if m.gated else 1) if m.renorm else 0, routed_scale=m.scale, groups=(m.groups, m.groups_kept, m.group_best))
        if lw.w13.fmt != "f32":
            return self.moe_local(lw, h, spec=m, rt=rt)
        ids, wts, pl = moe.route_plan(gemm.linear_f32(h, lw.router), m.top, m.n_experts, 64, **rt)
        gu = gemm.grouped_linear_f32(h, lw.w13.w.view(m.n_experts, -1, h.shape[1]), pl.seg_start, pl.seg_count, pl.capacity, pl.row_token)
        y = gemm.grouped_linear_f32(stream.act_mul(gu, "silu") if m.gated else stream.gelu_rows(gu), lw.w2.w.view(m.n_experts, -1, lw.w2.k), pl.seg_start, pl.seg_count, pl.capacity)
        return moe.PendingCombine(y, pl.pair_row, wts, h.shape[0], m.top)

    def plain_ffn(self, up: LinearWeight, down: LinearWeight, h: torch.Tensor):
        """down(gelu(up(h))), the exact GELU."""
        a = stream.gelu_rows(gemm.linear_f32(h, up.w)) if up.fmt == "f32" else gemm.linear(h, up.w, w_tiled=up.tiled, gelu=True)
        return apply_linear_stream(down, a)

    def ffn_parts(self, lw, sp: LayerSpec, h: torch.Tensor, gate: Optional[torch.Tensor]):
        """The feed-forward's results as parts of an ``Update``: with a shared expert two of them, its own times the tokens' ``gate``."""
        m = self.cfg.residual_mult
        if gate is None:
            return [(self.stream_ffn(lw, sp, h), m, None)]
        shared = self.branch(0, h, lambda: self.plain_ffn(lw.sh_up, lw.sh_down, h))
        y = self.stream_ffn(lw, sp, h)
        self.join_branch(0, h)
        return [(y, m, None), (shared, m, gate)]

    def stream_ffn(self, lw, sp: LayerSpec, h: torch.Tensor):
        if sp.moe is not None:
            return self.stream_moe(lw, sp.moe, h)
        gu = lw.w_gate_up
        if gu.fmt == "f32":
            return apply_linear_stream(lw.w_down, stream.act_mul(gemm.linear_f32(h, gu.w, gu.bias), sp.act, sp.act_cap))
        inter = gu.n // 2
        split = gemm.pick_partials_dual(inter, h.shape[0], (gu.k + 63) // 64 * 64, False) if SPLIT_PROJ and h.is_cuda else 1
        if split > 1:
            act = ew.silu_mul_partials(gemm.swiglu_partials(h, gu.w, split, w_tiled=gu.tiled), act=sp.act, cap=sp.act_cap, bias=gu.bias)
        else:
            act = gemm.linear_swiglu(h, gu.w, w_tiled=gu.tiled, act=sp.act, cap=sp.act_cap, bias=gu.bias)
        return apply_linear_stream(lw.w_down, act)

    def shared_expert(self, lw, h: torch.Tensor) -> torch.Tensor:
        """Always-on expert of the qwen35moe layers, scaled by sigmoid(h . g) (cuda/llm/cuda_llm_runner.c:11879-11897)."""
        if lw.sh_gate_up.fmt == "bf16":
            act = gemm.linear_swiglu(h, lw.sh_gate_up.w, w_tiled=lw.sh_gate_up.tiled)
            y = apply_linear(lw.sh_down, act)
        else:
            xm = ew.mx_quantize(h, sf_layout=32 if h.shape[0] <= 32 else 128)
            y = apply_linear(lw.sh_down, None, gemm.linear_mx_swiglu_quant(xm, lw.sh_gate_up.mx))
        if lw.sh_gate is not None:
            g = torch.sigmoid(moe.router_logits(h, lw.sh_gate) if h.is_cuda and h.shape[1] % 256 == 0 else h.float() @ lw.sh_gate.float().t())
            y = (y.float() * g).to(torch.bfloat16)
        return y

    def dense_ffn(self, lw, h: torch.Tensor, h_mx: Optional[MxTensor]) -> torch.Tensor:
        gu = lw.w_gate_up
        inter = gu.n // 2
        if gu.is_quant:
            return self.par.row_linear(lw.w_down, qlinear.linear_swiglu(h, gu.q))
        if gu.fmt == "bf16":
            sp = gemm.pick_partials_dual(inter, h.shape[0], gu.k, False) if (SPLIT_PROJ and h.is_cuda and inter % 128 == 0) else 1
            if sp > 1:      # decode-sized batch: the projection is cut along K to fill the GPU, the activation kernel adds the partials
                act = ew.silu_mul_partials(gemm.swiglu_partials(h, gu.w, sp, w_tiled=gu.tiled))
            else:
                act = gemm.linear_swiglu(h, gu.w, w_tiled=gu.tiled)
            return self.par.row_linear(lw.w_down, act)
        xm = h_mx if h_mx is not None else ew.mx_quantize(h, sf_layout=32 if h.shape[0] <= 32 else 128)
        sp = gemm.pick_partials_dual(inter, xm.rows, gu.k, True) if (SPLIT_PROJ and xm.data.is_cuda and inter % 128 == 0) else 1
        if sp > 1:
            act = ew.silu_mul_partials(gemm.swiglu_partials(xm, gu.mx, sp), quantize=True, sf_layout=xm.sf_layout)
        else:
            act = gemm.linear_mx_swiglu_quant(xm, gu.mx)
        return self.par.row_linear(lw.w_down, None, act)

    def moe_local(self, lw, h: torch.Tensor, h_mx: Optional[MxTensor] = None, local_range=None, spec: Optional[MoeSpec] = None, rt=None) -> torch.Tensor:
        """The experts held by this GPU over the rows ``h``: route -> plan -> (gather + quantise) -> gate/up -> down -> combine.
        ``local_range = (first expert, count)``: the weights are that slice of the experts; (token, expert) pairs routed
        elsewhere are dropped from the plan and contribute nothing to the pending sum (the caller adds the ranks' sums).
        ``spec`` / ``rt``: sizes and routing rule of one layer (models described layer by layer) instead of the model's."""
        cfg = self.cfg
        t = h.shape[0]
        e, k, inter, hid = (local_range[1] if local_range else cfg.n_experts), cfg.n_experts_used, cfg.expert_ffn, cfg.hidden
        n_exp = cfg.n_experts
        gated = True
        if spec is not None:
            e, n_exp, k, inter, hid, gated = spec.n_experts, spec.n_experts, spec.top, lw.w2.k, lw.w13.k, spec.gated
        rt = rt or dict(mode=cfg.router, bias=lw.router_bias, renorm=cfg.norm_topk, routed_scale=cfg.routed_scale, local_range=local_range)
        if self.mx:
            # token tile (= scale-atom layout) by the expected rows per expert: 32 for decode-sized batches
            tn = 32 if (t * k) // cfg.n_experts <= 24 else 128
            if tn == 32 and moe.can_prep(h, lw.router, k):
                # decode-sized batch: router projection, routing, plan and the quantised gather are one launch
                ids, wts, pl, xq = moe.prep_hidden(h, lw.router, k, e, tn, **rt)
            else:
                ids, wts, pl = moe.route_plan_hidden(h, lw.router, k, e, tn, **rt)
                # the RMSNorm before this block already quantised the tokens: gather bytes and scales (every token is quantised
                # once, not once per selected expert)
                xq = ew.mx_gather_rows(h_mx, pl.row_token, sf_layout=tn) if h_mx is not None else ew.mx_quantize(h, pl.row_token, sf_layout=tn)
            dev = h.device
            if tn == 32 and moe.can_fuse_ffn(xq, lw.w13, lw.w2, e, pl.capacity):
                y = moe.expert_ffn_fused(xq, lw.w13, lw.w2, e, pl)          # gate/up, activation and down as one persistent launch
            else:
                hq = torch.empty(pl.capacity, inter, dtype=torch.uint8, device=dev)
                hsf = ew.sf_alloc(pl.capacity, inter, dev, tn, init=False)
                expert_gate_up_mx(xq.data, xq.sf, lw.w13, e, pl.seg_start, pl.seg_count, tn, hq, hsf, pl.row_token)
                y = gemm.grouped_linear(hq, lw.w2.mx.data.view(e, hid, inter), pl.seg_start, pl.seg_count, tn, sfa=lw.w2.mx.sf, sfb=hsf,
                                        w_tiled=lw.w2.mx.tiled, pair_rows=(tn == 32 and PAIR_DOWN))
        else:
            per = max(1, (t * k + n_exp - 1) // n_exp)       # expected rows per expert
            tn = gemm.pick_tn(per, dual=True)
            wide = 256 if per >= 96 and tn == 128 else tn     # token tile of the products with one accumulator
            if moe.can_prep(h, lw.router, k):
                ids, wts, pl, xs = moe.prep_hidden(h, lw.router, k, e, tn, quantize=False, **rt)
            else:
                ids, wts, pl = moe.route_plan_hidden(h, lw.router, k, e, tn, **rt)
                xs = moe.gather_rows(h, pl.row_token)
            act = gemm.grouped_linear(xs, lw.w13.w.view(e, -1, hid), pl.seg_start, pl.seg_count, tn if gated else wide, dual=gated, gelu=not gated, w_tiled=lw.w13.tiled)
            y = gemm.grouped_linear(act, lw.w2.w.view(e, -1, inter), pl.seg_start, pl.seg_count, wide, w_tiled=lw.w2.tiled)
        return moe.PendingCombine(y, pl.pair_row, wts, t, k)

    # ------------------------------------------------------------------------------------------------
    def forward_hidden(self, fb: ForwardBatch, first_layer: int = 0, last_layer: Optional[int] = None,
                       x: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Residual stream after layers ``[first_layer, last_layer)`` (pipeline stages pass ``x`` in)."""
        cfg, w = self.cfg, self.w
        last_layer = len(self.runs) if last_layer is None else last_layer
        if x is None and self.stream_f32:
            x = stream.embed(fb.ids, w.embed, cfg.embed_scale) if fb.embeds is None else fb.embeds.float()
        elif x is None:
            x = fb.embeds if fb.embeds is not None else ew.embed(fb.ids, w.embed)
        delta = None
        first = x.clone() if any(r.again for r in self.runs) else None       # the embedding output, for later passes of a loop
        hist = torch.empty(last_layer, *x.shape, dtype=x.dtype, device=x.device) if cfg.depth_average else None      # it, and all layers' results but the last
        if hist is not None:
            hist[0].copy_(x)
        self._rotary = {}
        if hasattr(self.par, "_sp_ok"):
            # the fused tensor-parallel prefill path keeps the residual stream sharded by rows between the layers' GEMMs: only for
            # plain dense stacks (nothing reads the whole stream or the normalised rows outside a GEMM in between)
            self.par._sp_ok = not (cfg.is_moe or cfg.attn_output_gate or fb.deepstack is not None or self.snapshot_layers or
                                   any(l.ssm is not None for l in w.layers[first_layer:last_layer]))
        for li in range(first_layer, last_layer):           # li: the layer RUN, index of its cache (looped layers run several times)
            lw = w.layers[self.runs[li].layer]
            if cfg.parallel_ffn:
                delta = self.parallel_layer(li, lw, cfg.layer_specs[self.runs[li].layer], x, delta, first, fb)
                if li in self.snapshot_layers:
                    self.snapshots[li] = stream.settled(x, delta)
                continue
            if self.stream_f32:
                sp, step = cfg.layer_specs[self.runs[li].layer], self.runs[li].step
                h = stream.norm(x, lw.attn_norm, cfg.rms_eps, delta, add=w.loop_step[step] if step >= 0 else None, out_dtype=self.act_dtype)
                with profiler.region(sp.mixer, "block", "attention", li):
                    delta = self.mixer_blocks[sp.mixer](li, lw, sp, h, fb)
                if cfg.depth_average or cfg.residual_mult != 1.0:
                    delta = self.weighted_tail(li, lw, sp, x, stream.Update([(delta, cfg.residual_mult, None)]), hist)
                else:
                    if lw.attn_post is not None:
                        delta = stream.PostNormed(delta, lw.attn_post)
                    if sp.has_ffn:
                        h = stream.norm(x, lw.ffn_norm, cfg.rms_eps, delta, out_dtype=self.act_dtype)
                        with profiler.region("ffn", "block", "ffn", li):
                            delta = self.stream_ffn(lw, sp, h)
                        if lw.ffn_post is not None:
                            delta = stream.PostNormed(delta, lw.ffn_post)
                if li in self.snapshot_layers:
                    self.snapshots[li] = stream.settled(x, delta)
                continue
            lay = 32 if x.shape[0] <= 32 else 128
            par = self.par
            is_ssm = lw.ssm is not None
            if self.mx:
                h, h_mx = par.add_norm(delta if delta is not None else x, lw.attn_norm, cfg.rms_eps, x if delta is not None else None,
                                       quantize=True, want_bf16=is_ssm, sf_layout=lay)
            else:
                h, h_mx = par.add_norm(delta if delta is not None else x, lw.attn_norm, cfg.rms_eps, x if delta is not None else None), None
            with profiler.region("ssm" if is_ssm else "attention", "block", "attention", li):
                delta = self.ssm_block(li, lw, h, h_mx, fb) if is_ssm else self.attention_block(li, lw, h, h_mx, fb)
            need_bf16 = (not self.mx) or cfg.is_moe
            # a parallel context may name the buffer the normalised rows should land in (the staging buffer of its exchange)
            ob = par.ffn_in_buffer(x.shape[0], lw) if (hasattr(par, "ffn_in_buffer") and x.is_cuda) else None
            okw = {"out_buf": ob} if ob is not None else {}
            if self.mx:
                h, h_mx = par.add_norm(delta, lw.ffn_norm, cfg.rms_eps, x, quantize=True, want_bf16=need_bf16, sf_layout=lay, **okw)
            else:
                h, h_mx = par.add_norm(delta, lw.ffn_norm, cfg.rms_eps, x, **okw), None
            with profiler.region("moe" if lw.w13 is not None else "ffn", "block", "ffn", li):
                if lw.w13 is not None:
                    delta = self.par.moe_ffn(self, lw, h, h_mx)
                    if delta is None:
                        delta = self.moe_local(lw, h, h_mx)
                    if lw.sh_gate_up is not None:
                        delta = (self.par.materialize(delta).float() + self.shared_expert(lw, h).float()).to(torch.bfloat16)
                else:
                    delta = self.dense_ffn(lw, h, h_mx)
            if fb.deepstack is not None and li < fb.deepstack.shape[0]:
                # DeepStack (Qwen3-VL): vision features of deeper encoder layers join the stream after the first decoder layers
                delta = (self.par.materialize(delta).float() + fb.deepstack[li].float()).to(torch.bfloat16)
            if li in self.snapshot_layers:
                self.snapshots[li] = (x.float() + self.par.materialize(delta).float())
        # the last delta stays pending: the head (or the next pipeline stage) folds it into the stream
        if hasattr(self.par, "finish_residual"):
            self.par.finish_residual(x, delta)
        if self.stream_f32:
            self._last_delta = delta
            return x
        self._last_delta = self.par.materialize(delta) if delta is not None else None
        return x

    def forward(self, fb: ForwardBatch) -> torch.Tensor:
        """Logits ``f32 [len(logit_rows), V_local]``."""
        x = self.forward_hidden(fb)
        return self.head(x, fb)

    def _head_input(self, x: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        cfg, w = self.cfg, self.w
        delta = self._last_delta
        rows = fb.logit_rows
        if self.stream_f32:
            return stream.norm(x, w.final_norm, cfg.rms_eps, delta, rows=rows.long(), out_dtype=self.act_dtype)
        xr = x[rows]
        if delta is not None:
            xr = (xr.float() + delta[rows].float()).to(torch.bfloat16)
        return ew.rmsnorm(xr.contiguous(), w.final_norm, cfg.rms_eps)

    def head(self, x: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        if self.w.lm_head.is_quant:
            return qlinear.linear(self._head_input(x, fb), self.w.lm_head.q, out_dtype=torch.float32)
        if self.w.lm_head.fmt == "f32":
            return gemm.linear_f32(self._head_input(x, fb), self.w.lm_head.w)
        return gemm.linear(self._head_input(x, fb), self.w.lm_head.w, out_dtype=torch.float32, w_tiled=self.w.lm_head.tiled)

    def forward_greedy(self, fb: ForwardBatch, want_value: bool = False):
        """Greedy next tokens ``int32 [len(logit_rows)]``: the arg-max runs in the LM-head GEMM's epilogue, no logits are stored."""
        x = self.forward_hidden(fb)
        if self.w.lm_head.is_quant or self.w.lm_head.fmt == "f32":
            logits = self.head(x, fb)
            return sampling.argmax(logits, idx_offset=self.w.vocab_start, want_value=want_value)
        return gemm.linear_argmax(self._head_input(x, fb), self.w.lm_head.w, idx_offset=self.w.vocab_start, want_value=want_value,
                                  w_tiled=self.w.lm_head.tiled)

    def final_hidden(self, x: torch.Tensor) -> torch.Tensor:
        """Residual stream with the pending delta folded in (what a pipeline stage hands to the next)."""
        if self._last_delta is None:
            return x
        if self.stream_f32:
            return stream.settled(x, self._last_delta)
        return (x.float() + self._last_delta.float()).to(torch.bfloat16)


def greedy_tokens(logits: torch.Tensor, vocab_start: int = 0) -> torch.Tensor:
    return sampling.argmax(logits, idx_offset=vocab_start)
