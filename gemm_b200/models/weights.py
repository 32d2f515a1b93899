"""Weight containers and the synthetic (random-init) checkpoint generator.

A ``LinearWeight`` keeps one projection in the format the kernels consume:

* ``bf16``   row-major ``[N, K]``
* ``mxfp8``  e4m3 bytes + E8M0 scale atoms (``ops.mxfp8.MxTensor``)
* ``f32``    row-major ``[N, K]`` in 32-bit floats (models described layer by layer: the exact path the 16-bit one is checked against)

Grouped (expert) weights use the same class with ``groups > 0`` and rows stacked expert after expert.
Tensor-parallel and expert-parallel shards are cut when the weights are made or loaded, never at run
time (the reference slices TP rows out of the full matrix on every call, common/transformer.h:4239-4272).

Random init follows the benchmark recipe: N(0, 0.02) for matrices, ones for norms, seeded per tensor so
that a sharded model is a slice of the unsharded one.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import elementwise as ew
from ..ops import mxfp8
from ..ops.attention import LOG2E, cache_head_dims, distance_bias_table
from ..ops.stream import DynTanh, row_width
from ..ops.mxfp8 import MxTensor
from .config import ModelConfig


@dataclass
class LinearWeight:
    fmt: str                                  # "bf16" | "mxfp8" | "f32" | "q4_k" | "q8_0" (ggml blocks kept quantised in HBM)
    n: int                                    # output features (per group)
    k: int
    w: Optional[torch.Tensor] = None          # bf16 [rows, K]
    mx: Optional[MxTensor] = None
    q: Optional["QTensor"] = None             # tiled ggml blocks (``ops.qlinear.QTensor``)
    bias: Optional[torch.Tensor] = None       # f32 [n]
    groups: int = 0                           # > 0: expert-stacked, rows = groups * rows_per_group
    rows_per_group: int = 0
    tiled: bool = False                       # bf16 ``w`` is in the tiled layout (``mx.tiled`` for MXFP8)

    @property
    def is_quant(self) -> bool:
        return self.q is not None

    @property
    def is_tiled(self) -> bool:
        if self.is_quant:
            return True
        return self.tiled if self.fmt in ("bf16", "f32") else self.mx.tiled

    def tile_(self) -> "LinearWeight":
        """Re-lay the matrix in place into the GEMM kernel's tiled weight layout (``ops.mxfp8.tile_weight``)."""
        if self.is_quant or self.fmt == "f32":
            return self                       # ggml blocks are stored in their own tile order from the start
        t = self.w if self.fmt == "bf16" else self.mx.data
        if self.is_tiled or not mxfp8.can_tile(t) or (self.groups and self.rows_per_group % 128):
            return self
        t.copy_(mxfp8.tile_weight(t))
        if self.fmt == "bf16":
            self.tiled = True
        else:
            self.mx.tiled = True
        return self

    def rows(self, a: int, b: int) -> "LinearWeight":
        """The features ``a .. b - 1`` as a projection of their own (a view; of a tiled matrix ``a`` and ``b`` are multiples of 128, or ``b`` is its end)."""
        assert self.fmt in ("bf16", "f32") and not self.groups and (not self.tiled or (a % 128 == 0 and (b % 128 == 0 or b == self.n)))
        return LinearWeight(self.fmt, b - a, self.k, w=self.w[a:b], bias=self.bias[a:b] if self.bias is not None else None, tiled=self.tiled)

    def untiled_data(self) -> torch.Tensor:
        """Row-major copy of the stored matrix (bf16 values or e4m3 bytes)."""
        if self.fmt == "f32":
            return self.w
        t = self.w if self.fmt == "bf16" else self.mx.data
        return mxfp8.untile_weight(t) if self.is_tiled else t

    @property
    def device(self):
        if self.is_quant:
            return self.q.data.device
        return self.w.device if self.w is not None else self.mx.data.device

    def dequantized(self) -> torch.Tensor:
        """fp32 copy of the full matrix (tests and CPU reference paths)."""
        if self.is_quant:
            return self.q.dequantize()
        if self.fmt in ("bf16", "f32"):
            return self.untiled_data().float()
        return mxfp8.dequantize(self.mx)

    def nbytes(self) -> int:
        if self.is_quant:
            return self.q.nbytes()
        if self.fmt in ("bf16", "f32"):
            return self.w.numel() * self.w.element_size()
        return self.mx.data.numel() + self.mx.sf.numel()

    def to(self, device) -> "LinearWeight":
        return LinearWeight(self.fmt, self.n, self.k, w=self.w.to(device) if self.w is not None else None,
                            mx=self.mx.to(device) if self.mx is not None else None, q=self.q.to(device) if self.q is not None else None,
                            bias=self.bias.to(device) if self.bias is not None else None, groups=self.groups,
                            rows_per_group=self.rows_per_group, tiled=self.tiled)


QUANT_FMTS = {"q4_k": 12, "q8_0": 8}          # run-time formats that keep ggml blocks: name -> ggml type id


@dataclass
class QBlocks:
    """A matrix as row-major ggml blocks (the order of a GGUF file): ``raw`` uint8 ``[rows, row_bytes]``.  Supports what weight
    assembly needs without decoding: row ranges, column ranges on block boundaries, stacking along rows."""
    raw: torch.Tensor
    ggml_type: int
    k: int

    @property
    def shape(self):
        return (self.raw.shape[0], self.k)

    def _geom(self):
        from ..ops import ggml_torch as gt
        return gt.BLOCK[self.ggml_type]

    def rows(self, a: int, b: int) -> "QBlocks":
        return QBlocks(self.raw[a:b], self.ggml_type, self.k)

    def cols(self, a: int, b: int) -> "QBlocks":
        blk, nb = self._geom()
        if a % blk or b % blk:
            raise ValueError(f"column range [{a}, {b}) does not fall on {blk}-element block boundaries")
        return QBlocks(self.raw[:, a // blk * nb: b // blk * nb], self.ggml_type, b - a)

    def to(self, device) -> "QBlocks":
        return QBlocks(self.raw.to(device), self.ggml_type, self.k)

    def contiguous(self) -> "QBlocks":
        return QBlocks(self.raw.contiguous(), self.ggml_type, self.k)


def _mat(src, name: str, shape):
    """A projection matrix from a tensor source: its ggml blocks when the source can hand them out (``get_mat``), else floats."""
    return src.get_mat(name, shape) if hasattr(src, "get_mat") else src.get(name, shape)


def _rows(t, a: int, b: int):
    return t.rows(a, b) if isinstance(t, QBlocks) else t[a:b]


def _cols(t, a: int, b: int):
    return t.cols(a, b) if isinstance(t, QBlocks) else t[:, a:b]


def _cat(parts):
    """Stack matrices along rows; quantised parts must share type and width (a mixed list is decoded to float first)."""
    if all(isinstance(p, QBlocks) for p in parts) and len({(p.ggml_type, p.k) for p in parts}) == 1:
        return QBlocks(torch.cat([p.raw for p in parts]), parts[0].ggml_type, parts[0].k)
    return torch.cat([_to_float(p) for p in parts])


def _to_float(t):
    if isinstance(t, QBlocks):
        from ..ops import ggml_torch as gt
        return gt.dequantize(t.raw.contiguous(), t.ggml_type, t.raw.shape[0], t.k).to(torch.bfloat16)
    return t


def make_linear(w_f, fmt: str, bias: Optional[torch.Tensor] = None, groups: int = 0) -> LinearWeight:
    """Wrap a float / bf16 matrix ``[rows, K]`` (rows = groups * rows_per_group when grouped), or ggml blocks (``QBlocks``).

    ``fmt`` "q4_k" / "q8_0" keeps (or makes) ggml blocks and stores them tiled for the fused dequant kernels; blocks of a type
    without such a kernel, or with a width that is not a multiple of 256, are decoded to bf16.  Expert-stacked matrices have no
    quantised path and are stored as bf16 under these formats."""
    from ..ops.qlinear import QTensor
    if fmt in QUANT_FMTS or fmt == "ggml" or isinstance(w_f, QBlocks):
        rows, k = w_f.shape
        want = QUANT_FMTS.get(fmt)
        if groups == 0 and k % 256 == 0 and (want is not None or fmt == "ggml"):
            if isinstance(w_f, QBlocks) and w_f.ggml_type in QUANT_FMTS.values() and (fmt == "ggml" or w_f.ggml_type == want):
                name = {v: n for n, v in QUANT_FMTS.items()}[w_f.ggml_type]       # the file's own blocks, untouched
                return LinearWeight(name, rows, k, q=QTensor.from_blocks(w_f.raw.contiguous(), w_f.ggml_type, rows, k), bias=bias)
            if want is not None:
                return LinearWeight(fmt, rows, k, q=QTensor.from_float(_to_float(w_f).float(), want), bias=bias)
        w_f = _to_float(w_f)
        if fmt in QUANT_FMTS or fmt == "ggml":
            fmt = "bf16"
    rows, k = w_f.shape
    rpg = rows // groups if groups else 0
    n = rpg if groups else rows
    if fmt == "bf16":
        return LinearWeight("bf16", n, k, w=w_f.to(torch.bfloat16).contiguous(), bias=bias, groups=groups, rows_per_group=rpg)
    if fmt == "f32":
        return LinearWeight("f32", n, k, w=w_f.to(torch.float32).contiguous(), bias=bias, groups=groups, rows_per_group=rpg)
    if fmt == "mxfp8":
        if w_f.is_cuda:
            mx = ew.mx_quantize(w_f.to(torch.bfloat16).contiguous())
        else:
            mx = mxfp8.quantize(w_f.to(torch.bfloat16).float())
        return LinearWeight("mxfp8", n, k, mx=mx, bias=bias, groups=groups, rows_per_group=rpg)
    raise ValueError(f"unknown weight format {fmt!r}")


@dataclass
class SsmWeights:
    """A Delta-Net layer (GGUF names: attn_qkv, attn_gate, ssm_alpha, ssm_beta, ssm_conv1d, ssm_a, ssm_dt.bias, ssm_norm, ssm_out)."""
    w_in: LinearWeight            # rows [qkv (Q | K | V channels) ; z (d_inner)]
    w_ab: torch.Tensor            # bf16 [2 * n_heads_v, H]: alpha rows then beta rows
    conv_w: torch.Tensor          # f32 [qkv_dim, conv_k]
    a: torch.Tensor               # f32 [n_heads_v]
    dt_bias: torch.Tensor         # f32 [n_heads_v]
    norm: torch.Tensor            # f32 [head_dim]
    w_out: LinearWeight           # [H, d_inner]

    def to(self, device) -> "SsmWeights":
        return SsmWeights(self.w_in.to(device), self.w_ab.to(device), self.conv_w.to(device), self.a.to(device), self.dt_bias.to(device),
                          self.norm.to(device), self.w_out.to(device))


@dataclass
class LightningWeights:
    """A lightning-attention mixer."""
    w_in: LinearWeight            # rows [q ; k ; v ; gate]
    decay: torch.Tensor           # f32 [heads]
    norm: torch.Tensor            # f32 [heads * v_dim]
    w_out: LinearWeight           # [H, heads * v_dim]

    def to(self, device) -> "LightningWeights":
        return LightningWeights(self.w_in.to(device), self.decay.to(device), self.norm.to(device), self.w_out.to(device))


@dataclass
class Mamba2Weights:
    """A Mamba-2 mixer.  ``w_in`` rows: [z | x | B | C], padding up to ``dt_row`` (a multiple of 128), [dt]."""
    w_in: LinearWeight
    dt_row: int
    conv_w: torch.Tensor          # f32 [channels, taps]
    conv_b: torch.Tensor          # f32 [channels]
    dt_bias: torch.Tensor         # f32 [heads]
    a: torch.Tensor               # f32 [heads]: the state decays by exp(a dt)
    d: torch.Tensor               # f32 [heads]
    norm: torch.Tensor            # f32 [heads * v_dim]
    w_out: LinearWeight

    def to(self, device) -> "Mamba2Weights":
        return Mamba2Weights(self.w_in.to(device), self.dt_row, *(t.to(device) for t in (self.conv_w, self.conv_b, self.dt_bias, self.a, self.d, self.norm)),
                             self.w_out.to(device))


@dataclass
class GlaWeights:
    """A linear-attention mixer with a forget gate per key channel (HGRN2).  ``w_in`` rows: [q | v], padding up to ``f_row`` (a multiple of 128),
    [f]."""
    w_in: LinearWeight
    f_row: int
    f_bias: torch.Tensor          # f32 [heads * dim]
    lower: torch.Tensor           # f32 [heads * dim]
    norm: torch.Tensor            # f32 [v_dim]
    w_out: LinearWeight

    def to(self, device) -> "GlaWeights":
        return GlaWeights(self.w_in.to(device), self.f_row, self.f_bias.to(device), self.lower.to(device), self.norm.to(device), self.w_out.to(device))


@dataclass
class LatentWeights:
    """A latent-attention mixer.  ``w_a`` without a query latent: rows [q heads | kv latent | rotated key part | gate], each part starting at the column that
    ``cols`` names (multiples of 8).  ``w_kv`` expands cached latents to all heads' keys and values (prompts); ``w_uk`` / ``w_uv`` are the same matrices
    head by head, for attention over the latents themselves (decoding)."""
    w_a: LinearWeight             # rows [q latent | kv latent | rotated key part], or [q latent] alone
    q_norm: Optional[torch.Tensor]    # f32 [q_rank]
    kv_norm: Optional[torch.Tensor]   # f32 [kv_rank]
    w_qb: Optional[LinearWeight]  # [heads * (dim + rot_dim), q_rank]
    w_kv: Optional[LinearWeight]  # rows [heads * dim ; heads * v_dim], each head padded to 8 rows (bf16 only)
    w_uk: LinearWeight            # per head [rank, dim]
    w_uv: LinearWeight            # per head [v_dim, rank]
    sink: Optional[torch.Tensor]  # f32 [heads], times log2 e
    freq: torch.Tensor            # f64 [rot_dim / 2] rotary frequencies
    cols: Optional[Dict[str, int]] = None     # first columns of "kv" and "gate"

    def to(self, device) -> "LatentWeights":
        mv = lambda t: t.to(device) if t is not None else None
        return LatentWeights(self.w_a.to(device), mv(self.q_norm), mv(self.kv_norm), mv(self.w_qb), mv(self.w_kv), self.w_uk.to(device), self.w_uv.to(device),
                             mv(self.sink), mv(self.freq), self.cols)


@dataclass
class MinGruWeights:
    """A minGRU mixer.  ``w_in`` rows: [x | output gate], padding up to ``z_row`` (a multiple of 128), [z]."""
    w_in: LinearWeight
    z_row: int
    z_bias: torch.Tensor          # f32 [width]
    x_bias: torch.Tensor          # f32 [width]
    w_out: LinearWeight

    def to(self, device) -> "MinGruWeights":
        return MinGruWeights(self.w_in.to(device), self.z_row, self.z_bias.to(device), self.x_bias.to(device), self.w_out.to(device))


@dataclass
class RwkvWeights:
    """An RWKV-style mixer.  ``w_in``: the receptance, key, value and gate projections as four groups of rows, each over a mix of its own of the
    token's row and the one before it; ``w1`` / ``w2``: the decay's low-rank projection."""
    mu: torch.Tensor              # f32 [5, H]: r, k, v, g, decay
    w_in: LinearWeight
    w1: LinearWeight              # [rank, H]
    w2: LinearWeight              # [heads * dim, rank]
    w2_rows: Optional[torch.Tensor]   # bf16, the same row by row, for the step kernel (None in 32-bit)
    w0: torch.Tensor              # f32 [heads * dim]
    u: torch.Tensor               # f32 [heads * dim]: weight of the current token
    norm: torch.Tensor            # f32 [heads * v_dim]
    w_out: LinearWeight

    def to(self, device) -> "RwkvWeights":
        return RwkvWeights(*(t.to(device) for t in (self.mu, self.w_in, self.w1, self.w2)), self.w2_rows.to(device) if self.w2_rows is not None else None,
                           *(t.to(device) for t in (self.w0, self.u, self.norm, self.w_out)))


@dataclass
class SideWeights:
    """The token input of a layer: a gate on the stream, a projection back into it, a norm of the result."""
    gate: LinearWeight            # [dim, H]
    proj: LinearWeight            # [H, dim]
    norm: torch.Tensor            # f32 [H]

    def to(self, device) -> "SideWeights":
        return SideWeights(self.gate.to(device), self.proj.to(device), self.norm.to(device))


@dataclass
class LayerWeights:
    attn_norm: torch.Tensor                       # or DynTanh
    wqkv: Optional[LinearWeight]                  # rows [Q ; K ; V] (+ [gate] after V when the attention output is gated); None in SSM layers
    wo: Optional[LinearWeight]
    ffn_norm: torch.Tensor
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    w_gate_up: Optional[LinearWeight] = None      # dense FFN, rows [gate ; up]
    w_down: Optional[LinearWeight] = None
    router: Optional[torch.Tensor] = None         # bf16 [E, H]
    router_bias: Optional[torch.Tensor] = None    # f32 [E] (sigmoid router)
    w13: Optional[LinearWeight] = None            # experts, rows per expert [gate ; up] = 2I
    w2: Optional[LinearWeight] = None             # experts, rows per expert = H, K = I
    ssm: Optional[SsmWeights] = None              # Delta-Net layer (then wqkv / wo are None)
    sh_gate_up: Optional[LinearWeight] = None     # shared expert [gate ; up]
    sh_down: Optional[LinearWeight] = None
    sh_gate: Optional[torch.Tensor] = None        # bf16 [1, H]: sigmoid gate of the shared expert (absent = ungated)
    lin: Optional[LightningWeights] = None        # lightning-attention layer (then wqkv / wo are None)
    rel_bias: Optional[torch.Tensor] = None       # f32 [heads, 2 N] distance bias (ops.attention.distance_bias_table)
    attn_post: Optional[DynTanh] = None           # norm of the mixer's / feed-forward's result, with its per-channel scale folded in
    ffn_post: Optional[DynTanh] = None
    mamba: Optional[Mamba2Weights] = None
    gla: Optional[GlaWeights] = None
    latent: Optional[LatentWeights] = None        # (the output projection is wo)
    sink: Optional[torch.Tensor] = None           # f32 [heads], times log2 e: joins the softmax's sum (attention)
    conv_w: Optional[torch.Tensor] = None         # f32 [q and k channels, taps]: convolution of the projected q and k
    rot_freq: Optional[torch.Tensor] = None       # f64 [dims / 2] rotary frequencies
    rwkv: Optional[RwkvWeights] = None
    side: Optional[SideWeights] = None
    gru: Optional[MinGruWeights] = None
    log_bias: Optional[torch.Tensor] = None       # f32 [2, heads]: r1 and r2 of the logarithmic distance bias
    sh_up: Optional[LinearWeight] = None          # plain shared expert (its down projection is sh_down)
    sh_dot: Optional[torch.Tensor] = None         # f32 [H]: row that gates the shared expert, times the weight of the norm in front of the feed-forward
    depth_w: Optional[torch.Tensor] = None        # f32 [layer + 2]: weights of the embedding output and of every layer's result so far

    def linears(self) -> List[LinearWeight]:
        """Every projection matrix of the layer."""
        own = [self.wqkv, self.wo, self.w_gate_up, self.w_down, self.w13, self.w2, self.sh_gate_up, self.sh_down, self.sh_up]
        for part in (self.ssm, self.lin, self.mamba, self.gla, self.gru):
            if part is not None:
                own += [part.w_in, part.w_out]
        if self.rwkv is not None:
            own += [self.rwkv.w_in, self.rwkv.w1, self.rwkv.w2, self.rwkv.w_out]
        if self.side is not None:
            own += [self.side.gate, self.side.proj]
        if self.latent is not None:
            own += [self.latent.w_a, self.latent.w_qb, self.latent.w_kv, self.latent.w_uk, self.latent.w_uv]
        return [lw for lw in own if lw is not None]


@dataclass
class ModelWeights:
    cfg: ModelConfig
    embed: torch.Tensor                           # bf16 [V, H]
    layers: List[LayerWeights]
    final_norm: torch.Tensor
    lm_head: LinearWeight                         # bf16 [V(/tp), H]
    fmt: str = "bf16"
    tp_rank: int = 0
    tp_size: int = 1
    ep_rank: int = 0
    ep_size: int = 1
    vocab_start: int = 0                          # first vocabulary id of the LM-head shard
    loop_step: Optional[torch.Tensor] = None      # f32 [times, H]: vectors added in front of the passes of a layer loop
    side_embed: Optional[torch.Tensor] = None     # bf16 (f32) [V, layers * side_dim]: token inputs of the layers

    @property
    def kv_dtype(self) -> str:
        """The KV cache format that goes with the weights."""
        return "f32" if self.fmt == "f32" else "bf16"

    def to(self, device) -> "ModelWeights":
        def mv(x):
            return x.to(device) if x is not None else None
        layers = [LayerWeights(attn_norm=mv(l.attn_norm), wqkv=mv(l.wqkv), wo=mv(l.wo), ffn_norm=mv(l.ffn_norm), q_norm=mv(l.q_norm),
                               k_norm=mv(l.k_norm), w_gate_up=mv(l.w_gate_up), w_down=mv(l.w_down), router=mv(l.router),
                               router_bias=mv(l.router_bias), w13=mv(l.w13), w2=mv(l.w2), ssm=mv(l.ssm), sh_gate_up=mv(l.sh_gate_up),
                               sh_down=mv(l.sh_down), sh_gate=mv(l.sh_gate), lin=mv(l.lin), rel_bias=mv(l.rel_bias), attn_post=mv(l.attn_post),
                               ffn_post=mv(l.ffn_post), mamba=mv(l.mamba), gla=mv(l.gla), latent=mv(l.latent), sink=mv(l.sink), conv_w=mv(l.conv_w),
                               rot_freq=mv(l.rot_freq), rwkv=mv(l.rwkv), side=mv(l.side), gru=mv(l.gru), log_bias=mv(l.log_bias), sh_up=mv(l.sh_up), sh_dot=mv(l.sh_dot), depth_w=mv(l.depth_w)) for l in self.layers]
        return ModelWeights(cfg=self.cfg, embed=mv(self.embed), layers=layers, final_norm=mv(self.final_norm), lm_head=mv(self.lm_head),
                            fmt=self.fmt, tp_rank=self.tp_rank, tp_size=self.tp_size, ep_rank=self.ep_rank, ep_size=self.ep_size,
                            vocab_start=self.vocab_start, loop_step=mv(self.loop_step), side_embed=mv(self.side_embed))

    def tile_(self) -> "ModelWeights":
        """Put every projection matrix into the tiled weight layout (in place).  An LM head that shares its storage with
        the embedding table (tied embeddings) stays row-major: the embedding lookup reads rows."""
        for l in self.layers:
            for lw in l.linears():
                lw.tile_()
        if self.lm_head.w is not None and self.lm_head.w.data_ptr() != self.embed.data_ptr():
            self.lm_head.tile_()
        return self

    def nbytes(self) -> int:
        tot = self.embed.numel() * 2 + self.lm_head.nbytes()
        for l in self.layers:
            for lw in l.linears():
                tot += lw.nbytes()
        return tot


def ffn_shard(f: int, tp_size: int, tp_rank: int, fmt: str):
    """Column range of the FFN width owned by a tensor-parallel rank.  Formats that keep ggml blocks cut on 256-column boundaries
    (a K-quant super-block cannot be split), with the remainder going to the low ranks as in common/glm5.h:178-202 (its
    block-aligned variant); the others split evenly."""
    if (fmt in QUANT_FMTS or fmt == "ggml") and tp_size > 1 and f % 256 == 0:
        lo, hi = shard_range(f // 256, tp_size, tp_rank)
        return lo * 256, hi * 256
    assert f % tp_size == 0
    f_l = f // tp_size
    return tp_rank * f_l, (tp_rank + 1) * f_l


def shard_range(n: int, parts: int, idx: int):
    """Even split with the remainder to the low ranks (the rule of common/glm5.h:178-202)."""
    q, r = divmod(n, parts)
    lo = idx * q + min(idx, r)
    return lo, lo + q + (1 if idx < r else 0)


class RandomSource:
    """Tensor source of a random-init checkpoint: N(0, 0.02) matrices, unit norms, zero biases... every tensor
    (and every expert) has its own seed derived from its GGUF name, so shards are slices of the same model."""

    def __init__(self, cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02):
        self.cfg, self.seed, self.device, self.std = cfg, seed, torch.device(device), std
        self._gen = torch.Generator(device=self.device)

    def _randn(self, key: str, shape) -> torch.Tensor:
        self._gen.manual_seed((zlib.crc32(key.encode()) ^ (self.seed * 2654435761)) & 0x7FFFFFFF)
        return torch.randn(tuple(shape), generator=self._gen, device=self.device, dtype=torch.float32).mul_(self.std).to(torch.bfloat16)

    def has(self, name: str) -> bool:
        return True

    def get(self, name: str, shape) -> torch.Tensor:
        if name.endswith(".alpha"):
            return torch.full(tuple(shape), 0.75, dtype=torch.bfloat16, device=self.device)
        if name.endswith("post_scale.weight"):
            return torch.full(tuple(shape), 0.25, dtype=torch.bfloat16, device=self.device)
        if name.endswith("ssm_a_log"):                   # decay rates 1 .. 16 over the heads
            return torch.linspace(0.0, 2.75, shape[0], device=self.device).to(torch.bfloat16)
        if self.cfg.is_layered and name.endswith("ssm_dt.bias"):
            return (self._randn(name, shape).float() * 25 - 3.0).to(torch.bfloat16)
        if name.endswith("gla_lower"):
            return (self._randn(name, shape).float() * 5 + 0.5).clamp(0.0, 0.95).to(torch.bfloat16)
        if "rwkv_mu_" in name:
            return (self._randn(name, shape).float() * 10 + 0.5).clamp(0.0, 1.0).to(torch.bfloat16)
        if name.endswith("rwkv_w0"):                     # decays of about exp(-exp(-3))
            return (self._randn(name, shape).float() * 50 - 3.0).to(torch.bfloat16)
        if name.endswith("rwkv_u") or name.endswith(".conv"):
            return (self._randn(name, shape).float() * 25).to(torch.bfloat16)
        if name.endswith("depth_weights"):               # mostly the layer's own result
            w = self._randn(name, shape).float()
            w[-1] += 1.0
            return w.to(torch.bfloat16)
        if name.endswith("attn_r1") or name.endswith("attn_r2"):
            return (self._randn(name, shape).float().abs() * 10 + 0.1).to(torch.bfloat16)
        if name.endswith("gru_z.bias"):                  # states that hold for some ten to a hundred tokens
            return (self._randn(name, shape).float() * 50 - 3.0).to(torch.bfloat16)
        if name.endswith("_rows.norm"):
            return torch.ones(tuple(shape), dtype=torch.bfloat16, device=self.device)
        if name.endswith("norm.weight") and not name.endswith(("lin_norm.weight", "attn_kv_a_norm.weight")) and self.cfg.norm_offset:
            return torch.full(tuple(shape), 1.0 - self.cfg.norm_offset, dtype=torch.bfloat16, device=self.device)
        if name.endswith("norm.weight"):
            return torch.ones(tuple(shape), dtype=torch.bfloat16, device=self.device)
        if name.endswith("ssm_a"):                       # fixed decay constants are negative
            return -(self._randn(name, shape).float().abs() * 20 + 0.5).to(torch.bfloat16)
        if name.endswith("ssm_conv1d.weight") or name.endswith("ssm_alpha.weight") or name.endswith("ssm_beta.weight"):
            return (self._randn(name, shape).float() * 10).to(torch.bfloat16)
        if name.endswith(".bias"):
            return self._randn(name, shape)
        return self._randn(name, shape)

    def get_expert(self, name: str, e: int, shape) -> torch.Tensor:
        return self._randn(f"{name}#{e}", shape)


def _post_attn_norm_name(src, pre: str) -> str:
    """The norm before the FFN: ``ffn_norm`` (Qwen2/3) or ``post_attention_norm`` (Qwen3.5 GGUFs)."""
    if hasattr(src, "has") and not isinstance(src, RandomSource) and not src.has(pre + "ffn_norm.weight") and src.has(pre + "post_attention_norm.weight"):
        return "post_attention_norm.weight"
    return "ffn_norm.weight"


def _build_ffn(cfg, src, pre, lw, fmt, mv, dev, tp_rank, tp_size, ep_rank, ep_size) -> None:
    """Dense FFN or MoE (+ optional shared expert) of one layer into ``lw``."""
    h = cfg.hidden
    if cfg.is_moe:
        e, inter = cfg.n_experts, cfg.expert_ffn
        assert e % ep_size == 0
        e_l = e // ep_size
        lw.router = mv(src.get(pre + "ffn_gate_inp.weight", (e, h)).to(torch.bfloat16))
        if cfg.router == "sigmoid":
            lw.router_bias = torch.zeros(e, dtype=torch.float32, device=dev)
        w13 = torch.empty((e_l * 2 * inter, h), dtype=torch.bfloat16, device=dev)
        w2 = torch.empty((e_l * h, inter), dtype=torch.bfloat16, device=dev)
        for j in range(e_l):
            ge = ep_rank * e_l + j
            w13[j * 2 * inter: j * 2 * inter + inter] = mv(src.get_expert(pre + "ffn_gate_exps.weight", ge, (inter, h)))
            w13[j * 2 * inter + inter:(j + 1) * 2 * inter] = mv(src.get_expert(pre + "ffn_up_exps.weight", ge, (inter, h)))
            w2[j * h:(j + 1) * h] = mv(src.get_expert(pre + "ffn_down_exps.weight", ge, (h, inter)))
        lw.w13 = make_linear(w13, fmt, groups=e_l)
        lw.w2 = make_linear(w2, fmt, groups=e_l)
        del w13, w2
    else:
        f = cfg.ffn
        f0, f1 = ffn_shard(f, tp_size, tp_rank, fmt)
        wg = _rows(_mat(src, pre + "ffn_gate.weight", (f, h)), f0, f1)
        wu = _rows(_mat(src, pre + "ffn_up.weight", (f, h)), f0, f1)
        wd = _cols(_mat(src, pre + "ffn_down.weight", (h, f)), f0, f1)
        lw.w_gate_up = make_linear(mv(_cat([wg, wu])), fmt)
        lw.w_down = make_linear(mv(wd.contiguous()), fmt)
        del wg, wu, wd
    if cfg.is_moe and cfg.shared_expert_ffn > 0:
        fs = cfg.shared_expert_ffn
        lw.sh_gate_up = make_linear(mv(torch.cat([src.get(pre + "ffn_gate_shexp.weight", (fs, h)), src.get(pre + "ffn_up_shexp.weight", (fs, h))])), fmt)
        lw.sh_down = make_linear(mv(src.get(pre + "ffn_down_shexp.weight", (h, fs)).contiguous()), fmt)
        if not hasattr(src, "has") or src.has(pre + "ffn_gate_inp_shexp.weight"):
            lw.sh_gate = mv(src.get(pre + "ffn_gate_inp_shexp.weight", (h,)).to(torch.bfloat16).reshape(1, h).contiguous())


def build_weights(cfg: ModelConfig, src, fmt: str = "bf16", device="cuda", tp_rank: int = 0, tp_size: int = 1, ep_rank: int = 0,
                  ep_size: int = 1, shard_vocab: bool = False, n_layers: Optional[int] = None, layer_range=None,
                  tile: Optional[bool] = None) -> ModelWeights:
    """Assemble ``ModelWeights`` in format ``fmt`` from a tensor source that answers GGUF tensor names
    (``RandomSource``, ``loader.GGUFSource``, ``loader.SafetensorsSource``).  ``tile`` (default: on for CUDA devices) stores
    the projection matrices in the GEMM kernel's tiled layout.

    TP shards attention and the dense FFN Megatron style (q/k/v/gate/up by rows, o/down by columns; KV heads are
    replicated when ``n_kv_heads < tp_size``), EP keeps the experts ``[ep_rank * E/ep_size, (ep_rank+1) * E/ep_size)``."""
    if cfg.is_layered:
        if tp_size > 1 or ep_size > 1 or layer_range is not None or n_layers is not None:
            raise NotImplementedError("models described layer by layer run unsharded")
        return _build_layered(cfg, src, fmt, torch.device(device), tile)
    h, d = cfg.hidden, cfg.head_dim
    dev = torch.device(device)
    assert cfg.n_heads % tp_size == 0, "n_heads must divide by the TP size"
    hq_l = cfg.n_heads // tp_size
    if cfg.n_kv_heads >= tp_size:
        assert cfg.n_kv_heads % tp_size == 0
        hkv_l = cfg.n_kv_heads // tp_size
        kv_lo = tp_rank * hkv_l
    else:
        assert tp_size % cfg.n_kv_heads == 0
        hkv_l = 1
        kv_lo = tp_rank // (tp_size // cfg.n_kv_heads)
    q0, q1 = tp_rank * hq_l * d, (tp_rank + 1) * hq_l * d
    k0, k1 = kv_lo * d, (kv_lo + hkv_l) * d

    def mv(t):
        return t.to(dev)

    layers: List[LayerWeights] = []
    nl = n_layers if n_layers is not None else cfg.n_layers
    lo, hi = layer_range if layer_range is not None else (0, nl)       # pipeline stages keep a contiguous slice of layers
    for li in range(lo, hi):
        pre = f"blk.{li}."
        if cfg.is_ssm_layer(li):
            assert tp_size == 1, "Delta-Net layers are not tensor-parallel (the reference replicates them, test_transformer_parallel.c:351-364)"
            qd, di, hv = cfg.ssm_qkv_dim, cfg.ssm_d_inner, cfg.ssm_n_heads_v
            w_in = torch.cat([src.get(pre + "attn_qkv.weight", (qd, h)), src.get(pre + "attn_gate.weight", (di, h))])
            ssm = SsmWeights(
                w_in=make_linear(mv(w_in), fmt),
                w_ab=mv(torch.cat([src.get(pre + "ssm_alpha.weight", (hv, h)), src.get(pre + "ssm_beta.weight", (hv, h))]).to(torch.bfloat16).contiguous()),
                conv_w=mv(src.get(pre + "ssm_conv1d.weight", (qd, cfg.ssm_d_conv)).float().contiguous()),
                a=mv(src.get(pre + "ssm_a", (hv,)).float().contiguous()), dt_bias=mv(src.get(pre + "ssm_dt.bias", (hv,)).float().contiguous()),
                norm=mv(src.get(pre + "ssm_norm.weight", (cfg.ssm_head_dim,)).float().contiguous()),
                w_out=make_linear(mv(src.get(pre + "ssm_out.weight", (h, di)).contiguous()), fmt))
            del w_in
            lw = LayerWeights(attn_norm=mv(src.get(pre + "attn_norm.weight", (h,)).to(torch.bfloat16)), wqkv=None, wo=None,
                              ffn_norm=mv(src.get(pre + _post_attn_norm_name(src, pre), (h,)).to(torch.bfloat16)), ssm=ssm)
            _build_ffn(cfg, src, pre, lw, fmt, mv, dev, tp_rank, tp_size, ep_rank, ep_size)
            layers.append(lw)
            continue
        if cfg.attn_output_gate:
            # attn_q emits [Q_h | gate_h] per head (common/transformer.h:3857-3868): de-interleave, the gate rows go after V
            wqg = src.get(pre + "attn_q.weight", (2 * cfg.q_dim, h)).reshape(cfg.n_heads, 2, d, h)
            wq = wqg[:, 0].reshape(cfg.q_dim, h)[q0:q1]
            wgate = wqg[:, 1].reshape(cfg.q_dim, h)[q0:q1]
        else:
            wq = _rows(_mat(src, pre + "attn_q.weight", (cfg.q_dim, h)), q0, q1)
            wgate = None
        wk = _rows(_mat(src, pre + "attn_k.weight", (cfg.kv_dim, h)), k0, k1)
        wv = _rows(_mat(src, pre + "attn_v.weight", (cfg.kv_dim, h)), k0, k1)
        wo = _cols(_mat(src, pre + "attn_output.weight", (h, cfg.q_dim)), q0, q1)
        bias = None
        if cfg.qkv_bias:
            bias = torch.cat([src.get(pre + "attn_q.bias", (cfg.q_dim,))[q0:q1].float(), src.get(pre + "attn_k.bias", (cfg.kv_dim,))[k0:k1].float(),
                              src.get(pre + "attn_v.bias", (cfg.kv_dim,))[k0:k1].float()]).contiguous()
            bias = mv(bias)
        lw = LayerWeights(
            attn_norm=mv(src.get(pre + "attn_norm.weight", (h,)).to(torch.bfloat16)),
            wqkv=make_linear(mv(_cat([wq, wk, wv] + ([wgate] if wgate is not None else []))), fmt, bias=bias),
            wo=make_linear(mv(wo.contiguous()), fmt),
            ffn_norm=mv(src.get(pre + _post_attn_norm_name(src, pre), (h,)).to(torch.bfloat16)),
            q_norm=mv(src.get(pre + "attn_q_norm.weight", (d,)).to(torch.bfloat16)) if cfg.qk_norm else None,
            k_norm=mv(src.get(pre + "attn_k_norm.weight", (d,)).to(torch.bfloat16)) if cfg.qk_norm else None,
        )
        del wq, wk, wv, wo
        _build_ffn(cfg, src, pre, lw, fmt, mv, dev, tp_rank, tp_size, ep_rank, ep_size)
        layers.append(lw)
    embed_src = _mat(src, "token_embd.weight", (cfg.vocab, h))
    embed = mv(_to_float(embed_src).to(torch.bfloat16))          # the embedding lookup reads bf16 rows
    quant_head = fmt in QUANT_FMTS or fmt == "ggml"
    if cfg.tie_embeddings or not src.has("output.weight"):
        head_full = embed_src if (quant_head and isinstance(embed_src, QBlocks)) else embed
    else:
        head_src = _mat(src, "output.weight", (cfg.vocab, h))
        head_full = head_src if (quant_head and isinstance(head_src, QBlocks)) else mv(_to_float(head_src).to(torch.bfloat16))
    v0, v1 = (0, cfg.vocab)
    if shard_vocab and tp_size > 1:
        v0, v1 = shard_range(cfg.vocab, tp_size, tp_rank)
    head_rows = _rows(head_full, v0, v1).contiguous() if (v0, v1) != (0, cfg.vocab) else head_full
    # the LM head streams the largest matrix of a decode step: under the block formats it stays quantised too
    lm_head = make_linear(mv(head_rows), fmt if quant_head else "bf16")
    mw = ModelWeights(cfg=cfg, embed=embed, layers=layers, final_norm=mv(src.get("output_norm.weight", (h,)).to(torch.bfloat16)),
                      lm_head=lm_head, fmt=fmt, tp_rank=tp_rank, tp_size=tp_size, ep_rank=ep_rank, ep_size=ep_size, vocab_start=v0)
    if tile if tile is not None else dev.type == "cuda":
        mw.tile_()
    return mw


def _padded_linear(t: torch.Tensor, fmt: str, dev, bias: Optional[torch.Tensor] = None, groups: int = 0) -> LinearWeight:
    """A projection whose input rows are padded with zeros the way ``ops.stream`` pads them (``row_width``).  ``groups``: ``t`` is stacked group by
    group."""
    k = row_width(t.shape[1], torch.float32 if fmt == "f32" else torch.bfloat16)
    if k != t.shape[1]:
        t = torch.nn.functional.pad(t, (0, k - t.shape[1]))
    return make_linear(t.to(dev), fmt, bias=bias, groups=groups)


def _stack_at_128(a: torch.Tensor, b: torch.Tensor):
    """Rows of ``b`` behind those of ``a``, starting at a multiple of 128 (so that either part is a projection of its own in the tiled layout), the
    whole padded to a multiple of 128.  Returns (stack, first row of b)."""
    at = (a.shape[0] + 127) // 128 * 128
    out = torch.zeros((at + b.shape[0] + 127) // 128 * 128, a.shape[1], dtype=a.dtype, device=a.device)
    out[: a.shape[0]] = a
    out[at: at + b.shape[0]] = b
    return out, at


def _stack_at_8(parts: Dict[str, Optional[torch.Tensor]]):
    """Rows of the parts one behind the other, each starting at a multiple of 8 (zero rows in between).  Returns (stack, first row of each part)."""
    rows, at, n = [], {}, 0
    for name, t in parts.items():
        if t is not None:
            at[name] = n
            rows += [t] + ([t.new_zeros(-t.shape[0] % 8, t.shape[1])] if t.shape[0] % 8 else [])
            n += (t.shape[0] + 7) // 8 * 8
    return torch.cat(rows), at


class _LayeredBuilder:
    """Weights of a model described layer by layer.  Norm weights become f32 ``offset + w``; the factor of the logits is folded into the
    final norm's weight, the per-channel scale behind a post norm into that norm."""

    def __init__(self, cfg: ModelConfig, src, fmt: str, dev):
        self.cfg, self.src, self.fmt, self.dev, self.exact = cfg, src, fmt, dev, fmt == "f32"
        self.h = cfg.hidden

    def get(self, name, *shape):
        return self.src.get(name, shape)

    def f32(self, name, *shape):
        return self.get(name, *shape).float().contiguous().to(self.dev)

    def linear(self, t, **kw) -> LinearWeight:
        return _padded_linear(t, self.fmt, self.dev, **kw)

    def norm(self, name, scale=None):
        """A norm over the stream; ``scale``: name of a per-channel factor of its result."""
        w = (self.get(name + ".weight", self.h).float() + self.cfg.norm_offset).contiguous().to(self.dev)
        if self.cfg.norm_kind == "rms":
            return w
        b = self.f32(name + ".bias", self.h)
        if scale is not None:
            s = self.f32(scale, self.h)
            w, b = w * s, b * s                      # products of bf16 values: exact in f32
        return DynTanh(float(self.get(name + ".alpha").float()), w, b)

    def lightning(self, pre, sp, lw):
        h, nv = self.h, sp.n_heads * sp.v_dim
        w_in = torch.cat([self.get(pre + "lin_q.weight", sp.q_dim, h), self.get(pre + "lin_k.weight", sp.q_dim, h),
                          self.get(pre + "lin_v.weight", nv, h), self.get(pre + "lin_gate.weight", nv, h)])
        lw.lin = LightningWeights(w_in=self.linear(w_in), decay=torch.tensor(sp.decay, dtype=torch.float32, device=self.dev),
                                  norm=self.f32(pre + "lin_norm.weight", nv), w_out=self.linear(self.get(pre + "lin_out.weight", h, nv)))

    def mamba2(self, pre, sp, lw):
        h, nv, ch = self.h, sp.n_heads * sp.v_dim, sp.conv_channels
        w = self.get(pre + "ssm_in.weight", nv + ch + sp.n_heads, h)
        w_in, at = _stack_at_128(w[: nv + ch], w[nv + ch:])
        a = -torch.exp(self.get(pre + "ssm_a_log", sp.n_heads).double()).float().contiguous().to(self.dev)
        lw.mamba = Mamba2Weights(w_in=self.linear(w_in), dt_row=at, conv_w=self.f32(pre + "ssm_conv1d.weight", ch, sp.conv_taps), conv_b=self.f32(pre + "ssm_conv1d.bias", ch),
                                 dt_bias=self.f32(pre + "ssm_dt.bias", sp.n_heads), a=a, d=self.f32(pre + "ssm_d", sp.n_heads), norm=self.f32(pre + "ssm_norm.weight", nv),
                                 w_out=self.linear(self.get(pre + "ssm_out.weight", h, nv)))

    def hgrn2(self, pre, sp, lw):
        h, nv = self.h, sp.n_heads * sp.v_dim
        w_in, at = _stack_at_128(torch.cat([self.get(pre + "gla_q.weight", sp.q_dim, h), self.get(pre + "gla_v.weight", nv, h)]), self.get(pre + "gla_f.weight", sp.q_dim, h))
        lw.gla = GlaWeights(w_in=self.linear(w_in), f_row=at, f_bias=self.f32(pre + "gla_f.bias", sp.q_dim), lower=self.f32(pre + "gla_lower", sp.q_dim),
                            norm=self.f32(pre + "gla_norm.weight", sp.v_dim), w_out=self.linear(self.get(pre + "gla_out.weight", h, nv)))

    def latent(self, pre, sp, lw):
        h, hd, d, v, r, qr = self.h, sp.n_heads, sp.head_dim, sp.v_dim, sp.kv_rank, sp.q_rank
        order = torch.tensor(sp.rotary.pair_order())                     # pairs side by side, as the kernels rotate them
        turn = lambda w, at: torch.cat([w[..., :at, :], w[..., at + order.to(w.device), :]], -2)
        q_of = lambda w: turn(w.reshape(hd, d + sp.rot_dim, -1), d).reshape(w.shape)
        kv_a = turn(self.get(pre + "attn_kv_a.weight", r + sp.rot_dim, h), r) if sp.kv_from < 0 else None
        kv_norm = self.f32(pre + "attn_kv_a_norm.weight", r) if sp.kv_from < 0 else None
        w_qb = cols = None
        if qr:
            w_a = self.get(pre + "attn_q_a.weight", qr, h)
            w_a = torch.cat([w_a, kv_a]) if kv_a is not None else w_a
            w_qb = self.linear(q_of(self.get(pre + "attn_q_b.weight", hd * (d + sp.rot_dim), qr)))
        else:
            w_a, cols = _stack_at_8({"q": q_of(self.get(pre + "attn_q_direct.weight", hd * (d + sp.rot_dim), h)), "kv": kv_a,
                                     "gate": self.get(pre + "attn_gate.weight", hd * v, h) if sp.out_gate else None})
        uk, uv = self.get(pre + "attn_k_b.weight", hd * d, r).reshape(hd, d, r), self.get(pre + "attn_v_b.weight", hd * v, r).reshape(hd, v, r)
        w_kv, pad = None, torch.nn.functional.pad
        rows_k, v8 = r, v
        if not self.exact:
            d8, v8 = row_width(d, torch.bfloat16), row_width(v, torch.bfloat16)      # heads are padded; the output projection has zero columns there
            uv = pad(uv, (0, 0, 0, v8 - v))
            w_kv = self.linear(torch.cat([pad(uk, (0, 0, 0, d8 - d)).reshape(hd * d8, r), uv.reshape(hd * v8, r)]))
            rows_k = (r + 127) // 128 * 128          # whole 128-row tiles per head
        lw.latent = LatentWeights(
            w_a=self.linear(w_a), q_norm=self.f32(pre + "attn_q_a_norm.weight", qr) if qr else None, kv_norm=kv_norm, w_qb=w_qb, w_kv=w_kv, cols=cols,
            w_uk=self.linear(pad(uk.transpose(1, 2), (0, 0, 0, rows_k - r)).reshape(hd * rows_k, d), groups=hd),
            w_uv=self.linear(uv.reshape(hd * v8, r), groups=hd),
            sink=(self.get(pre + "attn_sink", hd).double() * LOG2E).float().contiguous().to(self.dev) if sp.sink else None,
            freq=torch.tensor(sp.rotary.frequencies(), dtype=torch.float64, device=self.dev))
        lw.wo = self.linear(pad(self.get(pre + "attn_output.weight", h, hd * v).reshape(h, hd, v), (0, v8 - v)).reshape(h, hd * v8))

    def attention(self, pre, sp, lw):
        h, nv = self.h, sp.n_heads * sp.v_dim
        nk, nkv = sp.n_kv_heads * sp.head_dim, sp.n_kv_heads * sp.v_dim
        rows = [("q", sp.q_dim), ("k", nk)] + ([] if sp.v_from_k else [("v", nkv)])
        bias = None
        if sp.qkv_bias:
            bias = [self.get(pre + f"attn_{c}.bias", n).float() for c, n in rows]
            bias = torch.cat(bias + ([bias[0].new_zeros(nv)] if sp.out_gate else [])).contiguous().to(self.dev)
        w = torch.cat([self.get(pre + f"attn_{c}.weight", n, h) for c, n in rows + ([("gate", nv)] if sp.out_gate else [])])
        lw.wqkv = self.linear(w, bias=bias)
        if sp.qk_norm_rows:
            lw.q_norm, lw.k_norm = self.f32(pre + "attn_q_rows.norm", sp.q_dim), self.f32(pre + "attn_k_rows.norm", nk)
        if sp.conv_taps:
            lw.conv_w = torch.cat([self.f32(pre + "attn_q.conv", sp.q_dim, sp.conv_taps), self.f32(pre + "attn_k.conv", nk, sp.conv_taps)]).contiguous()
        if sp.rotary is not None:
            lw.rot_freq = torch.tensor(sp.rotary.frequencies(), dtype=torch.float64, device=self.dev)
        if sp.sink:
            lw.sink = (self.get(pre + "attn_sink", sp.n_heads).double() * LOG2E).float().contiguous().to(self.dev)
        if sp.log_bias:
            lw.log_bias = torch.stack([self.f32(pre + "attn_r1", sp.n_heads), self.f32(pre + "attn_r2", sp.n_heads)]).contiguous()
        # the attention kernels emit heads of the cache's (padded) value width: the output projection has zero columns there
        wo = self.get(pre + "attn_output.weight", h, nv)
        dvp = cache_head_dims(sp.head_dim, sp.v_dim, torch.float32 if self.exact else torch.bfloat16)[1]
        wo = torch.nn.functional.pad(wo.reshape(h, sp.n_heads, sp.v_dim), (0, dvp - sp.v_dim)).reshape(h, sp.n_heads * dvp)
        lw.wo = self.linear(wo)
        if sp.rel_buckets:
            lw.rel_bias = distance_bias_table(self.get(pre + "attn_rel.weight", sp.rel_buckets, sp.n_heads).float().cpu(), sp.rel_max).to(self.dev)

    def mingru(self, pre, sp, lw):
        h, n = self.h, sp.v_dim
        w_in, at = _stack_at_128(torch.cat([self.get(pre + "gru_x.weight", n, h), self.get(pre + "gru_gate.weight", n, h)]), self.get(pre + "gru_z.weight", n, h))
        lw.gru = MinGruWeights(w_in=self.linear(w_in), z_row=at, z_bias=self.f32(pre + "gru_z.bias", n), x_bias=self.f32(pre + "gru_x.bias", n),
                               w_out=self.linear(self.get(pre + "gru_out.weight", h, n)))

    def rwkv(self, pre, sp, lw):
        h, nq, nv = self.h, sp.q_dim, sp.n_heads * sp.v_dim
        assert nq == nv, "the four projections of the mixes share a size"
        np_ = nq if self.exact else (nq + 127) // 128 * 128              # whole 128-row tiles per group
        w = [torch.nn.functional.pad(self.get(pre + f"rwkv_{c}.weight", nq, h), (0, 0, 0, np_ - nq)) for c in "rkvg"]
        w2 = self.get(pre + "rwkv_w2.weight", nq, sp.decay_rank)
        lw.rwkv = RwkvWeights(mu=torch.stack([self.f32(pre + f"rwkv_mu_{c}", h) for c in "rkvgw"]).contiguous(), w_in=self.linear(torch.cat(w), groups=4),
                              w1=self.linear(self.get(pre + "rwkv_w1.weight", sp.decay_rank, h)), w2=self.linear(w2), w2_rows=None if self.exact else w2.to(torch.bfloat16).contiguous().to(self.dev, copy=True),
                              w0=self.f32(pre + "rwkv_w0", nq), u=self.f32(pre + "rwkv_u", sp.n_heads, sp.head_dim).reshape(-1), norm=self.f32(pre + "rwkv_norm.weight", nv),
                              w_out=self.linear(self.get(pre + "rwkv_out.weight", h, nv)))

    def parallel(self, pre, sp, lw):
        """Both mixers' weights are parts of one layer's: they have no name in common."""
        for part, mx in (("left.", sp.left), ("right.", sp.right)):
            getattr(self, mx.mixer)(pre + part, mx, lw)

    def side(self, pre, lw):
        h, d = self.h, self.cfg.side_dim
        lw.side = SideWeights(gate=self.linear(self.get(pre + "side_gate.weight", d, h)), proj=self.linear(self.get(pre + "side_proj.weight", h, d)),
                              norm=self.f32(pre + "side_norm.weight", h))

    def dense_ffn(self, pre, sp, lw):
        h = self.h
        wg, wu = self.get(pre + "ffn_gate.weight", sp.ffn, h), self.get(pre + "ffn_up.weight", sp.ffn, h)
        wd = self.get(pre + "ffn_down.weight", h, sp.ffn)
        fp = sp.ffn if self.exact else (sp.ffn + 127) // 128 * 128       # the gate / up GEMM works on whole 128-row tiles
        pad = torch.nn.functional.pad
        bias = down_bias = None
        if sp.ffn_bias:
            bias = torch.cat([pad(self.f32(pre + f"ffn_{c}.bias", sp.ffn), (0, fp - sp.ffn)) for c in ("gate", "up")]).contiguous()
            down_bias = self.f32(pre + "ffn_down.bias", h)
        lw.w_gate_up = self.linear(torch.cat([pad(wg, (0, 0, 0, fp - sp.ffn)), pad(wu, (0, 0, 0, fp - sp.ffn))]), bias=bias)
        lw.w_down = self.linear(pad(wd, (0, fp - sp.ffn)), bias=down_bias)

    def moe_ffn(self, pre, sp, lw):
        """Expert weights with the expert width and, per expert, the rows of the down projection padded to whole 128-row tiles (bf16)."""
        h, m = self.h, sp.moe
        dt = torch.float32 if self.exact else torch.bfloat16
        up = lambda n: n if self.exact else (n + 127) // 128 * 128
        k, ip, hp, n_in = row_width(h, dt), up(m.ffn), up(h), 2 if m.gated else 1
        lw.router = torch.nn.functional.pad(self.get(pre + "ffn_gate_inp.weight", m.n_experts, h).to(dt), (0, k - h)).contiguous().to(self.dev)
        w13 = torch.zeros(m.n_experts, n_in, ip, k, dtype=dt, device=self.dev)
        w2 = torch.zeros(m.n_experts, hp, ip, dtype=dt, device=self.dev)
        for e in range(m.n_experts):
            if m.gated:
                w13[e, 0, : m.ffn, :h] = self.src.get_expert(pre + "ffn_gate_exps.weight", e, (m.ffn, h)).to(self.dev)
            w13[e, n_in - 1, : m.ffn, :h] = self.src.get_expert(pre + "ffn_up_exps.weight", e, (m.ffn, h)).to(self.dev)
            w2[e, :h, : m.ffn] = self.src.get_expert(pre + "ffn_down_exps.weight", e, (h, m.ffn)).to(self.dev)
        lw.w13 = make_linear(w13.reshape(-1, k), self.fmt, groups=m.n_experts)
        lw.w2 = make_linear(w2.reshape(-1, ip), self.fmt, groups=m.n_experts)
        if m.shared:
            pad, sp_ = torch.nn.functional.pad, up(m.shared)
            lw.sh_up = self.linear(pad(self.get(pre + "ffn_up_shexp.weight", m.shared, h), (0, 0, 0, sp_ - m.shared)))
            lw.sh_down = self.linear(pad(self.get(pre + "ffn_down_shexp.weight", h, m.shared), (0, sp_ - m.shared)))
            lw.sh_dot = (self.f32(pre + "ffn_gate_inp_shexp.weight", 1, h)[0] * lw.ffn_norm).contiguous()

    def layer(self, li: int, sp) -> LayerWeights:
        pre, post = f"blk.{li}.", self.cfg.post_norm
        lw = LayerWeights(attn_norm=self.norm(pre + "attn_norm"), wqkv=None, wo=None, ffn_norm=self.norm(pre + "ffn_norm") if sp.has_ffn else None)
        if post:
            lw.attn_post = self.norm(pre + "attn_post_norm", pre + "attn_post_scale.weight")
            lw.ffn_post = self.norm(pre + "ffn_post_norm", pre + "ffn_post_scale.weight") if sp.has_ffn else None
        getattr(self, sp.mixer)(pre, sp, lw)
        if sp.ffn:
            self.dense_ffn(pre, sp, lw)
        elif sp.moe is not None:
            self.moe_ffn(pre, sp, lw)
        if self.cfg.side_dim:
            self.side(pre, lw)
        if self.cfg.depth_average:
            lw.depth_w = self.f32(pre + "depth_weights", li + 2)
        return lw

    def model(self) -> ModelWeights:
        cfg, h, src = self.cfg, self.h, self.src
        layers = [self.layer(li, sp) for li, sp in enumerate(cfg.layer_specs)]
        dt = torch.float32 if self.exact else torch.bfloat16
        embed = self.get("token_embd.weight", cfg.vocab, h).to(dt).contiguous().to(self.dev)
        side = self.get("side_embd.weight", cfg.vocab, cfg.n_layers * cfg.side_dim).to(dt).contiguous().to(self.dev) if cfg.side_dim else None
        head = embed if (cfg.tie_embeddings or not src.has("output.weight")) else self.get("output.weight", cfg.vocab, h)
        step = self.f32("loop_step.weight", cfg.loop.times, h) if cfg.loop is not None and cfg.loop.add == "step" else None
        final = self.norm("output_norm")
        if cfg.norm_kind == "rms":
            final = final * cfg.logit_scale
        return ModelWeights(cfg=cfg, embed=embed, layers=layers, final_norm=final, lm_head=self.linear(head), fmt=self.fmt, loop_step=step, side_embed=side)


def _build_layered(cfg: ModelConfig, src, fmt: str, dev, tile: Optional[bool]) -> ModelWeights:
    if fmt not in ("bf16", "f32"):
        raise ValueError(f"models described layer by layer run in bf16 or f32, not {fmt!r}")
    mw = _LayeredBuilder(cfg, src, fmt, dev).model()
    if (tile if tile is not None else dev.type == "cuda") and fmt != "f32":
        mw.tile_()
    return mw


def synthetic_weights(cfg: ModelConfig, fmt: str = "bf16", device="cuda", seed: int = 0, tp_rank: int = 0, tp_size: int = 1,
                      ep_rank: int = 0, ep_size: int = 1, shard_vocab: bool = False, n_layers: Optional[int] = None,
                      layer_range=None) -> ModelWeights:
    """Random-init weights of ``cfg`` (generated on ``device``) in format ``fmt``."""
    return build_weights(cfg, RandomSource(cfg, seed, device), fmt, device, tp_rank, tp_size, ep_rank, ep_size, shard_vocab, n_layers,
                         layer_range)
