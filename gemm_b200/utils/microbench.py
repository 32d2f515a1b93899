"""Kernel micro-benchmarks: ``python -m gemm_b200.utils.microbench --case <name> [--iters N]``.

Every case times one op of the library on shapes of the Qwen3-30B-A3B benchmark configuration with CUDA events on the
launching stream, after warm-up, with the L2 flushed (a 256 MiB buffer is rewritten) before every timed launch, and
prints one JSON line per measurement: achieved TFLOP/s and GB/s of the bytes that must come from HBM.  ``--once`` runs
each op a single time without timing (the form to put under a profiler).

Cases
  gemm         dense projections: decode (64 tokens) and prefill (16384 tokens), bf16 and MXFP8
  moe_decode   grouped expert GEMMs (gate/up with SwiGLU + re-quantisation, down) for 64 tokens x top-8 of 128 experts, as two
               launches and as the one persistent launch
  moe_prefill  the same for 16384 tokens
  attn_decode  paged flash-decode, 64 sequences x 2048 cached tokens, 32 query / 4 KV heads
  attn_prefill causal prefill, 8 sequences x 2048 tokens
  lm_head      64 x 151936 x 2048 with the arg-max epilogue
  quant        ggml-quantised projections of the Qwen3-32B shape (Q4_K and Q8_0 blocks kept in HBM): fused dequant-GEMV for
               1 and 4 tokens, fused dequant-GEMM for 8, 64 and 4096 tokens
  small        the kernels around them: RMSNorm + residual + MXFP8 copy, QK-norm + RoPE + cache write (64 and 16384 tokens), the
               one-launch MoE front end, sampler and arg-max over 64 x 151936 logits, the Delta-Net recurrence (decode, prefill)
  layered      the kernels of models described layer by layer beside the like kernels of the other models at equal size: lightning
               attention (decode, prefill) and the Delta-Net recurrence; windowed attention with kept tokens and distance bias and the
               plain causal kernels; the f32-stream norm, Q / K unit norm and gated norm and their bf16-stream counterparts
  famepel      the kernels of Famepel at the sizes of ``famepel-30b-a3b`` beside the like kernels of the other models: Mamba-2 and HGRN2
               scans and Delta-Net; latent attention and plain attention; Dynamic-Tanh stream and RMSNorm, part norm, convolution, routing
  fidolix      the kernels of Fidolix at the sizes of ``fidolix-30b-a3b`` beside the like kernels of the other models: RWKV (HGRN2), token shift,
               convolution and rotation, norms of Q and K, capped scores and sinks (plain attention), the stream's norms and sums
  zedirax      the kernels of Zedirax at the sizes of ``zedirax-30b-a3b`` beside the like kernels of the other models: minGRU (HGRN2), logarithmic distance
               bias (a table of biases, plain attention), the average over earlier layers (the stream's norms and sums), GELU epilogues
  spec_verify  whole-model step over 1, 2, 3 and 5 positions per sequence (speculative verification against plain decode);
               builds the full Qwen3-30B-A3B shape, not part of ``all``

Counterpart in the reference: cuda/gemm/bench_log.md and cuda/fa2/bench_log.md are produced by stand-alone bench
programs of the same kind.
"""
from __future__ import annotations

import argparse
import json

import torch

from .. import _native
from ..ops import attention as att
from ..ops import elementwise as ew
from ..ops import gemm, moe, mxfp8

_flush = None


def _timeit(fn, iters: int, warm: int = 3) -> float:
    """Median milliseconds of ``fn`` (L2 flushed before each timed call)."""
    global _flush
    if _flush is None:
        _flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(warm):
        fn()
    ts = []
    for _ in range(iters):
        _flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    ts.sort()
    return ts[len(ts) // 2]


def _emit(name: str, ms: float, flops: float, hbm_bytes: float, **kw) -> None:
    print(json.dumps(dict(case=name, ms=round(ms, 5), tflops=round(flops / ms / 1e9, 1), hbm_gbs=round(hbm_bytes / ms / 1e6, 1), **kw)),
          flush=True)


def _run(name, fn, flops, hbm_bytes, args, **kw):
    if args.once:
        fn()
        torch.cuda.synchronize()
        print(json.dumps(dict(case=name, ran="once")), flush=True)
        return
    _emit(name, _timeit(fn, args.iters), flops, hbm_bytes, **kw)


def case_gemm(args):
    for (m, n, k) in [(64, 5120, 2048), (64, 2048, 4096), (16384, 5120, 2048), (16384, 2048, 4096), (8192, 8192, 8192)]:
        x = (torch.randn(m, k, device="cuda") * 0.5).bfloat16()
        w = (torch.randn(n, k, device="cuda") * 0.05).bfloat16()
        wt = mxfp8.tile_weight(w)
        _run(f"gemm_bf16_{m}x{n}x{k}", lambda: gemm.linear(x, wt, w_tiled=True), 2.0 * m * n * k, n * k * 2 + m * k * 2 + m * n * 2, args)
        if not args.once:
            _emit(f"torch_matmul_{m}x{n}x{k}", _timeit(lambda: torch.matmul(x, w.t()), args.iters), 2.0 * m * n * k, n * k * 2 + m * k * 2 + m * n * 2)
        xq = mxfp8.quantize(x.float(), sf_layout=32 if m <= 32 else 128)
        wq = mxfp8.quantize(w.float())
        wq = mxfp8.MxTensor(mxfp8.tile_weight(wq.data), wq.sf, wq.rows, wq.k, 128, tiled=True)
        _run(f"gemm_mxfp8_{m}x{n}x{k}", lambda: gemm.linear_mx(xq, wq), 2.0 * m * n * k, n * k + m * k + m * n * 2, args)


def _moe(args, t: int, name: str):
    e, kk, h, inter = 128, 8, 2048, 768
    tn = 32 if (t * kk) // e <= 24 else 128
    ids, _ = moe.route(torch.randn(t, e, device="cuda"), kk)
    pl = moe.plan(ids, e, tn)
    x = torch.randn(t, h, device="cuda").bfloat16()
    xq = ew.mx_quantize(x, pl.row_token, sf_layout=tn)
    w1 = mxfp8.quantize(torch.randn(e * 2 * inter, h, device="cuda") * 0.05)
    w2 = mxfp8.quantize(torch.randn(e * h, inter, device="cuda") * 0.05)
    d1, d2 = mxfp8.tile_weight(w1.data), mxfp8.tile_weight(w2.data)
    hq = torch.empty(pl.capacity, inter, dtype=torch.uint8, device="cuda")
    hsf = ew.sf_alloc(pl.capacity, inter, "cuda", tn, init=False)

    gu = torch.empty(pl.capacity, 2 * inter, dtype=torch.bfloat16, device="cuda") if tn == 128 else None

    def gate_up():
        if tn == 32:        # decode: SiLU(gate) * up and the re-quantisation run in the GEMM epilogue
            gemm.grouped_linear(xq.data, d1.view(e, 2 * inter, h), pl.seg_start, pl.seg_count, tn, out=hq, dual=True, sfa=w1.sf, sfb=xq.sf,
                                quant_out=True, out_sf=hsf, w_tiled=True)
        else:               # prefill: plain GEMM over the stacked rows (256-token tiles) + one fused activation / quantise pass
            gemm.grouped_linear(xq.data, d1.view(e, 2 * inter, h), pl.seg_start, pl.seg_count, tn, out=gu, sfa=w1.sf, sfb=xq.sf, w_tiled=True)
            ew.silu_mul_quant(gu, hq, hsf, pl.row_token, sf_layout=tn)

    def down():
        gemm.grouped_linear(hq, d2.view(e, h, inter), pl.seg_start, pl.seg_count, tn, sfa=w2.sf, sfb=hsf, w_tiled=True, pair_rows=(tn == 32))

    gate_up()
    touched = int((pl.seg_count > 0).sum())
    fl = 2.0 * t * kk * h * inter
    _run(f"{name}_gate_up", gate_up, 2 * fl, touched * 2 * h * inter + t * kk * h, args, tn=tn, experts_touched=touched)
    _run(f"{name}_down", down, fl, touched * h * inter + t * kk * inter + t * kk * h * 2, args, tn=tn, experts_touched=touched)
    if tn == 32:
        # the same two projections as one persistent launch
        from ..models.weights import LinearWeight
        lw1 = LinearWeight("mxfp8", 2 * inter, h, mx=mxfp8.MxTensor(d1, w1.sf, e * 2 * inter, h, 128, tiled=True), groups=e, rows_per_group=2 * inter)
        lw2 = LinearWeight("mxfp8", h, inter, mx=mxfp8.MxTensor(d2, w2.sf, e * h, inter, 128, tiled=True), groups=e, rows_per_group=h)
        if moe.can_fuse_ffn(xq, lw1, lw2, e, pl.capacity):
            _run(f"{name}_ffn_fused", lambda: moe.expert_ffn_fused(xq, lw1, lw2, e, pl), 3 * fl,
                 touched * 3 * h * inter + t * kk * h + t * kk * h * 2, args, tn=tn, experts_touched=touched)


def case_moe_decode(args):
    _moe(args, 64, "moe_decode")
    # what ONE rank of an 8-way expert-parallel group runs per layer: all 64 gathered tokens against its 16 local experts
    from ..models.weights import LinearWeight
    e_all, e_loc, kk, h, inter = 128, 16, 8, 2048, 768
    x = torch.randn(64, h, device="cuda").bfloat16()
    router = (torch.randn(e_all, h, device="cuda") * 0.05).bfloat16()
    w1 = mxfp8.quantize(torch.randn(e_loc * 2 * inter, h, device="cuda") * 0.05)
    w2 = mxfp8.quantize(torch.randn(e_loc * h, inter, device="cuda") * 0.05)
    lw1 = LinearWeight("mxfp8", 2 * inter, h, mx=mxfp8.MxTensor(mxfp8.tile_weight(w1.data), w1.sf, e_loc * 2 * inter, h, 128, tiled=True),
                       groups=e_loc, rows_per_group=2 * inter)
    lw2 = LinearWeight("mxfp8", h, inter, mx=mxfp8.MxTensor(mxfp8.tile_weight(w2.data), w2.sf, e_loc * h, inter, 128, tiled=True),
                       groups=e_loc, rows_per_group=h)
    if moe.can_prep(x, router, kk):
        ids, wts, pl, xq = moe.prep_hidden(x, router, kk, e_loc, 32, local_range=(32, e_loc))
        touched = int((pl.seg_count > 0).sum())
        pairs = int(pl.seg_count.sum())
        _run("moe_prep_ep8_rank", lambda: moe.prep_hidden(x, router, kk, e_loc, 32, local_range=(32, e_loc)), 0.0, e_all * h * 2 + 64 * h * 2, args,
             local_pairs=pairs)
        if moe.can_fuse_ffn(xq, lw1, lw2, e_loc, pl.capacity):
            _run("moe_ffn_fused_ep8_rank", lambda: moe.expert_ffn_fused(xq, lw1, lw2, e_loc, pl), 6.0 * pairs * h * inter,
                 touched * 3 * h * inter + pairs * h * 3, args, experts_touched=touched, local_pairs=pairs)


def case_moe_prefill(args):
    _moe(args, 16384, "moe_prefill")


def _attn(args, b: int, q_len: int, ctx: int, name: str):
    hq, hkv, d, page = args.hq, args.hkv, 128, args.page
    b = args.batch if args.batch > 0 else b
    ctx = args.ctx if args.ctx >= 0 else ctx
    pages_per = (ctx + q_len + page - 1) // page
    n_pages = b * pages_per + 1
    k = (torch.randn(n_pages * page, hkv, d, device="cuda") * 0.5).bfloat16()
    v = (torch.randn(n_pages * page, hkv, d, device="cuda") * 0.5).bfloat16()
    bt = (torch.arange(b * pages_per, device="cuda", dtype=torch.int32) + 1).reshape(b, pages_per)
    q = (torch.randn(b * q_len, hq, d, device="cuda") * 0.5 * ew.softmax_scale_log2(d)).bfloat16()
    q_lens = [q_len] * b
    cu = torch.tensor([i * q_len for i in range(b + 1)], device="cuda", dtype=torch.int32)
    kv_len = torch.full((b,), ctx + q_len, device="cuda", dtype=torch.int32)
    splits = att.pick_splits(b, hkv, ctx + q_len) if q_len == 1 else 1
    if args.splits > 0:
        splits = args.splits
    work = att.build_work(q_lens, hq, hkv, splits).to("cuda")

    def run():
        att.attention(q, k, v, cu, kv_len, bt, page, work, num_splits=splits, causal=True, decode=(q_len == 1))

    kv_bytes = b * (ctx + q_len) * hkv * d * 2 * 2
    if q_len == 1:
        flops = 4.0 * b * hq * (ctx + 1) * d
    else:
        flops = 4.0 * b * hq * d * (q_len * ctx + q_len * (q_len + 1) / 2)
    _run(name, run, flops, kv_bytes + b * q_len * hq * d * 4, args, splits=splits, batch=b, ctx=ctx, hq=hq, hkv=hkv, page=page)
    if q_len == 1:
        # the same pages as int8 + one scale per slot and head, read directly by the INT8 decode attention kernel
        kq, vq = torch.empty(k.shape, dtype=torch.int8, device="cuda"), torch.empty(v.shape, dtype=torch.int8, device="cuda")
        ks, vs = torch.empty(k.shape[:2], device="cuda"), torch.empty(v.shape[:2], device="cuda")
        att.kv_store_q8(k, v, None, torch.arange(k.shape[0], dtype=torch.int32, device="cuda"), kq, vq, ks, vs)
        sp8 = args.splits if args.splits > 0 else max(1, min(8, (148 * 4) // max(1, b * hkv)))
        _run(name + "_int8_kv", lambda: att.attention_decode_q8(q, kq, vq, ks, vs, kv_len, bt, page, num_splits=sp8), flops,
             kv_bytes // 2 + b * (ctx + 1) * hkv * 8 + b * hq * d * 4, args, splits=sp8, batch=b, ctx=ctx, hq=hq, hkv=hkv, page=page)


def case_attn_decode(args):
    _attn(args, 64, 1, 2048, "attn_decode")


def case_attn_prefill(args):
    _attn(args, 8, 2048, 0, "attn_prefill")


def case_lm_head(args):
    m, n, k = 64, 151936, 2048
    x = (torch.randn(m, k, device="cuda") * 0.5).bfloat16()
    w = mxfp8.tile_weight((torch.randn(n, k, device="cuda") * 0.05).bfloat16())
    _run("lm_head_argmax", lambda: gemm.linear_argmax(x, w, w_tiled=True), 2.0 * m * n * k, n * k * 2, args)


def case_spec_verify(args):
    """Cost of a speculative-decoding verify step (1 + gamma query positions per sequence through the chunked-prefill path)
    against a plain decode step, on the benchmark model: 64 sequences x 2048 cached tokens, MXFP8."""
    from ..models.config import get_config
    from ..models.transformer import ForwardBatch
    from ..models.weights import synthetic_weights
    from ..serve.engine import Engine
    name, b, ctx = "qwen3-30b-a3b", (args.batch or 64), (args.ctx if args.ctx >= 0 else 2048)
    cfg = get_config(name)
    dev = torch.device("cuda", torch.cuda.current_device())
    w = synthetic_weights(cfg, "mxfp8", device=dev, seed=0)
    eng = Engine(w, max_batch=b, max_seq_len=ctx + 16, page_size=128, max_prefill_tokens=16384)
    g = torch.Generator().manual_seed(0)
    prompts = torch.randint(0, cfg.vocab, (b, ctx), generator=g, dtype=torch.int32)
    eng.prefill([prompts[i] for i in range(b)], reserve=8)
    bt = eng._block_table(range(b))
    variants = {}
    for q in (1, 2, 3, 5):
        ids = torch.randint(0, cfg.vocab, (b * q,), generator=g, dtype=torch.int32)
        splits = att.pick_splits(b, eng.hkv_local, ctx + 8) if q == 1 else 1
        variants[q] = ForwardBatch.build([q] * b, [ctx] * b, ids, bt, 128, eng.hq_local, eng.hkv_local, dev, num_splits=splits, all_logits=True)

    def timed(fn):
        for _ in range(2):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(max(3, args.iters // 2)):
            a, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            e.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(e))
        ts.sort()
        return ts[len(ts) // 2]

    with torch.no_grad():
        base = None
        for q, fb in variants.items():
            ms = timed(lambda: eng.model.forward_greedy(fb))
            base = base or ms
            print(json.dumps(dict(case="spec_verify_eager", positions_per_seq=q, tokens=b * q, ms=round(ms, 3), vs_one=round(ms / base, 3))), flush=True)
        base = None
        for q, fb in variants.items():             # the same steps replayed from a CUDA graph (no host time between launches)
            try:
                gr = torch.cuda.CUDAGraph()
                with torch.cuda.graph(gr):
                    eng.model.forward_greedy(fb)
                ms = timed(gr.replay)
            except Exception as exc:               # a host read inside the step cannot be captured: the eager figure stands
                print(json.dumps(dict(case="spec_verify_graph", positions_per_seq=q, error=str(exc)[:120])), flush=True)
                break
            base = base or ms
            print(json.dumps(dict(case="spec_verify_graph", positions_per_seq=q, tokens=b * q, ms=round(ms, 3), vs_one=round(ms / base, 3))), flush=True)


def case_quant(args):
    from ..ops import ggml_torch as gt
    from ..ops import qlinear
    shapes = [("qkv", 10240, 5120), ("gate_up", 51200, 5120), ("down", 5120, 25600)]
    if args.once:
        shapes = shapes[1:2]
    for tname, t in (("q4_k", gt.Q4_K), ("q8_0", gt.Q8_0)):
        blk, nb = gt.BLOCK[t]
        for (pname, n, k) in shapes:
            w = qlinear.QTensor.from_float(torch.randn(n, k, device="cuda") * 0.02, t)
            wbytes = n * (k // blk) * nb
            for m in ((1,) if args.once else (1, 4)):
                x = torch.randn(m, k, device="cuda").bfloat16()
                sp = qlinear.pick_splits(n, k, m, t)
                out = torch.empty(sp, m, n, dtype=torch.float32, device="cuda")
                _run(f"qgemv_{tname}_{pname}_{m}x{n}x{k}", lambda: qlinear.gemv_partials(x, w, splits=sp, out=out), 2.0 * m * n * k, wbytes, args, splits=sp)
            for m in ((64,) if args.once else (8, 64, 4096)):
                if m == 4096 and pname != "qkv":
                    continue
                x = torch.randn(m, k, device="cuda").bfloat16()
                out = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
                sp = qlinear.pick_gemm_splits(n, k, m)
                if sp > 1:      # few row tiles: K is cut and the consumer adds the slabs (here: a sum, which the model folds into its next kernel)
                    _run(f"qgemm_{tname}_{pname}_{m}x{n}x{k}", lambda: qlinear.gemm_partials(x, w, sp), 2.0 * m * n * k,
                         wbytes + m * k * 2 + sp * m * n * 4, args, splits=sp)
                else:
                    _run(f"qgemm_{tname}_{pname}_{m}x{n}x{k}", lambda: qlinear.gemm(x, w, out=out), 2.0 * m * n * k, wbytes + m * k * 2 + m * n * 2, args)
            del w


def case_small(args):
    """The kernels around the GEMMs and attention at the benchmark's shapes: RMSNorm (+ residual + MXFP8 copy), QK-norm + RoPE +
    cache write, the one-launch MoE front end, the sampler, the Delta-Net recurrence; decode size (64 tokens) and, for the
    bandwidth-bound ones, a prefill chunk (16384 tokens, more than L2)."""
    from ..ops import deltanet as dn, sampling
    h, hq, hkv, d = 2048, 32, 4, 128
    nw = torch.ones(h, device="cuda", dtype=torch.bfloat16)
    for t in (64, 16384):
        x = torch.randn(t, h, device="cuda").bfloat16()
        res = torch.randn(t, h, device="cuda").bfloat16()
        _run(f"rmsnorm_add_quant_{t}x{h}", lambda: ew.rmsnorm(x, nw, 1e-6, residual=res, quantize=True, sf_layout=128), 0.0,
             t * h * (2 + 2 + 2 + 2 + 1), args)
        qkv = torch.randn(t, (hq + 2 * hkv) * d, device="cuda").bfloat16()
        pos = torch.arange(t, device="cuda", dtype=torch.int32) % 4096
        slots = torch.randperm(t, device="cuda").to(torch.int32)
        kc = torch.empty(t, hkv, d, device="cuda", dtype=torch.bfloat16)
        vc = torch.empty_like(kc)
        qw = torch.ones(d, device="cuda", dtype=torch.bfloat16)
        tab = ew.rope_table(4096, d, 1e6, "cuda")
        _run(f"qk_norm_rope_{t}", lambda: ew.qk_norm_rope(qkv, pos, slots, qw, qw, kc, vc, hq, hkv, d, 1e6, 1e-6, 1.0, table=tab), 0.0,
             2 * t * (hq + 2 * hkv) * d * 2, args)
    x = torch.randn(64, h, device="cuda").bfloat16()
    router = (torch.randn(128, h, device="cuda") * 0.05).bfloat16()
    if moe.can_prep(x, router, 8):
        _run("moe_prep_64x2048_top8of128", lambda: moe.prep_hidden(x, router, 8, 128, 32), 2.0 * 64 * 128 * h, 128 * h * 2 + 64 * h * 2 + 512 * h, args)
    logits = torch.randn(64, 151936, device="cuda")
    _run("sampler_top_p_64x151936", lambda: sampling.sample(logits, 0.8, 40, 0.95, seed=1, step=3), 0.0, logits.numel() * 4, args)
    _run("argmax_64x151936", lambda: sampling.argmax(logits), 0.0, logits.numel() * 4, args)
    # Delta-Net layer of the Qwen3.5 shape: 16 key / 32 value heads of 128, one state matrix per value head and sequence
    ng, hv, ds = 16, 32, 128
    for name, lens in (("decode_64", [1] * 64), ("prefill_8x512", [512] * 8)):
        t = sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device="cuda")
        sl = torch.arange(len(lens), dtype=torch.int32, device="cuda")
        qkv = (torch.randn(t, (2 * ng + hv) * ds, device="cuda") * 0.5).bfloat16()
        z = torch.randn(t, hv * ds, device="cuda").bfloat16()
        ab = torch.randn(t, 2 * hv, device="cuda")
        a = -(torch.rand(hv, device="cuda") * 2 + 0.1)
        bias = torch.randn(hv, device="cuda") * 0.5
        nwd = torch.rand(ds, device="cuda") + 0.5
        st = torch.randn(len(lens), hv, ds, ds, device="cuda") * 0.1
        _run(f"deltanet_{name}", lambda: dn.deltanet(qkv, z, ab, a, bias, nwd, st, cu, sl, ng, hv, ds, 1e-6), 4.0 * t * hv * ds * ds,
             2 * st.numel() * 4 + qkv.numel() * 2 + 2 * z.numel() * 2, args)


def case_layered(args):
    from ..ops import deltanet as dn
    from ..ops import lightning, stream
    dev, h, hd, d = "cuda", 4096, 32, 128
    # recurrent layers, 32 heads of 128 x 128
    for name, lens in (("decode_1", [1]), ("decode_64", [1] * 64), ("prefill_1x8192", [8192]), ("prefill_8x2048", [2048] * 8)):
        t = sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        sl = torch.arange(len(lens), dtype=torch.int32, device=dev)
        st = torch.randn(len(lens), hd, d, d, device=dev) * 0.1
        proj = (torch.randn(t, 4 * hd * d, device=dev) * 0.5).bfloat16()
        decay = torch.rand(hd, device=dev) * 0.5 + 0.499
        dec = t == len(lens)
        src = proj.float() if dec else proj
        _run(f"lightning_{name}", lambda: lightning.lightning(src, decay, st, cu, sl, hd, d, d, activated=not dec, max_tokens=max(lens)), 4.0 * t * hd * d * d,
             2 * st.numel() * 4 + t * 3 * hd * d * src.element_size() + t * hd * d * 4, args)
        o = torch.randn(t, hd * d, device=dev)
        nw = torch.ones(hd * d, device=dev)
        _run(f"gated_norm_{name}", lambda: stream.gated_norm(o, src, 3 * hd * d, nw, 1e-6), 0.0, t * hd * d * (4 + src.element_size() + 2), args)
        z = torch.randn(t, hd * d, device=dev).bfloat16()
        ab = torch.randn(t, 2 * hd, device=dev)
        a, bias, nwd = -(torch.rand(hd, device=dev) * 2 + 0.1), torch.randn(hd, device=dev) * 0.5, torch.rand(d, device=dev) + 0.5
        _run(f"deltanet_{name}", lambda: dn.deltanet(proj[:, : 3 * hd * d], z, ab, a, bias, nwd, st, cu, sl, hd, hd, d, 1e-6), 4.0 * t * hd * d * d,
             2 * st.numel() * 4 + t * 5 * hd * d * 2, args)
    # attention, 32 query heads over 8 key / value heads
    hq, hkv, page = 32, 8, 128
    for name, b, q_len, ctx, window, keep in (("decode_1x32768", 1, 1, 32767, 4096, 128), ("decode_64x2048", 64, 1, 2047, 4096, 128), ("decode_64x8192", 64, 1, 8191, 4096, 128),
                                              ("prefill_1x8192", 1, 8192, 0, 4096, 128), ("prefill_8x2048", 8, 2048, 0, 4096, 128)):
        kv = ctx + q_len
        pages = (kv + page - 1) // page
        k = (torch.randn((b * pages + 1) * page, hkv, d, device=dev) * 0.5).bfloat16()
        v = torch.randn_like(k)
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).reshape(b, pages) + 1
        q = (torch.randn(b * q_len, hq, d, device=dev) * 0.5 * ew.softmax_scale_log2(d)).bfloat16()
        cu = torch.tensor([i * q_len for i in range(b + 1)], device=dev, dtype=torch.int32)
        kvl = torch.full((b,), kv, device=dev, dtype=torch.int32)
        table = att.distance_bias_table(torch.randn(32, hq), 4096).to(dev)
        dec = q_len == 1
        seen = [min(i + 1, window + keep) for i in range(ctx, kv)]
        kv_bytes = b * min(kv, window + keep + q_len) * hkv * d * 4 + b * q_len * hq * d * 4
        splits = att.pick_splits(b, hkv, min(kv, window + keep + 128)) if dec else 1
        plan = (att.build_work([q_len] * b, hq, hkv, splits).to(dev), splits)
        _run(f"attn_masked_{name}", lambda: att.attention_masked(q, k, v, cu, kvl, bt, page, window, keep, table, plan, dec), 4.0 * b * hq * d * sum(seen), kv_bytes, args,
             splits=splits)
        _run(f"attn_window_{name}", lambda: att.attention(q, k, v, cu, kvl, bt, page, plan[0], num_splits=splits, window=window, decode=dec),
             4.0 * b * hq * d * sum(min(i + 1, window) for i in range(ctx, kv)), kv_bytes, args, splits=splits)
        del k, v
    for t in (1, 64, 8192):
        x, w = torch.randn(t, h, device=dev), torch.ones(h, device=dev)
        up = torch.randn(t, h, device=dev)
        _run(f"stream_norm_{t}x{h}", lambda: stream.norm(x, w, 1e-6, up), 0.0, t * h * (4 + 4 + 4 + 2), args)
        xb, wb = x.bfloat16(), w.bfloat16()
        _run(f"rmsnorm_add_{t}x{h}", lambda: ew.rmsnorm(xb, wb, 1e-6, residual=xb), 0.0, t * h * 8, args)
        qkv = torch.randn(t, (hq + 2 * hkv) * d, device=dev)
        qkvb = qkv.bfloat16()
        src = qkv if t <= 64 else qkvb
        slots = torch.randperm(t, device=dev).to(torch.int32)
        pos = torch.arange(t, device=dev, dtype=torch.int32) % 4096
        kc, vc = torch.empty(t, hkv, d, device=dev, dtype=torch.bfloat16), torch.empty(t, hkv, d, device=dev, dtype=torch.bfloat16)
        _run(f"qk_unit_{t}", lambda: stream.qk_unit(src, slots, kc, vc, hq, hkv, d, d, 1e-6, 0.1), 0.0, t * (hq + 2 * hkv) * d * (src.element_size() + 2), args)
        qw = torch.ones(d, device=dev, dtype=torch.bfloat16)
        tab = ew.rope_table(4096, d, 1e6, dev)
        _run(f"qk_norm_rope_{t}", lambda: ew.qk_norm_rope(qkvb, pos, slots, qw, qw, kc, vc, hq, hkv, d, 1e6, 1e-6, 1.0, table=tab), 0.0, t * (hq + 2 * hkv) * d * 4, args)
        xb = (torch.randn(t, h, device=dev) * 0.5).bfloat16()
        for nm, n, kk in (("in", 16384, 4096), ("out", 4096, 4096), ("down", 4096, 12288)):
            wt = mxfp8.tile_weight((torch.randn(n, kk, device=dev) * 0.02).bfloat16())
            xk = xb if kk == 4096 else xb.repeat(1, 3)
            _run(f"gemm_{nm}_bf16_{t}", lambda: gemm.linear(xk, wt, w_tiled=True), 2.0 * t * n * kk, n * kk * 2 + t * kk * 2 + t * n * 2, args)
            if nm == "in":
                if t > 64:                  # decode-sized batches leave the activation to the recurrence
                    _run(f"gemm_{nm}_silu_{t}", lambda: gemm.linear(xk, wt, w_tiled=True, silu_rows=12288), 2.0 * t * n * kk, n * kk * 2 + t * kk * 2 + t * n * 2, args)
            else:
                _run(f"gemm_{nm}_f32_{t}", lambda: gemm.linear(xk, wt, w_tiled=True, out_dtype=torch.float32), 2.0 * t * n * kk, n * kk * 2 + t * kk * 2 + t * n * 4, args)
            del wt
        wg = mxfp8.tile_weight((torch.randn(24576, h, device=dev) * 0.02).bfloat16())
        for act in ("silu", "gelu_tanh"):
            _run(f"gate_up_{act}_{t}", lambda: gemm.linear_swiglu(xb, wg, w_tiled=True, act=act), 2.0 * t * 24576 * h, 24576 * h * 2 + t * h * 2 + t * 12288 * 2, args)
        del wg


def case_famepel(args):
    from ..models.config import get_config
    from ..ops import deltanet as dn
    from ..ops import latent, recurrent, stream
    dev = "cuda"
    cfg = get_config("famepel-30b-a3b")
    spec = {sp.mixer: sp for sp in cfg.layer_specs}
    m, hg, la, h = spec["mamba2"], spec["hgrn2"], spec["latent"], cfg.hidden
    f32 = dict(device=dev, dtype=torch.float32)
    for name, lens in (("decode_1", [1]), ("decode_64", [1] * 64), ("prefill_1x8192", [8192]), ("prefill_8x2048", [2048] * 8)):
        t, b, dec = sum(lens), len(lens), len(lens) == sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        nv, ch = m.n_heads * m.v_dim, m.conv_channels
        at = (nv + ch + 127) // 128 * 128
        proj = torch.randn(t, at + 128, device=dev)
        rows = proj if dec else proj.bfloat16()
        es = rows.element_size()
        cw, cb, cst = torch.randn(ch, m.conv_taps, device=dev), torch.randn(ch, device=dev), torch.zeros(b, m.conv_taps - 1, ch, **f32)
        _run(f"causal_conv_{name}", lambda: recurrent.causal_conv(rows, nv, cw, cb, cst, cu, sl, max(lens)), 0.0, t * ch * (es + 2) + 2 * cst.numel() * 4, args)
        x = (torch.randn(t, ch, device=dev) * 0.5).bfloat16()
        if m.conv_taps <= 8:
            _run(f"ssm_conv_{name}", lambda: dn.conv_silu(x, cw, cst, cu, sl), 0.0, t * ch * 4 + 2 * cst.numel() * 4, args)
        st = torch.randn(b, m.n_heads, m.head_dim, m.v_dim, device=dev) * 0.1
        hv = [torch.randn(m.n_heads, device=dev) for _ in range(2)] + [-torch.rand(m.n_heads, device=dev) - 0.1]
        _run(f"ssd_{name}", lambda: recurrent.ssd(x, proj, at, hv[0], hv[2], hv[1], st, cu, sl, m.n_heads, m.state_groups, m.head_dim, m.v_dim, max(lens)),
             4.0 * t * m.n_heads * m.head_dim * m.v_dim, 2 * st.numel() * 4 + t * (ch * 2 + nv * 4), args)
        o, nw = torch.randn(t, nv, device=dev), torch.ones(nv, device=dev)
        _run(f"part_norm_gated_{name}", lambda: stream.part_norm(o, nw, m.norm_parts, 1e-5, rows), 0.0, t * nv * (4 + es + 2), args)
        _run(f"gated_norm_{name}", lambda: stream.gated_norm(o, rows, 0, nw, 1e-5), 0.0, t * nv * (4 + es + 2), args)
        del o, st
        nq, nv = hg.q_dim, hg.n_heads * hg.v_dim
        qv, z = torch.randn(t, nq + nv, device=dev), torch.randn(t, nq, device=dev) + 2
        qv = qv if dec else qv.bfloat16()
        st = torch.randn(b, hg.n_heads, hg.head_dim, hg.v_dim, device=dev) * 0.1
        fb, low = torch.zeros(nq, device=dev), torch.full((nq,), 0.3, device=dev)
        _run(f"gla_{name}", lambda: recurrent.gla(qv, z, 0, fb, low, st, cu, sl, hg.n_heads, hg.head_dim, hg.v_dim, not dec, max(lens)),
             4.0 * t * hg.n_heads * hg.head_dim * hg.v_dim, 2 * st.numel() * 4 + t * ((nq + nv) * qv.element_size() + nq * 4 + nv * 4), args)
        # Delta-Net with states of the same sizes: 16 and 32 heads of 128 x 128
        for hd in (16, 32):
            ds = 128
            qkv, zz, ab = torch.randn(t, 3 * hd * ds, device=dev).bfloat16(), torch.randn(t, hd * ds, device=dev).bfloat16(), torch.randn(t, 2 * hd, device=dev)
            a, bias, nwd = -(torch.rand(hd, device=dev) * 2 + 0.1), torch.randn(hd, device=dev) * 0.5, torch.ones(ds, device=dev)
            st = torch.randn(b, hd, ds, ds, device=dev) * 0.1
            _run(f"deltanet_{hd}_{name}", lambda: dn.deltanet(qkv, zz, ab, a, bias, nwd, st, cu, sl, hd, hd, ds, 1e-6), 4.0 * t * hd * ds * ds,
                 2 * st.numel() * 4 + t * 5 * hd * ds * 2, args)
        del qv, z, proj, rows, x, qkv, zz, st
    # latent attention: 32 heads, latents of 512 + 64 columns; plain attention with 32 heads over 4 key / value heads of 128
    hd, d, rd, v, r, page = la.n_heads, la.head_dim, la.rot_dim, la.v_dim, la.kv_rank, 128
    w = stream.row_width(r + rd, torch.bfloat16)

    class Batch:
        pass

    for name, b, q_len, ctx in (("decode_1x32768", 1, 1, 32767), ("decode_16x8192", 16, 1, 8191), ("decode_64x2048", 64, 1, 2047), ("decode_64x8192", 64, 1, 8191),
                                ("prefill_1x8192", 1, 8192, 0), ("prefill_8x2048", 8, 2048, 0)):
        kv, dec = ctx + q_len, q_len == 1
        pages = (kv + page - 1) // page
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).reshape(b, pages)
        cu, kvl = torch.tensor([i * q_len for i in range(b + 1)], device=dev, dtype=torch.int32), torch.full((b,), kv, device=dev, dtype=torch.int32)
        batch = Batch()
        batch.block_table, batch.kv_len, batch.cu_q = bt, kvl, cu
        cache = torch.randn(b * pages * page, 1, w, device=dev).bfloat16()
        sink = torch.zeros(hd, device=dev)
        plan = latent.make_plan([q_len] * b, [kv] * b, kv, dev, dec, True, [hd])
        seen = float(sum(range(ctx + 1, kv + 1)) * b)
        if dec:
            qa = (torch.randn(hd, plan.m, w, device=dev) * 0.1).bfloat16()
            _run(f"latent_{name}", lambda: latent.attend_latents(qa, cache, r, r + rd, plan, batch, page, sink), 2.0 * seen * hd * (2 * r + rd),
                 b * (kv * w * 2 + hd * (w + r) * 2), args, splits=plan.splits)
            qn = torch.randn(hd * plan.m, d, device=dev).bfloat16()
            uk, uv = torch.randn(hd, r, d, device=dev).bfloat16(), torch.randn(hd, v, r, device=dev).bfloat16()
            seg, cnt, rows = plan.groups(hd, dev)
            oo = torch.randn(hd * plan.m, r, device=dev).bfloat16()
            out = torch.empty(b * hd, v, device=dev, dtype=torch.bfloat16)
            _run(f"absorb_k_{name}", lambda: gemm.grouped_linear(qn, uk, seg, cnt, plan.tile, out=qa.view(-1, w), n_out=r), 2.0 * b * hd * d * r, hd * (d * r + b * (d + r)) * 2, args)
            _run(f"absorb_v_{name}", lambda: gemm.grouped_linear(oo, uv, seg, cnt, plan.tile, out=out, row_map=rows, n_out=v), 2.0 * b * hd * v * r,
                 hd * (v * r + b * (v + r)) * 2, args)
        else:
            en, er = torch.randn(b * q_len, hd, d, device=dev).bfloat16() * 0.1, torch.randn(b * q_len, hd, rd, device=dev).bfloat16() * 0.1
            kvx = torch.randn(b * kv, hd * (d + v), device=dev).bfloat16()
            out = torch.empty(b * q_len, hd, v, device=dev, dtype=torch.bfloat16)
            rows = latent.gather_latents(cache, plan, bt, page)
            _run(f"latent_{name}", lambda: latent.attend_expanded(en, er, kvx, rows, r, plan, sink, out), 2.0 * seen * hd * (d + rd + v),
                 (kvx.numel() + out.numel() + en.numel() + er.numel() + rows.numel()) * 2, args)
            _run(f"latent_gather_{name}", lambda: latent.gather_latents(cache, plan, bt, page), 0.0, b * kv * w * 4, args)
            del kvx
        hkv = 4
        k, vv = (torch.randn(b * pages * page, hkv, 128, device=dev).bfloat16() for _ in range(2))
        q = (torch.randn(b * q_len, hd, 128, device=dev) * 0.1).bfloat16()
        splits = att.pick_splits(b, hkv, kv) if dec else 1
        work = att.build_work([q_len] * b, hd, hkv, splits).to(dev)
        _run(f"attn_{name}", lambda: att.attention(q, k, vv, cu, kvl, bt, page, work, num_splits=splits, decode=dec), 4.0 * seen * hd * 128, b * (kv * hkv * 512 + q_len * hd * 512),
             args, splits=splits)
        del k, vv, cache
    for t in (1, 64, 8192):
        x, u = torch.randn(t, h, device=dev), torch.randn(t, h, device=dev)
        n1, n2 = (stream.DynTanh(0.5, torch.ones(h, device=dev), torch.zeros(h, device=dev)) for _ in range(2))
        _run(f"stream_dyt_{t}x{h}", lambda: stream.norm(x, n1, 1e-5, stream.PostNormed(u, n2)), 0.0, t * h * 14, args)
        _run(f"stream_norm_{t}x{h}", lambda: stream.norm(x, n1.weight, 1e-5, u), 0.0, t * h * 14, args)
        k, e = 8, 128
        y = torch.randn(t * k, h, device=dev).bfloat16()
        pend = moe.PendingCombine(y, torch.randperm(t * k, device=dev).to(torch.int32), torch.rand(t, k, device=dev), t, k)
        _run(f"stream_dyt_moe_{t}x{h}", lambda: stream.norm(x, n1, 1e-5, stream.PostNormed(pend, n2)), 0.0, t * h * (10 + 2 * k), args)
        xb = x.bfloat16()
        _run(f"rmsnorm_moe_{t}x{h}", lambda: ew.rmsnorm(pend, n1.weight.bfloat16(), 1e-5, residual=xb), 0.0, t * h * (6 + 2 * k), args)
        z = torch.randn(t, e, device=dev)
        for groups in ((1, 1), (8, 4)):
            _run(f"route_{groups[0]}_groups_{t}", lambda: moe.route(z, k, "sigmoid", None, 2, 2.5, None, groups), 0.0, t * (e * 4 + k * 8), args)
        nk = hd * (d + rd)
        qf = torch.randn(t, nk, device=dev)
        qf = qf if t <= 64 else qf.bfloat16()
        pos = torch.arange(t, device=dev, dtype=torch.int32)
        freq = torch.tensor(la.rotary.frequencies(), dtype=torch.float64, device=dev)
        en, er = torch.empty(t, hd, d, device=dev, dtype=torch.bfloat16), torch.empty(t, hd, rd, device=dev, dtype=torch.bfloat16)
        _run(f"latent_q_{t}", lambda: latent.latent_q(qf, pos, freq, 1.0, 0.1, None, (en, er), None, hd, d, rd), 0.0, t * nk * (qf.element_size() + 2), args)
        a = torch.randn(t, la.q_rank + r + rd, device=dev)
        a = a if t <= 64 else a.bfloat16()
        cache = torch.empty(t, 1, w, device=dev, dtype=torch.bfloat16)
        qn, kn = torch.ones(la.q_rank, device=dev), torch.ones(r, device=dev)
        _run(f"latent_store_{t}", lambda: latent.latent_store(a, pos, pos, qn, kn, freq, 1.0, cache, la.q_rank, r, rd, 1e-5, torch.bfloat16), 0.0,
             t * (la.q_rank + r + rd) * (a.element_size() + 2), args)
        qkv = torch.randn(t, (hd + 8) * 128, device=dev).bfloat16()
        kc, vc = (torch.empty(t, 4, 128, device=dev, dtype=torch.bfloat16) for _ in range(2))
        tab, qw = ew.rope_table(8192, 128, 1e6, dev), torch.ones(128, device=dev, dtype=torch.bfloat16)
        _run(f"qk_norm_rope_{t}", lambda: ew.qk_norm_rope(qkv, pos, pos, qw, qw, kc, vc, hd, 4, 128, 1e6, 1e-6, 1.0, table=tab), 0.0, t * (hd + 8) * 128 * 4, args)


def case_fidolix(args):
    from ..models.config import get_config
    from ..ops import recurrent, stream
    dev, page = "cuda", 128
    cfg = get_config("fidolix-30b-a3b")
    spec = {sp.mixer: sp for sp in cfg.layer_specs}
    at, lf, rw, h = spec["attention"], spec["parallel"].left, spec["parallel"].right, cfg.hidden
    f32 = dict(device=dev, dtype=torch.float32)
    for name, lens in (("decode_1", [1]), ("decode_64", [1] * 64), ("prefill_1x8192", [8192]), ("prefill_8x2048", [2048] * 8)):
        t, b, dec = sum(lens), len(lens), len(lens) == sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        n, hd, d = rw.q_dim, rw.n_heads, rw.head_dim
        dt = torch.float32 if dec else torch.bfloat16
        es = 4 if dec else 2
        # recurrence, beside HGRN2 of the same sizes
        pad = recurrent.shift_pad(t)
        rkvg, z = torch.randn(4, pad, n, device=dev).to(dt), torch.randn(t, n, device=dev) - 3
        st = torch.randn(b, hd, d, d, device=dev) * 0.1
        w0, u, low = torch.zeros(n, device=dev), torch.randn(n, device=dev), torch.full((n,), 0.3, device=dev)
        _run(f"rwkv_{name}", lambda: recurrent.rwkv(rkvg, z, w0, u, st, cu, sl, hd, d, d, t, max(lens)), 4.0 * t * hd * d * d, 2 * st.numel() * 4 + t * (3 * n * es + n * 4 + n * 4), args)
        qv = torch.randn(t, 2 * n, device=dev).to(dt)
        _run(f"gla_{name}", lambda: recurrent.gla(qv, z, 0, w0, low, st, cu, sl, hd, d, d, not dec, max(lens)), 4.0 * t * hd * d * d,
             2 * st.numel() * 4 + t * (2 * n * es + n * 4 + n * 4), args)
        del st, qv
        x = torch.randn(t, h, device=dev).bfloat16()
        mu, sh = torch.rand(5, h, device=dev), torch.zeros(b, 1, h, **f32)
        _run(f"token_shift_{name}", lambda: recurrent.token_shift(x, h, mu, sh, cu, sl, pad, max(lens)), 0.0, t * h * 12, args)
        lr = torch.randn(t, rw.decay_rank, device=dev)
        _run(f"tanh_rows_{name}", lambda: recurrent.tanh_rows(lr, rw.decay_rank), 0.0, lr.numel() * 6, args)
        o, nw = torch.randn(t, n, device=dev), torch.ones(n, device=dev)
        gate = rkvg[3, :t]
        _run(f"part_norm_gate_after_{name}", lambda: stream.part_norm(o, nw, hd, 1e-5, gate, gate_after=True), 0.0, t * n * (4 + es + 2), args)
        _run(f"part_norm_gated_{name}", lambda: stream.part_norm(o, nw, hd, 1e-5, gate), 0.0, t * n * (4 + es + 2), args)
        wg = (torch.randn(4, n, h, device=dev) * 0.02).bfloat16()
        seg, cnt = torch.arange(4, dtype=torch.int32, device=dev) * pad, torch.full((4,), t, dtype=torch.int32, device=dev)
        mix = torch.randn(4 * pad, h, device=dev).bfloat16()
        wt = mxfp8.tile_weight(wg.view(4 * n, h)).view(4, n, h)
        _run(f"grouped_rkvg_{name}", lambda: gemm.grouped_linear(mix, wt, seg, cnt, recurrent.shift_tile(pad), out=rkvg.view(4 * pad, n), w_tiled=True), 8.0 * t * n * h,
             4 * n * h * 2 + 4 * t * h * 2 + 4 * t * n * es, args)
        _run(f"gemm_same_size_{name}", lambda: gemm.linear(x, wt.view(4 * n, h), w_tiled=True, out_dtype=dt), 8.0 * t * n * h, 4 * n * h * 2 + t * h * 2 + 4 * t * n * es, args)
        del rkvg, mix, o, z
        # from projection to attention
        ch = lf.conv_channels
        rows, cw, cst = torch.randn(t, ch, device=dev).to(dt), torch.randn(ch, lf.conv_taps, device=dev), torch.zeros(b, lf.conv_taps - 1, ch, **f32)
        pos = torch.arange(t, device=dev, dtype=torch.int32)
        freq = torch.tensor(lf.rotary.frequencies(), dtype=torch.float64, device=dev)
        tab = stream.rotary_table(pos, freq, 1.1)
        kc, vc = (torch.empty(t, lf.n_kv_heads, lf.head_dim, device=dev, dtype=torch.bfloat16) for _ in range(2))
        nk = lf.n_kv_heads * lf.head_dim
        _run(f"rotary_table_{name}", lambda: stream.rotary_table(pos, freq, 1.1), 0.0, tab.numel() * 4, args)
        _run(f"conv_rotary_{name}", lambda: stream.conv_rotary(rows, tab, pos, cw, cst, cu, sl, kc, vc, lf.n_heads, lf.n_kv_heads, lf.head_dim, 0.1, max(lens)), 0.0,
             t * (ch * (es + 2) + nk * 2 + tab.shape[1] * 8) + 2 * cst.numel() * 4, args)
        cb = torch.zeros(ch, device=dev)
        _run(f"causal_conv_{name}", lambda: recurrent.causal_conv(rows, 0, cw, cb, cst, cu, sl, max(lens)), 0.0, t * ch * (es + 2) + 2 * cst.numel() * 4, args)
        nq, nk, nv = at.q_dim, at.n_kv_heads * at.head_dim, at.n_heads * at.v_dim
        rows = torch.randn(t, nq + 2 * nk + nv, device=dev).to(dt)
        qn, kn = torch.ones(nq, device=dev), torch.ones(nk, device=dev)
        kc, vc = (torch.empty(t, at.n_kv_heads, at.head_dim, device=dev, dtype=torch.bfloat16) for _ in range(2))
        by = t * (nq + 2 * nk) * (es + 2)
        _run(f"qk_rows_{name}", lambda: stream.qk_rows(rows, pos, qn, kn, kc, vc, at.n_heads, at.n_kv_heads, at.head_dim, at.v_dim, 1e-5, 0.1), 0.0, by, args)
        _run(f"qk_unit_{name}", lambda: stream.qk_unit(rows, pos, kc, vc, at.n_heads, at.n_kv_heads, at.head_dim, at.v_dim, 1e-5, 0.1), 0.0, by, args)
        a = torch.randn(t, at.n_heads, at.v_dim, device=dev).bfloat16()
        _run(f"sigmoid_gate_{name}", lambda: stream.sigmoid_gate(a, rows, nq + 2 * nk, at.v_dim), 0.0, t * nv * (4 + es), args)
        del rows, a
    # attention: capped scores over everything, sinks over a window, and the plain and biased forms of the same sizes
    for name, b, q_len, ctx in (("decode_1x32768", 1, 1, 32767), ("decode_64x2048", 64, 1, 2047), ("decode_64x8192", 64, 1, 8191), ("prefill_1x8192", 1, 8192, 0), ("prefill_8x2048", 8, 2048, 0)):
        for sp, win in ((at, 0), (lf, lf.window)):
            hq, hkv, d = sp.n_heads, sp.n_kv_heads, sp.head_dim
            kv, dec = ctx + q_len, q_len == 1
            pages = (kv + page - 1) // page
            k, v = ((torch.randn((b * pages + 1) * page, hkv, d, device=dev) * 0.5).bfloat16() for _ in range(2))
            bt = torch.arange(b * pages, device=dev, dtype=torch.int32).reshape(b, pages) + 1
            cu, kvl = torch.tensor([i * q_len for i in range(b + 1)], device=dev, dtype=torch.int32), torch.full((b,), kv, device=dev, dtype=torch.int32)
            seen = float(sum(min(i + 1, win or kv) for i in range(ctx, kv)) * b)
            by = b * min(kv, (win or kv) + q_len) * hkv * d * 4 + b * q_len * hq * d * 4
            splits = att.pick_splits(b, hkv, min(kv, win + 128) if win else kv) if dec else 1
            plan = (att.build_work([q_len] * b, hq, hkv, splits).to(dev), splits)
            sink = torch.zeros(hq, device=dev)
            q = (torch.randn(b * q_len, hq, d, device=dev) * 0.5 * d ** -0.5).bfloat16()
            run = lambda nm, qq, **kw: _run(f"attn_{nm}_{name}", lambda: att.attention_masked(qq, k, v, cu, kvl, bt, page, win, plan=plan, decode=dec, **kw), 4.0 * seen * hq * d, by, args,
                                            splits=splits)
            if win:
                run("window_sink", q * att.LOG2E, sink=sink)
                _run(f"attn_window_{name}", lambda: att.attention(q, k, v, cu, kvl, bt, page, plan[0], num_splits=splits, window=win, decode=dec), 4.0 * seen * hq * d, by, args, splits=splits)
            else:
                run("capped", (q / at.softcap).bfloat16(), softcap=at.softcap)                                   # scores well within the cap
                run("capped_wide", (q * 40.0 / at.softcap).bfloat16(), softcap=at.softcap)                       # ... and around it
                _run(f"attn_{name}", lambda: att.attention(q, k, v, cu, kvl, bt, page, plan[0], num_splits=splits, decode=dec), 4.0 * seen * hq * d, by, args, splits=splits)
            del k, v
    for t in (1, 64, 8192):
        x, u = torch.randn(t, h, device=dev), torch.randn(t, h, device=dev)
        w1, w2, w3 = (torch.ones(h, device=dev) for _ in range(3))
        _run(f"stream_rms2_{t}x{h}", lambda: stream.norm2(x, w1, 1e-5, stream.RmsPosted(u, w3, 1e-5), weight2=w2), 0.0, t * h * 16, args)
        _run(f"stream_norm_{t}x{h}", lambda: stream.norm(x, w1, 1e-5, u), 0.0, t * h * 14, args)
        k, e = 8, 128
        y = torch.randn(t * k, h, device=dev).bfloat16()
        pend = moe.PendingCombine(y, torch.randperm(t * k, device=dev).to(torch.int32), torch.rand(t, k, device=dev), t, k)
        u2 = torch.randn(t, h, device=dev)
        _run(f"stream_join_moe_{t}x{h}", lambda: stream.join(x, [(u, 1.0), (u2, 1.0), (pend, 1.0)], torch.bfloat16), 0.0, t * h * (18 + 2 * k), args)
        xb = x.bfloat16()
        _run(f"rmsnorm_moe_{t}x{h}", lambda: ew.rmsnorm(pend, w1.bfloat16(), 1e-5, residual=xb), 0.0, t * h * (6 + 2 * k), args)
        z, sd = torch.randn(t, cfg.side_dim, device=dev), cfg.side_dim
        table, ids = torch.randn(4096, 45 * sd, device=dev).bfloat16(), torch.randint(0, 4096, (t,), device=dev, dtype=torch.int32)
        _run(f"token_gate_{t}", lambda: stream.token_gate(z, ids, table, 3 * sd, sd), 0.0, t * sd * 8, args)
        z = torch.randn(t, e, device=dev)
        for best in (1, 2):
            _run(f"route_8_groups_best{best}_{t}", lambda: moe.route(z, k, "softmax", None, 2, 1.0, None, (8, 4, best)), 0.0, t * (e * 4 + k * 8), args)
        ff = 6144
        wg = mxfp8.tile_weight((torch.randn(2 * ff, h, device=dev) * 0.02).bfloat16())
        for act in ("silu", "capped"):
            _run(f"gate_up_{act}_{t}", lambda: gemm.linear_swiglu(xb, wg, w_tiled=True, act=act, cap=7.0), 4.0 * t * ff * h, 2 * ff * h * 2 + t * h * 2 + t * ff * 2, args)
        del wg


def case_zedirax(args):
    from ..models.config import get_config
    from ..ops import latent, recurrent, stream
    dev, page = "cuda", 128
    cfg = get_config("zedirax-30b-a3b")
    spec = {sp.mixer: sp for sp in cfg.layer_specs}
    gr, at, la, h = spec["mingru"], spec["attention"], spec["latent"], cfg.hidden
    for name, lens in (("decode_1", [1]), ("decode_64", [1] * 64), ("prefill_1x1024", [1024]), ("prefill_1x8192", [8192]), ("prefill_8x2048", [2048] * 8)):
        t, b, dec = sum(lens), len(lens), len(lens) == sum(lens)
        cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        pos = torch.arange(t, device=dev, dtype=torch.int32)
        n, dt = gr.v_dim, torch.float32 if dec else torch.bfloat16
        es = 4 if dec else 2
        xg, z = torch.randn(t, 2 * n, device=dev).to(dt), torch.randn(t, n, device=dev) - 3
        zero, st = torch.zeros(n, device=dev), torch.zeros(b, 1, 1, n, device=dev)
        _run(f"mingru_{name}", lambda: recurrent.mingru(xg, z, 0, zero, zero, st, cu, sl, n, max(lens)), 0.0, t * n * (2 * es + 4 + 2) + 2 * st.numel() * 4, args)
        hd, d = 16, 128
        n2 = hd * d
        qv, f, s2 = xg[:, : 2 * n2].contiguous(), z[:, :n2].contiguous(), torch.zeros(b, hd, d, d, device=dev)
        low = torch.full((n2,), 0.3, device=dev)
        _run(f"gla_{name}", lambda: recurrent.gla(qv, f, 0, zero[:n2], low, s2, cu, sl, hd, d, d, not dec, max(lens)), 4.0 * t * hd * d * d,
             2 * s2.numel() * 4 + t * (2 * n2 * es + n2 * 4 + n2 * 4), args)
        del xg, z, qv, f
        nq, nk = at.q_dim, at.n_kv_heads * at.head_dim
        rows = torch.randn(t, nq + 2 * nk, device=dev).to(dt)
        kc, vc = (torch.empty(t, at.n_kv_heads, at.head_dim, device=dev, dtype=torch.bfloat16) for _ in range(2))
        by = t * (nq + 2 * nk) * (es + 2)
        for nm, kw in (("temperature", dict(unit=False, positions=pos, temp=(0.1, 8192.0))), ("unit", {})):
            _run(f"qk_{nm}_{name}", lambda: stream.qk_unit(rows, pos, kc, vc, at.n_heads, at.n_kv_heads, at.head_dim, at.v_dim, 1e-5, 0.1, **kw), 0.0, by, args)
        del rows
        r, rd, qn = la.kv_rank, la.rot_dim, la.n_heads * (la.head_dim + la.rot_dim)
        rows = torch.randn(t, qn + r + rd + la.n_heads * la.v_dim, device=dev).to(dt)
        cache, freq = torch.empty(t, 1, r + rd, device=dev, dtype=torch.bfloat16), torch.tensor(la.rotary.frequencies(), dtype=torch.float64, device=dev)
        one = torch.ones(1536, device=dev)
        _run(f"latent_store_alone_{name}", lambda: latent.latent_store(rows, pos, pos, None, one[:r], freq, 1.0, cache, 0, r, rd, 1e-5, torch.bfloat16, qn), 0.0, t * (r + rd) * (es + 2), args)
        _run(f"latent_store_with_q_{name}", lambda: latent.latent_store(rows, pos, pos, one, one[:r], freq, 1.0, cache, 1536, r, rd, 1e-5, torch.bfloat16), 0.0, t * (1536 + r + rd) * (es + 2), args)
        a = torch.randn(t, la.n_heads, la.v_dim, device=dev).bfloat16()
        _run(f"sigmoid_gate_{name}", lambda: stream.sigmoid_gate(a, rows, qn + r + rd, la.v_dim), 0.0, a.numel() * (4 + es), args)
        del rows, a
    for name, b, q_len, ctx in (("decode_1x32768", 1, 1, 32767), ("decode_64x2048", 64, 1, 2047), ("decode_64x8192", 64, 1, 8191), ("prefill_1x8192", 1, 8192, 0), ("prefill_8x2048", 8, 2048, 0)):
        hq, hkv, d = at.n_heads, at.n_kv_heads, at.head_dim
        kv, dec = ctx + q_len, q_len == 1
        pages = (kv + page - 1) // page
        k, v = ((torch.randn((b * pages + 1) * page, hkv, d, device=dev) * 0.5).bfloat16() for _ in range(2))
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).reshape(b, pages) + 1
        cu, kvl = torch.tensor([i * q_len for i in range(b + 1)], device=dev, dtype=torch.int32), torch.full((b,), kv, device=dev, dtype=torch.int32)
        seen = float(sum(i + 1 for i in range(ctx, kv)) * b)
        by = b * kv * hkv * d * 4 + b * q_len * hq * d * 4
        splits = att.pick_splits(b, hkv, kv) if dec else 1
        plan = (att.build_work([q_len] * b, hq, hkv, splits).to(dev), splits)
        q = (torch.randn(b * q_len, hq, d, device=dev) * 0.5 * d ** -0.5 * att.LOG2E).bfloat16()
        table = att.distance_bias_table(torch.randn(32, hq), 8192).to(dev)
        lb = torch.rand(2, hq, device=dev)
        run = lambda nm, **kw: _run(f"attn_{nm}_{name}", lambda: att.attention_masked(q, k, v, cu, kvl, bt, page, plan=plan, decode=dec, **kw), 4.0 * seen * hq * d, by, args, splits=splits)
        run("log_bias", log_bias=lb)
        run("table_bias", bias=table)
        _run(f"attn_{name}", lambda: att.attention(q, k, v, cu, kvl, bt, page, plan[0], num_splits=splits, decode=dec), 4.0 * seen * hq * d, by, args, splits=splits)
        del k, v
    for t in (1, 64, 8192):
        x, u = torch.randn(t, h, device=dev), torch.randn(t, h, device=dev)
        w1 = torch.ones(h, device=dev)
        _run(f"stream_norm_gate_{t}x{h}", lambda: stream.norm_gate(x, w1, 1e-5, stream.Update([(u, 0.5, None)]), w1), 0.0, t * h * 14, args)
        _run(f"stream_norm_{t}x{h}", lambda: stream.norm(x, w1, 1e-5, u), 0.0, t * h * 14, args)
        k, places = 8, 46
        y = torch.randn(t * k, h, device=dev).bfloat16()
        pend = moe.PendingCombine(y, torch.randperm(t * k, device=dev).to(torch.int32), torch.rand(t, k, device=dev), t, k)
        hist, gate = torch.randn(places, t, h, device=dev), torch.rand(t, device=dev)
        coef = [torch.full((p + 1,), 0.02, device=dev) for p in range(places)]
        bs = stream.depth_base(hist, 41, coef[41:46])
        for nm, p, base, first in (("1_place", 1, None, 0), ("8_places", 8, None, 0), ("41_and_4_places", 45, bs[4], 41)):
            _run(f"stream_depth_moe_{nm}_{t}x{h}", lambda: stream.norm(x, w1, 1e-5, stream.Update([(pend, 0.5, None), (u, 0.5, gate)], stream.Depth(hist, p, coef[p], base, first))), 0.0,
                 t * h * (4 * (4 + p - first + (base is not None)) + 2 * k + 2), args)
        ones = [torch.full((46,), 0.02, device=dev) for _ in range(8)]
        _run(f"depth_base_41_places_{t}x{h}", lambda: stream.depth_base(hist, 41, ones), 0.0, t * h * 4 * (41 + 8), args)
        _run(f"stream_join_moe_{t}x{h}", lambda: stream.join(x, [(u, 1.0), (pend, 1.0)], torch.bfloat16), 0.0, t * h * (14 + 2 * k), args)
        xb = x.bfloat16()
        _run(f"rmsnorm_moe_{t}x{h}", lambda: ew.rmsnorm(pend, w1.bfloat16(), 1e-5, residual=xb), 0.0, t * h * (6 + 2 * k), args)
        del hist, y, pend
        ff = 6144
        wg = mxfp8.tile_weight((torch.randn(2 * ff, h, device=dev) * 0.02).bfloat16())
        bias = torch.randn(2 * ff, device=dev)
        for nm, kw in (("gelu_biased", dict(bias=bias)), ("gelu", {})):
            _run(f"gate_up_{nm}_{t}", lambda: gemm.linear_swiglu(xb, wg, w_tiled=True, act="gelu_tanh", **kw), 4.0 * t * ff * h, 2 * ff * h * 2 + t * h * 2 + t * ff * 2, args)
        for nm, kw in (("gelu_erf", dict(gelu=True)), ("plain", {})):
            _run(f"gemm_{nm}_{t}", lambda: gemm.linear(xb, wg, w_tiled=True, **kw), 4.0 * t * ff * h, 2 * ff * h * 2 + t * h * 2 + 2 * t * ff * 2, args)
        del wg
        # experts: plain ones of 1152, gated ones of 768
        e, mo = 128, la.moe
        tn = gemm.pick_tn(max(1, (t * k + e - 1) // e), dual=True)
        _, _, pl = moe.route_plan(torch.randn(t, e, device=dev), k, e, tn)
        xs = moe.gather_rows(xb, pl.row_token)
        used = min(t * k, e)
        for nm, rows, kw in (("plain_gelu", mo.ffn, dict(gelu=True)), ("plain", mo.ffn, {}), ("gated_silu", 2 * 768, dict(dual=True))):
            we = mxfp8.tile_weight((torch.randn(e * rows, h, device=dev) * 0.02).bfloat16()).view(e, rows, h)
            _run(f"experts_up_{nm}_{t}", lambda: gemm.grouped_linear(xs, we, pl.seg_start, pl.seg_count, tn, w_tiled=True, **kw), 2.0 * t * k * rows * h, used * rows * h * 2 + t * k * (h + rows) * 2, args)
            del we


MODEL_CASES = {"spec_verify": case_spec_verify}      # build the whole benchmark model: not part of --case all
CASES = {"gemm": case_gemm, "moe_decode": case_moe_decode, "moe_prefill": case_moe_prefill, "attn_decode": case_attn_decode,
         "attn_prefill": case_attn_prefill, "lm_head": case_lm_head, "quant": case_quant, "small": case_small, "layered": case_layered,
         "famepel": case_famepel, "fidolix": case_fidolix, "zedirax": case_zedirax}


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--case", default="all", choices=["all"] + sorted(CASES) + sorted(MODEL_CASES))
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--splits", type=int, default=0, help="attention cases: force the number of KV splits")
    ap.add_argument("--hq", type=int, default=32)
    ap.add_argument("--hkv", type=int, default=4)
    ap.add_argument("--page", type=int, default=128, help="attention cases: KV page size")
    ap.add_argument("--batch", type=int, default=0, help="attention cases: number of sequences (0 = the case's default)")
    ap.add_argument("--ctx", type=int, default=-1, help="attention cases: cached tokens per sequence (-1 = the case's default)")
    ap.add_argument("--once", action="store_true", help="run each op once, untimed (for use under a profiler)")
    args = ap.parse_args(argv)
    torch.manual_seed(0)
    for name in (sorted(CASES) if args.case == "all" else [args.case]):
        (CASES.get(name) or MODEL_CASES[name])(args)
    print(json.dumps(dict(kernel_status=_native.read_status()["what"])), flush=True)


if __name__ == "__main__":
    main()
