"""The mechanisms of Famepel alone, each op against the plain reference of ``famepel_oracle`` in float64, on the CPU references of the ops and, on a GPU
box, on the kernels.  Inputs are made so that a fault shows: single keys that stand out, gates near 0 and near 1, steps that forget everything."""
import math

import pytest
import torch

from . import famepel_oracle as O
from gemm_b200.models.config import RotarySpec
from gemm_b200.ops import attention as att
from gemm_b200.ops import gemm, latent, moe, recurrent, stream

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
LENS = [[1], [16], [17, 1, 130], [300, 5], [129, 128, 64]]


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, s=1.0):
    return torch.randn(*shape, generator=g) * s


def check_status(device):
    if device == "cuda":
        from gemm_b200 import _native
        _native.assert_status_ok()


def rel(got, ref):
    return float((got.double().cpu() - ref).abs().max() / ref.abs().max())


def batch(lens, device):
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=device)
    slots = torch.tensor([(3 * i + 2) % (len(lens) + 3) for i in range(len(lens))], dtype=torch.int32)
    if len(set(slots.tolist())) < len(lens):
        slots = torch.arange(len(lens), dtype=torch.int32)
    return cu, slots.to(device)


# ------------------------------------------------------------------------------------------ convolution
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolution(taps, dtype, device):
    """Unequal sequences in two portions (the second cut inside the history), channels in the middle of wider rows, partial sums."""
    for ch in (24, 37):
        g = gen(taps * 100 + ch)
        lens = [40, 3, 71, 2]
        w, b = rnd(g, ch, taps), rnd(g, ch)
        xs = [rnd(g, n, ch).to(dtype).float() for n in lens]
        state = torch.randn(6, taps - 1, ch, generator=g)
        slots = [4, 0, 5, 2]
        state[slots] = 0
        keep = state[1].clone()
        state, wd, bd = state.to(device).contiguous(), w.to(device), b.to(device)
        got = [[] for _ in lens]
        for part in ([min(n, 33) if i != 1 else 1 for i, n in enumerate(lens)], None):
            done = [sum(len(y) for y in o) for o in got]
            part = part or [n - d for n, d in zip(lens, done)]
            rows = torch.cat([xs[i][done[i]: done[i] + part[i]] for i in range(4)])
            wide = torch.full((rows.shape[0], ch + 16), 99.0)
            wide[:, 8: 8 + ch] = rows
            cu = torch.tensor([0] + list(torch.tensor(part).cumsum(0)), dtype=torch.int32, device=device)
            src = wide.to(device).to(dtype)
            if dtype == torch.float32:
                src = gemm.PendingPartials(torch.stack([0.25 * src, 0.75 * src]).contiguous())
            y = recurrent.causal_conv(src, 8, wd, bd, state, cu, torch.tensor(slots, dtype=torch.int32, device=device), max(part), dtype)
            at = 0
            for i, n in enumerate(part):
                got[i].append(y[at: at + n, :ch].float().cpu())
                at += n
        for i in range(4):
            ref = O.causal_conv_silu(xs[i].double(), w.double(), b.double())
            assert rel(torch.cat(got[i]), ref) < (1e-2 if dtype == torch.bfloat16 else 2e-6)
        assert torch.equal(state[1].cpu(), keep)


# ------------------------------------------------------------------------------------------ Mamba-2
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", ["f32", "bf16"])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 2, 128, 64), (6, 3, 24, 40), (1, 1, 8, 8), (3, 1, 13, 11), (2, 2, 72, 200)])
def test_ssd(heads, groups, dim, vdim, fmt, device):
    dt_ = torch.float32 if fmt == "f32" else torch.bfloat16
    for lens in LENS:
        g = gen(sum(lens) + heads)
        t = sum(lens)
        nv = heads * vdim
        xbc = rnd(g, t, nv + 2 * groups * dim, s=0.5).to(dt_)
        dt = rnd(g, t, heads, s=2.0)
        dt[::7] = 6.0                                    # a step that forgets nearly everything
        dt[3::11] = -30.0                                # ... and one that does nothing
        bias, a_log, d = rnd(g, heads), torch.linspace(-3, 2.5, heads), rnd(g, heads)
        cu, slots = batch(lens, device)
        state = torch.zeros(len(lens) + 3, heads, dim, vdim, device=device)
        wide = torch.zeros(t, heads + 5)
        wide[:, 3: 3 + heads] = dt
        half = torch.stack([0.5 * wide, 0.5 * wide]).to(device).contiguous()
        pad = (-xbc.shape[1]) % 8
        rows = torch.nn.functional.pad(xbc, (0, pad)).to(device).contiguous()
        args = (3, bias.to(device), -torch.exp(a_log).to(device), d.to(device), state, cu, slots, heads, groups, dim, vdim)
        got = recurrent.ssd(rows, gemm.PendingPartials(half), *args, max(lens)).cpu()
        check_status(device)
        for i, n in enumerate(lens):
            lo = int(cu[i])
            y = xbc[lo: lo + n].double()
            ref = O.ssd_recurrence(y[:, :nv].reshape(n, heads, vdim), y[:, nv: nv + groups * dim].reshape(n, groups, dim), y[:, nv + groups * dim:].reshape(n, groups, dim),
                                   O.softplus(dt[lo: lo + n].double() + bias.double()), a_log.double(), d.double())
            assert rel(got[lo: lo + n], ref.reshape(n, -1)) < 1e-4, (lens, i)


def _ssd_pieces(cuts, device, fmt):
    g = gen(5)
    heads, groups, dim, vdim, t = 2, 1, 64, 64, 290
    xbc = rnd(g, t, heads * vdim + 2 * groups * dim, s=0.5).to(fmt).to(device)
    dt = rnd(g, t, heads).to(device)
    state = torch.zeros(2, heads, dim, vdim, device=device)
    out, at = [], 0
    for n in cuts:
        cu = torch.tensor([0, n], dtype=torch.int32, device=device)
        out.append(recurrent.ssd(xbc[at: at + n].contiguous(), dt[at: at + n].contiguous(), 0, torch.zeros(heads, device=device), torch.tensor([-0.1, -0.02], device=device),
                                 torch.ones(heads, device=device), state, cu, torch.tensor([1], dtype=torch.int32, device=device), heads, groups, dim, vdim, n))
        at += n
    return torch.cat(out), state


@pytest.mark.parametrize("device", DEVICES)
def test_ssd_portions_do_not_matter(device):
    whole, s0 = _ssd_pieces([290], device, torch.bfloat16)
    for cuts in ([2] * 145, [127, 2, 128, 33], [16, 17, 256, 1]):
        got, s1 = _ssd_pieces(cuts, device, torch.bfloat16)
        assert rel(got, whole.double().cpu()) < 5e-5 and rel(s1, s0.double().cpu()) < 5e-5
    check_status(device)


# ------------------------------------------------------------------------------------------ HGRN2
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", ["f32", "bf16"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 128, 128), (3, 24, 40), (1, 8, 8), (3, 10, 9), (2, 64, 72), (1, 72, 200)])
def test_gla(heads, dim, vdim, fmt, device):
    """Gates from 1e-9 to nearly 1, in blocks of both and mixed."""
    act = fmt == "bf16"
    for lens in LENS:
        g = gen(sum(lens) + heads)
        t, nq, nv = sum(lens), heads * dim, heads * vdim
        q, v = rnd(g, t, nq), rnd(g, t, nv)
        z = rnd(g, t, nq, s=3.0)
        z[20:60] += 6.0                                  # remembers
        z[64:90, ::3] = -20.0                            # forgets at once, on every third channel
        z[100:103] = -25.0
        low = (torch.rand(nq, generator=g) * 0.9)
        low[::3] = 0.0
        bias = rnd(g, nq)
        cu, slots = batch(lens, device)
        state = torch.zeros(len(lens) + 3, heads, dim, vdim, device=device)
        src = torch.cat([O.silu(q) if act else q, v], 1)
        src = torch.nn.functional.pad(src, (0, (-src.shape[1]) % 8)).to(torch.bfloat16 if act else torch.float32)
        wide = torch.zeros(t, nq + 4)
        wide[:, 4:] = z
        if act:
            qq, vv, rows = src[:, :nq].double(), src[:, nq: nq + nv].double(), src.to(device).contiguous()
        else:
            qq, vv, rows = O.silu(q.double()), v.double(), gemm.PendingPartials(torch.stack([0.5 * src, 0.5 * src]).to(device).contiguous())
        got = recurrent.gla(rows, wide.to(device), 4, bias.to(device), low.to(device), state, cu, slots, heads, dim, vdim, act, max(lens)).cpu()
        check_status(device)
        f = low.double() + (1 - low.double()) * torch.sigmoid(z.double() + bias.double())
        for i, n in enumerate(lens):
            lo = int(cu[i])
            r = slice(lo, lo + n)
            ref = O.gated_recurrence(qq[r].reshape(n, heads, dim), f[r].reshape(n, heads, dim), vv[r].reshape(n, heads, vdim)).reshape(n, -1)
            assert rel(got[r], ref) < 1e-4, (lens, i)


@pytest.mark.parametrize("device", DEVICES)
def test_gla_portions_do_not_matter(device):
    g = gen(8)
    heads, dim, vdim, t = 2, 128, 64, 290
    qv = rnd(g, t, heads * (dim + vdim)).bfloat16().to(device)
    z = (rnd(g, t, heads * dim, s=2.0) + 2).to(device)
    low = torch.full((heads * dim,), 0.1, device=device)

    def run(cuts):
        state = torch.zeros(2, heads, dim, vdim, device=device)
        out, at = [], 0
        for n in cuts:
            cu = torch.tensor([0, n], dtype=torch.int32, device=device)
            out.append(recurrent.gla(qv[at: at + n].contiguous(), z[at: at + n].contiguous(), 0, torch.zeros_like(low), low, state, cu,
                                     torch.tensor([1], dtype=torch.int32, device=device), heads, dim, vdim, True, n))
            at += n
        return torch.cat(out), state

    whole, s0 = run([290])
    for cuts in ([2] * 145, [127, 2, 128, 33], [16, 17, 256, 1]):
        got, s1 = run(cuts)
        assert rel(got, whole.double().cpu()) < 5e-5 and rel(s1, s0.double().cpu()) < 5e-5
    check_status(device)


# ------------------------------------------------------------------------------------------ latent attention
def test_rotation_frequencies():
    for rot in ({"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}}, {"dims": 16, "base": 1e4},
                {"dims": 6, "base": 300.0, "scaling": {"factor": 2.0, "original": 40, "fast": 4.0, "slow": 4.0}},
                {"dims": 32, "base": 1e4, "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}}):
        f, mag = O.rotary_frequencies(rot)
        sc = rot.get("scaling")
        spec = RotarySpec(rot["dims"], rot["base"], *(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ())
        assert spec.frequencies() == pytest.approx(f, rel=1e-14) and spec.magnitude == pytest.approx(mag, rel=1e-14)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_store_and_queries(dtype, device):
    """Norms, rotation (also at large positions) and where the rows go."""
    g = gen(3)
    t, qr, r, rd, hd, d = 70, 56, 72, 16, 3, 24
    rot = {"dims": rd, "base": 1e4, "scaling": {"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0}}
    spec = RotarySpec(rd, 1e4, 4.0, 64, 32.0, 1.0)
    freq = torch.tensor(spec.frequencies(), dtype=torch.float64, device=device)
    pos = torch.arange(t, dtype=torch.int32)
    pos[60:] += 100003
    slots = torch.randperm(t, generator=g).to(torch.int32)
    slots[5] = -1
    rows = rnd(g, t, qr + r + rd).to(dtype)
    qn, kn = rnd(g, qr), rnd(g, r)
    w = stream.row_width(r + rd, dtype)
    cache = torch.full((t, 1, w), 7.0, dtype=dtype, device=device)
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    got = latent.latent_store(rows.to(device), pos.to(device), slots.to(device), qn.to(device), kn.to(device), freq, spec.magnitude, cache, qr, r, rd, 1e-5, dtype).cpu()
    x = rows.double()
    assert rel(got[:, :qr], O.rms(x[:, :qr], 1e-5) * qn.double()) < tol
    ref = torch.cat([O.rms(x[:, qr: qr + r], 1e-5) * kn.double(), O.rotate(x[:, qr + r:], pos, rot)], -1)
    ok = slots >= 0
    assert rel(cache.cpu()[slots[ok].long(), 0, : r + rd], ref[ok]) < tol
    untouched = (set(range(t)) - set(slots[ok].tolist())).pop()              # of the token that is not stored
    assert bool((cache.cpu()[untouched] == 7.0).all())
    q = rnd(g, t, hd * (d + rd)).to(dtype)
    dst = torch.tensor([(i // 2) if i % 2 == 0 else -1 - i // 2 for i in range(t)], dtype=torch.int32)
    dp, rp = stream.row_width(d, dtype) + 8, stream.row_width(rd, dtype)
    mk = lambda *s: torch.full(s, 5.0, dtype=dtype, device=device)
    an, ar, mn, mr = mk(hd, 40, dp), mk(hd, 40, w), mk(35, hd, dp), mk(35, hd, rp)
    latent.latent_q(q.to(device), pos.to(device), freq, spec.magnitude, 0.3, dst.to(device), (an.transpose(0, 1), ar[:, :, r:].transpose(0, 1)), (mn, mr), hd, d, rd)
    y = q.double().reshape(t, hd, d + rd)
    n_ref, r_ref = y[..., :d] * 0.3, O.rotate(y[..., d:], pos, rot) * 0.3
    assert rel(an.cpu()[:, :35, :d].transpose(0, 1), n_ref[::2]) < tol and rel(ar.cpu()[:, :35, r: r + rd].transpose(0, 1), r_ref[::2]) < tol
    assert rel(mn.cpu()[..., :d], n_ref[1::2]) < tol and rel(mr.cpu()[..., :rd], r_ref[1::2]) < tol
    assert not an.cpu()[:, :35, d:].any() and not mn.cpu()[..., d:].any() and bool((an.cpu()[:, 35:] == 5).all())


class _Fb:
    pass


def _latent_case(g, lens, ctx, heads, d, rd, v, r, page, dtype, loud):
    """Cached rows in shuffled pages, queries, projections.  ``loud``: per sequence, one key that the last query of each head asks for."""
    kv = [a + b for a, b in zip(lens, ctx)]
    w = stream.row_width(r + rd, dtype)
    per = [(n + page - 1) // page for n in kv]
    pages = torch.randperm(sum(per) + 2, generator=g)
    bt = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    cache = rnd(g, (sum(per) + 2) * page, 1, w).to(dtype)
    cache[..., r + rd:] = 0
    seqs, at = [], 0
    for i, n in enumerate(kv):
        bt[i, : per[i]] = pages[at: at + per[i]].to(torch.int32)
        at += per[i]
        pos = torch.arange(n)
        seqs.append(bt[i].long()[pos // page] * page + pos % page)
    t = sum(lens)
    uk, uv = rnd(g, heads, d, r, s=r ** -0.5).to(dtype), rnd(g, heads, v, r, s=r ** -0.5).to(dtype)
    qn, qr = rnd(g, t, heads, d, s=0.4), rnd(g, t, heads, rd, s=0.4)
    at = 0
    for i, n in enumerate(lens):
        for h in range(heads):
            c = cache[seqs[i][loud[i]], 0].float()
            qr[at + n - 1, h] = c[r: r + rd] * (14.0 / float(c[r: r + rd].pow(2).sum()))      # a score that stands out
        at += n
    return kv, bt, cache, seqs, uk, uv, qn.to(dtype), qr.to(dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,d,rd,v,r,page", [(4, 128, 64, 128, 512, 64), (3, 24, 16, 40, 72, 64), (20, 64, 32, 64, 136, 16), (37, 32, 8, 24, 200, 128), (1, 8, 2, 8, 8, 64),
                                                 (2, 16, 6, 9, 30, 24)])
def test_latent_attention(heads, d, rd, v, r, page, dtype, device):
    """Both forms against expanded keys and values: prompts on top of a context, short portions and single tokens in one batch; the key that stands out
    lies at the first and last place of a page, of a 128-key block, and at the ends of the sequence; sinks from negligible to dominant."""
    lens, ctx = [150, 1, 17, 2, 1, 300], [0, 0, 128, 191, 700, 45]
    loud = [0, 0, 127, 64, 63, 128]
    g = gen(heads * 1000 + r)
    kv, bt, cache, seqs, uk, uv, qn, qr = _latent_case(g, lens, ctx, heads, d, rd, v, r, page, dtype, loud)
    sink = torch.linspace(-6.0, 9.0, heads) if heads > 1 else torch.tensor([2.0])
    t = sum(lens)
    spec = _Fb()
    spec.head_dim, spec.rot_dim, spec.v_dim, spec.kv_rank = d, rd, v, r
    refs, at = [], 0
    for i, n in enumerate(lens):
        c = cache[seqs[i], 0].double()
        k = torch.cat([torch.einsum("kr,hdr->khd", c[:, :r], uk.double()), c[:, None, r: r + rd].expand(-1, heads, rd)], -1)
        val = torch.einsum("kr,hvr->khv", c[:, :r], uv.double())
        q = torch.zeros(kv[i], heads, d + rd, dtype=torch.float64)
        q[-n:] = torch.cat([qn[at: at + n], qr[at: at + n]], -1).double()
        refs.append(O.sink_attention(q, k, val, 1.0, sink.double())[-n:])
        at += n
    ref = torch.cat(refs)
    fb = _Fb()
    fb.block_table, fb.kv_len = bt.to(device), torch.tensor(kv, dtype=torch.int32, device=device)
    fb.cu_q = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=device)
    cache, sk = cache.to(device), (sink * att.LOG2E).to(device)
    w, dp, rp, vp = cache.shape[2], stream.row_width(d, dtype), stream.row_width(rd, dtype), stream.row_width(v, dtype)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    pad = torch.nn.functional.pad
    for expand in ([False, True] if dtype == torch.bfloat16 and latent.can_expand(spec) else [False]):
        plan = latent.make_plan(lens, kv, max(kv), device, False, expand, [heads])
        out = torch.zeros(t, heads, vp, dtype=dtype)
        dst = plan.dst.cpu().long()
        assert sorted(dst.tolist()) == list(range(-plan.n_exp, plan.n_abs))
        if plan.n_abs:
            qa = torch.zeros(heads, plan.m, w, dtype=dtype)
            for tok in range(t):
                if dst[tok] >= 0:
                    ql = torch.einsum("hd,hdr->hr", qn[tok].float(), uk.float())
                    qa[:, dst[tok], : r + rd] = (torch.cat([ql, qr[tok].float()], -1) * att.LOG2E).to(dtype)
            for splits in (1, 3):
                plan.splits = splits
                o = latent.attend_latents(qa.to(device), cache, r, r + rd, plan, fb, page, sk).float().cpu()
                for tok in range(t):
                    if dst[tok] >= 0:
                        got = torch.einsum("hr,hvr->hv", o[:, dst[tok], :r].double(), uv.double())
                        assert (got - ref[tok]).abs().max() < tol * ref.abs().max(), (tok, splits, expand)
        if plan.n_exp:
            kvx = torch.cat([torch.einsum("kr,hdr->khd", cache[torch.cat([seqs[s] for s in plan.seqs.tolist()]).to(device), 0, :r].float().cpu(), pad(uk, (0, 0, 0, dp - d)).float())
                             .reshape(plan.n_kv, -1), torch.einsum("kr,hvr->khv", cache[torch.cat([seqs[s] for s in plan.seqs.tolist()]).to(device), 0, :r].float().cpu(),
                                                                   pad(uv, (0, 0, 0, vp - v)).float()).reshape(plan.n_kv, -1)], 1).to(dtype).to(device)
            rows = latent.gather_latents(cache, plan, fb.block_table, page)
            tok = plan.exp_tok.cpu().long()
            en, er = pad(qn[tok].float() * att.LOG2E, (0, dp - d)).to(dtype).to(device), pad(qr[tok].float() * att.LOG2E, (0, rp - rd)).to(dtype).to(device)
            res = torch.zeros(t, heads, vp, dtype=dtype, device=device)
            latent.attend_expanded(en.contiguous(), er.contiguous(), kvx, rows, r, plan, sk, res)
            assert (res.cpu()[tok][..., :v].double() - ref[tok]).abs().max() < tol * ref.abs().max()
            assert not res.cpu()[dst >= 0].any()
    check_status(device)


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("e,top,count,keep", [(16, 4, 4, 2), (12, 4, 3, 2), (9, 2, 9, 3), (8, 8, 1, 1), (128, 8, 8, 4), (300, 6, 100, 40), (1, 1, 1, 1), (6, 6, 3, 3), (256, 16, 128, 60)])
def test_routing(e, top, count, keep, device):
    g = gen(e + top)
    for t in (1, 33, 300):
        z = rnd(g, t, e, s=2.0)
        groups = {"count": count, "keep": keep} if count > 1 else None
        want_ids, want_w = O.route(z.double(), top, groups, 1.7)
        got = [moe.route(z.to(device), top, "sigmoid", None, 2, 1.7, None, (count, keep))]
        got.append(moe.route_plan(z.to(device), top, e, 64, mode="sigmoid", renorm=2, routed_scale=1.7, groups=(count, keep))[:2])
        for ids, w in got:
            same = (ids.cpu().long() == want_ids).all(1)
            assert same.float().mean() > 0.98                                # (ties by rounding)
            assert rel(w[same.to(w.device)], want_w[same]) < 1e-5
    z = torch.full((3, e), -60.0)                                            # scores that underflow nearly to zero: the sum's offset matters
    _, w = moe.route(z.to(device), top, "sigmoid", None, 2, 1.0, None, (count, keep))
    s = torch.sigmoid(z.double())[0, 0]
    assert rel(w, torch.full((3, top), float(s / (s * top + 1e-20)), dtype=torch.float64)) < 1e-3


@pytest.mark.gpu
@pytest.mark.parametrize("groups", [(1, 1), (8, 3)])
def test_fused_front_end_routes_by_groups(groups):
    """The one-launch router + plan + gather of decode-sized batches."""
    g = gen(4)
    h, w = rnd(g, 50, 512).bfloat16().cuda(), rnd(g, 64, 512, s=0.1).bfloat16().cuda()
    assert moe.can_prep(h, w, 6)
    ids, wt, pl, rows = moe.prep_hidden(h, w, 6, 64, 16, "sigmoid", renorm=2, routed_scale=2.5, quantize=False, groups=groups)
    z = h.double().cpu() @ w.double().cpu().t()
    want_ids, want_w = O.route(z, 6, {"count": groups[0], "keep": groups[1]}, 2.5)
    same = (ids.cpu().long() == want_ids).all(1)
    assert same.float().mean() > 0.9 and rel(wt[same.cuda()], want_w[same]) < 1e-4
    assert torch.equal(rows[pl.pair_row.long()].cpu(), h.cpu().repeat_interleave(6, dim=0))


@pytest.mark.parametrize("device", DEVICES)
def test_f32_products(device):
    g = gen(6)
    x, w = rnd(g, 3, 70, 37), rnd(g, 3, 50, 37)
    out = torch.zeros(70, 3, 60, device=device)
    gemm.batched_linear_f32(x.to(device), w.to(device), out[:, :, 5:55].transpose(0, 1))
    assert rel(out[:, :, 5:55].transpose(0, 1), torch.bmm(x.double(), w.double().transpose(1, 2))) < 1e-6 and not out[:, :, :5].any()
    start, count = torch.tensor([0, 64, 192], dtype=torch.int32), torch.tensor([3, 100, 0], dtype=torch.int32)
    src = torch.randint(0, 70, (256,), generator=g).to(torch.int32)
    src[130:] = -1
    got = gemm.grouped_linear_f32(x[0].to(device), w.to(device), start.to(device), count.to(device), 256, src.to(device)).cpu()
    for i in range(2):
        s, c = int(start[i]), int(count[i])
        ref = (x[0].double()[src[s: s + c].long().clamp_min(0)] * (src[s: s + c] >= 0).unsqueeze(1)) @ w[i].double().t()
        assert rel(got[s: s + c], ref) < 1e-6


# ------------------------------------------------------------------------------------------ stream and norms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [136, 90, 1300])
def test_dynamic_tanh_stream(width, device):
    """Update through its own norm, stream, next norm in one step; plain, partial-sum and expert updates; selected rows."""
    g = gen(width)
    t, k = 21, 3
    t_ = {}
    for nm in ("n", "p"):
        t_[nm], t_[nm + ".b"], t_[nm + ".alpha"] = rnd(g, width), rnd(g, width), torch.tensor(0.3 + 0.4 * (nm == "p"))
    mk = lambda nm: stream.DynTanh(float(t_[nm + ".alpha"]), t_[nm].to(device), t_[nm + ".b"].to(device))
    td = {a: b.double() for a, b in t_.items()}
    x0 = rnd(g, t, width, s=3.0)
    pad = (-width) % 8
    y = rnd(g, 80, width + pad)
    pair = torch.randperm(80, generator=g)[: t * k].to(torch.int32)
    pair[4] = -1
    wts = torch.rand(t, k, generator=g)
    moe_ref = sum(wts[:, j: j + 1].double() * torch.where(pair.reshape(t, k)[:, j: j + 1] >= 0, y.double()[pair.reshape(t, k)[:, j].clamp_min(0).long()], torch.zeros(1).double()) for j in range(k))
    u = rnd(g, t, width)
    for upd, ref_u in ((None, None), (u.to(device), u.double()), (gemm.PendingPartials(torch.stack([u, 2 * u]).to(device).contiguous()), 3 * u.double()),
                       (moe.PendingCombine(y.to(device), pair.to(device), wts.to(device), t, k), moe_ref[:, :width]),
                       (moe.PendingCombine(y.bfloat16().to(device), pair.to(device), wts.to(device), t, k), None)):
        if ref_u is None and upd is not None:
            yb = y.bfloat16().double()
            ref_u = sum(wts[:, j: j + 1].double() * torch.where(pair.reshape(t, k)[:, j: j + 1] >= 0, yb[pair.reshape(t, k)[:, j].clamp_min(0).long()], torch.zeros(1).double())
                        for j in range(k))[:, :width]
        for post in (False, True):
            if upd is None and post:
                continue
            xr = x0.double() if upd is None else x0.double() + (O.dyn_tanh(ref_u, td, "p") if post else ref_u)
            d = stream.PostNormed(upd, mk("p")) if post else upd
            for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
                x = x0.clone().to(device)
                o = stream.norm(x, mk("n"), 1e-5, d, out_dtype=dtype)
                assert rel(x, xr) < 3e-6 and rel(o[:, :width], O.dyn_tanh(xr, td, "n")) < tol and not o[:, width:].any()
            rows = torch.tensor([7, 0, 20], device=device)
            x = x0.clone().to(device)
            o = stream.norm(x, mk("n"), 1e-5, d, rows=rows, out_dtype=torch.float32)
            assert torch.equal(x.cpu(), x0) and rel(o, O.dyn_tanh(xr[[7, 0, 20]], td, "n")) < 3e-6
    e = stream.embed(torch.tensor([3, 1], dtype=torch.int32, device=device), y.bfloat16().to(device), 5.5)
    assert rel(e, y.bfloat16().double()[[3, 1]] * 5.5) < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n,parts", [(96, 4), (96, 1), (33, 3), (40, 40), (2048, 2), (4096, 1)])
def test_part_norm(n, parts, device):
    g = gen(n + parts)
    o, z, w = rnd(g, 19, n), rnd(g, 19, n + 7, s=2.0), rnd(g, n)
    ref = O.gated_group_norm(o.double(), z[:, 5: 5 + n].double(), w.double(), parts, 1e-5)
    got = stream.part_norm(o.to(device), w.to(device), parts, 1e-5, gemm.PendingPartials(torch.stack([0.5 * z, 0.5 * z]).to(device).contiguous()), 5, torch.float32)
    assert rel(got, ref) < 3e-6
    got = stream.part_norm(o.to(device), w.to(device), parts, 1e-5, z.bfloat16().to(device), 5)
    assert rel(got[:, :n], O.gated_group_norm(o.double(), z.bfloat16()[:, 5: 5 + n].double(), w.double(), parts, 1e-5)) < 8e-3 and not got[:, n:].any()
    short = w[: n // parts]
    got = stream.part_norm(o.to(device), short.to(device), parts, 1e-5, out_dtype=torch.float32)
    assert rel(got, O.rms(o.double().reshape(19, parts, -1), 1e-5).reshape(19, n) * short.double().repeat(parts)) < 3e-6
    assert math.isfinite(float(got.sum()))
