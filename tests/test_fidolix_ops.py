"""The mechanisms of Fidolix alone, each op against the plain reference of ``fidolix_oracle`` in float64, on the CPU references of the ops and, on a GPU
box, on the kernels.  Inputs are made so that a fault shows: single keys that stand out at the edges of windows, pages and key blocks, scores on both sides
of the cap, decays that forget at once and that hold."""
import pytest
import torch

from . import fidolix_oracle as O
from gemm_b200.models.config import RotarySpec
from gemm_b200.ops import attention as att
from gemm_b200.ops import elementwise as ew
from gemm_b200.ops import gemm, moe, recurrent, stream

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = [torch.float32, torch.bfloat16]
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


def halves(x, device):
    """``x`` as the partial sums of a projection."""
    return gemm.PendingPartials(torch.stack([0.25 * x, 0.75 * x]).to(device).contiguous())


def cum(lens, device):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=device)


def batch(lens, device):
    slots = torch.tensor([(3 * i + 2) % (len(lens) + 3) for i in range(len(lens))], dtype=torch.int32)
    if len(set(slots.tolist())) < len(lens):
        slots = torch.arange(len(lens), dtype=torch.int32)
    return cum(lens, device), slots.to(device)


# ------------------------------------------------------------------------------------------ attention
def _attention_case(g, lens, ctx, hq, hkv, dk, dv, page, dtype, padded):
    """Cached keys and values in shuffled pages, and queries."""
    kv = [a + b for a, b in zip(lens, ctx)]
    dkp, dvp = att.cache_head_dims(dk, dv, dtype) if padded else (dk, dv)
    per = [(n + page - 1) // page for n in kv]
    pages = torch.randperm(sum(per) + 2, generator=g)
    bt = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    rows = (sum(per) + 2) * page
    k, v = torch.zeros(rows, hkv, dkp), torch.zeros(rows, hkv, dvp)
    k[..., :dk], v[..., :dv] = rnd(g, rows, hkv, dk, s=0.5), rnd(g, rows, hkv, dv)
    seqs, at = [], 0
    for i, n in enumerate(kv):
        bt[i, : per[i]] = pages[at: at + per[i]].to(torch.int32)
        at += per[i]
        pos = torch.arange(n)
        seqs.append(bt[i].long()[pos // page] * page + pos % page)
    q = torch.zeros(sum(lens), hq, dkp)
    q[..., :dk] = rnd(g, sum(lens), hq, dk, s=0.5)
    return kv, bt, k, v, seqs, q


def _run_attention(lens, ctx, hq, hkv, dk, dv, page, dtype, device, window=0, softcap=0.0, sink=None, loud=None, scale=1.0):
    """(result, reference) of one batch; ``loud``: position -> key position which the query of the first head of each group asks for."""
    g = gen(hq * 100 + dk + window)
    kv, bt, k, v, seqs, q = _attention_case(g, lens, ctx, hq, hkv, dk, dv, page, dtype, True)
    per, at = hq // hkv, 0
    for i, n in enumerate(lens):
        for x in range(n):
            pos = ctx[i] + x
            for j in (loud(pos) if loud else []):
                if 0 <= j <= pos:
                    for h in range(0, hq, per):
                        key = k[seqs[i][j], h // per]
                        q[at + x, h] = key * (9.0 / scale / float(key.pow(2).sum()))
        at += n
    q, k, v = q.to(dtype).float(), k.to(dtype), v.to(dtype)
    factor = scale / softcap if softcap else scale * att.LOG2E
    decode = all(n == 1 for n in lens)
    splits = [1, 3] if decode and device == "cuda" and dtype == torch.bfloat16 else [1]
    refs, at = [], 0
    for i, n in enumerate(lens):
        full = torch.zeros(kv[i], hq, dk, dtype=torch.float64)
        qs = (q[at: at + n, :, :dk] * factor).to(dtype).double() / factor
        full[-n:] = qs
        ks, vs = k[seqs[i]][..., :dk].double(), v[seqs[i]][..., :dv].double()
        refs.append(O.attend(full, ks, vs, scale, window=window or None, softcap=softcap or None, sink=sink.double() if sink is not None else None)[-n:])
        at += n
    outs = []
    for sp in splits:
        plan = (att.build_work(lens, hq, hkv, sp).to(device), sp) if device == "cuda" else None
        o = att.attention_masked((q * factor).to(dtype).to(device), k.to(device), v.to(device), cum(lens, device), torch.tensor(kv, dtype=torch.int32, device=device), bt.to(device), page,
                                 window=window, plan=plan, decode=decode, softcap=softcap, sink=(sink * att.LOG2E).to(device) if sink is not None else None)
        outs.append(o.float().cpu()[..., :dv])
    check_status(device)
    return outs, torch.cat(refs)


SHAPES = [(8, 2, 128, 128, 64), (6, 3, 40, 40, 64), (5, 1, 64, 64, 16), (3, 3, 24, 100, 128), (16, 1, 128, 64, 64), (2, 1, 160, 136, 64), (2, 2, 16, 16, 24)]
BATCHES = [([150, 1, 17, 2, 300], [0, 300, 128, 191, 45]), ([1, 1, 1, 1], [0, 63, 128, 700]), ([2, 2], [126, 0])]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,dk,dv,page", SHAPES)
def test_capped_scores(hq, hkv, dk, dv, page, dtype, device):
    """Scores far below the cap, around it and far above; keys that stand out at the start, at page and block borders and next to the query."""
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    for (lens, ctx), (cap, scale) in zip(BATCHES, ((30.0, 1.0), (4.0, 0.7), (1.0, 2.5))):
        outs, ref = _run_attention(lens, ctx, hq, hkv, dk, dv, page, dtype, device, softcap=cap, scale=scale, loud=lambda p: [(p * 37) % (p + 1)] if p % 3 else [0])
        for got in outs:
            assert rel(got, ref) < tol


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 17, 64, 129, 0])
@pytest.mark.parametrize("hq,hkv,dk,dv,page", SHAPES)
def test_windows_with_sinks(hq, hkv, dk, dv, page, window, dtype, device):
    """The key that stands out is the oldest one in the window, or the first one outside of it; sinks from negligible to dominant."""
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2
    sink = torch.linspace(-6.0, 8.0, hq)
    w = window or 10 ** 6
    for lens, ctx in BATCHES:
        outs, ref = _run_attention(lens, ctx, hq, hkv, dk, dv, page, dtype, device, window=window, sink=sink, loud=lambda p: [p - w + 1] if p % 2 else [p - w])
        for got in outs:
            assert rel(got, ref) < tol
    off = _run_attention(*BATCHES[0], hq, hkv, dk, dv, page, torch.float32, "cpu", window=w - 1 if window > 1 else 2, sink=sink, loud=lambda p: [p - w + 1] if p % 2 else [p - w])[1] \
        if window else None
    if off is not None:                                                       # such a key makes a window that is one off show
        assert rel(off, _run_attention(*BATCHES[0], hq, hkv, dk, dv, page, torch.float32, "cpu", window=window, sink=sink,
                                       loud=lambda p: [p - w + 1] if p % 2 else [p - w])[1]) > 0.05


@pytest.mark.parametrize("device", DEVICES)
def test_capped_scores_with_sinks(device):
    sink = torch.tensor([3.0, -2.0, 0.5, 6.0])
    for dtype in DTYPES:
        for lens, ctx in BATCHES:
            outs, ref = _run_attention(lens, ctx, 4, 2, 64, 64, 64, dtype, device, window=40, softcap=5.0, sink=sink, loud=lambda p: [p - 39])
            for got in outs:
                assert rel(got, ref) < (1e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,dk,dv", [(4, 2, 40, 24), (3, 1, 10, 9), (8, 8, 128, 128), (32, 4, 128, 128), (3, 3, 7, 13)])
def test_norm_over_all_heads(hq, hkv, dk, dv, dtype, device):
    g = gen(hq + dk)
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    dkp, dvp = att.cache_head_dims(dk, dv, dtype)
    t = 21
    x = rnd(g, t, nq + nk + nv + 5, s=2.0).to(dtype)
    qn, kn = rnd(g, nq), rnd(g, nk)
    slots = torch.randperm(40, generator=g)[:t].to(torch.int32)
    slots[3] = -1
    mk = lambda w: torch.full((40, hkv, w), 7.0, dtype=dtype, device=device)
    kc, vc = mk(dkp), mk(dvp)
    src = halves(x, device) if dtype == torch.float32 else x.to(device)
    q = stream.qk_rows(src, slots.to(device), qn.to(device), kn.to(device), kc, vc, hq, hkv, dk, dv, 1e-3, 0.37).cpu()
    y, tol, ok = x.double(), 3e-6 if dtype == torch.float32 else 8e-3, slots >= 0
    rq, rk = O.rms(y[:, :nq], 1e-3) * qn.double() * 0.37, O.rms(y[:, nq: nq + nk], 1e-3) * kn.double()
    at = slots[ok].long()
    assert rel(q[..., :dk], rq.reshape(t, hq, dk)) < tol and not q[..., dk:].any()
    assert rel(kc.cpu()[at, :, :dk], rk.reshape(t, hkv, dk)[ok]) < tol and not kc.cpu()[at, :, dk:].any()
    assert rel(vc.cpu()[at, :, :dv], y[:, nq + nk: nq + nk + nv].reshape(t, hkv, dv)[ok]) < tol and not vc.cpu()[at, :, dv:].any()
    rest = [i for i in range(40) if i not in at.tolist()]
    assert bool((kc.cpu()[rest] == 7).all()) and bool((vc.cpu()[rest] == 7).all())


def test_rotation_frequencies():
    for rot in ({"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}}, {"dims": 16, "base": 1e4},
                {"dims": 6, "base": 300.0, "scaling": {"factor": 2.0, "original": 40, "fast": 4.0, "slow": 4.0}}):
        f, mag = O.rotary_table(rot)
        sc = rot.get("scaling")
        spec = RotarySpec(rot["dims"], rot["base"], *(sc[k] for k in ("factor", "original", "fast", "slow")) if sc else ())
        assert spec.frequencies() == pytest.approx(f, rel=1e-14) and spec.magnitude == pytest.approx(mag, rel=1e-14)


@pytest.mark.parametrize("device", DEVICES)
def test_rotary_table_at_large_positions(device):
    freq = torch.tensor([1.0, 0.3, 1e-4], dtype=torch.float64)
    pos = torch.tensor([0, 1, 7, 100003, 1048575], dtype=torch.int32)
    got = stream.rotary_table(pos.to(device), freq.to(device), 1.25).cpu().double()
    a = pos.double().unsqueeze(1) * freq
    assert (got - torch.stack([torch.cos(a), torch.sin(a)], -1) * 1.25).abs().max() < 3e-7


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,dims,taps", [(6, 3, 40, 24, 4), (1, 1, 8, 2, 1), (4, 2, 7, 6, 5), (3, 3, 13, 10, 3), (8, 2, 128, 128, 2), (2, 1, 64, 32, 16)])
def test_convolution_and_rotation(hq, hkv, d, dims, taps, dtype, device):
    """Unequal sequences in two portions (the second cut inside the history), from zero and on the state left behind."""
    g = gen(taps * 10 + d)
    rot = {"dims": dims, "base": 500.0, "scaling": {"factor": 2.0, "original": 32, "fast": 8.0, "slow": 1.0}}
    spec = RotarySpec(dims, 500.0, 2.0, 32, 8.0, 1.0)
    freq = torch.tensor(spec.frequencies(), dtype=torch.float64, device=device)
    ch, lens = (hq + hkv) * d, [40, 3, 71, 2]
    dkp, dvp = att.cache_head_dims(d, d, dtype)
    w = rnd(g, ch, taps)
    xs = [rnd(g, n, ch).to(dtype) for n in lens]
    state = torch.randn(6, taps - 1, ch, generator=g)
    seq_slots = [4, 0, 5, 2]
    state[seq_slots] = 0
    keep = state[1].clone()
    state = state.to(device).contiguous()
    kc, vc = torch.full((200, hkv, dkp), 7.0, dtype=dtype, device=device), torch.full((200, hkv, dvp), 7.0, dtype=dtype, device=device)
    place = torch.randperm(200, generator=g)
    got, where = [[] for _ in lens], [[] for _ in lens]
    at = 0
    for part in ([min(n, 33) if i != 1 else 1 for i, n in enumerate(lens)], None):
        done = [sum(len(y) for y in o) for o in got]
        part = part or [n - x for n, x in zip(lens, done)]
        rows = torch.cat([xs[i][done[i]: done[i] + part[i]] for i in range(4)])
        pos = torch.cat([torch.arange(done[i], done[i] + part[i]) for i in range(4)]).to(torch.int32).to(device)
        n = rows.shape[0]
        slots = place[at: at + n]
        at += n
        wide = torch.full((n, ch + 8), 99.0).to(dtype)
        wide[:, :ch] = rows
        src = halves(wide, device) if dtype == torch.float32 else wide.to(device)
        q = stream.conv_rotary(src, stream.rotary_table(pos, freq, spec.magnitude), slots.to(torch.int32).to(device), w.to(device), state, cum(part, device),
                               torch.tensor(seq_slots, dtype=torch.int32, device=device), kc, vc, hq, hkv, d, 0.3, max(part)).cpu()
        assert not q[..., d:].any()
        p = 0
        for i, c in enumerate(part):
            got[i].append(q[p: p + c, :, :d])
            where[i].append(slots[p: p + c])
            p += c
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    for i in range(4):
        h = O.short_conv(xs[i].double(), w.double()).reshape(lens[i], hq + hkv, d)
        r, s = O.rotate(h, rot), torch.cat(where[i])
        assert rel(torch.cat(got[i]), r[:, :hq] * 0.3) < tol
        assert rel(kc.cpu()[s, :, :d], r[:, hq:]) < tol and rel(vc.cpu()[s, :, :d], h[:, hq:]) < tol
        assert not kc.cpu()[s, :, d:].any() and not vc.cpu()[s, :, d:].any()
    assert torch.equal(state[1].cpu(), keep) and bool((kc.cpu()[place[at:]] == 7).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dv,pad", [(4, 24, 40), (3, 9, 7), (8, 128, 0), (1, 1, 63)])
def test_output_gate(heads, dv, pad, dtype, device):
    g = gen(heads + dv)
    t = 13
    a = rnd(g, t, heads, dv + pad).to(dtype)
    z = rnd(g, t, heads * dv + 8, s=3.0).to(dtype)
    src = halves(z, device) if dtype == torch.float32 else z.to(device)
    got = stream.sigmoid_gate(a.clone().to(device), src, 4 if dtype == torch.float32 else 8, dv).cpu()
    col = 4 if dtype == torch.float32 else 8
    ref = a[..., :dv].double() * torch.sigmoid(z[:, col: col + heads * dv].double()).reshape(t, heads, dv)
    assert rel(got[..., :dv], ref) < (2e-6 if dtype == torch.float32 else 8e-3) and torch.equal(got[..., dv:], a[..., dv:])


# ------------------------------------------------------------------------------------------ RWKV
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [136, 90, 1300])
def test_token_shift(width, dtype, device):
    """Unequal sequences in portions, among them single tokens; the first token of a sequence has zeros in front of it."""
    g = gen(width)
    lens = [40, 3, 71, 2]
    mu = torch.rand(5, width, generator=g)
    ld = stream.row_width(width, dtype)
    xs = [torch.nn.functional.pad(rnd(g, n, width).to(dtype), (0, ld - width)) for n in lens]
    state = torch.randn(6, 1, width, generator=g)
    slots = [4, 0, 5, 2]
    state[slots] = 0
    keep = state[1].clone()
    state = state.to(device)
    got, done = [[] for _ in lens], [0] * 4
    for part in ([1, 1, 1, 1], [8, 1, 33, 0], [31, 1, 37, 1]):
        cu = cum(part, device)
        rows = torch.cat([xs[i][done[i]: done[i] + part[i]] for i in range(4)]).to(device)
        pad = recurrent.shift_pad(rows.shape[0])
        y = recurrent.token_shift(rows, width, mu.to(device), state, cu, torch.tensor(slots, dtype=torch.int32, device=device), pad, max(part)).cpu()
        assert y.shape == (5, pad, ld) and not y[:, : rows.shape[0], width:].any()
        for i in range(4):
            got[i].append(y[:, int(cu[i]): int(cu[i + 1]), :width])
            done[i] += part[i]
    for i in range(4):
        ref = torch.stack([O.shift_mix(xs[i][:, :width].double(), m.double()) for m in mu])
        assert done[i] == lens[i] and rel(torch.cat(got[i], 1), ref) < (1e-6 if dtype == torch.float32 else 8e-3)
        assert torch.equal(state[slots[i], 0].cpu(), xs[i][-1, :width].float())
    assert torch.equal(state[1].cpu(), keep)


def _rwkv_inputs(g, t, heads, dim, dtype):
    n = heads * dim
    r, k, v = (rnd(g, t, n).to(dtype) for _ in range(3))
    z = rnd(g, t, n, s=1.5) - 2.0
    z[20:60] -= 6.0                                      # holds
    z[64:90, ::3] = 5.0                                  # forgets at once, on every third channel
    z[100:103] = 6.0
    return r, k, v, z


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(2, 128), (3, 24), (1, 8), (3, 9), (2, 64), (1, 136), (5, 40)])
def test_rwkv(heads, dim, dtype, device):
    for lens in LENS:
        g = gen(sum(lens) + dim)
        t, n = sum(lens), heads * dim
        r, k, v, z = _rwkv_inputs(g, t, heads, dim, dtype)
        w0, u = rnd(g, n, s=0.5), rnd(g, n)
        cu, slots = batch(lens, device)
        pad, ld = recurrent.shift_pad(t), stream.row_width(n, dtype)
        rkv = torch.full((4, pad, ld), 99.0, dtype=dtype)
        for i, x in enumerate((r, k, v)):
            rkv[i, :t, :n] = x
        state = torch.zeros(len(lens) + 3, heads, dim, dim, device=device)
        zs = halves(torch.nn.functional.pad(z, (0, 3)), device)
        got = recurrent.rwkv(rkv.to(device), zs, w0.to(device), u.to(device), state, cu, slots, heads, dim, dim, t, max(lens)).cpu()
        check_status(device)
        w = torch.exp(-torch.exp(z.double() + w0.double()))
        for i, m in enumerate(lens):
            s = slice(int(cu[i]), int(cu[i]) + m)
            sh = lambda x: x[s].double().reshape(m, heads, dim)
            ref = O.time_recurrence(sh(r), sh(k), sh(v), sh(w), u.double().reshape(heads, dim)).reshape(m, n)
            assert rel(got[s], ref) < 1e-4, (lens, i)


@pytest.mark.parametrize("device", DEVICES)
def test_rwkv_portions_do_not_matter(device):
    g = gen(8)
    heads, dim, t = 2, 128, 290
    n = heads * dim
    r, k, v, z = _rwkv_inputs(g, t, heads, dim, torch.bfloat16)
    rkv, z = torch.stack([r, k, v]).to(device), z.to(device)
    w0, u = torch.zeros(n, device=device), rnd(g, n).to(device)

    def run(cuts):
        state = torch.zeros(2, heads, dim, dim, device=device)
        out, at = [], 0
        for m in cuts:
            out.append(recurrent.rwkv(rkv[:, at: at + m].contiguous(), z[at: at + m].contiguous(), w0, u, state, cum([m], device), torch.tensor([1], dtype=torch.int32, device=device),
                                      heads, dim, dim, m, m))
            at += m
        return torch.cat(out), state

    whole, s0 = run([290])
    for cuts in ([2] * 145, [127, 2, 128, 33], [16, 17, 256, 1], [1] * 290):
        got, s1 = run(cuts)
        assert rel(got, whole.double().cpu()) < 5e-5 and rel(s1, s0.double().cpu()) < 5e-5
    check_status(device)


@pytest.mark.parametrize("device", DEVICES)
def test_decay_projection_and_head_norm(device):
    g = gen(2)
    z = rnd(g, 9, 15, s=2.0)
    for n in (12, 8):
        got = recurrent.tanh_rows(halves(z, device), n)
        assert got.shape[1] == stream.row_width(n, torch.bfloat16) and rel(got[:, :n], torch.tanh(z[:, :n].double())) < 5e-3 and not got[:, n:].any()
        assert rel(recurrent.tanh_rows(z.to(device), n, torch.float32), torch.tanh(z[:, :n].double())) < 1e-6
    for n, parts in ((96, 4), (33, 3), (40, 40), (2048, 16), (272, 2), (1024, 2)):
        o, gate, w = rnd(g, 19, n), rnd(g, 19, n + 4, s=2.0), rnd(g, n)
        ref = O.rms(o.double().reshape(19, parts, -1), 1e-3).reshape(19, n) * w.double() * O.silu(gate[:, 4:].double())
        got = stream.part_norm(o.to(device), w.to(device), parts, 1e-3, halves(gate, device), 4, torch.float32, gate_after=True)
        assert rel(got, ref) < 3e-6
        got = stream.part_norm(o.to(device), w.to(device), parts, 1e-3, gate.bfloat16().to(device), 4, gate_after=True)
        assert rel(got[:, :n], O.rms(o.double().reshape(19, parts, -1), 1e-3).reshape(19, n) * w.double() * O.silu(gate.bfloat16()[:, 4:].double())) < 8e-3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("t", [1, 5, 16, 70, 200, 600])
def test_projections_of_the_mixes(t, device):
    """One grouped product for four mixes: f32 and 16-bit results, feature counts off and on the tiles, rows behind the tokens left over."""
    g = gen(t)
    for n, k in ((72, 136), (256, 64)):
        pad, np_ = recurrent.shift_pad(t), (n + 127) // 128 * 128
        x = torch.full((4, pad, k), 3.0).bfloat16()
        x[:, :t] = rnd(g, 4, t, k).bfloat16()
        w = torch.zeros(4, np_, k).bfloat16()
        w[:, :n] = rnd(g, 4, n, k, s=k ** -0.5).bfloat16()
        seg, cnt = torch.arange(4, dtype=torch.int32, device=device) * pad, torch.full((4,), t, dtype=torch.int32, device=device)
        ref = torch.bmm(x[:, :t].double(), w[:, :n].double().transpose(1, 2))
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
            out = torch.zeros(4, pad, n + 8, dtype=dtype, device=device)
            for tn in {min(pad, 128), 256 if pad >= 256 else min(pad, 128)}:
                gemm.grouped_linear(x.to(device).view(4 * pad, k), w.to(device), seg, cnt, tn, out=out.view(4 * pad, n + 8), n_out=n)
                assert rel(out[:, :t, :n], ref) < tol and not out[:, :, n:].any()
                out.zero_()
    check_status(device)


# ------------------------------------------------------------------------------------------ feed-forward
def _capped(g, u, cap):
    g, u = g.double().clamp(max=cap), u.double().clamp(-cap, cap)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cap", [0.7, 2.5])
def test_capped_feed_forward(cap, device):
    """The 32-bit form, the GEMM's epilogue and the one over K-split partial sums; values on both sides of the bounds."""
    g = gen(11)
    inter, k = 128, 72
    gu = rnd(g, 9, 2 * inter, s=2.0)
    ref = _capped(gu[:, :inter], gu[:, inter:], cap)
    assert rel(stream.act_mul(gu.to(device), "capped", cap), ref) < 2e-6
    part = gemm.PendingPartials(torch.stack([0.25 * gu, 0.75 * gu]).to(device).contiguous())
    assert rel(ew.silu_mul_partials(part, act="capped", cap=cap), ref) < 8e-3
    for t in (1, 40, 300):
        x, w = rnd(g, t, k).bfloat16(), rnd(g, 2 * inter, k, s=2.0 * k ** -0.5).bfloat16()
        y = x.double() @ w.double().t()
        assert rel(gemm.linear_swiglu(x.to(device), w.to(device), act="capped", cap=cap), _capped(y[:, :inter], y[:, inter:], cap)) < 8e-3
    check_status(device)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("e,top,count,keep", [(16, 4, 4, 2), (12, 4, 3, 2), (9, 2, 9, 3), (8, 8, 1, 1), (128, 8, 8, 4), (300, 6, 100, 40), (1, 1, 1, 1), (6, 6, 3, 3), (256, 16, 128, 60), (16, 1, 2, 1)])
def test_routing(e, top, count, keep, device):
    """Softmax over all experts, groups ranked by their best score; the two rankings differ here."""
    g = gen(e + top)
    for t in (1, 33, 300):
        z = rnd(g, t, e, s=2.0)
        groups = {"count": count, "keep": keep} if count > 1 else None
        want_ids, want_w = O.route(z.double(), top, groups)
        got = [moe.route(z.to(device), top, "softmax", None, 2, 1.0, None, (count, keep, 1))]
        got.append(moe.route_plan(z.to(device), top, e, 64, mode="softmax", renorm=2, groups=(count, keep, 1))[:2])
        for ids, w in got:
            same = (ids.cpu().long() == want_ids).all(1)
            assert same.float().mean() > 0.98                                # (ties by rounding)
            assert rel(w[same.to(w.device)], want_w[same]) < 1e-5
        if 1 < keep < count <= 8 and t == 300:
            two, _ = moe.route(z.to(device), top, "softmax", None, 2, 1.0, None, (count, keep))
            assert (two.cpu().long() != want_ids).any()


@pytest.mark.gpu
@pytest.mark.parametrize("groups", [(1, 1, 1), (8, 3, 1)])
def test_fused_front_end_routes_by_groups(groups):
    """The one-launch router + plan + gather of decode-sized batches."""
    g = gen(4)
    h, w = rnd(g, 50, 512).bfloat16().cuda(), rnd(g, 64, 512, s=0.1).bfloat16().cuda()
    assert moe.can_prep(h, w, 6)
    ids, wt, pl, rows = moe.prep_hidden(h, w, 6, 64, 16, "softmax", renorm=2, quantize=False, groups=groups)
    z = h.double().cpu() @ w.double().cpu().t()
    want_ids, want_w = O.route(z, 6, {"count": groups[0], "keep": groups[1]})
    same = (ids.cpu().long() == want_ids).all(1)
    assert same.float().mean() > 0.9 and rel(wt[same.cuda()], want_w[same]) < 1e-4
    assert torch.equal(rows[pl.pair_row.long()].cpu(), h.cpu().repeat_interleave(6, dim=0))


# ------------------------------------------------------------------------------------------ stream
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [136, 90, 1300, 2048, 5000])
def test_stream_with_a_normed_update(width, device):
    """Update through its own norm, a row per token, the stream, two sets of normalised rows; partial sums; selected rows."""
    g = gen(width)
    t = 21
    x0, u, add, post, w1, w2 = rnd(g, t, width, s=3.0), rnd(g, t, width), rnd(g, t, width), rnd(g, width), rnd(g, width), rnd(g, width)
    d = lambda z: z.to(device)
    ud = O.rms(u.double(), 1e-2) * post.double()
    for upd, up_ref in ((None, 0), (d(u), ud), (halves(u, device), ud), (d(u.bfloat16()), O.rms(u.bfloat16().double(), 1e-2) * post.double())):
        delta = stream.RmsPosted(upd, d(post), 1e-2) if upd is not None else None
        for extra in (None, add):
            ref = x0.double() + up_ref + (extra.double() if extra is not None else 0)
            n = O.rms(ref, 1e-3)
            for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
                x = d(x0.clone())
                a, b = stream.norm2(x, d(w1), 1e-3, delta, d(extra) if extra is not None else None, weight2=d(w2), out_dtype=dtype)
                assert rel(x, ref) < 3e-6
                for o, w in ((a, w1), (b, w2)):
                    assert rel(o[:, :width], n * w.double()) < tol and not o[:, width:].any()
            x = d(x0.clone())
            (a,) = stream.norm2(x, d(w1), 1e-3, delta, d(extra) if extra is not None else None, out_dtype=torch.float32)
            assert rel(x, ref) < 3e-6 and rel(a, n * w1.double()) < 3e-6
            rows = torch.tensor([7, 0, 20], device=device)
            x = d(x0.clone())
            (a,) = stream.norm2(x, d(w1), 1e-3, delta, d(extra) if extra is not None else None, rows=rows, out_dtype=torch.float32)
            assert torch.equal(x.cpu(), x0) and rel(a, (n * w1.double())[[7, 0, 20]]) < 3e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [136, 90, 1300])
def test_join(width, device):
    """Several results with factors of their own: tensors, partial sums, the weighted sum of expert rows."""
    g = gen(width)
    t, k, pad = 21, 3, (-width) % 8
    x0, u, v = rnd(g, t, width, s=3.0), rnd(g, t, width + pad), rnd(g, t, width)
    y = rnd(g, 80, width + pad)
    pair = torch.randperm(80, generator=g)[: t * k].to(torch.int32)
    pair[4] = -1
    wts = torch.rand(t, k, generator=g)

    def expert_sum(rows):
        p = pair.reshape(t, k)
        return sum(wts[:, j: j + 1].double() * torch.where(p[:, j: j + 1] >= 0, rows.double()[p[:, j].clamp_min(0).long()], torch.zeros(1).double()) for j in range(k))[:, :width]

    d = lambda z: z.to(device)
    cases = [([(d(u), 0.7)], 0.7 * u.double()[:, :width]), ([(halves(u, device), -1.3), (d(v.bfloat16()), 0.5)], -1.3 * u.double()[:, :width] + 0.5 * v.bfloat16().double()),
             ([(d(v), 1.0), (halves(u, device), 0.25), (moe.PendingCombine(d(y.bfloat16()), d(pair), d(wts), t, k), 1.0)], v.double() + 0.25 * u.double()[:, :width] + expert_sum(y.bfloat16())),
             ([(moe.PendingCombine(d(y), d(pair), d(wts), t, k), 2.0)], 2.0 * expert_sum(y))]
    for parts, upd in cases:
        ref = x0.double() + upd
        for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3), (None, 0)):
            x = d(x0.clone())
            o = stream.join(x, parts, dtype)
            assert rel(x, ref) < 3e-6
            if dtype is not None:
                assert o.shape[1] == stream.row_width(width, dtype) and rel(o[:, :width], ref) < tol and not o[:, width:].any()
            else:
                assert o is None


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n", [1, 11, 64])
def test_token_gate(n, device):
    g = gen(n)
    table = rnd(g, 30, 3 * n + 2)
    ids = torch.tensor([3, 0, 29, 3, 17], dtype=torch.int32)
    z = rnd(g, 5, n + 6, s=2.0)
    for col in (0, n, 2 * n + 2):
        ref = O.gelu_tanh(z[:, :n].double()) * table.double()[ids.long(), col: col + n]
        assert rel(stream.token_gate(halves(z, device), ids.to(device), table.to(device), col, n, torch.float32), ref) < 3e-6
        got = stream.token_gate(z.to(device), ids.to(device), table.bfloat16().to(device), col, n)
        ref = O.gelu_tanh(z[:, :n].double()) * table.bfloat16().double()[ids.long(), col: col + n]
        assert got.shape[1] == stream.row_width(n, torch.bfloat16) and rel(got[:, :n], ref) < 8e-3 and not got[:, n:].any()


# ------------------------------------------------------------------------------------------ fused steps of decoding
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,dim,rank", [(2, 128, 64), (3, 24, 12), (1, 8, 1), (2, 136, 32), (4, 40, 256), (5, 9, 48)])
def test_rwkv_with_its_low_rank_decay(heads, dim, rank, device):
    """The step forms the decays itself: single tokens and short portions."""
    for lens in ([1] * 9, [1], [3, 1, 15, 2]):
        g = gen(rank + len(lens))
        t, n = sum(lens), heads * dim
        r, k, v = (rnd(g, t, n) for _ in range(3))
        w0, u, w2, z = rnd(g, n) - 2.0, rnd(g, n), rnd(g, n, rank, s=1.5 * rank ** -0.5).bfloat16(), rnd(g, t, rank, s=2.0)
        cu, slots = batch(lens, device)
        state = torch.zeros(len(lens) + 3, heads, dim, dim, device=device)
        s0 = rnd(g, len(lens), heads, dim, dim)
        state[slots.long()] = s0.to(device)
        assert recurrent.can_fuse_decay(t, max(lens), rank)
        got = recurrent.rwkv(torch.stack([r, k, v]).to(device), halves(z, device), w0.to(device), u.to(device), state, cu, slots, heads, dim, dim, t, max(lens), w2.to(device)).cpu()
        w = torch.exp(-torch.exp(torch.tanh(z.double()) @ w2.double().t() + w0.double()))
        for i, m in enumerate(lens):
            s = slice(int(cu[i]), int(cu[i]) + m)
            sh = lambda x: x[s].double().reshape(m, heads, dim)
            ref = O.time_recurrence(sh(r), sh(k), sh(v), sh(w), u.double().reshape(heads, dim))
            decay = torch.cumprod(torch.cat([torch.ones(1, heads, dim, dtype=torch.float64), sh(w)[:-1]]), 0)
            ref = ref + torch.einsum("hde,thd->the", s0[i].double(), decay * sh(r))                # what the state in front of the portion adds
            assert rel(got[s], ref.reshape(m, n)) < 1e-4
