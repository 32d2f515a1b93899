"""The mechanisms of Zedirax alone, each op against the plain reference of ``zedirax_oracle`` in float64, on the CPU references of the ops and, on a GPU
box, on the kernels.  Inputs are made so that a fault shows: single keys that stand out against a steep distance bias, gates that hold, that replace the
state at once and that sit in between, candidates on both sides of zero."""
import math

import pytest
import torch

from . import zedirax_oracle as O
from gemm_b200.models.config import RotarySpec
from gemm_b200.ops import attention as att
from gemm_b200.ops import elementwise as ew
from gemm_b200.ops import gemm, latent, moe, mxfp8, recurrent, stream

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = [torch.float32, torch.bfloat16]


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


# ------------------------------------------------------------------------------------------ minGRU
def gru_inputs(g, t, n):
    z, x = rnd(g, t, n, s=2.0) - 1.0, rnd(g, t, n, s=1.5)
    z[t // 4: t // 2] -= 9.0                             # holds
    z[t // 2: t // 2 + 3, ::3] = 30.0                    # the candidate replaces the state, on every third channel
    z[t // 2 + 5: t // 2 + 9, 1::4] = -40.0
    x[::7, ::2] = 0.0                                    # the candidate's two halves meet
    x[3::11, 1::2] = -25.0
    return z, x, rnd(g, t, n, s=2.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 24, 136, 90, 257, 1030])
def test_mingru(n, dtype, device):
    """Unequal sequences from zero; other slots stay as they are; K-split partial sums (32-bit) and 16-bit rows beside 32-bit gates."""
    for lens in ([1], [16], [17, 1, 130], [300, 5], [129, 128, 64, 2], [1300]):
        g = gen(n + sum(lens))
        t, b = sum(lens), len(lens)
        z, x, gate = gru_inputs(g, t, n)
        xb, zb = rnd(g, n), rnd(g, n, s=0.5)
        x, gate = x.to(dtype), gate.to(dtype)
        ld = 2 * n + 6 + 2 * n % 2
        rows = torch.full((t, ld + ld % 2), 9.0).to(dtype)
        rows[:, :n], rows[:, n: 2 * n] = x, gate
        zs = torch.nn.functional.pad(z, (4, 2 + n % 2))
        state = torch.randn(b + 2, 1, 1, n, generator=g)
        slots = torch.randperm(b + 2, generator=g)[:b].to(torch.int32)
        state[slots.long()] = 0
        other = [i for i in range(b + 2) if i not in slots.tolist()]
        keep = state[other].clone()
        state = state.to(device)
        for parts in ([False, True] if dtype == torch.float32 else [False]):
            st = state.clone()
            args = (halves(rows, device), halves(zs, device)) if parts else (rows.to(device), zs.to(device))
            got = recurrent.mingru(*args, 4, xb.to(device), zb.to(device), st, cum(lens, device), slots.to(device), n, max(lens), dtype).cpu()
            check_status(device)
            assert got.shape == (t, stream.row_width(n, dtype)) and not got[:, n:].any()
            at, tol = 0, 3e-6 if dtype == torch.float32 else 6e-3
            for i, m in enumerate(lens):
                s = slice(at, at + m)
                ref = O.gru_recurrence(z[s].double() + zb.double(), x[s].double() + xb.double())
                assert rel(got[s, :n], ref * O.silu(gate[s].double())) < tol, (lens, i)
                assert rel(st[int(slots[i])].reshape(-1), ref[-1]) < 2e-5, (lens, i)
                at += m
            assert torch.equal(st[other].cpu(), keep)


@pytest.mark.parametrize("device", DEVICES)
def test_mingru_portions_do_not_matter(device):
    """The scan and the step agree wherever the tokens are cut, and on what they leave behind; batches of other sequences do not matter."""
    g = gen(5)
    n, t = 200, 700
    z, x, gate = gru_inputs(g, t, n)
    rows, zs = torch.cat([x, gate], 1).bfloat16().to(device), z.to(device)
    xb, zb = rnd(g, n).to(device), rnd(g, n).to(device)

    def run(cuts, beside=0):
        state = torch.zeros(3, 1, 1, n, device=device)
        out, at = [], 0
        for m in cuts:
            r, q = rows[at: at + m], zs[at: at + m]
            lens, sl = [m], [1]
            if beside:
                r, q, lens, sl = torch.cat([rows[:beside], r]), torch.cat([zs[:beside], q]), [beside, m], [0, 1]
            y = recurrent.mingru(r.contiguous(), q.contiguous(), 0, xb, zb, state, cum(lens, device), torch.tensor(sl, dtype=torch.int32, device=device), n, max(lens))
            out.append(y[-m:])
            at += m
        return torch.cat(out), state[1].clone()

    whole, s0 = run([700])
    for cuts in ([2] * 350, [127, 2, 128, 443], [16, 17, 256, 1, 410], [1] * 700):
        for beside in (0, 40):
            if beside and len(cuts) > 10:
                continue
            got, s1 = run(cuts, beside)
            assert rel(got, whole.double().cpu()) < 8e-3 and rel(s1, s0.double().cpu()) < 1e-5
    check_status(device)


# ------------------------------------------------------------------------------------------ attention
def _attention_case(g, lens, ctx, hq, hkv, dk, dv, page, dtype):
    """Cached keys and values in shuffled pages, and queries."""
    kv = [a + b for a, b in zip(lens, ctx)]
    dkp, dvp = att.cache_head_dims(dk, dv, dtype)
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


SHAPES = [(8, 2, 128, 128, 64), (6, 3, 40, 40, 64), (5, 1, 64, 64, 16), (3, 3, 24, 100, 128), (16, 1, 128, 64, 64), (2, 1, 160, 136, 64), (2, 2, 16, 16, 24), (40, 1, 16, 72, 64)]
BATCHES = [([150, 1, 17, 2, 300], [0, 300, 128, 191, 45]), ([1, 1, 1, 1], [0, 63, 128, 900]), ([2, 2], [126, 0])]


def _loud_keys(q, k, seqs, lens, ctx, per, hq, r1, r2, which, scale):
    """Queries that ask for the key at position ``which(p)`` with a score that stands out above the bias there."""
    at = 0
    for i, n in enumerate(lens):
        for x in range(n):
            p = ctx[i] + x
            j = which(p)
            if not 0 <= j <= p:
                continue
            for h in range(0, hq, max(1, per // 2)):
                key = k[seqs[i][j], h // per]
                q[at + x, h] = key * ((7.0 + float(r1[h]) * math.log(1 + float(r2[h]) * (p - j))) / scale / float(key.pow(2).sum()))
        at += n


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,dk,dv,page", SHAPES)
def test_logarithmic_distance_bias(hq, hkv, dk, dv, page, dtype, device):
    """Slight and steep biases by head; the key that stands out is the first one, one at a page or block border, or the query's own; prompts on top of a context,
    short portions, single tokens, split key ranges."""
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    r1, r2 = torch.linspace(0.0, 3.0, hq), torch.linspace(2.0, 0.01, hq)
    if hq > 2:
        r1[1], r2[2] = -0.3, 0.0                         # grows with the distance; none at all
    scale, per = 0.7, hq // hkv
    for bi, (lens, ctx) in enumerate(BATCHES):
        for which in (lambda p: 0, lambda p: (p // 64) * 64 - 1, lambda p: (p * 37) % (p + 1), lambda p: p):
            g = gen(hq * 100 + dk + bi)
            kv, bt, k, v, seqs, q = _attention_case(g, lens, ctx, hq, hkv, dk, dv, page, dtype)
            _loud_keys(q, k, seqs, lens, ctx, per, hq, r1, r2, which, scale)
            q, k, v = q.to(dtype).float(), k.to(dtype), v.to(dtype)
            qs = (q * scale * att.LOG2E).to(dtype)
            refs, at = [], 0
            for i, n in enumerate(lens):
                full = torch.zeros(kv[i], hq, dk, dtype=torch.float64)
                full[-n:] = qs[at: at + n, :, :dk].double() / att.LOG2E
                refs.append(O.attend(full, k[seqs[i]][..., :dk].double(), v[seqs[i]][..., :dv].double(), 1.0, r1.double(), r2.double())[-n:])
                at += n
            ref = torch.cat(refs)
            decode = all(n == 1 for n in lens)
            for sp in ([1, 3] if decode and device == "cuda" and dtype == torch.bfloat16 else [1]):
                plan = (att.build_work(lens, hq, hkv, sp).to(device), sp) if device == "cuda" else None
                got = att.attention_masked(qs.to(device), k.to(device), v.to(device), cum(lens, device), torch.tensor(kv, dtype=torch.int32, device=device), bt.to(device), page, plan=plan,
                                           decode=decode, log_bias=torch.stack([r1, r2]).to(device)).float().cpu()[..., :dv]
                assert rel(got, ref) < tol, (bi, sp)
    check_status(device)


def test_a_wrong_distance_shows():
    """The case above tells a distance that is one off, and a logarithm of another base, from the right one."""
    g = gen(1)
    q, k, v = rnd(g, 60, 2, 16).double(), rnd(g, 60, 1, 16).double(), rnd(g, 60, 1, 16).double()
    r1, r2 = torch.tensor([2.0, 0.7]).double(), torch.tensor([0.5, 2.0]).double()
    ref = O.attend(q, k, v, 0.3, r1, r2)
    assert rel(O.attend(q, k, v, 0.3, r1 * math.log(2), r2), ref) > 0.1 and rel(O.attend(q, k, v, 0.3, r1, r2 * 1.5), ref) > 0.02


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,dk,dv,every", [(4, 2, 40, 24, 7), (3, 1, 160, 9, 64), (8, 8, 128, 128, 1), (2, 1, 10, 13, 2.5)])
def test_query_temperature(hq, hkv, dk, dv, every, dtype, device):
    """Positions around every step of the temperature, and far away; keys and values stay as they are."""
    g = gen(hq + dk)
    nq, nk, nv = hq * dk, hkv * dk, hkv * dv
    pos = torch.tensor(list(range(20)) + [62, 63, 64, 126, 127, 128, 99999, 1048575], dtype=torch.int32)
    t = pos.numel()
    x = rnd(g, t, nq + nk + nv, s=2.0).to(dtype)
    dkp, dvp = att.cache_head_dims(dk, dv, dtype)
    kc, vc = torch.zeros(t, hkv, dkp, dtype=dtype, device=device), torch.zeros(t, hkv, dvp, dtype=dtype, device=device)
    slots = torch.randperm(t, generator=g).to(torch.int32)
    src = halves(x, device) if dtype == torch.float32 else x.to(device)
    q = stream.qk_unit(src, slots.to(device), kc, vc, hq, hkv, dk, dv, 1e-5, 0.37, unit=False, positions=pos.to(device), temp=(0.4, float(every))).cpu()
    f = torch.tensor([1 + 0.4 * math.log((p + 1) // every + 1) for p in pos.tolist()], dtype=torch.float64)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    ref = x[:, :nq].double().reshape(t, hq, dk) * f.reshape(-1, 1, 1) * 0.37
    assert ((q[..., :dk].double() - ref).abs() <= tol * ref.abs() + 1e-9).all() and not q[..., dk:].any()
    assert torch.equal(kc.cpu()[slots.long(), :, :dk], x[:, nq: nq + nk].reshape(t, hkv, dk).to(dtype)) or dtype == torch.float32
    assert rel(kc[slots.long().to(device), :, :dk], x[:, nq: nq + nk].double().reshape(t, hkv, dk)) < tol
    assert rel(vc[slots.long().to(device), :, :dv], x[:, nq + nk:].double().reshape(t, hkv, dv)) < tol
    assert [O.temperature(200, 0.4, every)[p].item() for p in (0, 62, 63, 64)] == pytest.approx([1 + 0.4 * math.log((p + 1) // every + 1) for p in (0, 62, 63, 64)])


def test_pairs_of_halves_as_neighbours():
    """Rows of a projection in ``pair_order`` turn as neighbours by what the halves turn: the rotated vector is the same up to that order."""
    for n in (2, 8, 64):
        spec = RotarySpec(n, 300.0, halves=True)
        order = spec.pair_order()
        assert sorted(order) == list(range(n)) and RotarySpec(n, 300.0).pair_order() == list(range(n))
        x = torch.randn(50, 3, n, dtype=torch.float64)
        freq = torch.tensor(spec.frequencies(), dtype=torch.float64)
        got = latent.rotate_ref(x[..., order].float(), torch.arange(50), freq, 1.0)
        assert rel(got, O.rotate_halves(x, 300.0)[..., order]) < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_latents_without_a_query_latent(dtype, device):
    """Latent and rotated key part from columns behind the queries; nothing else is written."""
    g = gen(9)
    t, r, rd, col = 40, 72, 8, 24
    rows = rnd(g, t, col + r + rd + 16).to(dtype)
    spec, kn = RotarySpec(rd, 500.0), rnd(g, r)
    freq = torch.tensor(spec.frequencies(), dtype=torch.float64, device=device)
    pos, slots = torch.arange(t, dtype=torch.int32), torch.randperm(t + 5, generator=g)[:t].to(torch.int32)
    cache = torch.full((t + 5, 1, stream.row_width(r + rd, dtype)), 7.0, dtype=dtype, device=device)
    src = halves(rows, device) if dtype == torch.float32 else rows.to(device)
    assert latent.latent_store(src, pos.to(device), slots.to(device), None, kn.to(device), freq, 1.0, cache, 0, r, rd, 1e-4, dtype, col) is None
    x = rows.double()[:, col:]
    order = RotarySpec(rd, 500.0, halves=True).pair_order()
    back = torch.argsort(torch.tensor(order))
    ref = torch.cat([O.unit(x[:, :r], 1e-4) * kn.double(), O.rotate_halves(x[:, r: r + rd][:, back], 500.0)[:, order]], -1)
    assert rel(cache.cpu()[slots.long(), 0, : r + rd], ref) < (3e-6 if dtype == torch.float32 else 8e-3)
    rest = [i for i in range(t + 5) if i not in slots.tolist()]
    assert bool((cache.cpu()[rest] == 7).all())


# ------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("device", DEVICES)
def test_biased_gelu_pair(device):
    """Biases of both products in front of the activation: the 32-bit form, the GEMM's epilogue, the one over K-split partial sums."""
    g = gen(21)
    inter, k = 128, 72
    b = rnd(g, 2 * inter, s=1.5)
    act = lambda y: O.gelu_tanh(y[:, :inter]) * y[:, inter:]
    for t in (1, 9, 40, 300):
        x, w = rnd(g, t, k).bfloat16(), rnd(g, 2 * inter, k, s=1.5 * k ** -0.5).bfloat16()
        y = x.double() @ w.double().t() + b.double()
        for tiled in ((False, True) if device == "cuda" else (False,)):
            wd = mxfp8.tile_weight(torch.nn.functional.pad(w, (0, 56))).to(device) if tiled else w.to(device)
            xd = torch.nn.functional.pad(x, (0, 56)).to(device) if tiled else x.to(device)
            assert rel(gemm.linear_swiglu(xd, wd, act="gelu_tanh", bias=b.to(device), w_tiled=tiled), act(y)) < 8e-3
        part = halves((x.float() @ w.float().t()), device)
        assert rel(ew.silu_mul_partials(part, act="gelu_tanh", bias=b.to(device)), act(y)) < 8e-3
        f = stream.act_mul(gemm.linear_f32(x.float().to(device), w.float().to(device), b.to(device)), "gelu_tanh")
        assert rel(f, act(y)) < 2e-6
    check_status(device)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("t", [1, 20, 60, 200, 700])
def test_exact_gelu_in_the_epilogue(t, device):
    """Of one product and of grouped ones, feature counts off and on the tiles; far from the form with a tanh where the two differ most."""
    g = gen(t)
    for n, k in ((72, 136), (256, 64)):
        x, w = rnd(g, t, k, s=2.0).bfloat16(), rnd(g, n, k, s=k ** -0.5).bfloat16()
        y = x.double() @ w.double().t()
        assert rel(gemm.linear(x.to(device), w.to(device), gelu=True), O.gelu_erf(y)) < 5e-3
        assert rel(stream.gelu_rows(y.float().to(device)), O.gelu_erf(y.float().double())) < 1e-6
        groups, tn = 3, gemm.pick_tn(t, dual=True)
        pad = (t + tn - 1) // tn * tn
        xs = torch.zeros(groups * pad, k).bfloat16()
        ws = rnd(g, groups, 256, k, s=k ** -0.5).bfloat16()
        cnt = [t, 0, max(1, t // 2)]
        for i in range(groups):
            xs[i * pad: i * pad + cnt[i]] = rnd(g, cnt[i], k).bfloat16()
        seg = torch.arange(groups, dtype=torch.int32, device=device) * pad
        got = gemm.grouped_linear(xs.to(device), ws.to(device), seg, torch.tensor(cnt, dtype=torch.int32, device=device), tn, gelu=True).cpu()
        for i in range(groups):
            if cnt[i]:
                s = slice(i * pad, i * pad + cnt[i])
                assert rel(got[s], O.gelu_erf(xs[s].double() @ ws[i].double().t())) < 5e-3
    z = torch.linspace(-4, 4, 4001, dtype=torch.float64)
    assert (O.gelu_erf(z) - O.gelu_tanh(z)).abs().max() > 4e-4 and (stream.gelu_rows(z.float().to(device)).cpu().double() - O.gelu_erf(z.float().double())).abs().max() < 3e-6
    check_status(device)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("e,top", [(10, 3), (16, 1), (5, 5), (128, 8), (1, 1)])
def test_softmax_over_the_chosen(e, top, device):
    """Large logits, too: the weights are relative to the best one."""
    g = gen(e)
    for s in (1.0, 40.0):
        z = rnd(g, 77, e, s=s)
        ids, w = moe.route(z.to(device), top, "softmax", renorm=1)
        ref_i, ref_w = O.route(z.double(), top)
        full = lambda i, v: torch.zeros(77, e, dtype=torch.float64).scatter_add(1, i.cpu().long(), v.cpu().double())
        assert (full(ids, w) - full(ref_i, ref_w)).abs().max() < 2e-6
        assert s > 1 or torch.equal(ids.cpu().long(), ref_i)                 # (weights of far smaller logits vanish, and so does their order)


# ------------------------------------------------------------------------------------------ stream
def expert_sum(g, t, k, w, dtype, device):
    """Pending expert outputs, some of the pairs dropped, and their sum."""
    y = rnd(g, t * k + 3, w).to(dtype)
    rows = torch.randperm(t * k + 3, generator=g)[: t * k].to(torch.int32)
    rows[1::9] = -1
    wts = torch.rand(t, k, generator=g)
    ref = (y.double()[rows.long().clamp_min(0)] * (rows >= 0).unsqueeze(1)).reshape(t, k, w) * wts.double().unsqueeze(-1)
    return moe.PendingCombine(y.to(device), rows.to(device), wts.to(device), t, k), ref.sum(1)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [8, 136, 90, 33, 1030, 2048, 5000])
def test_norm_with_a_factor_and_a_gate(width, device):
    """The update's factor; one number per token from the normalised row; the same through a sum of several results."""
    g = gen(width)
    t = 11
    x0, w, sg = rnd(g, t, width, s=2.0), 1 + rnd(g, width, s=0.3), rnd(g, width, s=width ** -0.5)
    u = rnd(g, t, width + 3 + width % 2)
    dot = (sg * w).to(device)
    shared, ref_pend = rnd(g, t, width).bfloat16(), None
    pend, ref_pend = expert_sum(g, t, 3, width, torch.bfloat16, device)
    row = torch.rand(t, generator=g)
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        for parts, ref_u in (([(halves(u, device), 0.7, None)], 0.7 * u[:, :width].double()),
                             ([(pend, 0.4, None), (shared.to(device), 0.4, row.to(device))], 0.4 * ref_pend + 0.4 * row.double().unsqueeze(1) * shared.double())):
            x = x0.clone().to(device)
            h, gate = stream.norm_gate(x, w.to(device), 1e-4, stream.Update(parts), dot, dtype)
            y = x0.double() + ref_u
            n = O.unit(y, 1e-4) * w.double()
            assert rel(x, y) < 1e-6 and rel(h[:, :width], n) < tol and not h[:, width:].any()
            assert rel(gate, O.sigmoid((n * sg.double()).sum(-1))) < 3e-6
    check_status(device)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [8, 136, 90, 33, 1030, 2048, 5000])
def test_average_over_earlier_places(width, device):
    """Every place in turn, with sums of several results in front of it: what is kept, what goes on, the normed rows (all, or some without touching anything), and
    the sums over the places so far that are formed ahead."""
    g = gen(width + 1)
    t, places = 7, 2 * stream.DEPTH_BLOCK + 3
    w = 1 + rnd(g, width, s=0.3)
    first = rnd(g, t, width)
    hist = torch.full((places, t, width), float("nan"), device=device)
    hist[0] = first
    ref = [first.double()]
    x, cur = first.clone().to(device), first.double()
    coef = [rnd(g, i + 2, s=0.4) for i in range(places)]
    base, at0 = None, 0
    rows = torch.tensor([5, 0, 5])
    for at in range(1, places):
        c = coef[at - 1]
        if at > 1 and (at - 1) % stream.DEPTH_BLOCK == 0:
            base, at0 = stream.depth_base(hist, at, [q.to(device) for q in coef[at - 1: at - 1 + stream.DEPTH_BLOCK]]), at
        y, pend = rnd(g, t, width).bfloat16(), expert_sum(g, t, 2, width, torch.bfloat16, device)
        row = torch.rand(t, generator=g)
        parts = [(halves(rnd(g, t, width), device), 0.5, None)] if at % 3 == 0 else [(pend[0], 0.5, None), (y.to(device), 0.5, row.to(device))]
        add = 0.5 * parts[0][0].buf.double().cpu().sum(0) if at % 3 == 0 else 0.5 * pend[1] + 0.5 * row.double().unsqueeze(1) * y.double()
        upd = stream.Update(parts, stream.Depth(hist, at, c.to(device), base[at - at0] if base is not None else None, at0))
        ref.append(cur + add)
        cur = O.depth_average(ref, c.double())
        n = O.unit(cur, 1e-4) * w.double()
        before = x.clone()
        got = stream.norm(x, w.to(device), 1e-4, upd, rows=rows.to(device), out_dtype=torch.float32)
        assert rel(got, n[rows]) < 1e-5 and torch.equal(x, before) and bool(torch.isnan(hist[at]).all())
        assert rel(stream.settled(x, upd), cur) < 3e-6
        dtype = torch.float32 if at % 2 else torch.bfloat16
        got = stream.norm(x, w.to(device), 1e-4, upd, out_dtype=dtype)
        assert rel(got[:, :width], n) < (1e-5 if at % 2 else 8e-3) and not got[:, width:].any()
        assert rel(x, cur) < 3e-6 and rel(hist[at], ref[-1]) < 3e-6
        cur, ref[-1] = x.double().cpu(), hist[at].double().cpu()
    check_status(device)
