"""The mechanisms of models described layer by layer, each alone, against ``layerspec_oracle`` (float64).  On a GPU box the kernels run (the
tcgen05 forms and the any-size forms), else their CPU references.

Where random data would hide a fault (a key just outside a window among hundreds, one bias bucket), one query and key are made to
stand out, so that seeing the key or not changes the whole output."""
import math

import pytest
import torch

from gemm_b200.ops import attention as att
from gemm_b200.ops import gemm, lightning, stream
from gemm_b200.ops.elementwise import silu_mul_partials

from . import layerspec_oracle as O

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = [torch.float32, torch.bfloat16]


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def status_ok(device):
    if device == "cuda":
        from gemm_b200 import _native
        _native.assert_status_ok()


# ------------------------------------------------------------------------------------------ attention
class Cache:
    """A paged cache filled with the keys and values of some sequences, pages in shuffled order, stale values everywhere else."""

    def __init__(self, ks, vs, dtype, device, page, seed=0):
        g = torch.Generator().manual_seed(seed)
        hkv, dk, dv = ks[0].shape[1], ks[0].shape[2], vs[0].shape[2]
        dkp, dvp = att.cache_head_dims(dk, dv, dtype)
        per = [(k.shape[0] + page - 1) // page for k in ks]
        order = torch.randperm(sum(per) + 2, generator=g).tolist()
        n = len(order) * page
        self.k = torch.randn(n, hkv, dkp, generator=g) * 3
        self.v = torch.randn(n, hkv, dvp, generator=g) * 30
        self.bt = torch.zeros(len(ks), max(per), dtype=torch.int32)
        for s, (k, v) in enumerate(zip(ks, vs)):
            for p in range(per[s]):
                pg = self.bt[s, p] = order.pop()
                kk, vv = k[p * page: (p + 1) * page], v[p * page: (p + 1) * page]
                rows = slice(int(pg) * page, int(pg) * page + kk.shape[0])
                self.k[rows], self.v[rows] = 0, 0
                self.k[rows, :, :dk], self.v[rows, :, :dv] = kk.float(), vv.float()
        self.k, self.v, self.bt = self.k.to(dtype).to(device), self.v.to(dtype).to(device), self.bt.to(device)
        self.dkp, self.dvp, self.page, self.dtype, self.device = dkp, dvp, page, dtype, device


def run_attention(cache, qs, kv_lens, scale, rel_table, bias_max, window, keep, decode=False, splits=1, kernel="flash"):
    """qs: per sequence the queries [n, Hq, dk] of its last n positions.  Returns per sequence [n, Hq, dv]."""
    hq, dk = qs[0].shape[1], qs[0].shape[2]
    hkv = cache.k.shape[1]
    q = torch.nn.functional.pad(torch.cat(qs).float() * scale * att.LOG2E, (0, cache.dkp - dk)).to(cache.dtype).to(cache.device)
    lens = [x.shape[0] for x in qs]
    cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32, device=cache.device)
    kvl = torch.tensor(kv_lens, dtype=torch.int32, device=cache.device)
    bias = att.distance_bias_table(rel_table.float(), bias_max).to(cache.device) if rel_table is not None else None
    plan = (att.build_work(lens, hq, hkv, splits).to(cache.device), splits) if kernel == "flash" else None
    out = att.attention_masked(q, cache.k, cache.v, cu, kvl, cache.bt, cache.page, window, keep, bias, plan, decode)
    status_ok(cache.device)
    return torch.split(out.float().cpu(), lens)


def bf(x):
    return x.bfloat16().double()


ATT = [  # hq, hkv, dk, dv, window, keep, rel rows, bias_max
    (8, 2, 128, 128, 100, 30, 32, 140),
    (4, 4, 32, 64, 129, 1, 8, 500),
    (6, 3, 80, 88, 64, 64, 32, 64.5),
    (3, 1, 64, 128, 0, 0, 16, 200),
    (5, 5, 40, 24, 1, 0, 2, 40),
    (14, 2, 128, 64, 128, 129, 0, 0),
    (32, 1, 16, 16, 17, 200, 33, 90),
]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kernel,dtype", [("flash", torch.bfloat16), ("any", torch.bfloat16), ("any", torch.float32)])
@pytest.mark.parametrize("case", range(len(ATT)))
def test_attention(case, kernel, dtype, device):
    """Prompts, later portions, single decoded tokens and split decoding of unequal sequences."""
    hq, hkv, dk, dv, window, keep, rows, bmax = ATT[case]
    torch.manual_seed(case)
    n = [333, 129, 40, 1]
    scale = 0.7 * dk ** -0.5
    ks, vs = [bf(torch.randn(x, hkv, dk)) for x in n], [bf(torch.randn(x, hkv, dv)) for x in n]
    qs = [torch.randn(x, hq, dk).double() for x in n]
    table = bf(torch.randn(rows, hq) * 2) if rows else None
    ref = [O.attention_core(q, k, v, scale, table, bmax, window or None, keep) for q, k, v in zip(qs, ks, vs)]
    c = Cache(ks, vs, dtype, device, 64, case)
    tol = 1e-5 if dtype == torch.float32 else 1.5e-2

    def check(take, **kw):
        got = run_attention(c, [q[-t:] for q, t in zip(qs, take)], n, scale, table, bmax, window, keep, kernel=kernel, **kw)
        for g, r, t in zip(got, ref, take):
            assert rel(g[:, :, :dv], r[-t:]) < tol
            assert not g[:, :, dv:].any()

    check([333, 129, 40, 1])
    check([70, 2, 1, 1])
    if kernel == "flash" and hq // hkv <= 16:
        check([1, 1, 1, 1], decode=True)
        check([1, 1, 1, 1], decode=True, splits=3)
    else:
        check([1, 1, 1, 1])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kernel,dtype", [("flash", torch.bfloat16), ("any", torch.float32)])
@pytest.mark.parametrize("window,keep", [(44, 12), (128, 1), (64, 64), (129, 0), (200, 130), (1, 1), (65, 0)])
def test_window_edges(window, keep, kernel, dtype, device):
    """One key answers one query so loudly that the output says whether it is seen: distances just inside and just outside the window, the last
    kept token and the next one, page and block borders, in prompts and in decoding."""
    dk, dv, hq, hkv, n = 64, 64, 2, 1, 420
    far = n - 1 - window
    places = {n - 1, n - window, far, far + 1, keep - 1, keep, 0, 1, 63, 64, 127, 128, 129, n - 64, n - 65, n - 128, n - 129, 255, 256}
    torch.manual_seed(1)
    k0 = torch.randn(n, hkv, dk)
    k0[:, :, 0] = 0
    for j in sorted(p for p in places if 0 <= p < n):
        k = k0.clone()
        k[j] = 0
        k[j, :, 0] = 8.0
        v = torch.zeros(n, hkv, dv)
        v[j] = 1.0
        q = torch.zeros(n, hq, dk)
        q[:, :, 0] = 4.0
        c = Cache([bf(k)], [bf(v)], dtype, device, 64)
        rows = sorted(i for i in {j, j + window - 1, j + window, n - 1, n - 2} if j <= i < n)
        whole = run_attention(c, [q], [n], 1.0, None, 0, window, keep, kernel=kernel)[0]
        dec = {i: run_attention(c, [q[i: i + 1]], [i + 1], 1.0, None, 0, window, keep, decode=True, kernel=kernel)[0][0] for i in rows}
        for i in rows:
            seen = 1.0 if O.visible(i, j, window, keep) else 0.0
            for got in (whole[i], dec[i]):
                assert (got[:, :dv] - seen).abs().max() < 2e-2, (i, j)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kernel,dtype", [("flash", torch.bfloat16), ("any", torch.float32)])
def test_every_distance_has_its_bucket(kernel, dtype, device):
    """Keys of score 0 and values that tell the distance apart: with a bias of log(weight) per bucket the output is a known mixture; a bucket border one
    token off shifts it."""
    n, rows, bmax, hq = 300, 16, 150, 4
    v = torch.zeros(n, 1, 64)
    border = [d for d in range(1, n) if O.distance_bucket(d, rows, bmax) != O.distance_bucket(d - 1, rows, bmax)]
    assert len(border) == rows - 1 and max(border) < 150
    table = torch.full((rows, hq), -30.0).double()
    for h in range(hq):
        for b in range(rows):
            if (b + h) % 2:
                table[b, h] = 0.0
    c_k = torch.zeros(n, 1, 64)
    for x in range(64):
        for d in border[x % len(border):: 5]:
            v[n - 1 - d, 0, x] = 1.0
            v[n - d, 0, x] = -1.0
    q = torch.zeros(n, hq, 64)
    ref = O.attention_core(q.double(), c_k.double(), bf(v), 1.0, table, bmax, None, 0)
    c = Cache([c_k], [bf(v)], dtype, device, 64)
    got = run_attention(c, [q], [n], 1.0, table, bmax, 0, 0, kernel=kernel)[0]
    one = run_attention(c, [q[-1:]], [n], 1.0, table, bmax, 0, 0, decode=True, kernel=kernel)[0]
    assert rel(got, ref) < 1e-2 and rel(one, ref[-1:]) < 1e-2


@pytest.mark.parametrize("buckets,dmax", [(32, 150), (32, 4096), (2, 40), (8, 64), (33, 90), (16, 16.5), (64, 32 * 2 ** 5), (6, 3 * 3 ** 3)])
def test_distance_buckets(buckets, dmax):
    prev = 0
    for n in range(0, 5000, 1 if dmax < 1000 else 7):
        b = att.distance_bucket(n, buckets, dmax)
        assert b == O.distance_bucket(n, buckets, dmax) and prev <= b <= buckets - 1
        prev = b
    # a power hits its bucket's first distance exactly
    half = buckets // 2
    if buckets == 64:
        assert [att.distance_bucket(half * 2 ** e, buckets, half * 2 ** 4) for e in range(5)] == [32, 40, 48, 56, 63]
    if buckets == 6:
        assert [att.distance_bucket(d, 6, 81) for d in (8, 9, 26, 27, 80, 81)] == [3, 4, 4, 5, 5, 5]
    t = att.distance_bias_table(torch.randn(buckets, 3), dmax)
    n = t.shape[1] // 2
    for d in (0, 1, n // 2, n - 1):
        assert torch.equal(t[:, n + d], t[:, d: min(n, d + 128)].max(dim=1).values)


# ------------------------------------------------------------------------------------------ lightning attention
LIGHT = [(3, 24, 40), (2, 64, 64), (2, 128, 128), (1, 80, 72), (2, 8, 8), (4, 130, 20), (2, 7, 9), (1, 256, 256)]


def lightning_inputs(heads, dim, vdim, lens, seed):
    g = torch.Generator().manual_seed(seed)
    t = sum(lens)
    raw = torch.randn(t, 2 * heads * dim + 2 * heads * vdim, generator=g).bfloat16()
    state = torch.randn(5, heads, dim, vdim, generator=g)
    decay = (torch.rand(heads, generator=g) * 0.9 + 0.1)
    decay[0] = 0.9995
    return raw, state, decay


def lightning_want(raw, state, decay, lens, slots, heads, dim, vdim, activated=False):
    y = raw.double()[:, : 2 * heads * dim + heads * vdim]
    y = y if activated else O.silu(y)
    out, st, at = [], state.double().clone(), 0
    for n, s in zip(lens, slots):
        r = y[at: at + n]
        q, k = r[:, : heads * dim].reshape(n, heads, dim), r[:, heads * dim: 2 * heads * dim].reshape(n, heads, dim)
        o, st[s] = O.lightning_recurrence(q, k, r[:, 2 * heads * dim:].reshape(n, heads, vdim), decay.double(), st[s])
        out.append(o.reshape(n, -1))
        at += n
    return torch.cat(out), st


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("sizes", LIGHT)
def test_lightning_step(sizes, device):
    """Pre-activation rows in bf16, f32 and as K-split partial sums; slots in any order; a slot nobody uses keeps its state."""
    heads, dim, vdim = sizes
    lens, slots = [1, 13, 1, 6], [3, 0, 4, 2]
    raw, state, decay = lightning_inputs(heads, dim, vdim, lens, 1)
    cu = torch.tensor([0, 1, 14, 15, 21], dtype=torch.int32, device=device)
    sl = torch.tensor(slots, dtype=torch.int32, device=device)
    want, wst = lightning_want(raw, state, decay, lens, slots, heads, dim, vdim)
    a = torch.randn(raw.shape, generator=torch.Generator().manual_seed(5))
    pend = gemm.PendingPartials(torch.stack([a, raw.float() - a]).to(device))
    for proj in (raw.to(device), raw.float().to(device), pend):
        st = state.clone().to(device)
        got = lightning.lightning(proj, decay.to(device), st, cu, sl, heads, dim, vdim)
        assert rel(got, want) < 2e-5 and rel(st, wst) < 2e-5
        assert torch.equal(st[1].cpu(), state[1])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("sizes", LIGHT)
def test_lightning_prompt(sizes, device):
    """Activated rows of a prefill: chunk borders at every place, lengths around a chunk, a long decay and short ones, state carried on."""
    heads, dim, vdim = sizes
    lens, slots = [300, 1, 128, 129, 2], [1, 0, 4, 2, 3]
    raw, state, decay = lightning_inputs(heads, dim, vdim, lens, 2)
    rows = torch.nn.functional.silu(raw.float()).bfloat16()
    want, wst = lightning_want(rows, state, decay, lens, slots, heads, dim, vdim, activated=True)
    st = state.clone().to(device)
    cu = torch.tensor([0, 300, 301, 429, 558, 560], dtype=torch.int32, device=device)
    sl = torch.tensor(slots, dtype=torch.int32, device=device)
    got = lightning.lightning(rows.to(device), decay.to(device), st, cu, sl, heads, dim, vdim, activated=True, max_tokens=300)
    status_ok(device)
    assert rel(got, want) < 5e-5 and rel(st, wst) < 5e-5
    # the same prompt in two launches
    st = state.clone().to(device)
    outs = []
    for lo, hi in ((0, 101), (101, 300)):
        outs.append(lightning.lightning(rows[lo:hi].to(device), decay.to(device), st, torch.tensor([0, hi - lo], dtype=torch.int32, device=device), sl[:1],
                                        heads, dim, vdim, activated=True, max_tokens=hi - lo))
    assert rel(torch.cat(outs), want[:300]) < 5e-5 and rel(st[1], wst[1]) < 5e-5


@pytest.mark.parametrize("device", DEVICES)
def test_lightning_remembers_the_first_token(device):
    """With a decay near one a token hundreds of positions back still decides the output; with a small one it is gone."""
    heads, dim, vdim, n = 2, 64, 64, 700
    rows = torch.zeros(n, 2 * heads * dim + heads * vdim)
    rows[0, heads * dim: 2 * heads * dim] = 1.0           # k of the first token
    rows[0, 2 * heads * dim:] = 1.0                        # its v
    rows[-1, : heads * dim] = 1.0                          # q of the last token
    decay = torch.tensor([0.999, 0.5])
    st = torch.zeros(1, heads, dim, vdim, device=device)
    one = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    o = lightning.lightning(rows.bfloat16().to(device), decay.to(device), st, one([0, n]), one([0]), heads, dim, vdim, activated=True, max_tokens=n).cpu()
    assert (o[-1, :vdim] / (dim * 0.999 ** (n - 1)) - 1).abs().max() < 1e-3
    assert o[-1, vdim:].abs().max() < 1e-30 and not o[1:-1].any()


# ------------------------------------------------------------------------------------------ norms, activations, products
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width", [64, 90, 1028, 4096, 5000, 16384, 20000])
def test_stream_norm(width, device):
    g = torch.Generator().manual_seed(width)
    x, w, add = torch.randn(5, width, generator=g), torch.randn(width, generator=g), torch.randn(width, generator=g)
    d = torch.randn(3, 5, width, generator=g)
    eps = 0.3
    for delta, total in ((None, 0), (d[0].bfloat16(), d[0].bfloat16()), (d[0], d[0]), (gemm.PendingPartials(d.to(device)), d.sum(0))):
        delta = delta.to(device) if isinstance(delta, torch.Tensor) else delta
        for out_dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 4e-3)):
            want_x = x.double() + (total.double() if torch.is_tensor(total) else 0) + add.double()
            xx = x.clone().to(device)
            got = stream.norm(xx, (1 + w).to(device), eps, delta, add=add.to(device), out_dtype=out_dtype)
            assert rel(xx, want_x) < 1e-6 and rel(got[:, :width], O.norm_zero_centred(want_x, w.double(), eps)) < tol
            assert not got[:, width:].any() and got.shape[1] == stream.row_width(width, out_dtype)
            xx = x.clone().to(device)
            rows = torch.tensor([4, 1, 1], device=device)
            got = stream.norm(xx, (1 + w).to(device), eps, delta, rows=rows, out_dtype=out_dtype)
            assert torch.equal(xx.cpu(), x)
            assert rel(got[:, :width], O.norm_zero_centred((want_x - add.double())[[4, 1, 1]], w.double(), eps)) < tol


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,dk,dv,unit", [(4, 2, 40, 56, True), (3, 3, 130, 20, True), (6, 1, 128, 64, True), (2, 1, 1, 3, True), (4, 4, 64, 200, False)])
def test_qk_unit_norm_and_cache_store(hq, hkv, dk, dv, unit, dtype, device):
    g = torch.Generator().manual_seed(hq)
    n, eps, scale = 6, 0.2, 0.37
    y = torch.randn(n, (hq + hkv) * dk + hkv * dv, generator=g)
    slots = torch.tensor([7, 0, 3, -1, 11, 5], dtype=torch.int32)
    dkp, dvp = att.cache_head_dims(dk, dv, dtype)
    ins = [y.to(device)] + ([y.bfloat16().to(device)] if dtype == torch.bfloat16 else [])
    a = torch.randn(y.shape, generator=g)
    ins.append(gemm.PendingPartials(torch.stack([y - a, a]).to(device)))
    for x in ins:
        kc, vc = torch.full((12, hkv, dkp), 9.0, dtype=dtype, device=device), torch.full((12, hkv, dvp), 9.0, dtype=dtype, device=device)
        q = stream.qk_unit(x, slots.to(device), kc, vc, hq, hkv, dk, dv, eps, scale, unit=unit)
        r = y.bfloat16().double() if isinstance(x, torch.Tensor) and x.dtype == torch.bfloat16 else y.double()
        wq, wk = r[:, : hq * dk].reshape(n, hq, dk), r[:, hq * dk: (hq + hkv) * dk].reshape(n, hkv, dk)
        if unit:
            wq, wk = O.rms(wq, eps), O.rms(wk, eps)
        wv = r[:, (hq + hkv) * dk:].reshape(n, hkv, dv)
        tol = 2e-6 if dtype == torch.float32 else 4e-3
        assert rel(q[:, :, :dk], wq * scale) < tol and not q[:, :, dk:].any()
        ok = [i for i in range(n) if slots[i] >= 0]
        at = slots[ok].long().to(device)
        assert rel(kc[at][:, :, :dk], wk[ok]) < tol and rel(vc[at][:, :, :dv], wv[ok]) < tol
        assert not kc[at][:, :, dk:].any() and not vc[at][:, :, dv:].any()
        rest = [i for i in range(12) if i not in slots.tolist()]
        assert bool((kc[rest] == 9).all()) and bool((vc[rest] == 9).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n", [72, 120, 2050, 4096, 6000])
def test_gated_norm(n, device):
    g = torch.Generator().manual_seed(n)
    o, proj, w, eps = torch.randn(4, n, generator=g), torch.randn(4, 30 + 2 * n, generator=g) * 3, torch.randn(n, generator=g), 0.1
    col = 24
    for p in (proj.to(device), proj.bfloat16().to(device), gemm.PendingPartials(torch.stack([proj / 2, proj / 2]).to(device))):
        r = proj.bfloat16().double() if isinstance(p, torch.Tensor) and p.dtype == torch.bfloat16 else proj.double()
        want = O.rms(o.double(), eps) * w.double() / (1 + torch.exp(-r[:, col: col + n]))
        for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 4e-3)):
            got = stream.gated_norm(o.to(device), p, col, w.to(device), eps, dt)
            assert rel(got[:, :n], want) < tol and not got[:, n:].any()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("m", [1, 7, 64, 130, 300])
def test_gelu_feed_forward(m, device):
    """The gated feed-forward's forms: epilogue of the gate / up GEMM, K-split partial sums, and 32-bit."""
    g = torch.Generator().manual_seed(m)
    k, inter = 192, 256
    x, w = (torch.randn(m, k, generator=g) * 1.5).bfloat16(), (torch.randn(2 * inter, k, generator=g) * k ** -0.5 * 2).bfloat16()
    y = x.double() @ w.double().t()
    want = O.gelu_tanh(y[:, :inter]) * y[:, inter:]
    assert rel(gemm.linear_swiglu(x.to(device), w.to(device), act="gelu_tanh"), want) < 4e-3
    y32 = gemm.linear_f32(x.float().to(device), w.float().to(device))
    assert rel(y32, y) < 1e-6 and rel(stream.act_mul(y32, "gelu_tanh"), want) < 2e-6
    assert rel(stream.act_mul(y32, "silu"), O.silu(y[:, :inter]) * y[:, inter:]) < 2e-6
    if m <= 64:
        a = torch.randn(m, 2 * inter, generator=g)
        pend = gemm.PendingPartials(torch.stack([a, y.float() - a]).to(device))
        assert rel(silu_mul_partials(pend, act="gelu_tanh"), want) < 4e-3
    extreme = torch.tensor([[-1e4, -30.0, 0.0, 30.0, 1e4, 1.0, 1.0, 1.0, 1.0, 1.0]], device=device)
    assert stream.act_mul(extreme, "gelu_tanh").tolist() == [[0.0, 0.0, 0.0, 30.0, 1e4]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("m,n,k", [(1, 1, 1), (3, 65, 17), (64, 64, 64), (130, 100, 90)])
def test_linear_f32(m, n, k, device):
    g = torch.Generator().manual_seed(m)
    x, w, b = torch.randn(m, k, generator=g), torch.randn(n, k, generator=g), torch.randn(n, generator=g)
    assert rel(gemm.linear_f32(x.to(device), w.to(device), b.to(device)), x.double() @ w.double().t() + b.double()) < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("m", [5, 100, 129, 600])
def test_linear_with_silu_on_leading_features(m, device):
    g = torch.Generator().manual_seed(m)
    k, n, rows = 128, 328, 200
    x, w, b = torch.randn(m, k, generator=g).bfloat16(), (torch.randn(n, k, generator=g) * k ** -0.5).bfloat16(), torch.randn(n, generator=g)
    y = x.double() @ w.double().t() + b.double()
    want = torch.cat([O.silu(y[:, :rows]), y[:, rows:]], dim=1)
    assert rel(gemm.linear(x.to(device), w.to(device), bias=b.to(device), silu_rows=rows), want) < 4e-3
    assert rel(gemm.linear(x.to(device), w.to(device), bias=b.to(device), silu_rows=rows, out_dtype=torch.float32), want) < 1e-5


@pytest.mark.parametrize("device", DEVICES)
def test_embedding_stream(device):
    for dt in DTYPES:
        e = torch.randn(20, 90).to(dt)
        ids = torch.tensor([3, 19, 0, 3], dtype=torch.int32)
        assert torch.equal(stream.embed(ids.to(device), e.to(device)).cpu(), e[ids.long()].float())


def test_oracle_bucket_formula():
    """The oracle against the formula evaluated directly, away from the borders."""
    for n in (17, 40, 99, 130, 1000):
        x = math.log(n / 16) / math.log(150 / 16) * 16
        assert O.distance_bucket(n, 32, 150) == min(31, 16 + math.floor(x))
