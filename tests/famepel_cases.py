"""Small random Famepel models for the tests.

The routers of a 16-bit run must not flip between two nearly equal experts, or every comparison would be one of luck.  So the first dimensions of the
stream hold a code per token that no layer changes (their layer scales are zero) and the routers read almost nothing else; the codes are drawn so
that every choice, of groups and of experts, is clear."""
import json
import os

import torch

from gemm_b200.models import loader


def moe(experts, top, ff, scale, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def mamba2(heads, state, vdim, groups, conv, parts, mlp):
    return {"type": "mamba2", "mixer": {"heads": heads, "state": state, "vdim": vdim, "groups": groups, "conv": conv, "norm_groups": parts}, "mlp": mlp}


def hgrn2(heads, dim, vdim, mlp):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def latent(heads, dim, rot, vdim, kv_rank, q_rank, scale, base, mlp, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


# name -> (width, vocab, embedding scale, eps, layers)
_A, _B = moe(10, 3, 48, 1.7, 5, 2), moe(12, 4, 40, 2.2, 3, 2)
CASES = {
    # attention first, unequal sizes, two layers that read another's cache, layers without a feed-forward
    "mixed": (136, 211, 3.0, 1e-5, [latent(3, 24, 16, 40, 72, 56, 0.21, 1e4, _A, (4.0, 64, 32.0, 1.0)), mamba2(4, 40, 24, 2, 4, 2, _B), hgrn2(3, 24, 40, None),
                                    latent(5, 16, 16, 24, 72, 40, 0.3, 1e4, _B, (4.0, 64, 32.0, 1.0), 0), mamba2(6, 16, 32, 3, 2, 6, None),
                                    latent(2, 32, 8, 48, 48, 24, 0.15, 500.0, None, (2.5, 100, 8.0, 2.0)), hgrn2(2, 40, 16, _A),
                                    latent(4, 40, 8, 16, 48, 32, 0.25, 500.0, _A, (2.5, 100, 8.0, 2.0), 5)]),
    # sizes equal to 1: one head, one group, one tap, one expert per token out of one group; rotation without scaling
    "ones": (64, 97, 1.0, 1e-6, [mamba2(1, 8, 8, 1, 1, 1, moe(4, 1, 16, 1.0)), latent(1, 8, 2, 8, 8, 8, 0.5, 100.0, moe(3, 3, 8, 0.6, 3, 3)), hgrn2(1, 8, 8, moe(1, 1, 24, 1.0)),
                                 latent(1, 16, 2, 24, 8, 16, 0.4, 100.0, None, None, 1)]),
    # widths that are no multiples of 8 or 4
    "odd": (90, 131, 7.3, 1e-5, [hgrn2(3, 10, 9, moe(9, 4, 33, 2.5, 3, 2)), latent(3, 10, 6, 9, 30, 22, 0.3, 3000.0, moe(6, 2, 21, 1.3, 2, 1), (8.0, 32, 16.0, 1.0)),
                                 mamba2(3, 13, 11, 1, 3, 3, moe(9, 4, 33, 2.5, 3, 2)), mamba2(4, 7, 10, 4, 5, 1, None), latent(2, 14, 6, 18, 30, 10, 0.25, 3000.0, None, (8.0, 32, 16.0, 1.0), 1)]),
    # sizes of the tcgen05 kernels
    "wide": (256, 301, 2.0, 1e-6, [mamba2(4, 128, 64, 2, 4, 4, moe(16, 4, 128, 2.5, 4, 2)), hgrn2(2, 128, 128, moe(16, 4, 128, 2.5, 4, 2)),
                                   latent(4, 128, 64, 128, 512, 192, 192 ** -0.5, 5e5, moe(16, 2, 128, 1.0), (8.0, 128, 32.0, 1.0)), hgrn2(3, 64, 64, None),
                                   latent(40, 64, 32, 64, 512, 64, 0.1, 1e4, None), latent(8, 64, 64, 64, 512, 64, 0.125, 5e5, None, (8.0, 128, 32.0, 1.0), 2)]),
}


def _clear(z, r):
    """Whether a router that sees the logits z [E] chooses with a margin."""
    s = torch.sigmoid(z[: r["experts"]].double())
    cnt, keep = r["groups"]["count"], r["groups"]["keep"]
    if keep < cnt:
        g = s.reshape(cnt, -1).sort(dim=-1, descending=True).values[:, :2].sum(-1)
        o = g.sort(descending=True)
        if o.values[keep - 1] - o.values[keep] < 0.06:
            return False
        ok = torch.zeros(cnt, dtype=torch.bool)
        ok[o.indices[:keep]] = True
        s = s[ok.repeat_interleave(r["experts"] // cnt)]
    o = s.sort(descending=True).values
    return r["top"] == len(o) or bool(o[r["top"] - 1] - o[r["top"]] > 0.03)


def make_model(name, seed=0):
    """``{"config": ..., "t": ...}`` in the oracle's form; the values are bf16-representable, so that a bf16 checkpoint holds them exactly."""
    width, vocab, escale, eps, layers = CASES[name]
    g = torch.Generator().manual_seed(seed + 31)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def uni(n, lo, hi):
        return (torch.rand(n, generator=g) * (hi - lo) + lo).bfloat16()

    routers = [sp["mlp"]["router"] for sp in layers if sp["mlp"]]
    code = max(r["experts"] for r in routers)
    alpha, gain = torch.tensor(0.5).bfloat16(), 2.5
    t = {"embed": rnd(vocab, width, s=1.0 / escale)}
    for v in range(vocab):
        for _ in range(2000):
            x = (torch.rand(code, generator=g) * 5 - 2.5) / escale
            x = x.bfloat16()
            if all(_clear(gain * torch.tanh(alpha.float() * x.float() * escale), r) for r in routers):
                break
        else:
            raise RuntimeError("no clear code found")
        t["embed"][v, :code] = x

    def norm(nm, plain=False):
        t[nm], t[nm + ".b"], t[nm + ".alpha"] = (1 + rnd(width, s=0.3).float()).bfloat16(), rnd(width, s=0.2), uni(1, 0.4, 0.9).reshape(())
        if plain:
            t[nm][:code], t[nm + ".b"][:code], t[nm + ".alpha"] = 1.0, 0.0, alpha

    norm("final.norm")
    t["head"] = rnd(vocab, width, s=width ** -0.5)
    w = width ** -0.5
    for i, sp in enumerate(layers):
        m, p = sp["mixer"], f"l{i}."
        for nm in ("norm1", "norm1b") + (("norm2", "norm2b") if sp["mlp"] else ()):
            norm(p + nm, nm == "norm2")
        for nm in ("ls1",) + (("ls2",) if sp["mlp"] else ()):
            t[p + nm] = uni(width, 0.3, 1.0)
            t[p + nm][:code] = 0
        hd, v, p = m["heads"], m["vdim"], p + "mix."
        if sp["type"] == "mamba2":
            inner, gn = hd * v, m["groups"] * m["state"]
            t[p + "in"] = rnd(2 * inner + 2 * gn + hd, width, s=1.5 * w)
            t[p + "conv"], t[p + "conv.b"] = rnd(inner + 2 * gn, m["conv"], s=0.8), rnd(inner + 2 * gn, s=0.2)
            t[p + "dt_bias"], t[p + "A_log"], t[p + "D"] = uni(hd, -4.0, 0.5), uni(hd, -2.0, 2.0), rnd(hd)
            t[p + "norm"], t[p + "o"] = (1 + rnd(inner, s=0.3).float()).bfloat16(), rnd(width, inner, s=1.5 * inner ** -0.5)
        elif sp["type"] == "hgrn2":
            nq = hd * m["dim"]
            for nm, n in (("q", nq), ("f", nq), ("v", hd * v)):
                t[p + nm] = rnd(n, width, s=1.5 * w)
            t[p + "f.b"], t[p + "lower"] = uni(nq, -2.0, 5.0), uni(nq, 0.0, 0.95)
            t[p + "norm"], t[p + "o"] = (1 + rnd(v, s=0.3).float()).bfloat16(), rnd(width, hd * v, s=1.5 * (hd * v) ** -0.5)
        else:
            d, r, kr, qr = m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"]
            t[p + "dq"], t[p + "dq.norm"] = rnd(qr, width, s=1.5 * w), (1 + rnd(qr, s=0.3).float()).bfloat16()
            t[p + "uq"] = rnd(hd * (d + r), qr, s=1.6 * qr ** -0.5)
            if m.get("kv_from") is None:
                t[p + "dkv"], t[p + "dkv.norm"] = rnd(kr + r, width, s=1.5 * w), (1 + rnd(kr, s=0.3).float()).bfloat16()
            t[p + "uk"], t[p + "uv"] = rnd(hd * d, kr, s=1.6 * kr ** -0.5), rnd(hd * v, kr, s=kr ** -0.5)
            t[p + "sink"], t[p + "o"] = rnd(hd, s=2.0), rnd(width, hd * v, s=1.5 * (hd * v) ** -0.5)
        if sp["mlp"]:
            p, r, ff = f"l{i}.mlp.", sp["mlp"]["router"], sp["mlp"]["expert"]["ff"]
            t[p + "router"] = rnd(r["experts"], width, s=0.003)
            t[p + "router"][:, :code] = 0
            t[p + "router"][torch.arange(r["experts"]), torch.arange(r["experts"])] = gain
            for e in range(r["experts"]):
                t[f"{p}e{e}.gate"], t[f"{p}e{e}.up"] = rnd(ff, width, s=1.5 * w), rnd(ff, width, s=1.5 * w)
                t[f"{p}e{e}.down"] = rnd(width, ff, s=1.5 * ff ** -0.5)
    cfg = {"architecture": "Famepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": escale}, "layers": layers}
    return {"config": cfg, "t": t}


def save_model(model, path):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(model["config"], fh)
    loader.save_safetensors(model["t"], os.path.join(path, "model.safetensors"))
