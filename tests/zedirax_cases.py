"""Small random Zedirax models for the tests.

The routers of a 16-bit run must not flip between two nearly equal experts, or every comparison would be one of luck.  So the first dimensions of the
stream hold a code per token that no layer changes but for a positive factor (nothing is projected there, norms and averages only scale it), the routers
read almost nothing else, and the codes are drawn so that every choice of experts is clear."""
import json
import os

import torch

from gemm_b200.models import loader


def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {**m, "shared": {"ff": shared}} if shared else m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def mingru(width, mlp):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, base, scale, mlp):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "rot_dim": rot_dim,
                                                              "rot": {"base": base, "dims": rot_dim}, "scale": scale}}


def attention(heads, kv_heads, dim, vdim, scale, coef, every, mlp):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "q_temp": {"coef": coef, "every": every}}}


# name -> (width, vocab, eps, factor of every sublayer, layers)
CASES = {
    # all kinds beside each other, uneven sizes, layers without a feed-forward, experts with and without a shared one
    "mixed": (136, 211, 1e-2, 0.6, [mingru(200, moe(10, 3, 48, 72)), attention(6, 3, 40, 24, 0.25, 0.3, 17, dense(200)), latent(3, 24, 8, 40, 72, 1e4, 0.2, moe(12, 4, 40)),
                                    attention(4, 1, 24, 48, 0.3, 0.7, 50, None), mingru(72, None), latent(5, 40, 24, 16, 56, 500.0, 0.15, dense(72))]),
    # sizes equal to 1: one head, one expert, a state of one number, a latent of few numbers
    "ones": (64, 97, 0.3, 1.0, [latent(1, 8, 2, 8, 8, 100.0, 0.5, moe(1, 1, 16, 8)), mingru(1, moe(4, 1, 24)), attention(1, 1, 8, 8, 0.5, 0.2, 1, dense(1)), attention(2, 1, 16, 8, 0.4, 0.0, 5, None)]),
    # widths that are no multiples of 8 or 4, odd heads and ranks
    "odd": (90, 131, 1e-2, 1.3, [attention(3, 1, 10, 9, 0.3, 0.5, 3, moe(9, 4, 33, 21)), mingru(77, dense(50)), latent(3, 13, 6, 9, 30, 3000.0, 0.25, moe(6, 2, 21, 50)), mingru(90, None)]),
    # sizes of the tcgen05 kernels
    "wide": (256, 301, 1e-3, 0.5, [latent(4, 128, 64, 128, 256, 5e5, 192 ** -0.5, moe(16, 4, 128, 256)), attention(8, 2, 128, 128, 128 ** -0.5, 0.2, 64, dense(256)), mingru(512, moe(16, 2, 128)),
                                   attention(4, 4, 64, 64, 0.125, 0.4, 100, moe(16, 4, 256, 128)), latent(8, 64, 32, 64, 128, 1e4, 96 ** -0.5, dense(384))]),
    # many layers: averages over many places
    "deep": (72, 101, 1e-2, 0.4, [mingru(40, None), attention(2, 1, 16, 16, 0.3, 0.3, 20, None), latent(2, 16, 8, 16, 24, 1e3, 0.2, None)] * 7 + [mingru(64, dense(40))]),
}


def _clear(code, r):
    """Whether a router that sees the logits ``code``, times any positive factor, chooses with a margin."""
    o = code[: r["experts"]].double().sort(descending=True).values
    return r["top"] == len(o) or bool(o[r["top"] - 1] - o[r["top"]] > 0.12)


def make_model(name, seed=0):
    """``{"config": ..., "t": ...}`` in the oracle's form; the values are bf16-representable, so that a bf16 checkpoint holds them exactly."""
    width, vocab, eps, by, layers = CASES[name]
    g = torch.Generator().manual_seed(seed + 53)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def uni(n, lo, hi):
        return (torch.rand(n, generator=g) * (hi - lo) + lo).bfloat16()

    routers = [sp["mlp"]["router"] for sp in layers if sp["mlp"] and sp["mlp"]["kind"] == "moe"]
    code = max((r["experts"] for r in routers), default=0)
    t = {"embed": rnd(vocab, width), "final.norm": rnd(width, s=0.3), "head": rnd(vocab, width, s=width ** -0.5)}
    for v in range(vocab if code else 0):
        for _ in range(4000):
            x = (torch.rand(code, generator=g) * 4 - 2).bfloat16()
            if all(_clear(x.float(), r) for r in routers):
                break
        else:
            raise RuntimeError("no clear code found")
        t["embed"][v, :code] = x
    w = width ** -0.5

    def out(n):                                     # a projection into the stream leaves the code alone
        o = rnd(width, n, s=1.5 * n ** -0.5)
        o[:code] = 0
        return o

    for i, sp in enumerate(layers):
        m, p = sp["mixer"], f"l{i}.mix."
        t[f"l{i}.norm1"] = rnd(width, s=0.3)
        a = rnd(i + 2, s=0.35 * (i + 1) ** -0.5)
        a[-1] = 1.3
        t[f"l{i}.dwa"] = a
        if sp["type"] == "mingru":
            n = m["width"]
            for c in "zxg":
                t[p + c] = rnd(n, width, s=1.5 * w)
            t[p + "z.b"], t[p + "x.b"], t[p + "o"] = uni(n, -6.0, 1.0), rnd(n, s=0.5), out(n)
        elif sp["type"] == "latent_attention":
            hd, r, rd = m["heads"], m["kv_rank"], m["rot_dim"]
            t[p + "q"], t[p + "dkv"] = rnd(hd * (m["dim"] + rd), width, s=1.5 * w), rnd(r + rd, width, s=1.5 * w)
            t[p + "dkv.norm"] = (1 + rnd(r, s=0.3).float()).bfloat16()
            t[p + "uk"], t[p + "uv"] = rnd(hd * m["dim"], r, s=1.5 * r ** -0.5), rnd(hd * m["vdim"], r, s=1.5 * r ** -0.5)
            t[p + "g"], t[p + "o"] = rnd(hd * m["vdim"], width, s=1.5 * w), out(hd * m["vdim"])
        else:
            for c, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                t[p + c] = rnd(n, width, s=1.5 * w)
            t[p + "r1"], t[p + "r2"], t[p + "o"] = uni(m["heads"], 0.0, 2.0), uni(m["heads"], 0.05, 1.5), out(m["heads"] * m["vdim"])
        if sp["mlp"]:
            p, mlp = f"l{i}.mlp.", sp["mlp"]
            t[f"l{i}.norm2"] = rnd(width, s=0.3)
            t[f"l{i}.norm2"][:code] = 0
            if mlp["kind"] == "dense":
                ff = mlp["ff"]
                for c in ("gate", "up"):
                    t[p + c], t[p + c + ".b"] = rnd(ff, width, s=1.5 * w), rnd(ff, s=0.7)
                t[p + "down"], t[p + "down.b"] = out(ff), rnd(width, s=0.5)
                t[p + "down.b"][:code] = 0
                continue
            n = mlp["router"]["experts"]
            sizes = {f"e{e}.": mlp["expert"]["ff"] for e in range(n)}
            if mlp.get("shared"):
                sizes["shared."] = mlp["shared"]["ff"]
                t[p + "shared.sg"] = rnd(1, width, s=1.5 * w)
            for e, ff in sizes.items():
                t[p + e + "up"], t[p + e + "down"] = rnd(ff, width, s=2.0 * w), out(ff)
            t[p + "router"] = rnd(n, width, s=0.0003)
            t[p + "router"][:, :code] = 0
            t[p + "router"][torch.arange(n), torch.arange(n)] = 1.0
    return {"config": {"architecture": "Zedirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": by, "layers": layers}, "t": t}


def save_model(model, path):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(model["config"], fh)
    loader.save_safetensors(model["t"], os.path.join(path, "model.safetensors"))
