"""Small random Fidolix models for the tests.

The routers of a 16-bit run must not flip between two nearly equal experts, or every comparison would be one of luck.  So the first dimensions of the
stream hold a code per token that no layer changes (nothing is projected there, and a norm only scales it, which keeps the order of the logits), the routers
read almost nothing else, and the codes are drawn so that every choice, of groups and of experts, is clear.  The norms' eps is large enough that a vector
which happens to be nearly zero does not blow up its rounding."""
import json
import os

import torch

from gemm_b200.models import loader


def moe(experts, top, ff, count=0, keep=0):
    r = {"experts": experts, "top": top}
    if count:
        r["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def attention(heads, kv_heads, dim, vdim, scale, softcap, mlp):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}, "mlp": mlp}


def parallel(heads, kv_heads, dim, conv, window, rot, scale, right, rank, scales, mlp):
    """``rot`` (dims, base, scaling or None), ``right`` (heads, dim); ``rank``: of the decay's projection."""
    r = {"dims": rot[0], "base": rot[1]}
    if rot[2]:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "mask": {"size": window} if window else None, "rot": r, "scale": scale}
    return {"type": "parallel", "rank": rank, "mlp": mlp,
            "mixer": {"left": left, "right": {"heads": right[0], "dim": right[1]}, "left_scale": scales[0], "right_scale": scales[1]}}


_Y = (4.0, 64, 32.0, 1.0)
# name -> (width, vocab, embedding scale, eps, token input, loop, layers)
CASES = {
    # a looped middle, uneven sizes, part of the head rotated, layers without a feed-forward
    "mixed": (136, 211, 3.0, 1e-2, 20, {"start": 1, "stop": 4, "times": 3},
              [parallel(6, 3, 40, 4, 33, (24, 1e4, _Y), 0.2, (3, 24), 12, (0.7, 1.3), dense(200, 1.1)), attention(4, 2, 40, 24, 0.3, 9.0, moe(10, 3, 48, 5, 2)),
               parallel(5, 1, 32, 2, 70, (32, 500.0, (2.5, 100, 8.0, 2.0)), 0.25, (2, 40), 20, (1.2, -0.6), moe(12, 4, 40, 3, 2)), attention(6, 1, 24, 48, 0.25, 3.0, None),
               parallel(3, 3, 16, 3, 17, (8, 300.0, None), 0.3, (4, 16), 8, (0.5, 0.9), None), attention(3, 3, 16, 16, 0.5, 40.0, dense(72, 0.4))]),
    # sizes equal to 1: one head, one tap, one key in the window, one expert per token, a loop of one pass, a token input of one number
    "ones": (64, 97, 1.0, 0.05, 1, {"start": 0, "stop": 2, "times": 1},
             [parallel(1, 1, 8, 1, 1, (2, 100.0, None), 0.5, (1, 8), 1, (1.0, 1.0), moe(4, 1, 16)), attention(1, 1, 8, 8, 0.5, 1.0, moe(1, 1, 24)),
              attention(2, 1, 16, 8, 0.4, 5.0, dense(8, 1.0))]),
    # widths that are no multiples of 8 or 4, odd heads, no window, no loop
    "odd": (90, 131, 7.3, 1e-2, 11, None,
            [attention(3, 1, 10, 9, 0.3, 7.0, moe(9, 4, 33, 3, 2)), parallel(4, 2, 7, 5, 0, (6, 3000.0, (8.0, 32, 16.0, 1.0)), 0.3, (3, 9), 5, (0.8, 0.8), dense(50, 2.0)),
             parallel(3, 3, 13, 3, 21, (10, 3000.0, None), 0.25, (5, 11), 6, (1.0, 0.4), moe(6, 2, 21)), attention(2, 2, 14, 18, 0.3, 30.0, None)]),
    # sizes of the tcgen05 kernels, the whole model looped
    "wide": (256, 301, 2.0, 1e-3, 64, {"start": 0, "stop": 3, "times": 2},
             [attention(8, 2, 128, 64, 128 ** -0.5, 12.0, moe(16, 4, 128, 4, 2)), parallel(8, 2, 128, 4, 129, (64, 5e5, (8.0, 128, 32.0, 1.0)), 128 ** -0.5, (2, 128), 32, (0.9, 1.1), dense(256, 3.0)),
              parallel(4, 4, 64, 2, 64, (64, 1e4, None), 0.125, (4, 64), 16, (1.0, 1.0), moe(16, 2, 128, 2, 1))]),
}


def _clear(code, r):
    """Whether a router that sees the logits ``code`` [E], times any positive factor, chooses with a margin."""
    z = code[: r["experts"]].double()
    g = r.get("groups")
    if g and g["keep"] < g["count"]:
        o = z.reshape(g["count"], -1).max(-1).values.sort(descending=True)
        if o.values[g["keep"] - 1] - o.values[g["keep"]] < 0.12:
            return False
        ok = torch.zeros(g["count"], dtype=torch.bool)
        ok[o.indices[: g["keep"]]] = True
        z = z[ok.repeat_interleave(r["experts"] // g["count"])]
    o = z.sort(descending=True).values
    return r["top"] == len(o) or bool(o[r["top"] - 1] - o[r["top"]] > 0.12)


def make_model(name, seed=0):
    """``{"config": ..., "t": ...}`` in the oracle's form; the values are bf16-representable, so that a bf16 checkpoint holds them exactly."""
    width, vocab, escale, eps, side, loop, layers = CASES[name]
    g = torch.Generator().manual_seed(seed + 41)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    def uni(n, lo, hi):
        return (torch.rand(n, generator=g) * (hi - lo) + lo).bfloat16()

    def near_one(n):
        return (1 + rnd(n, s=0.3).float()).bfloat16()

    routers = [sp["mlp"]["router"] for sp in layers if sp["mlp"] and sp["mlp"]["kind"] == "moe"]
    code = max((r["experts"] for r in routers), default=0)
    t = {"embed": rnd(vocab, width, s=1.0 / escale), "side.embed": rnd(vocab, side * len(layers)), "final.norm": near_one(width), "head": rnd(vocab, width, s=width ** -0.5)}
    for v in range(vocab if code else 0):
        for _ in range(4000):
            x = (torch.rand(code, generator=g) * 4 - 2).bfloat16()
            if all(_clear(x.float(), r) for r in routers):
                break
        else:
            raise RuntimeError("no clear code found")
        t["embed"][v, :code] = (x.float() / escale).bfloat16()
    w = width ** -0.5

    def out(n):                                     # a projection into the stream leaves the code alone
        o = rnd(width, n, s=1.5 * n ** -0.5)
        o[:code] = 0
        return o

    def att(p, m, names):
        for nm in names:
            n = m["heads" if nm == "q" else "kv_heads"] * m["vdim" if nm == "v" else "dim"]
            t[p + nm], t[p + nm + ".b"] = rnd(n, width, s=1.5 * w), rnd(n, s=0.5)
        t[p + "o"] = out(m["heads"] * m["vdim"])

    for i, sp in enumerate(layers):
        m, p = sp["mixer"], f"l{i}.mix."
        t[f"l{i}.norm1"], t[f"l{i}.norm2"] = near_one(width), near_one(width)
        t[f"l{i}.norm2"][:code] = 1
        if sp["type"] == "attention":
            att(p, m, "qkv")
            for nm, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"])):
                t[p + nm + ".norm"] = near_one(n)
            t[p + "g"] = rnd(m["heads"] * m["vdim"], width, s=1.5 * w)
        else:
            q, l, r = p + "right.", m["left"], m["right"]
            att(p + "left.", l, "qk")
            for nm, n in (("q", l["heads"] * l["dim"]), ("k", l["kv_heads"] * l["dim"])):
                t[f"{p}left.{nm}.conv"] = rnd(n, l["conv"], s=0.8)
            t[p + "left.sink"] = rnd(l["heads"], s=2.0)
            n = r["heads"] * r["dim"]
            for nm in "rkvg":
                t[q + nm] = rnd(n, width, s=1.5 * w)
            for nm in "rkvgw":
                t[q + "mu." + nm] = uni(width, 0.0, 1.0)
            t[q + "w1"], t[q + "w2"], t[q + "w0"] = rnd(sp["rank"], width, s=1.5 * w), rnd(n, sp["rank"], s=0.7 * sp["rank"] ** -0.5), uni(n, -5.0, 1.0)
            t[q + "u"], t[q + "norm"], t[q + "o"] = rnd(r["heads"], r["dim"]), near_one(n), out(n)
        if sp["mlp"]:
            p, mlp = f"l{i}.mlp.", sp["mlp"]
            ff = mlp["ff"] if mlp["kind"] == "dense" else mlp["expert"]["ff"]
            for e in [""] if mlp["kind"] == "dense" else [f"e{e}." for e in range(mlp["router"]["experts"])]:
                t[p + e + "gate"], t[p + e + "up"], t[p + e + "down"] = rnd(ff, width, s=1.5 * w), rnd(ff, width, s=1.5 * w), out(ff)
            if mlp["kind"] == "moe":
                n = mlp["router"]["experts"]
                t[p + "router"] = rnd(n, width, s=0.0003)
                t[p + "router"][:, :code] = 0
                t[p + "router"][torch.arange(n), torch.arange(n)] = 1.0
        p = f"l{i}.side."
        t[p + "gate"], t[p + "proj"], t[p + "norm"] = rnd(side, width, s=w), rnd(width, side, s=1.5 * side ** -0.5), uni(width, 0.3, 0.9)
        t[p + "norm"][:code] = 0
    cfg = {"architecture": "Fidolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": escale}, "token_side": {"dim": side},
           "layers": [{k: v for k, v in sp.items() if k != "rank"} for sp in layers]}
    if loop:
        cfg["loop"] = loop
    return {"config": cfg, "t": t}


def save_model(model, path):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(model["config"], fh)
    loader.save_safetensors(model["t"], os.path.join(path, "model.safetensors"))
