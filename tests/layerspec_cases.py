"""Small random models and schedules for the tests of models described layer by layer."""
import json
import os

import torch

from gemm_b200.models import loader


def lightning_layer(heads, dim, vdim, ff, decays):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decays}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention_layer(heads, kv_heads, dim, vdim, ff, size, keep, bias_max, rel, scale):
    return {"type": "attention", "rel": rel, "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
                      "mask": {"size": size, "keep_first": keep}}}


# name -> (width, vocab, layers, loop, logit_scale, eps)
CASES = {
    # lightning first, uneven sizes, a loop over two layers, no feed-forward in one layer
    "mixed": (136, 211, [lightning_layer(3, 24, 40, 200, [0.31, 0.83, 0.997]),
                         attention_layer(4, 2, 40, 56, 144, 33, 5, 90, 12, 0.5),
                         lightning_layer(2, 72, 24, 0, [0.9, 0.5]),
                         attention_layer(6, 1, 64, 128, 96, 70, 0, 300, 32, 0.3)], {"start": 1, "stop": 3, "times": 3}, 0.7, 1e-5),
    # sizes equal to 1: one head, one key/value head, a loop of one pass, two bias rows
    "ones": (64, 97, [attention_layer(1, 1, 16, 8, 32, 1, 1, 50, 2, 1.1), lightning_layer(1, 8, 8, 24, [0.75]),
                      attention_layer(2, 2, 8, 16, 0, 20, 3, 17, 6, 0.9)], {"start": 0, "stop": 1, "times": 1}, 1.0, 1e-6),
    # no loop; widths that are no multiple of 8 or 4; heads wider than the flash kernels' 128 columns; an odd number of bias rows
    "odd": (90, 131, [lightning_layer(2, 10, 12, 50, [1.0, 0.6]), attention_layer(3, 3, 130, 20, 70, 50, 9, 64, 8, 0.2),
                      lightning_layer(5, 7, 9, 33, [0.1, 0.3, 0.5, 0.7, 0.9])], None, 1.3, 1e-5),
    # whole-model sizes of the tcgen05 kernels: 128-wide heads, groups of four, page and window edges at multiples of 64 and off them
    "wide": (256, 301, [attention_layer(8, 2, 128, 64, 256, 129, 70, 200, 32, 0.12), lightning_layer(2, 128, 128, 256, [0.95, 0.9995]),
                        attention_layer(4, 4, 64, 128, 0, 64, 64, 33, 32, 0.4)], {"start": 0, "stop": 2, "times": 2}, 0.5, 1e-6),
}


def make_model(name, seed=0):
    """``{"config": ..., "t": ...}`` in the oracle's form; the values are bf16-representable, so that a bf16 checkpoint holds them exactly."""
    width, vocab, layers, loop, logit_scale, eps = CASES[name]
    g = torch.Generator().manual_seed(seed + 17)

    def rnd(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s).bfloat16()

    t = {"embed": rnd(vocab, width), "final.norm": rnd(width, s=0.2)}
    if loop:
        t["loop.step"] = rnd(loop["times"], width, s=0.7)
    for i, sp in enumerate(layers):
        m, p = sp["mixer"], f"l{i}."
        t[p + "norm1"] = rnd(width, s=0.3)
        w = width ** -0.5
        if sp["type"] == "lightning":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for nm, n in (("q", hd), ("k", hd), ("v", hv), ("g", hv)):
                t[p + "mix." + nm] = rnd(n, width, s=1.5 * w)
            t[p + "mix.norm"] = (1 + rnd(hv, s=0.3).float()).bfloat16()
            t[p + "mix.o"] = rnd(width, hv, s=1.5 * hv ** -0.5)
        else:
            for nm, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                t[p + "mix." + nm] = rnd(n, width, s=1.5 * w)
                t[p + "mix." + nm + ".b"] = rnd(n, s=0.5)
            t[p + "mix.rel"] = rnd(sp["rel"], m["heads"], s=1.5)
            hv = m["heads"] * m["vdim"]
            t[p + "mix.o"] = rnd(width, hv, s=1.5 * hv ** -0.5)
        if sp["mlp"]:
            ff = sp["mlp"]["ff"]
            t[p + "norm2"] = rnd(width, s=0.3)
            t[p + "mlp.gate"] = rnd(ff, width, s=1.5 * w)
            t[p + "mlp.up"] = rnd(ff, width, s=w)
            t[p + "mlp.down"] = rnd(width, ff, s=ff ** -0.5)
    cfg = {"architecture": "Zogavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "layers": [{k: v for k, v in sp.items() if k != "rel"} for sp in layers]}
    if loop:
        cfg["loop"] = loop
    return {"config": cfg, "t": t}


def save_model(model, path):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(model["config"], fh)
    loader.save_safetensors(model["t"], os.path.join(path, "model.safetensors"))


def tokens(model, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, model["config"]["vocab"], (n,), generator=g).tolist()


def cuts(n, sizes):
    """Portions of a prompt of n tokens: the sizes in turn, around and around."""
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


def replay_one(rep, toks, portions, rid="r"):
    """All logits [n, vocab] of one request fed in the given portions."""
    got, at = [], 0
    for i, n in enumerate(portions):
        got.append(rep.step([{"id": rid, "tokens": toks[at: at + n], "want": list(range(n))}], [rid] if at + n == len(toks) else []))
        at += n
    assert at == len(toks)
    return torch.cat(got)


def err(got, want):
    """Root mean square of the difference per position (means taken off), over the root mean square of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
