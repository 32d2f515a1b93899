"""Plain, slow reference of Famepel: Mamba-2, HGRN2 and latent-attention mixers, grouped mixture of experts, Dynamic-Tanh norms around every
sublayer.  One function per mechanism, whole sequences at a time, nothing shared with the product code.

Every function works in the dtype of its inputs (the tests use float64).  ``model`` is a dict: ``config`` (the parsed config.json) and
``t`` (tensor name -> tensor)."""
import math

import torch


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp_min(z, 0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dyn_tanh(x, t, name):
    return torch.tanh(t[name + ".alpha"] * x) * t[name] + t[name + ".b"]


# ---------------------------------------------------------------------------------------------- rotation
def rotary_frequencies(rot):
    """(frequency of each pair, factor of cos and sin)."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, positions, rot):
    """x [T, ..., dims]: neighbours 2i and 2i + 1 turned by position * frequency."""
    f, mag = rotary_frequencies(rot)
    n = rot["dims"]
    a = positions.double().reshape(-1, *([1] * (x.dim() - 1))) * torch.tensor(f, dtype=torch.float64)
    c, s = (torch.cos(a) * mag).to(x.dtype), (torch.sin(a) * mag).to(x.dtype)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y = x.clone()
    y[..., 0:n:2] = u * c - v * s
    y[..., 1:n:2] = v * c + u * s
    return y


# ---------------------------------------------------------------------------------------------- recurrent mixers
def causal_conv_silu(x, w, b):
    """x [T, C], w [C, taps] (the last tap meets the current token), b [C]."""
    taps = w.shape[1]
    xp = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return silu(sum(w[:, k] * xp[k: k + x.shape[0]] for k in range(taps)) + b)


def ssd_recurrence(x, bm, cm, dt, a_log, d):
    """x [T, H, E], bm / cm [T, G, N], dt [T, H] (after softplus) -> [T, H, E]."""
    t, h, e = x.shape
    g, n = bm.shape[1:]
    s = torch.zeros(h, n, e, dtype=x.dtype)
    of = [hh // (h // g) for hh in range(h)]
    out = []
    for i in range(t):
        dec = torch.exp(-torch.exp(a_log) * dt[i]).reshape(h, 1, 1)
        s = dec * s + dt[i].reshape(h, 1, 1) * bm[i][of].unsqueeze(-1) * x[i].unsqueeze(1)
        out.append((s * cm[i][of].unsqueeze(-1)).sum(1) + d.reshape(h, 1) * x[i])
    return torch.stack(out)


def gated_group_norm(y, z, w, parts, eps):
    y = y * silu(z)
    return rms(y.reshape(y.shape[0], parts, -1), eps).reshape(y.shape) * w


def mamba2_mixer(h, t, pre, m, eps):
    hd, e, n, g = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = hd * e
    p = h @ t[pre + "in"].t()
    z, xbc, dt = p[:, :inner], p[:, inner: 2 * inner + 2 * g * n], p[:, 2 * inner + 2 * g * n:]
    xbc = causal_conv_silu(xbc, t[pre + "conv"], t[pre + "conv.b"])
    x = xbc[:, :inner].reshape(-1, hd, e)
    bm, cm = xbc[:, inner: inner + g * n].reshape(-1, g, n), xbc[:, inner + g * n:].reshape(-1, g, n)
    y = ssd_recurrence(x, bm, cm, softplus(dt + t[pre + "dt_bias"]), t[pre + "A_log"], t[pre + "D"])
    return gated_group_norm(y.reshape(-1, inner), z, t[pre + "norm"], m["norm_groups"], eps) @ t[pre + "o"].t()


def gated_recurrence(q, f, v):
    """q, f [T, H, D], v [T, H, E]: S <- diag(f) S + (1 - f) v^T, o = S^T q."""
    t, h, d = q.shape
    s = torch.zeros(h, d, v.shape[2], dtype=q.dtype)
    out = []
    for i in range(t):
        s = f[i].unsqueeze(-1) * s + (1 - f[i]).unsqueeze(-1) * v[i].unsqueeze(1)
        out.append((s * q[i].unsqueeze(-1)).sum(1))
    return torch.stack(out)


def hgrn2_mixer(h, t, pre, m, eps):
    hd, d, e = m["heads"], m["dim"], m["vdim"]
    q, v = silu(h @ t[pre + "q"].t()), h @ t[pre + "v"].t()
    low = t[pre + "lower"]
    f = low + (1 - low) * torch.sigmoid(h @ t[pre + "f"].t() + t[pre + "f.b"])
    o = gated_recurrence(q.reshape(-1, hd, d), f.reshape(-1, hd, d), v.reshape(-1, hd, e))
    return (rms(o, eps) * t[pre + "norm"]).reshape(-1, hd * e) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- latent attention
def sink_attention(q, k, v, scale, sink):
    """q, k [T, H, D], v [T, H, E], causal; exp(sink) joins each head's sum of weights."""
    t, h, _ = q.shape
    see = torch.ones(t, t, dtype=torch.bool).tril()
    out = torch.empty(t, h, v.shape[2], dtype=q.dtype)
    for i in range(h):
        s = ((q[:, i] @ k[:, i].t()) * scale).masked_fill(~see, float("-inf"))
        m = torch.maximum(s.max(-1, keepdim=True).values, sink[i])
        p = torch.exp(s - m)
        out[:, i] = (p @ v[:, i]) / (p.sum(-1, keepdim=True) + torch.exp(sink[i] - m))
    return out


def latent_cache(h, t, pre, m, eps):
    """(latent [T, rank], rotated key part [T, rot_dim]) of every token."""
    d = h @ t[pre + "dkv"].t()
    r = m["kv_rank"]
    return rms(d[:, :r], eps) * t[pre + "dkv.norm"], rotate(d[:, r:], torch.arange(h.shape[0]), m["rot"])


def latent_attention_mixer(h, t, pre, m, eps, cache):
    hd, d, rd, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = cache
    n = h.shape[0]
    q = ((rms(h @ t[pre + "dq"].t(), eps) * t[pre + "dq.norm"]) @ t[pre + "uq"].t()).reshape(n, hd, d + rd)
    q = torch.cat([q[..., :d], rotate(q[..., d:], torch.arange(n), m["rot"])], -1)
    k = torch.cat([(c @ t[pre + "uk"].t()).reshape(n, hd, d), kr.unsqueeze(1).expand(n, hd, rd)], -1)
    v = (c @ t[pre + "uv"].t()).reshape(n, hd, e)
    return sink_attention(q, k, v, m["scale"], t[pre + "sink"]).reshape(n, hd * e) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- experts
def route(z, top, groups, scale):
    """z [T, E] -> (chosen experts [T, top], their weights)."""
    s = torch.sigmoid(z)
    n, e = s.shape
    ok = torch.ones_like(s, dtype=torch.bool)
    if groups:
        cnt, keep = groups["count"], groups["keep"]
        per = s.reshape(n, cnt, e // cnt)
        best2 = per.sort(dim=-1, descending=True).values[..., :2].sum(-1)
        rank = best2.sort(dim=-1, descending=True, stable=True).indices[:, :keep]
        ok = torch.zeros(n, cnt, dtype=torch.bool).scatter(1, rank, True).repeat_interleave(e // cnt, dim=1)
    ids = s.masked_fill(~ok, -1.0).sort(dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20) * scale


def experts(h, t, pre, mlp):
    r = mlp["router"]
    ids, w = route(h @ t[pre + "router"].t(), r["top"], r.get("groups"), r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        tok, place = (ids == e).nonzero(as_tuple=True)
        if tok.numel():
            x = h[tok]
            y = (silu(x @ t[f"{pre}e{e}.gate"].t()) * (x @ t[f"{pre}e{e}.up"].t())) @ t[f"{pre}e{e}.down"].t()
            out[tok] += w[tok, place].unsqueeze(-1) * y
    return out


def forward(model, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of a whole sequence; ``capture`` (a list) receives the stream after every layer."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["t"].items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    caches = {}
    for li, spec in enumerate(cfg["layers"]):
        pre, m = f"l{li}.", spec["mixer"]
        h = dyn_tanh(x, t, pre + "norm1")
        if spec["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                caches[li] = latent_cache(h, t, pre + "mix.", m, eps)
            y = latent_attention_mixer(h, t, pre + "mix.", m, eps, caches[li if src is None else src])
        else:
            y = {"mamba2": mamba2_mixer, "hgrn2": hgrn2_mixer}[spec["type"]](h, t, pre + "mix.", m, eps)
        x = x + dyn_tanh(y, t, pre + "norm1b") * t[pre + "ls1"]
        if spec.get("mlp"):
            y = experts(dyn_tanh(x, t, pre + "norm2"), t, pre + "mlp.", spec["mlp"])
            x = x + dyn_tanh(y, t, pre + "norm2b") * t[pre + "ls2"]
        if capture is not None:
            capture.append(x.clone())
    return dyn_tanh(x, t, "final.norm") @ t["head"].t()
