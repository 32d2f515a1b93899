"""Plain, slow reference of Zedirax: minGRU recurrences, latent attention with a gate on its heads, attention with a query temperature and a logarithmic
distance bias, biased GELU feed-forwards, mixtures of plain (ungated) experts with a shared one, and a weighted average over all earlier layers behind
every layer.  One function per mechanism, whole sequences at a time, nothing shared with the product code.

Every function works in the dtype of its inputs (the tests use float64).  ``model`` is a dict: ``config`` (the parsed config.json) and
``t`` (tensor name -> tensor)."""
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit(x, eps) * (1 + w)


# ---------------------------------------------------------------------------------------------- minGRU
def gru_recurrence(z, u):
    """z (a gate's logit) and u [T, N]: the states after every token, from zero."""
    s = torch.zeros_like(z[0])
    out = []
    for t in range(z.shape[0]):
        a = sigmoid(z[t])
        cand = torch.where(u[t] >= 0, u[t] + 0.5, sigmoid(u[t]))
        s = (1 - a) * s + a * cand
        out.append(s)
    return torch.stack(out)


def gru_mixer(h, t, pre):
    s = gru_recurrence(h @ t[pre + "z"].t() + t[pre + "z.b"], h @ t[pre + "x"].t() + t[pre + "x.b"])
    return (s * silu(h @ t[pre + "g"].t())) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- attention
def rotate_halves(x, base):
    """x [T, ..., n], token t at position t: dimension i turns with dimension i + n / 2."""
    n = x.shape[-1]
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64).reshape([-1] + [1] * (x.dim() - 1)) * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., : n // 2], x[..., n // 2:]
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def causal_softmax(s):
    """s [T, T]: the weights of keys j <= i."""
    n = s.shape[0]
    i = torch.arange(n)
    s = s.masked_fill(i.unsqueeze(0) > i.unsqueeze(1), -math.inf)
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    return p / p.sum(-1, keepdim=True)


def latent_attend(q, c, kr, uk, uv, scale, base):
    """q [T, H, dim + rot], latents c [T, r], the heads' common key part kr [T, rot], uk [H, dim, r], uv [H, vdim, r] -> [T, H, vdim]."""
    heads, dim = uk.shape[0], uk.shape[1]
    kr = rotate_halves(kr, base)
    out = []
    for h in range(heads):
        k, v = c @ uk[h].t(), c @ uv[h].t()
        s = (q[:, h, :dim] @ k.t() + rotate_halves(q[:, h, dim:], base) @ kr.t()) * scale
        out.append(causal_softmax(s) @ v)
    return torch.stack(out, 1)


def latent_mixer(h, t, pre, m, eps):
    n, hd, r = h.shape[0], m["heads"], m["kv_rank"]
    low = h @ t[pre + "dkv"].t()
    c = unit(low[:, :r], eps) * t[pre + "dkv.norm"]
    o = latent_attend((h @ t[pre + "q"].t()).reshape(n, hd, -1), c, low[:, r:], t[pre + "uk"].reshape(hd, -1, r), t[pre + "uv"].reshape(hd, -1, r), m["scale"], m["rot"]["base"])
    return (o.reshape(n, -1) * sigmoid(h @ t[pre + "g"].t())) @ t[pre + "o"].t()


def temperature(n, coef, every):
    """Factor of the queries at positions 0 .. n - 1."""
    return torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in range(n)], dtype=torch.float64)


def attend(q, k, v, scale, r1, r2, first=0):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; a score loses r1 ln(1 + r2 distance).  Only rows from ``first`` on mean anything to the caller."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    i = torch.arange(n)
    dist = (i.unsqueeze(1) - i.unsqueeze(0)).clamp_min(0).to(q.dtype)
    return torch.stack([causal_softmax((q[:, h] @ k[:, h // per].t()) * scale - r1[h] * torch.log(1 + r2[h] * dist)) @ v[:, h // per] for h in range(heads)], 1)


def attention_mixer(h, t, pre, m):
    n = h.shape[0]
    q, k, v = ((h @ t[pre + c].t()).reshape(n, m["heads" if c == "q" else "kv_heads"], -1) for c in "qkv")
    tmp = temperature(n, m["q_temp"]["coef"], m["q_temp"]["every"]).to(h.dtype)
    return attend(q * tmp.reshape(-1, 1, 1), k, v, m["scale"], t[pre + "r1"], t[pre + "r2"]).reshape(n, -1) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- feed-forward
def biased_gelu(h, t, pre):
    g, u = (h @ t[pre + c].t() + t[pre + c + ".b"] for c in ("gate", "up"))
    return (gelu_tanh(g) * u) @ t[pre + "down"].t() + t[pre + "down.b"]


def plain_expert(h, t, pre):
    return gelu_erf(h @ t[pre + "up"].t()) @ t[pre + "down"].t()


def route(z, top):
    """z [T, E] -> (chosen experts [T, top], their weights)."""
    o = z.sort(dim=-1, descending=True, stable=True)
    w = torch.exp(o.values[:, :top] - o.values[:, :1])
    return o.indices[:, :top], w / w.sum(-1, keepdim=True)


def experts(h, t, pre, mlp):
    r = mlp["router"]
    ids, w = route(h @ t[pre + "router"].t(), r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        tok, place = (ids == e).nonzero(as_tuple=True)
        out[tok] += w[tok, place].unsqueeze(-1) * plain_expert(h[tok], t, f"{pre}e{e}.")
    if mlp.get("shared"):
        out = out + sigmoid(h @ t[pre + "shared.sg"].t()) * plain_expert(h, t, pre + "shared.")
    return out


# ---------------------------------------------------------------------------------------------- model
def mixer(h, t, pre, spec, eps):
    m = spec["mixer"]
    if spec["type"] == "mingru":
        return gru_mixer(h, t, pre)
    return latent_mixer(h, t, pre, m, eps) if spec["type"] == "latent_attention" else attention_mixer(h, t, pre, m)


def depth_average(xs, w):
    return sum(w[j] * x for j, x in enumerate(xs))


def forward(model, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of a whole sequence; ``capture`` (a list) receives what every layer hands on."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["t"].items()}
    eps, by = cfg["norm"]["eps"], cfg["residual_mult"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    xs = [x]
    for i, spec in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + by * mixer(norm(x, t[pre + "norm1"], eps), t, pre + "mix.", spec, eps)
        if spec.get("mlp"):
            h = norm(x, t[pre + "norm2"], eps)
            x = x + by * (biased_gelu(h, t, pre + "mlp.") if spec["mlp"]["kind"] == "dense" else experts(h, t, pre + "mlp.", spec["mlp"]))
        xs.append(x)
        x = depth_average(xs, t[pre + "dwa"])
        if capture is not None:
            capture.append(x.clone())
    return norm(x, t["final.norm"], eps) @ t["head"].t()
