"""Plain, slow reference of Fidolix: softcapped gated attention, a windowed attention with sinks beside an RWKV-style recurrence, dense and
mixture-of-experts feed-forwards next to the mixer, a looped middle and a per-layer token input.  One function per mechanism, whole sequences at
a time, nothing shared with the product code.

Every function works in the dtype of its inputs (the tests use float64).  ``model`` is a dict: ``config`` (the parsed config.json) and
``t`` (tensor name -> tensor)."""
import math

import torch


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ---------------------------------------------------------------------------------------------- rotation
def rotary_table(rot):
    """(frequency of each pair, factor of cos and sin)."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return freq, 1.0
    at = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), n - 1)
    ramp = [min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001))) for i in range(n // 2)]
    return [f / sc["factor"] * r + f * (1 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot):
    """x [T, heads, dim], token t at position t: dimensions 2i and 2i + 1 below rot.dims are turned."""
    freq, mag = rotary_table(rot)
    n = rot["dims"]
    a = torch.arange(x.shape[0], dtype=torch.float64).reshape(-1, 1, 1) * torch.tensor(freq, dtype=torch.float64)
    c, s = (torch.cos(a) * mag).to(x.dtype), (torch.sin(a) * mag).to(x.dtype)
    y = x.clone()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2], y[..., 1:n:2] = u * c - v * s, v * c + u * s
    return y


def short_conv(u, w):
    """u [T, C], w [C, taps]; the last tap meets the current token."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] += w[:, j] * u[: n - back]
    return y


# ---------------------------------------------------------------------------------------------- attention
def attend(q, k, v, scale, window=None, softcap=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    i = torch.arange(n)
    dist = i.unsqueeze(1) - i.unsqueeze(0)
    see = dist >= 0
    if window is not None:
        see &= dist < window
    out = torch.empty(n, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        s = (q[:, h] @ k[:, h // per].t()) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~see, -math.inf)
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp_min(top, float(sink[h]))
        p = torch.exp(s - top)
        total = p.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[h] - top)
        out[:, h] = (p / total) @ v[:, h // per]
    return out


def attention_mixer(h, t, pre, m, eps):
    n, hd, g = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (h @ t[pre + c].t() + t[pre + c + ".b"] for c in "qkv")
    q, k = rms(q, eps) * t[pre + "q.norm"], rms(k, eps) * t[pre + "k.norm"]
    o = attend(q.reshape(n, hd, -1), k.reshape(n, g, -1), v.reshape(n, g, -1), m["scale"], softcap=m["softcap"]).reshape(n, -1)
    return (o * torch.sigmoid(h @ t[pre + "g"].t())) @ t[pre + "o"].t()


def left_mixer(h, t, pre, m):
    n, hd, g = h.shape[0], m["heads"], m["kv_heads"]
    q, k = (short_conv(h @ t[pre + c].t() + t[pre + c + ".b"], t[pre + c + ".conv"]) for c in "qk")
    q, k = q.reshape(n, hd, -1), k.reshape(n, g, -1)
    window = m["mask"]["size"] if m.get("mask") else None
    o = attend(rotate(q, m["rot"]), rotate(k, m["rot"]), k, m["scale"], window=window, sink=t[pre + "sink"])
    return o.reshape(n, -1) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- RWKV-style recurrence
def shift_mix(h, mu):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def time_recurrence(r, k, v, w, u):
    """r, k, w [T, H, D], v [T, H, E], u [H, D]: the current token counts with the bonus u, then enters the state."""
    s = torch.zeros(r.shape[1], r.shape[2], v.shape[2], dtype=r.dtype)
    out = []
    for i in range(r.shape[0]):
        kv = k[i].unsqueeze(-1) * v[i].unsqueeze(1)
        out.append(((s + u.unsqueeze(-1) * kv) * r[i].unsqueeze(-1)).sum(1))
        s = w[i].unsqueeze(-1) * s + kv
    return torch.stack(out)


def right_mixer(h, t, pre, m, eps):
    n, hd = h.shape[0], m["heads"]
    mixed = {c: shift_mix(h, t[pre + "mu." + c]) for c in "rkvgw"}
    r, k, v, g = (mixed[c] @ t[pre + c].t() for c in "rkvg")
    w = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ t[pre + "w1"].t()) @ t[pre + "w2"].t() + t[pre + "w0"]))
    o = time_recurrence(*(z.reshape(n, hd, -1) for z in (r, k, v, w)), t[pre + "u"])
    return (rms(o, eps).reshape(n, -1) * t[pre + "norm"] * silu(g)) @ t[pre + "o"].t()


# ---------------------------------------------------------------------------------------------- feed-forward, token input
def capped_swiglu(h, t, pre, limit):
    g = torch.clamp_max(h @ t[pre + "gate"].t(), limit)
    u = torch.clamp(h @ t[pre + "up"].t(), -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ t[pre + "down"].t()


def route(z, top, groups):
    """z [T, E] -> (chosen experts [T, top], their weights)."""
    s = torch.softmax(z, -1)
    n, e = s.shape
    ok = torch.ones_like(s, dtype=torch.bool)
    if groups:
        best = s.reshape(n, groups["count"], -1).max(-1).values
        kept = best.sort(dim=-1, descending=True, stable=True).indices[:, : groups["keep"]]
        ok = torch.zeros(n, groups["count"], dtype=torch.bool).scatter(1, kept, True).repeat_interleave(e // groups["count"], dim=1)
    ids = s.masked_fill(~ok, -1.0).sort(dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def experts(h, t, pre, mlp):
    r = mlp["router"]
    ids, w = route(h @ t[pre + "router"].t(), r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        tok, place = (ids == e).nonzero(as_tuple=True)
        x = h[tok]
        y = (silu(x @ t[f"{pre}e{e}.gate"].t()) * (x @ t[f"{pre}e{e}.up"].t())) @ t[f"{pre}e{e}.down"].t()
        out[tok] += w[tok, place].unsqueeze(-1) * y
    return out


def token_input(x, e, t, pre, eps):
    y = (gelu_tanh(x @ t[pre + "gate"].t()) * e) @ t[pre + "proj"].t()
    return x + rms(y, eps) * t[pre + "norm"]


def mixer(h, t, pre, spec, eps):
    m = spec["mixer"]
    if spec["type"] == "attention":
        return attention_mixer(h, t, pre, m, eps)
    return m["left_scale"] * left_mixer(h, t, pre + "left.", m["left"]) + m["right_scale"] * right_mixer(h, t, pre + "right.", m["right"], eps)


def feed_forward(h, t, pre, mlp):
    return capped_swiglu(h, t, pre, mlp["limit"]) if mlp["kind"] == "dense" else experts(h, t, pre, mlp)


def layer_order(cfg):
    """(layer, whether the embedding output is added in front of it) in the order of execution."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    body = list(range(lp["start"], lp["stop"]))
    order = [(i, False) for i in range(lp["start"])]
    for p in range(lp["times"]):
        order += [(i, p > 0 and i == body[0]) for i in body]
    return order + [(i, False) for i in range(lp["stop"], n)]


def forward(model, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of a whole sequence; ``capture`` (a list) receives the stream after every layer run."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["t"].items()}
    eps, dim = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    first = t["embed"][ids] * cfg["embedding"]["scale"]
    side = t["side.embed"][ids]
    x = first
    for i, again in layer_order(cfg):
        pre, spec = f"l{i}.", cfg["layers"][i]
        if again:
            x = x + first
        y = mixer(rms(x, eps) * t[pre + "norm1"], t, pre + "mix.", spec, eps)
        if spec.get("mlp"):
            y = y + feed_forward(rms(x, eps) * t[pre + "norm2"], t, pre + "mlp.", spec["mlp"])
        x = token_input(x + y, side[:, i * dim: (i + 1) * dim], t, pre + "side.", eps)
        if capture is not None:
            capture.append(x.clone())
    return (rms(x, eps) * t["final.norm"]) @ t["head"].t()
