"""Plain, slow reference of models described layer by layer (lightning attention, windowed attention with kept first tokens and a
learned distance bias, looped layers): one function per mechanism, whole sequences at a time, nothing shared with the product code.

Every function works in the dtype of its inputs (the tests use float64).  ``model`` is a dict: ``config`` (the parsed config.json) and
``t`` (tensor name -> tensor)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def distance_bucket(n, buckets, bias_max):
    """Bucket of the distance n >= 0: exact below half of the buckets, then logarithmic up to bias_max."""
    half = buckets // 2
    if n < half:
        return n
    x = math.log(n / half) / math.log(bias_max / half) * (buckets - half)
    if abs(x - round(x)) < 1e-9:            # a bucket's first distance is hit exactly
        x = round(x)
    return min(buckets - 1, half + math.floor(x))


def visible(i, j, size, keep_first):
    """Whether position i sees position j: a causal window plus the first tokens of the sequence."""
    return j <= i and (size is None or i - j < size or j < keep_first)


def lightning_recurrence(q, k, v, decay, state=None):
    """q, k [T, H, D], v [T, H, E]: S <- decay_h S + k v^T, o = S^T q.  Returns (o [T, H, E], state [H, D, E])."""
    t, h, d = q.shape
    s = torch.zeros(h, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    dec = torch.as_tensor(decay, dtype=q.dtype).reshape(h, 1, 1)
    out = []
    for i in range(t):
        s = dec * s + k[i].unsqueeze(-1) * v[i].unsqueeze(1)
        out.append((s * q[i].unsqueeze(-1)).sum(1))
    return torch.stack(out), s


def lightning_mixer(h, t, pre, m, eps):
    hd, d, e = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ t[pre + "q"].t()).reshape(-1, hd, d)
    k = silu(h @ t[pre + "k"].t()).reshape(-1, hd, d)
    v = silu(h @ t[pre + "v"].t()).reshape(-1, hd, e)
    o, _ = lightning_recurrence(q, k, v, m["decay"])
    o = rms(o.reshape(-1, hd * e), eps) * t[pre + "norm"]
    return (o / (1 + torch.exp(-(h @ t[pre + "g"].t())))) @ t[pre + "o"].t()


def attention_core(q, k, v, scale, rel, bias_max, size, keep_first):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]: softmax over the visible keys of (q . k) scale + rel[bucket(i - j), h]."""
    t, hq, _ = q.shape
    g = hq // k.shape[1]
    idx = torch.arange(t)
    dist = idx.unsqueeze(1) - idx.unsqueeze(0)
    see = torch.tensor([[visible(i, j, size, keep_first) for j in range(t)] for i in range(t)])
    bk = torch.tensor([distance_bucket(n, rel.shape[0], bias_max) for n in range(t)]) if rel is not None else None
    out = torch.empty(t, hq, v.shape[2], dtype=q.dtype)
    for h in range(hq):
        s = (q[:, h] @ k[:, h // g].t()) * scale
        if rel is not None:
            s = s + rel[bk[dist.clamp_min(0)], h]
        s = s.masked_fill(~see, float("-inf"))
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h // g]
    return out


def attention_mixer(h, t, pre, m, eps):
    hq, hk, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ t[pre + "q"].t() + t[pre + "q.b"]).reshape(-1, hq, d), eps)
    k = rms((h @ t[pre + "k"].t() + t[pre + "k.b"]).reshape(-1, hk, d), eps)
    v = (h @ t[pre + "v"].t() + t[pre + "v.b"]).reshape(-1, hk, e)
    mask = m["mask"]
    o = attention_core(q, k, v, m["scale"], t[pre + "rel"], m["bias_max"], mask["size"], mask["keep_first"])
    return o.reshape(-1, hq * e) @ t[pre + "o"].t()


def feed_forward(h, t, pre):
    return (gelu_tanh(h @ t[pre + "gate"].t()) * (h @ t[pre + "up"].t())) @ t[pre + "down"].t()


def layer_runs(config):
    """(layer, pass number at whose start this run stands or None) in the order of execution."""
    n = len(config["layers"])
    lp = config.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(lp["start"])]
    for p in range(lp["times"]):
        runs += [(i, p if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, None) for i in range(lp["stop"], n)]


def forward(model, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of a whole sequence; ``capture`` (a list) receives the stream after every layer run."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["t"].items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for li, step in layer_runs(cfg):
        spec, pre = cfg["layers"][li], f"l{li}."
        if step is not None:
            x = x + t["loop.step"][step]
        mixer = {"lightning": lightning_mixer, "attention": attention_mixer}[spec["type"]]
        x = x + mixer(norm_zero_centred(x, t[pre + "norm1"], eps), t, pre + "mix.", spec["mixer"], eps)
        if spec.get("mlp"):
            x = x + feed_forward(norm_zero_centred(x, t[pre + "norm2"], eps), t, pre + "mlp.")
        if capture is not None:
            capture.append(x.clone())
    return (norm_zero_centred(x, t["final.norm"], eps) @ t["embed"].t()) * cfg["logit_scale"]
