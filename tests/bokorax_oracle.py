"""Plain, slow statement of the Bokorax design in float64, one function per mechanism.  Works on a whole sequence at
once, no cache, no padding, one query or token at a time; shares no code with the package."""

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def norm_around_zero(x, weight, eps):
    """The stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + weight)


# ---------------------------------------------------------------------------------------------- positions
def frequencies(rot):
    """Radians per position of every rotated pair, all slowed down alike when a factor is given."""
    slow = (rot.get("scaling") or {"factor": 1.0})["factor"]
    return torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) / slow for i in range(rot["dims"] // 2)], dtype=torch.float64)


def rotate(x, rot, first=0):
    """x [T, heads, dim]: pair (i, i + dims / 2) of the first ``dims`` columns turns by position times frequency."""
    half = rot["dims"] // 2
    angle = (first + torch.arange(x.shape[0], dtype=torch.float64))[:, None] * frequencies(rot)
    c, s = angle.cos()[:, None], angle.sin()[:, None]
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


# ---------------------------------------------------------------------------------------------- attention
def capped(score, cap):
    return score if not cap else cap * torch.tanh(score / cap)


def attend(q, k, v, scale, *, window=None, cap=0.0, sink=None, first=0):
    """q [T, H, d] at positions ``first ..``, k [N, G, d], v [N, G, e] -> [T, H, e].  ``sink [H]``: a score that takes
    part in the denominator only."""
    share = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, 1), v.repeat_interleave(share, 1)
    out = []
    for t in range(q.shape[0]):
        i = first + t
        lo = 0 if window is None else max(0, i - window + 1)
        s = capped(torch.einsum("hd,jhd->hj", q[t], k[lo:i + 1]) * scale, cap)
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[:, None])
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[:, None] - top)
        out.append(torch.einsum("hj,jhe->he", e / total, v[lo:i + 1]))
    return torch.stack(out)


def tied_value_attention(h, w, p, m, eps, shared):
    """Windowed attention whose values are the keys as projected; norm over the whole query and key rows."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    raw = h @ w[p + "k"].T
    k = rms(raw, eps) * w[p + "k.norm"]
    kv = rotate(k.view(T, G, d), m["rot"]), raw.view(T, G, d)
    o = attend(rotate(q.view(T, H, d), m["rot"]), *kv, m["scale"], window=m["mask"]["size"])
    return o.reshape(T, -1) @ w[p + "o"].T, kv


def sink_attention(h, w, p, m, eps, shared):
    """Causal attention with per-head norms, capped scores, a sink and a gate per head; ``shared``: keys and values of
    another layer instead of its own."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rotate(rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"], m["rot"])
    if shared is None:
        k = rotate(rms((h @ w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"], m["rot"])
        shared = k, (h @ w[p + "v"].T).view(T, G, m["vdim"])
    o = attend(q, *shared, m["scale"], cap=m["softcap"], sink=w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T, shared


# --------------------------------------------------------------------------------------------- recurrence
def shifted(h):
    """The previous token's row, zeros in front of the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def decay(z, w, p):
    return torch.exp(-torch.exp(torch.tanh(z @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))


def recurrence(r, k, v, d, u, state=None):
    """r, k, d [T, H, n], v [T, H, m], u [H, n] -> outputs [T, H, m] and the state [H, n, m] behind the last token."""
    T, H, n = r.shape
    S = torch.zeros(H, n, v.shape[2], dtype=r.dtype) if state is None else state
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnm,hn->hm", S + u[:, :, None] * kv, r[t]))
        S = d[t][:, :, None] * S + kv
    return torch.stack(out), S


def time_mix(h, w, p, m, eps, shared):
    T, H, n = h.shape[0], m["heads"], m["dim"]
    mixed = {s: h + (shifted(h) - h) * w[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).view(T, H, n) for s in "rkv")
    o, _ = recurrence(r, k, v, decay(mixed["w"], w, p).view(T, H, n), w[p + "u"])
    return (rms(o, eps).reshape(T, -1) * w[p + "norm"] * silu(mixed["g"] @ w[p + "g"].T)) @ w[p + "o"].T, None


MIXERS = {"attention": tied_value_attention, "attention_2": sink_attention, "wkv": time_mix}


# ------------------------------------------------------------------------------------------- feed-forward
def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, router):
    """Logits of one token -> [(expert, weight)].  Chosen by score plus correction inside the best groups, weighted by
    the score alone."""
    s = torch.softmax(z, -1)
    choice = (s + correction).tolist()
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = len(choice) // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(choice[g * size:(g + 1) * size]))[:groups["keep"]]
    open_to = [e for e in range(len(choice)) if e // size in best]
    chosen = sorted(open_to, key=lambda e: -choice[e])[:router["top"]]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return [(e, float(s[e]) / total * router.get("scale", 1.0)) for e in chosen]


def mixture(h, w, p, mlp):
    y = torch.zeros_like(h)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, weight in route(z[t], w[p + "correction"], mlp["router"]):
            y[t] += weight * (glu(h[t], w, f"{p}e{e}.") if e < mlp["router"]["experts"] else h[t])
    if mlp.get("shared"):
        y = y + glu(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return y


# -------------------------------------------------------------------------------------------------- model
def forward(tokens, weights, cfg):
    """Logits [T, vocab] and the stream after every layer [layers, T, width], float64."""
    w = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    states, kept = [], {}
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        y, kept[i] = MIXERS[entry["type"]](x, w, p + "mix.", m, eps, kept.get(m.get("kv_from", -1)))
        x = x + norm_around_zero(y, w[p + "norm1"], eps)
        if entry["mlp"] is not None:
            x = x + norm_around_zero(mixture(x, w, p + "mlp.", entry["mlp"]), w[p + "norm2"], eps)
        states.append(x)
    return norm_around_zero(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"], torch.stack(states)
