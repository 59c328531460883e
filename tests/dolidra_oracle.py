"""Plain, slow statement of the Dolidra design in float64, one function per mechanism.  Works on a whole sequence at
once, no cache, no padding, one query at a time; shares no code with the package."""

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps):
    return rms(x, eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


# ---------------------------------------------------------------------------------------------- positions
def frequencies(rot):
    """Radians per position of every rotated pair, with the three-band scaling when one is given."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s is not None:
            turns = s["original"] * f / (2.0 * math.pi)   # full turns over the original context
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                t = (turns - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, rot, first=0):
    """x [T, heads, dim]: pair (i, i + dims / 2) of the first ``dims`` columns turns by position times frequency."""
    half = rot["dims"] // 2
    angle = (first + torch.arange(x.shape[0], dtype=torch.float64))[:, None] * frequencies(rot)
    c, s = angle.cos()[:, None], angle.sin()[:, None]
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


# ---------------------------------------------------------------------------------------------- attention
def visible(i, window, keep_first=0):
    """Key positions that query position ``i`` sees."""
    return [j for j in range(i + 1) if i - j < window or j < keep_first]


def masked_attention(q, k, v, scale, window, keep_first=0, first=0):
    """q [T, H, d] at positions ``first ..``, k [N, G, d], v [N, G, e] -> [T, H, e]."""
    share = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, 1), v.repeat_interleave(share, 1)
    out = []
    for i in range(q.shape[0]):
        seen = visible(first + i, window, keep_first)
        s = torch.einsum("hd,jhd->hj", q[i], k[seen]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append(torch.einsum("hj,jhe->he", e / e.sum(-1, keepdim=True), v[seen]))
    return torch.stack(out)


def difference_weight(w, p, diff):
    dot = lambda a, b: float((w[p + a] * w[p + b]).sum())  # noqa: E731
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, p, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = linear(h, w, p + "q").view(T, H, 2, d)
    k = linear(h, w, p + "k").view(T, G, 2, d)
    v = linear(h, w, p + "v").view(T, G, m["vdim"])
    maps = [masked_attention(rotate(q[:, :, i], m["rot"]), rotate(k[:, :, i], m["rot"]), v, m["scale"], m["mask"]["size"])
            for i in range(2)]
    o = combine_maps(maps[0], maps[1], difference_weight(w, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, -1) @ w[p + "o"].T


def gated_attention(h, w, p, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = norm(linear(h, w, p + "q"), w[p + "q.norm"], eps).view(T, H, d)
    k = norm(linear(h, w, p + "k"), w[p + "k.norm"], eps).view(T, G, d)
    v = linear(h, w, p + "v").view(T, G, m["vdim"])
    o = masked_attention(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    o = o * sigmoid(linear(h, w, p + "g"))[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


MIXERS = {"attention": differential_attention, "attention_2": gated_attention}


# ------------------------------------------------------------------------------------------- feed-forward
def glu(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w_router, top):
    """For every token: [(expert, weight)], the largest logits with the softmax over those alone."""
    out = []
    for z in h @ w_router.T:
        best = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
        e = [math.exp(float(z[b] - z[best[0]])) for b in best]
        out.append([(b, x / sum(e)) for b, x in zip(best, e)])
    return out


def mixture(h, w, p, mlp):
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(h, w[p + "router"], mlp["router"]["top"])):
        for e, weight in chosen:
            y[t] += weight * glu(h[t], w, f"{p}e{e}.", silu)
    if mlp.get("shared"):
        y = y + glu(h, w, p + "shared.", silu)
    return y


def feed_forward(h, w, p, mlp):
    return glu(h, w, p, gelu_tanh) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# -------------------------------------------------------------------------------------------------- layers
def token_side(x, tokens, w, i, cfg):
    """What the layer's own token table adds to the stream."""
    p, dim = f"l{i}.side.", cfg["token_side"]["dim"]
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    g = gelu_tanh(x @ w[p + "gate"].T) * e
    return norm(g @ w[p + "proj"].T, w[p + "norm"], cfg["norm"]["eps"])


def layer(x, tokens, w, i, cfg):
    p, eps = f"l{i}.", cfg["norm"]["eps"]
    entry = cfg["layers"][i]
    y = MIXERS[entry["type"]](norm(x, w[p + "norm1"], eps), w, p + "mix.", entry["mixer"], eps)
    x = x + norm(y, w[p + "norm1b"], eps)
    if entry["mlp"] is not None:
        y = feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.", entry["mlp"])
        x = x + norm(y, w[p + "norm2b"], eps)
    return x + token_side(x, tokens, w, i, cfg)


def layer_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    return (list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n)))


def forward(tokens, weights, cfg):
    """Logits [T, vocab] and the stream after every layer run [runs, T, width], float64."""
    w = {k: v.double() for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens]
    states = []
    for i in layer_order(cfg):
        x = layer(x, tokens, w, i, cfg)
        states.append(x)
    return norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T, torch.stack(states)
