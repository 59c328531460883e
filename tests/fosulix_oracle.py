"""Plain, slow statement of the Fosulix design in float64, one function per mechanism.  Works on a whole sequence at once, no
cache, no padding, one query or token at a time; shares no code with the package."""

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ----------------------------------------------------------------------------------------- input convolution
def short_conv(h, weight):
    """h [T, C], weight [C, taps]: a causal sum over the last ``taps`` rows on every channel, zeros in front of the first row;
    the last tap meets the row itself."""
    taps = weight.shape[1]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += weight[:, j] * h[s]
    return out


# ---------------------------------------------------------------------------------------------- positions
def frequencies(rot):
    """Radians per position of every pair, and the factor on both cosine and sine."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def turns(t):
        """Pair index at which ``original`` positions make ``t`` turns."""
        return dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / s["factor"] * slow + v * (1.0 - slow))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot, first=0):
    """x [T, heads, d]: pairs (2 i, 2 i + 1) of the first ``dims`` columns turn by position times frequency."""
    f, size = frequencies(rot)
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(rot["dims"] // 2):
            a = float((first + t) * f[i])
            c, s = math.cos(a) * size, math.sin(a) * size
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i], out[t, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------- attention
def attend(q, k, v, scale, *, window=None, first=0):
    """q [T, H, d] at positions ``first ..``, k [N, H, d], v [N, H, e] -> [T, H, e]."""
    out = []
    for t in range(q.shape[0]):
        i = first + t
        lo = 0 if window is None else max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[t], k[lo:i + 1]) * scale
        out.append(torch.einsum("hj,jhe->he", torch.softmax(s, -1), v[lo:i + 1]))
    return torch.stack(out)


def latent_rows(h, w, p, m, eps):
    """What a layer with a projection of its own caches: latents [T, R] and the rotated key part [T, r] all heads share."""
    y = h @ w[p + "dkv"].T
    R = m["kv_rank"]
    return rms(y[:, :R], eps) * w[p + "dkv.norm"], rotate(y[:, None, R:], m["rot"])[:, 0]


def latent_attention(h, w, p, m, eps, shared):
    T, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"])], -1)
    c, kr = latent_rows(h, w, p, m, eps) if shared is None else shared
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr[:, None].expand(T, H, r)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    o = attend(q, k, v, m["scale"], window=(m.get("mask") or {}).get("size"))
    return o.reshape(T, -1) @ w[p + "o"].T, (c, kr)


# --------------------------------------------------------------------------------------------- recurrence
def forget(z, lower):
    return lower + (1.0 - lower) * sigmoid(z)


def recurrence(q, f, v, state=None):
    """q, f [T, H, n], v [T, H, m] -> outputs [T, H, m] and the state [H, n, m] behind the last token."""
    T, H, n = q.shape
    S = torch.zeros(H, n, v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnm,hn->hm", S, q[t]))
    return torch.stack(out), S


def gated_linear_attention(h, w, p, m, eps, shared):
    T, H, n = h.shape[0], m["heads"], m["dim"]
    q = silu(h @ w[p + "q"].T).view(T, H, n)
    f = forget(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).view(T, H, n)
    o, _ = recurrence(q, f, (h @ w[p + "v"].T).view(T, H, m["vdim"]))
    return (rms(o, eps) * w[p + "norm"]).reshape(T, -1) @ w[p + "o"].T, None


MIXERS = {"latent_attention": latent_attention, "hgrn2": gated_linear_attention}


# ------------------------------------------------------------------------------------------- feed-forward
def bounded_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, p, limit):
    return bounded_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def route(z, router):
    """Logits of one token -> [(expert, weight)]."""
    s = sigmoid(z).tolist()
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = len(s) // groups["count"]
    worth = [sum(sorted(s[g * size:(g + 1) * size])[-2:]) for g in range(groups["count"])]
    best = sorted(range(groups["count"]), key=lambda g: -worth[g])[:groups["keep"]]
    open_to = [e for e in range(len(s)) if e // size in best]
    return [(e, s[e] * router.get("scale", 1.0)) for e in sorted(open_to, key=lambda e: -s[e])[:router["top"]]]


def mixture(h, w, p, mlp):
    y = torch.zeros_like(h)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, weight in route(z[t], mlp["router"]):
            y[t] += weight * expert(h[t], w, f"{p}e{e}.", mlp["expert"]["limit"])
    return y


# -------------------------------------------------------------------------------------------------- model
def depth_average(rows, weight):
    """rows: the embedding and every layer's result so far, [T, W] each."""
    return sum(weight[j] * r for j, r in enumerate(rows))


def forward(tokens, weights, cfg):
    """Logits [T, vocab] and the averaged stream behind every layer [layers, T, width], float64."""
    w = {k: v.double() for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    rows, states, kept = [x], [], {}
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        h = rms(x, eps) * w[p + "norm1"]
        h = h + short_conv(h, w[p + "canon1"])
        source = m.get("kv_from")
        y, kept[i] = MIXERS[entry["type"]](h, w, p + "mix.", m, eps, None if source is None else kept[source])
        x = x + mult * y
        if entry["mlp"] is not None:
            x = x + mult * mixture(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", entry["mlp"])
        rows.append(x)
        x = depth_average(rows, w[p + "dwa"])
        states.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T, torch.stack(states)
