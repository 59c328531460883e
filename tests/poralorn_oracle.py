"""Plain, slow statement of the Poralorn design in float64, one function per mechanism.  Works on a whole sequence
at once, no cache, no padding, no absorption; shares no code with the package."""

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    return rms(x, eps) * gain


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_exact(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def latent(h, w_dkv, weight, eps):
    return rms(h @ w_dkv.T, eps) * weight


def causal_softmax_attention(q, k, v, scale):
    """q, k [T, H, d], v [T, H, e] -> [T, H, e]; one query at a time."""
    out = []
    for i in range(q.shape[0]):
        s = torch.einsum("hd,jhd->hj", q[i], k[: i + 1]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        p = e / e.sum(-1, keepdim=True)
        out.append(torch.einsum("hj,jhe->he", p, v[: i + 1]))
    return torch.stack(out)


def latent_attention(h, w, p, mixer, eps):
    T, H = h.shape[0], mixer["heads"]
    q = (h @ w[p + "q"].T).view(T, H, mixer["dim"])
    c = latent(h, w[p + "dkv"], w[p + "dkv.norm"], eps)
    k = (c @ w[p + "uk"].T).view(T, H, mixer["dim"])
    v = (c @ w[p + "uv"].T).view(T, H, mixer["vdim"])
    o = causal_softmax_attention(q, k, v, mixer["scale"]).reshape(T, -1)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h, w, p):
    return gelu_exact(h @ w[p + "up"].T) @ w[p + "down"].T


def gated(y, h, w, name):
    return y * sigmoid(h @ w[name].T + w[name + ".b"])


def layer(x, w, i, cfg):
    p, eps = f"l{i}.", cfg["norm"]["eps"]
    entry = cfg["layers"][i]
    h = scalar_norm(x, w[p + "norm1"], eps)
    delta = gated(latent_attention(h, w, p + "mix.", entry["mixer"], eps), h, w, p + "rg1")
    if entry["mlp"] is not None:
        h = scalar_norm(x, w[p + "norm2"], eps)
        delta = delta + gated(feed_forward(h, w, p + "mlp."), h, w, p + "rg2")
    return x + cfg["residual_mult"] * delta


def loop_input(x, x0, w, t):
    return torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


def softcap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(tokens, weights, cfg):
    """Logits [T, vocab] and the stream after every layer run [runs, T, width], float64."""
    w = {k: v.double() for k, v in weights.items()}
    x0 = x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    states = []
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    for i in range(loop["start"]):
        x = layer(x, w, i, cfg)
        states.append(x)
    for t in range(loop["times"]):
        x = loop_input(x, x0, w, t)
        for i in range(loop["start"], loop["stop"]):
            x = layer(x, w, i, cfg)
            states.append(x)
    for i in range(loop["stop"], len(cfg["layers"])):
        x = layer(x, w, i, cfg)
        states.append(x)
    logits = scalar_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    return softcap(logits, cfg["logit_softcap"]), torch.stack(states)


def greedy(prompt, n, weights, cfg):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(tokens, weights, cfg)[0][-1].argmax()))
    return tokens[len(prompt):]
