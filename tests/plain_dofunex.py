"""Plain, slow statement of the Dofunex design, one function per mechanism, in the precision of its inputs: no cache, no batching, a
sequence in, the logits (and the residual rows after every layer run) out. Shares no code with the package; the tests compare the
engine with it.

`cfg` is the parsed config.json, `w` maps tensor names to tensors.
"""
import math

import torch


# ---- shared pieces -------------------------------------------------------------------------------------------------------

def rms(x, eps):
    """Divide rows by their root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---- attention with positions, key values, normed queries and keys, a sink --------------------------------------------------

def frequencies(rot, dtype=torch.float64):
    """Angle per position of every rotated pair, long wavelengths stretched by `scaling`."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=dtype)


def rotate(x, freq):
    """x [n, heads, dim], row = position: pairs (0, 1), (2, 3), ... of the first 2 len(freq) columns turn by position * freq."""
    n, d = x.shape[0], 2 * freq.numel()
    a = torch.arange(n, dtype=freq.dtype)[:, None] * freq[None, :]
    c, s = a.cos().to(x.dtype)[:, None, :], a.sin().to(x.dtype)[:, None, :]
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    out = x.clone()
    out[..., 0:d:2] = u * c - v * s
    out[..., 1:d:2] = v * c + u * s
    return out


def sink_softmax(scores, sink):
    """scores [heads, n, n] -> weights over the keys 0 .. i; exp(sink[h]) is part of every denominator."""
    n = scores.shape[-1]
    seen = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    s = scores.masked_fill(~seen, -math.inf)
    s = torch.cat([s, sink[:, None, None].expand(-1, n, 1)], -1)
    return torch.softmax(s, -1)[..., :n]


def attention(m, w, p, h, eps):
    """m: the layer's sizes; p: prefix of its tensors."""
    H, G, D, n = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    q = (h @ w[p + "q"].t() + w[p + "q.b"]).reshape(n, H, D)
    k = (h @ w[p + "k"].t() + w[p + "k.b"]).reshape(n, G, D)
    v = k
    if m.get("rot"):
        f = frequencies(m["rot"])
        q, k = rotate(q, f), rotate(k, f)
    q, k = rms(q, eps), rms(k, eps)
    own = [j // (H // G) for j in range(H)]
    scores = torch.einsum("ihd,jhd->hij", q, k[:, own]) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", sink_softmax(scores, w[p + "sink"]), v[:, own])
    return o.reshape(n, H * D) @ w[p + "o"].t() + w[p + "o.b"]


# ---- delta rule with a decay per key channel --------------------------------------------------------------------------------

def short_conv(x, taps):
    """x [n, channels], taps [channels, K]: y[t] = sum_j taps[:, j] x[t - (K - 1) + j]."""
    n, K = x.shape[0], taps.shape[1]
    xp = torch.cat([x.new_zeros(K - 1, x.shape[1]), x])
    return sum(xp[j:j + n] * taps[:, j] for j in range(K))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decays(h, w, p, heads, dim):
    """Factor of every state row, [n, heads, dim]."""
    z = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "dt_bias"]
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(-1, heads, dim))


def delta_scan(q, k, v, beta, g):
    """q, k, g [n, heads, dim], v [n, heads, vdim], beta [n, heads] -> reads [n, heads, vdim], from a zero state."""
    n, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    out = []
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_delta(m, w, p, h, eps):
    H, G, D, V, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(short_conv(h @ w[p + c].t(), w[p + c + ".conv"])) for c in "qkv")
    own = [j // (H // G) for j in range(H)]
    q, k = unit(q.reshape(n, G, D))[:, own] * D ** -0.5, unit(k.reshape(n, G, D))[:, own]
    o = delta_scan(q, k, v.reshape(n, H, V), sigmoid(h @ w[p + "b"].t()), decays(h, w, p, H, D))
    o = rms_norm(o, w[p + "norm"], eps) * sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t()).reshape(n, H, V)
    return o.reshape(n, H * V) @ w[p + "o"].t()


# ---- model ---------------------------------------------------------------------------------------------------------------

def feed_forward(w, p, h):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


MIXERS = {"attention": attention, "channel_delta": channel_delta}


def layer(cfg, w, i, x):
    e, p, eps, m = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["residual_mult"]
    y = MIXERS[e["type"]](e["mixer"], w, p + "mix.", rms_norm(x, w[p + "norm1"], eps), eps)
    x = x + m * rms_norm(y, w[p + "norm1b"], eps)
    if e.get("mlp"):
        x = x + m * rms_norm(feed_forward(w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
    return x


def order(cfg):
    """(layer, number of the pass when the layer opens one, else None) in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(lp["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, dtype=torch.float64):
    """Returns (logits [n, vocab], residual rows after every layer run [runs, n, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    x = x0 = w["embed"][torch.tensor(list(tokens))]
    after = []
    for i, t in order(cfg):
        if t is not None:
            x = torch.cat([x, x0], -1) @ w["loop.in"].t() + w["loop.step"][t]
        x = layer(cfg, w, i, x)
        after.append(x)
    return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].t() * cfg["logit_scale"], torch.stack(after)


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, w, seq)[0][-1].argmax()))
    return seq[len(prompt):]
