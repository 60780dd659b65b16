"""The Rakizen design stated plainly: one function per mechanism, whole sequences at once, no cache, no batch, float64 unless the
caller passes something else. Shares no code with the package."""
import math

import torch


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def layer_norm(x, w, b, eps):
    """Mean off, divided by the root of the mean squared deviation (eps inside the root), times w, plus b."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def rotate(x, base, dims, positions=None):
    """x [tokens, heads, dim]: pairs (0, 1), (2, 3), ... of the first `dims` columns turned by position * base^(-2i / dims)."""
    n = x.shape[0]
    pos = torch.arange(n, dtype=torch.float64) if positions is None else positions.double()
    out = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def chunk_mask(n, size):
    """[row, key]: the key is not later than the row and in the row's chunk, chunks counted from position 0."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (j <= i) & (i // size == j // size)


def window_mask(n, size):
    """[row, key]: the row itself and the size - 1 tokens before it."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (i - j >= 0) & (i - j < size)


def capped(scores, cap):
    return cap * torch.tanh(scores / cap)


def attend(q, k, v, mask, scale, cap):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]: query head h over key head h // (H / G), softmax over what the mask shows."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = capped(q[:, h] @ k[:, g].t() * scale, cap).masked_fill(~mask, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def difference(a1, a2, lam, diff, eps):
    """The two maps' outputs per head [n, H, e]: their weighted difference, divided by its root mean square, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def route(z, top, groups, keep, scale):
    """Router logits [experts] -> [(expert, weight)]: the `top` best sigmoid scores among the `keep` groups whose two best scores sum
    highest, divided by their sum and scaled."""
    s = torch.sigmoid(z)
    per = len(s) // groups
    of_group = [sum(sorted(s[g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: -of_group[g])[:keep]
    allowed = [e for e in range(len(s)) if e // per in best]
    chosen = sorted(allowed, key=lambda e: -float(s[e]))[:top]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return [(e, float(s[e]) / total * scale) for e in chosen]


def gated_mlp(h, gate, up, down):
    return (silu(h @ gate.t()) * (h @ up.t())) @ down.t()


# ---- sublayers ----------------------------------------------------------------------------------------------------------

def difference_attention(m, w, p, h, eps):
    """Mixer type "attention": two maps per head over shared values, chunked, no positions, gated output."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].t()).view(n, H, 2, d)
    k = (h @ w[p + "k"].t()).view(n, G, 2, d)
    v = (h @ w[p + "v"].t()).view(n, G, e)
    mask = chunk_mask(n, m["mask"]["size"])
    a = [attend(q[:, :, j], k[:, :, j], v, mask, m["scale"], m["softcap"]) for j in (0, 1)]
    lam = difference_weight(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    o = difference(a[0], a[1], lam, m["diff"], eps).reshape(n, H * e)
    return (o * torch.sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def window_attention(m, w, p, h, eps):
    """Mixer type "attention_2": queries and keys normed over the whole projection, rotated, a sliding window."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].t(), eps) * w[p + "q.norm"]).view(n, H, d)
    k = (rms(h @ w[p + "k"].t(), eps) * w[p + "k.norm"]).view(n, G, d)
    v = (h @ w[p + "v"].t()).view(n, G, e)
    q, k = rotate(q, m["rot"]["base"], m["rot"]["dims"]), rotate(k, m["rot"]["base"], m["rot"]["dims"])
    o = attend(q, k, v, window_mask(n, m["mask"]["size"]), m["scale"], m["softcap"])
    return o.reshape(n, H * e) @ w[p + "o"].t()


def experts(f, w, p, h):
    """Every token through its chosen experts."""
    r = f["router"]
    out = torch.zeros_like(h)
    z = h @ w[p + "router"].t()
    for t in range(h.shape[0]):
        for e, g in route(z[t], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"]):
            out[t] += g * gated_mlp(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    return out


MIXERS = {"attention": difference_attention, "attention_2": window_attention}


# ---- model --------------------------------------------------------------------------------------------------------------

def order(cfg):
    """Layer numbers as they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg, weights, ids, dtype=torch.float64):
    """(logits [n, vocab], residual rows after every layer run)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(ids)]
    after = []
    for i in order(cfg):
        l, p = cfg["layers"][i], f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        y = MIXERS[l["type"]](l["mixer"], w, p + "mix.", h, eps)
        f = l["mlp"]
        if f and f["kind"] == "dense":
            y = y + gated_mlp(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
        elif f:
            y = y + experts(f, w, p + "mlp.", h)
        x = x + y
        after.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].t(), after


def greedy(cfg, weights, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, weights, ids)[0][-1].argmax()))
    return ids[len(prompt):]
