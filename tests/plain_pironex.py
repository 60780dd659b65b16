"""The Pironex design stated plainly: one function per mechanism, whole sequences at once, no cache, no batch, float64 unless the
caller passes something else. Shares no code with the package."""
import math

import torch


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def layer_norm(x, w, eps):
    """Mean off, divided by the root of the mean squared deviation (eps inside the root), times w."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x, w):
    """x [tokens, channels], w [channels, taps]: the last column meets the row itself, zeros before the first row."""
    out = torch.zeros_like(x)
    taps = w.shape[1]
    for j in range(taps):
        back = taps - 1 - j
        if back < x.shape[0]:
            out[back:] += x[:x.shape[0] - back] * w[:, j]
    return out


def input_conv(h, w):
    return h + causal_conv(h, w)


def depth_average(xs, w):
    """Weighted sum over the embedding output and the results of the layers so far."""
    return sum(w[j] * x for j, x in enumerate(xs))


def silu(z):
    return z * torch.sigmoid(z)


def turn(u, v, base, dims, i, positions):
    a = positions * base ** (-2.0 * i / dims)
    c, s = torch.cos(a).to(u.dtype)[:, None], torch.sin(a).to(u.dtype)[:, None]
    return u * c - v * s, v * c + u * s


def rotate_half(x, base, dims, positions=None):
    """x [tokens, heads, dim]: column i turned with column i + dims / 2, the columns from `dims` on stay."""
    pos = torch.arange(x.shape[0], dtype=torch.float64) if positions is None else positions.double()
    out = x.clone()
    for i in range(dims // 2):
        out[..., i], out[..., i + dims // 2] = turn(x[..., i], x[..., i + dims // 2], base, dims, i, pos)
    return out


def rotate_pairs(x, base, dims, positions=None):
    """x [tokens, heads, dim]: column 2 i turned with column 2 i + 1."""
    pos = torch.arange(x.shape[0], dtype=torch.float64) if positions is None else positions.double()
    out = x.clone()
    for i in range(dims // 2):
        out[..., 2 * i], out[..., 2 * i + 1] = turn(x[..., 2 * i], x[..., 2 * i + 1], base, dims, i, pos)
    return out


def window_mask(n, size):
    """[row, key]: the row itself and the size - 1 tokens before it."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (i - j >= 0) & (i - j < size)


def block_means(x, pool):
    """x [n, heads, d] -> [n // pool, heads, d]: means over whole blocks of `pool` rows."""
    b = x.shape[0] // pool
    return x[:b * pool].reshape(b, pool, *x.shape[1:]).mean(1)


def block_mask(n, size, pool):
    """[row, block]: the block's last token has left the row's window."""
    i, b = torch.arange(n)[:, None], torch.arange(n // pool)[None]
    return b * pool + pool - 1 <= i - size


def capped(scores, cap):
    return cap * torch.tanh(scores / cap) if cap else scores


def pooled_attention(q, k, v, size, pool, scale, cap):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]: a window of tokens and the means of the blocks before it in one softmax."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    keys, values = torch.cat([k, block_means(k, pool)]), torch.cat([v, block_means(v, pool)])
    mask = torch.cat([window_mask(n, size), block_mask(n, size, pool)], 1)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = capped(q[:, h] @ keys[:, g].t() * scale, cap).masked_fill(~mask, -math.inf)
        out.append(torch.softmax(s, -1) @ values[:, g])
    return torch.stack(out, 1)


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(h, gate, up, down, limit):
    return clamped_glu(h @ gate.t(), h @ up.t(), limit) @ down.t()


def route(z, top):
    """Router logits [experts] -> [(expert, weight)]: softmax over the `top` largest."""
    chosen = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    w = torch.softmax(z[chosen], 0)
    return [(e, w[j]) for j, e in enumerate(chosen)]


def ssm(x, B, C, dt, A_log, D):
    """x [n, heads, e], B, C [n, groups, N], dt [n, heads] (positive): y [n, heads, e] of the recurrence with a decay per head."""
    n, H, e = x.shape
    G = B.shape[1]
    S = torch.zeros(H, B.shape[2], e, dtype=x.dtype)
    own = [h // (H // G) for h in range(H)]
    out = []
    for t in range(n):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t][own][:, :, None] * x[t][:, None, :]
        out.append((S * C[t][own][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(out)


def group_norm_gated(y, z, w, groups, eps):
    """Gate first, then the root mean square of each of `groups` equal parts, then the weights."""
    y = y * silu(z)
    return rms(y.reshape(y.shape[0], groups, -1), eps).reshape(y.shape) * w


# ---- sublayers ----------------------------------------------------------------------------------------------------------

def attention(m, w, p, h, eps, shared):
    """Queries and keys normed over the whole projection and rotated; with `kv_from` the keys and values of that layer."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = rotate_half((rms(h @ w[p + "q"].t(), eps) * w[p + "q.norm"]).view(n, H, d), rot["base"], rot["dims"])
    if m.get("kv_from") is None:
        k = rotate_half((rms(h @ w[p + "k"].t(), eps) * w[p + "k.norm"]).view(n, G, d), rot["base"], rot["dims"])
        v = (h @ w[p + "v"].t()).view(n, G, e)
        shared[int(p[1:p.index(".")])] = (k, v)
    else:
        k, v = shared[m["kv_from"]]
    o = pooled_attention(q, k, v, m["mask"]["size"], m["mask"]["pool"], m["scale"], m.get("softcap"))
    return o.reshape(n, H * e) @ w[p + "o"].t()


def latent_attention(m, w, p, h, eps, shared):
    """Keys and values made out of one normed latent per token, beside one rotated key part for all heads."""
    n, H, d, r, e, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].t()).view(n, H, d + r)
    ckv = h @ w[p + "dkv"].t()
    c = rms(ckv[:, :L], eps) * w[p + "dkv.norm"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    kr = rotate_pairs(ckv[:, None, L:], base, dims)[:, 0]
    qr = rotate_pairs(q[..., d:], base, dims)
    k, v = (c @ w[p + "uk"].t()).view(n, H, d), (c @ w[p + "uv"].t()).view(n, H, e)
    mask = window_mask(n, m["mask"]["size"])
    out = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].t() + qr[:, i] @ kr.t()) * m["scale"]
        out.append(torch.softmax(s.masked_fill(~mask, -math.inf), -1) @ v[:, i])
    return torch.cat(out, 1) @ w[p + "o"].t()


def mamba2(m, w, p, h, eps, shared):
    n, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = torch.split(h @ w[p + "in"].t(), [inner, inner + 2 * G * N, H], 1)
    x, B, C = torch.split(silu(causal_conv(xbc, w[p + "conv"]) + w[p + "conv.b"]), [inner, G * N, G * N], 1)
    dt = dt + w[p + "dt_bias"]
    dt = torch.where(dt > 30, dt, torch.log1p(torch.exp(torch.clamp(dt, max=30.0))))
    y = ssm(x.view(n, H, e), B.view(n, G, N), C.view(n, G, N), dt, w[p + "A_log"], w[p + "D"])
    return (group_norm_gated(y.reshape(n, inner), z, w[p + "norm"], m["norm_groups"], eps)) @ w[p + "o"].t()


def feed_forward(f, w, p, h):
    out = torch.zeros_like(h)
    z = h @ w[p + "router"].t()
    for t in range(h.shape[0]):
        for e, g in route(z[t], f["router"]["top"]):
            out[t] += g * expert(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], f["expert"]["limit"])
    s = p + "shared."
    if f.get("shared"):
        out = out + torch.sigmoid(h @ w[s + "sg"].t()) * expert(h, w[s + "gate"], w[s + "up"], w[s + "down"], f["shared"]["limit"])
    return out


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mamba2": mamba2}


# ---- model --------------------------------------------------------------------------------------------------------------

def forward(cfg, weights, ids, dtype=torch.float64):
    """(logits [n, vocab], residual rows after every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(ids)] * cfg["embedding"]["scale"]
    xs, after, shared = [x], [], {}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_conv(layer_norm(x, w[p + "norm1"], eps), w[p + "canon1"])
        x = x + layer_norm(MIXERS[l["type"]](l["mixer"], w, p + "mix.", h, eps, shared), w[p + "norm1b"], eps)
        if l["mlp"]:
            h = input_conv(layer_norm(x, w[p + "norm2"], eps), w[p + "canon2"])
            x = x + layer_norm(feed_forward(l["mlp"], w, p + "mlp.", h), w[p + "norm2b"], eps)
        xs.append(x)
        x = depth_average(xs, w[p + "dwa"])
        after.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].t(), after


def greedy(cfg, weights, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, weights, ids)[0][-1].argmax()))
    return ids[len(prompt):]
