"""Plain, slow statement of the latent-attention design with output norms ("Zototar"), one function per mechanism, in the
precision of its inputs. No cache, no batching: a sequence in, the logits (and the residual rows after every layer) out.
Shares no code with the package; the tests compare the engine with it.

`cfg` is the parsed config.json, `w` maps tensor names to tensors.
"""
import math

import torch


def rms(x, eps):
    """Divide rows by their root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token of a sequence that starts with tokens[0]."""
    rows = [buckets]
    for a, b in zip(tokens, tokens[1:]):
        rows.append((a * mul_prev + b * mul_cur) % buckets)
    return rows


def embed(cfg, w, tokens):
    e = cfg["embedding"]
    x = w["embed"][torch.tensor(tokens)] * e["scale"]
    if e.get("bigram"):
        b = e["bigram"]
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


def latent(h, w_dkv, norm_w, eps):
    """What the cache holds of a token."""
    return rms_norm(h @ w_dkv.t(), norm_w, eps)


def queries(h, w_dq, norm_w, w_uq, eps, heads, dim):
    return (rms_norm(h @ w_dq.t(), norm_w, eps) @ w_uq.t()).reshape(-1, heads, dim)


def causal_softmax(scores):
    """scores [heads, n, n]: row i over the keys 0 .. i."""
    n = scores.shape[-1]
    seen = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    return torch.softmax(scores.masked_fill(~seen, -math.inf), -1)


def attend(q, c, w_uk, w_uv, scale, heads, dim, vdim):
    """q [n, heads, dim], latents c [n, rank] -> [n, heads * vdim], keys and values written out."""
    k = (c @ w_uk.t()).reshape(-1, heads, dim)
    v = (c @ w_uv.t()).reshape(-1, heads, vdim)
    p = causal_softmax(torch.einsum("ihd,jhd->hij", q, k) * scale)
    return torch.einsum("hij,jhv->ihv", p, v).reshape(q.shape[0], heads * vdim)


def mixer(cfg, w, i, h, latents):
    m, p, eps = cfg["layers"][i]["mixer"], f"l{i}.mix.", cfg["norm"]["eps"]
    if m.get("kv_from") is None:
        latents[i] = latent(h, w[p + "dkv"], w[p + "dkv.norm"], eps)
        c = latents[i]
    else:
        c = latents[m["kv_from"]]
    q = queries(h, w[p + "dq"], w[p + "dq.norm"], w[p + "uq"], eps, m["heads"], m["dim"])
    return attend(q, c, w[p + "uk"], w[p + "uv"], m["scale"], m["heads"], m["dim"], m["vdim"]) @ w[p + "o"].t()


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def feed_forward(w, i, h):
    return relu_squared(h @ w[f"l{i}.mlp.up"].t()) @ w[f"l{i}.mlp.down"].t()


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, w, tokens, dtype=torch.float64):
    """Returns (logits [n, vocab], residual rows after every layer [layers, n, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(cfg, w, list(tokens))
    latents, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        x = x + rms_norm(mixer(cfg, w, i, x, latents), w[f"l{i}.norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(feed_forward(w, i, x), w[f"l{i}.norm2"], eps)
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].t()
    if cfg.get("logit_softcap"):
        logits = softcap(logits, cfg["logit_softcap"])
    return logits, torch.stack(after)


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, w, seq)[0][-1].argmax()))
    return seq[len(prompt):]
