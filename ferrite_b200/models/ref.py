"""Plain PyTorch fp32 reference of every model family: the oracle for the CUDA kernels and the CPU path.

Numerics follow the reference's written conventions (the design notes of `crates/fe-xe`, lines 44-60): RMSNorm with (1 + w),
per-head q/k norm and partial RoPE with a sigmoid output gate on attention, Gated DeltaNet with a causal
depthwise conv (tap 0 = oldest), `g = exp(-exp(A_log) * softplus(a + dt_bias))`, `beta = sigmoid(b)`,
`S = S g; delta = (v - S^T k) beta; S += k (x) delta; y = S^T q`, gated RMSNorm `rmsnorm(y) * w * silu(z)`.
It processes one sequence token by token, holding its own KV / conv / recurrent state, so it is slow and
obviously right; the CPU oracles of the reference play the same role (`crates/fe-dsc/src/refmodel.rs`,
`crates/fe-exl3/src/cpu.rs`).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

from ..config import ModelConfig
from .weights import Weights, rope_frequencies


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, centred: bool = True) -> torch.Tensor:
    x = x.float()
    r = torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return x * r * ((1.0 + w.float()) if centred else w.float())


def rope_tables(positions: torch.Tensor, rotary_dim: int, theta: float) -> tuple:
    half = rotary_dim // 2
    inv = theta ** (-torch.arange(half, dtype=torch.float64) / half)
    ang = positions.double()[:, None] * inv[None, :]
    return ang.cos().float(), ang.sin().float()


def apply_rope(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, rotary_dim: int) -> torch.Tensor:
    """x: [rows, heads, hd]; rotate-half pairing (i, i + rotary_dim/2) over the first rotary_dim dims."""
    half = rotary_dim // 2
    a, b = x[..., :half], x[..., half:rotary_dim]
    c, s = cos[:, None, :], sin[:, None, :]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., rotary_dim:]], -1)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.where(x > 20, x, torch.log1p(torch.exp(torch.clamp(x, max=20.0))))


def swiglu(gu: torch.Tensor) -> torch.Tensor:
    i = gu.shape[-1] // 2
    return F.silu(gu[..., :i]) * gu[..., i:]


def route(cfg: ModelConfig, logits: torch.Tensor, bias: Optional[torch.Tensor]):
    """Top-k routing. softmax: softmax over experts, top-k (ties to the lower id), renormalise.
    sigmoid_group: scores = sigmoid(logits); choice by scores + bias restricted to the best `topk_groups`
    groups (group score = sum of its top-2 biased scores); weights = picked scores / sum * route_scale
    (reference routers: `kernels/k-fnext/src/fast.rs:393`, `kernels/k-ds/src/moe.rs:11`)."""
    logits = logits.float()
    if cfg.router == "softmax":
        p = torch.softmax(logits, -1)
        val, idx = torch.sort(p, dim=-1, descending=True, stable=True)
        val, idx = val[..., :cfg.top_k], idx[..., :cfg.top_k]
        return idx, val / val.sum(-1, keepdim=True) * cfg.route_scale
    s = torch.sigmoid(logits)
    sb = s + (bias.float() if bias is not None else 0.0)
    n, e = sb.shape
    g = cfg.n_groups
    grp = sb.view(n, g, e // g)
    gscore = grp.topk(min(2, e // g), -1).values.sum(-1)
    _, gi = torch.sort(gscore, dim=-1, descending=True, stable=True)
    gmask = torch.zeros(n, g, dtype=torch.bool)
    gmask.scatter_(1, gi[:, :cfg.topk_groups], True)
    masked = torch.where(gmask[:, :, None].expand(n, g, e // g).reshape(n, e), sb, torch.full_like(sb, float("-inf")))
    _, idx = torch.sort(masked, dim=-1, descending=True, stable=True)
    idx = idx[:, :cfg.top_k]
    val = s.gather(1, idx)
    return idx, val / (val.sum(-1, keepdim=True) + 1e-20) * cfg.route_scale


class RefState:
    def __init__(self, cfg: ModelConfig):
        self.cfg = cfg
        self.pos = 0
        self.prev: Optional[int] = None          # last token (hashed bigram embeddings)
        self.k: List[List[torch.Tensor]] = [[] for _ in range(cfg.n_layers)]
        self.v: List[List[torch.Tensor]] = [[] for _ in range(cfg.n_layers)]
        self.conv = [torch.zeros(cfg.conv_dim, cfg.conv_k - 1) for _ in range(cfg.n_layers)]
        self.rec = [torch.zeros(cfg.lin_v_heads, cfg.lin_dk, cfg.lin_dv) for _ in range(cfg.n_layers)]
        self.run: Dict[tuple, object] = {}       # rows and states of the runs of listed layers, by (what, run)

    def clone(self) -> "RefState":
        s = RefState(self.cfg)
        s.pos, s.prev = self.pos, self.prev
        s.k = [list(x) for x in self.k]
        s.v = [list(x) for x in self.v]
        s.conv = [x.clone() for x in self.conv]
        s.rec = [x.clone() for x in self.rec]
        s.run = {k: list(x) if isinstance(x, list) else x for k, x in self.run.items()}
        return s


class RefModel:
    """fp32 oracle. `forward(tokens, state)` appends the tokens to the sequence held by `state` and returns
    logits [len(tokens), vocab] (and the per-layer hidden taps when asked)."""

    def __init__(self, cfg: ModelConfig, weights: Weights):
        self.cfg = cfg
        self.w = {k: v.detach().float().cpu() for k, v in weights.items()}

    def new_state(self) -> RefState:
        return RefState(self.cfg)

    # ---- mixers ------------------------------------------------------------------------------------
    def _gdn(self, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        c, w = self.cfg, self.w
        p = f"l{i}."
        nk, nv, dk, dv = c.lin_k_heads, c.lin_v_heads, c.lin_dk, c.lin_dv
        proj = w[p + "in_proj"] @ x
        qkv, z, b, a = torch.split(proj, [c.conv_dim, nv * dv, nv, nv])
        win = torch.cat([st.conv[i], qkv[:, None]], 1)             # [conv_dim, conv_k], tap 0 oldest
        st.conv[i] = win[:, 1:].clone()
        qkv = F.silu((win * w[p + "conv_w"]).sum(1))
        q, k, v = torch.split(qkv, [nk * dk, nk * dk, nv * dv])
        q = q.view(nk, dk)
        k = k.view(nk, dk)
        v = v.view(nv, dv)
        q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + c.eps) / math.sqrt(dk)
        k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + c.eps)
        rep = nv // nk
        q = q.repeat_interleave(rep, 0)
        k = k.repeat_interleave(rep, 0)
        g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(a + w[p + "dt_bias"]))
        beta = torch.sigmoid(b)
        S = st.rec[i] * g[:, None, None]
        kv = torch.einsum("hkv,hk->hv", S, k)
        delta = (v - kv) * beta[:, None]
        S = S + torch.einsum("hk,hv->hkv", k, delta)
        st.rec[i] = S
        y = torch.einsum("hkv,hk->hv", S, q)
        y = rmsnorm(y, w[p + "gnorm_w"], c.eps, centred=False) * F.silu(z.view(nv, dv))
        return w[p + "out_proj"] @ y.reshape(-1)

    def _attn(self, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        c, w = self.cfg, self.w
        p = f"l{i}."
        hd, nq, nkv = c.head_dim, c.n_q, c.n_kv
        proj = w[p + "in_proj"] @ x
        qd = c.attn_q_dim
        qg = proj[:qd].view(nq, -1)
        q = qg[:, :hd]
        gate = qg[:, hd:] if c.attn_gate else None
        k = proj[qd:qd + nkv * hd].view(nkv, hd)
        v = proj[qd + nkv * hd:].view(nkv, hd)
        q = rmsnorm(q, w[p + "q_norm"], c.eps)
        k = rmsnorm(k, w[p + "k_norm"], c.eps)
        cos, sin = rope_tables(torch.tensor([st.pos]), c.rotary_dim, c.rope_theta)
        q = apply_rope(q[None], cos, sin, c.rotary_dim)[0]
        k = apply_rope(k[None], cos, sin, c.rotary_dim)[0]
        st.k[i].append(k)
        st.v[i].append(v)
        K = torch.stack(st.k[i], 0)                                # [T, nkv, hd]
        V = torch.stack(st.v[i], 0)
        grp = nq // nkv
        qh = q.view(nkv, grp, hd)
        s = torch.einsum("kgd,tkd->kgt", qh, K) / math.sqrt(hd)
        pr = torch.softmax(s, -1)
        o = torch.einsum("kgt,tkd->kgd", pr, V).reshape(nq, hd)
        if gate is not None:
            o = o * torch.sigmoid(gate)
        return w[p + "out_proj"] @ o.reshape(-1)

    def _mla(self, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        c, w = self.cfg, self.w
        p = f"l{i}."
        nq, dn, dr, dvh = c.n_q, c.nope_head_dim, c.rope_head_dim, c.v_head_dim
        qa = rmsnorm(w[p + "q_a"] @ x, w[p + "q_a_norm"], c.eps)
        q = (w[p + "q_b"] @ qa).view(nq, dn + dr)
        kva = w[p + "kv_a"] @ x
        lat = rmsnorm(kva[:c.kv_lora], w[p + "kv_a_norm"], c.eps)
        kr = kva[c.kv_lora:]
        cos, sin = rope_tables(torch.tensor([st.pos]), dr, c.rope_theta)
        qr = apply_rope(q[None, :, dn:], cos, sin, dr)[0]
        kr = apply_rope(kr[None, None, :], cos, sin, dr)[0, 0]
        st.k[i].append(lat)
        st.v[i].append(kr)
        L = torch.stack(st.k[i], 0)                                # [T, kv_lora]
        R = torch.stack(st.v[i], 0)                                # [T, dr]
        kvb = w[p + "kv_b"].view(nq, dn + dvh, c.kv_lora)
        kn = torch.einsum("hdl,tl->thd", kvb[:, :dn], L)
        vv = torch.einsum("hdl,tl->thd", kvb[:, dn:], L)
        s = (torch.einsum("hd,thd->ht", q[:, :dn], kn) + torch.einsum("hd,td->ht", qr, R)) / math.sqrt(dn + dr)
        pr = torch.softmax(s, -1)
        o = torch.einsum("ht,thd->hd", pr, vv)
        return w[p + "out_proj"] @ o.reshape(-1)

    def _latent(self, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        """Latent attention; a layer with `kv_from` reads the rows that layer appended for this token."""
        l, w, p, eps = self.cfg.layers[i], self.w, f"l{i}.", self.cfg.eps
        if not l.q_rank:
            return self._latent_rotated(i, x, st)
        q = (w[p + "q_b"] @ rmsnorm(w[p + "q_a"] @ x, w[p + "q_a_norm"], eps, False)).view(l.heads, l.dim)
        if l.kv_from is None:
            st.k[i].append(rmsnorm(w[p + "kv_a"] @ x, w[p + "kv_a_norm"], eps, False))
        lat = torch.stack(st.k[i if l.kv_from is None else l.kv_from], 0)                  # [T, kv_rank]
        k = (lat @ w[p + "k_b"].t()).view(-1, l.heads, l.dim)
        v = (lat @ w[p + "v_b"].t()).view(-1, l.heads, l.vdim)
        pr = torch.softmax(torch.einsum("hd,thd->ht", q, k) * l.scale, -1)
        return w[p + "out_proj"] @ torch.einsum("ht,thv->hv", pr, v).reshape(-1)

    def _latent_rotated(self, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        """Latent attention under a window with one rotated key part for all heads beside the latent."""
        l, w, p, R = self.cfg.layers[i], self.w, f"l{i}.", self.cfg.layers[i].rot_dims
        ang = st.pos * rope_frequencies(l)
        c, s = ang.cos().float(), ang.sin().float()
        turned = lambda z: torch.stack([z[..., 0::2] * c - z[..., 1::2] * s, z[..., 1::2] * c + z[..., 0::2] * s], -1).flatten(-2)
        q, kva = (w[p + "q"] @ x).view(l.heads, l.dim + R), w[p + "kv_a"] @ x
        st.k[i].append(rmsnorm(kva[:l.kv_rank], w[p + "kv_a_norm"], self.cfg.eps, False))
        st.v[i].append(turned(kva[l.kv_rank:]))
        first = max(0, st.pos - l.window + 1) if l.window else 0
        lat, kr = torch.stack(st.k[i][first:]), torch.stack(st.v[i][first:])
        k, v = (lat @ w[p + "k_b"].t()).view(-1, l.heads, l.dim), (lat @ w[p + "v_b"].t()).view(-1, l.heads, l.vdim)
        sc = torch.einsum("hd,thd->ht", q[:, :l.dim], k) + torch.einsum("hd,td->ht", turned(q[:, l.dim:]), kr)
        return w[p + "out_proj"] @ torch.einsum("ht,thv->hv", torch.softmax(sc * l.scale, -1), v).reshape(-1)

    def _ssm(self, r: int, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        """State-space recurrence with one decay per head; run r's state and convolution inputs are its own."""
        l, w, p = self.cfg.layers[i], self.w, f"l{i}."
        H, V, N, G = l.heads, l.vdim, l.dim, l.kv_heads
        z, xbc, dt = torch.split(w[p + "in"] @ x, [H * V, H * V + 2 * G * N, H])
        buf = st.run.setdefault(("xbc", r), [])
        buf.append(xbc)
        c = F.silu(sum(b * w[p + "xbc_conv"][:, l.conv - 1 - j] for j, b in enumerate(reversed(buf[-l.conv:]))) + w[p + "xbc_bias"])
        xs, B, C = torch.split(c, [H * V, G * N, G * N])
        own = torch.arange(H) // (H // G)
        xs, B, C, dt = xs.view(H, V), B.view(G, N)[own], C.view(G, N)[own], softplus(dt + w[p + "dt_bias"])
        S = st.run.get(("rec", r), torch.zeros(H, N, V)) * torch.exp(-torch.exp(w[p + "A_log"]) * dt)[:, None, None]
        S = st.run["rec", r] = S + (dt[:, None] * B)[:, :, None] * xs[:, None, :]
        y = (torch.einsum("hnv,hn->hv", S, C) + w[p + "skip"][:, None] * xs).reshape(-1) * F.silu(z)
        y = (y.view(l.norm_groups, -1) * torch.rsqrt(y.view(l.norm_groups, -1).pow(2).mean(-1, keepdim=True) + self.cfg.eps)).reshape(-1)
        return w[p + "out_proj"] @ (y * w[p + "gnorm_w"])

    def _gqa(self, r: int, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        """Grouped-query attention of listed layers; run r's keys and values are its own, or those of the layer it names."""
        l, w, p = self.cfg.layers[i], self.w, f"l{i}."
        own_kv = l.kv_from is None
        proj = {n: w[p + n] @ x + (w[p + n + "_bias"] if l.bias else 0.0)
                for n in ("q",) + (("k",) if own_kv else ()) + (("v",) if own_kv and not l.key_values else ())}
        if l.row_norm:
            proj.update({n: rmsnorm(proj[n], w[p + n + "_norm"], self.cfg.eps, False) for n in "qk" if n in proj})
        ang = st.pos * rope_frequencies(l)
        c, s = ang.cos().float(), ang.sin().float()

        def turned(z):
            z, half = z.clone(), l.rot_dims // 2
            u, v = (slice(0, half), slice(half, l.rot_dims)) if l.rot_half else (slice(0, l.rot_dims, 2), slice(1, l.rot_dims, 2))
            a, b = z[:, u].clone(), z[:, v].clone()
            z[:, u], z[:, v] = a * c - b * s, b * c + a * s
            return z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + self.cfg.eps) if l.qk_norm else z
        H, M = l.heads, l.maps
        q = turned(proj["q"].view(H * M, l.dim))
        if own_kv:
            k = proj["k"].view(l.kv_heads * M, l.dim)
            st.run.setdefault(("k", r), []).append(turned(k))
            st.run.setdefault(("v", r), []).append(k if l.key_values else proj["v"].view(l.kv_heads, l.vdim))
        else:
            r = max(x.index for x in self.cfg.layer_runs[:r] if x.layer == l.kv_from)
        own = torch.arange(H) // (H // l.kv_heads)
        first = max(0, st.pos - l.window + 1) if l.window else st.pos - st.pos % l.chunk if l.chunk else 0
        blocks = [slice(b * l.pool, (b + 1) * l.pool) for b in range(first // l.pool)] if l.pool else []
        seen = lambda rows: torch.stack([torch.stack(rows[b]).mean(0) for b in blocks] + rows[first:])
        K, V = seen(st.run["k", r]), seen(st.run["v", r])[:, own]
        maps = []
        for m in range(M):
            sc = torch.einsum("hd,thd->ht", q[m::M], K[:, m::M][:, own]) * l.scale
            e = torch.exp(l.softcap * torch.tanh(sc / l.softcap) if l.softcap else sc)
            pr = e / (e.sum(-1, keepdim=True) + (torch.exp(w[p + "sink"])[:, None] if l.sink else 0.0))
            maps.append(torch.einsum("ht,thd->hd", pr, V))
        o = maps[0]
        if M == 2:
            lam = torch.exp(w[p + "lq1"] @ w[p + "lk1"]) - torch.exp(w[p + "lq2"] @ w[p + "lk2"]) + l.diff
            o = o - lam * maps[1]
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + self.cfg.eps) * (1 - l.diff)
        if l.out_gate:
            o = o * torch.sigmoid(w[p + "g"] @ x).view(H, l.vdim)
        return w[p + "out_proj"] @ o.reshape(-1) + (w[p + "out_bias"] if l.bias else 0.0)

    def _cdelta(self, r: int, i: int, x: torch.Tensor, st: RefState) -> torch.Tensor:
        """Delta rule with a decay per key channel; run r's state and convolution inputs are its own."""
        l, w, p = self.cfg.layers[i], self.w, f"l{i}."
        H, G, D, V = l.heads, l.kv_heads, l.dim, l.vdim
        out = {}
        for n in "qkv":
            buf = st.run.setdefault((n + "_conv", r), [])
            buf.append(w[p + n] @ x)
            out[n] = F.silu(sum(z * w[p + n + "_conv"][:, l.conv - 1 - j] for j, z in enumerate(reversed(buf[-l.conv:]))))
        own = torch.arange(H) // (H // G)
        unit = lambda z: z * torch.rsqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6)
        q, k = unit(out["q"].view(G, D))[own] / math.sqrt(D), unit(out["k"].view(G, D))[own]
        g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * softplus(w[p + "a2"] @ (w[p + "a1"] @ x) + w[p + "dt_bias"]).view(H, D))
        S = st.run.get(("rec", r), torch.zeros(H, D, V)) * g[:, :, None]
        u = torch.sigmoid(w[p + "b"] @ x)[:, None] * (out["v"].view(H, V) - torch.einsum("hdv,hd->hv", S, k))
        S = st.run["rec", r] = S + k[:, :, None] * u[:, None, :]
        o = rmsnorm(torch.einsum("hdv,hd->hv", S, q), w[p + "gnorm_w"], self.cfg.eps, False)
        return w[p + "out_proj"] @ (o * torch.sigmoid(w[p + "g2"] @ (w[p + "g1"] @ x)).view(H, V)).reshape(-1)

    def _experts(self, i: int, h: torch.Tensor) -> torch.Tensor:
        """Routed feed-forward of listed layers."""
        l, w, p = self.cfg.layers[i], self.w, f"l{i}."
        if l.act == "clamped_glu":
            def expert(gate_up, down, limit):
                g, u = (gate_up @ h).chunk(2)
                g, u = g.clamp(max=limit), u.clamp(-limit, limit)
                return down @ (g * torch.sigmoid(1.702 * g) * (u + 1))
            val, idx = torch.sort(w[p + "router"] @ h, descending=True, stable=True)
            out = sum(g * expert(w[p + "experts_gate_up"][e], w[p + "experts_down"][e], l.limit)
                      for e, g in zip(idx[:l.top].tolist(), torch.softmax(val[:l.top], -1)))
            if l.shared_ff:
                out = out + torch.sigmoid(w[p + "shared_gate"] @ h) * expert(w[p + "shared_gate_up"][0], w[p + "shared_down"][0], l.shared_limit)
            return out
        rc = ModelConfig(router="sigmoid_group", top_k=l.top, n_groups=l.groups, topk_groups=l.keep_groups, route_scale=l.route_scale)
        idx, wt = route(rc, (w[p + "router"] @ h)[None], None)
        return sum(g * (w[p + "experts_down"][e] @ swiglu(w[p + "experts_gate_up"][e] @ h)) for e, g in zip(idx[0].tolist(), wt[0].tolist()))

    def _token_conv(self, t: int, st: RefState, tap: list) -> torch.Tensor:
        """One token through a model of layer norms, convolved operands and averages over depth: the row before the final norm."""
        c, w = self.cfg, self.w
        x = w["embed"][t] * c.embed_scale
        xs = [x]
        norm = lambda z, name: F.layer_norm(z, z.shape, w[name], None, c.eps)

        def operand(name, conv, key):
            h = norm(x, name)
            if not c.canon:
                return h
            buf = st.run.setdefault(key, [])
            buf.append(h)
            return h + sum(b * w[conv][:, c.canon - 1 - j] for j, b in enumerate(reversed(buf[-c.canon:])))
        for run in c.layer_runs:
            i, l, p, r = run.layer, c.layers[run.layer], f"l{run.layer}.", run.index
            h = operand(p + "pre_norm", p + "mix_canon", ("mix", r))
            y = self._latent(i, h, st) if l.mixer == "latent" else (self._gqa if l.mixer == "gqa" else self._ssm)(r, i, h, st)
            x = x + norm(y, p + "mix_norm")
            if l.ff:
                x = x + norm(self._experts(i, operand(p + "ffn_pre_norm", p + "ffn_canon", ("ffn", r))), p + "ffn_norm")
            if c.depth_average:
                xs.append(x)
                x = sum(g * z for g, z in zip(w[p + "dwa"], xs))
            if i in c.tap_layers:
                tap.append(x.clone())
        return x

    def _token_parallel(self, t: int, st: RefState, tap: list) -> torch.Tensor:
        """One token through a model of parallel blocks: the row before the final norm."""
        c, w = self.cfg, self.w
        x = w["embed"][t] * c.embed_scale
        for run in c.layer_runs:
            i, l, p = run.layer, c.layers[run.layer], f"l{run.layer}."
            h = F.layer_norm(x, x.shape, w[p + "pre_norm"], w[p + "pre_norm_bias"], c.eps)
            y = self._gqa(run.index, i, h, st)
            if l.experts:
                y = y + self._experts(i, h)
            elif l.ff:
                y = y + w[p + "down"] @ (F.silu(w[p + "gate"] @ h) * (w[p + "up"] @ h))
            x = x + y
            if i in c.tap_layers and not any(q.layer == i and q.index > run.index for q in c.layer_runs):
                tap.append(x.clone())
        return x

    def _token_out_norm(self, t: int, st: RefState, tap: list) -> torch.Tensor:
        """One token through a model with norms on the sublayers' outputs: the row before the final norm."""
        c, w = self.cfg, self.w
        x = w["embed"][t] * c.embed_scale
        if c.gram_buckets:
            x = x + w["bigram"][c.gram_buckets if st.prev is None else (st.prev * c.gram_mul_prev + t * c.gram_mul_cur) % c.gram_buckets]
        st.prev, x0 = t, x
        before = lambda name: rmsnorm(x, w[name], c.eps, False) if c.pre_norm else x
        for run in c.layer_runs:
            i, l = run.layer, c.layers[run.layer]
            p = f"l{i}."
            if run.enter is not None:
                x = w["loop_in"] @ torch.cat([x, x0]) + w["loop_step"][run.enter]
            h = before(p + "pre_norm")
            y = self._latent(i, h, st) if l.mixer == "latent" else (self._gqa if l.mixer == "gqa" else self._cdelta)(run.index, i, h, st)
            x = x + c.residual_mult * rmsnorm(y, w[p + "mix_norm"], c.eps, False)
            if l.ff:
                h = before(p + "ffn_pre_norm")
                act = F.silu(w[p + "gate"] @ h) * (w[p + "up"] @ h) if l.act == "swiglu" else torch.relu(w[p + "up"] @ h).square()
                x = x + c.residual_mult * rmsnorm(w[p + "down"] @ act, w[p + "ffn_norm"], c.eps, False)
            if i in c.tap_layers and not any(q.layer == i and q.index > run.index for q in c.layer_runs):
                tap.append(x.clone())
        return x

    def _ffn(self, i: int, x: torch.Tensor) -> torch.Tensor:
        c, w = self.cfg, self.w
        p = f"l{i}."
        if not c.is_moe(i):
            return w[p + "down"] @ swiglu(w[p + "gate_up"] @ x)
        idx, wt = route(c, (w[p + "router"] @ x)[None], w.get(p + "router_bias"))
        out = torch.zeros_like(x)
        for e, g in zip(idx[0].tolist(), wt[0].tolist()):          # fixed pair order: rank of the pick
            out = out + g * (w[p + "experts_down"][e] @ swiglu(w[p + "experts_gate_up"][e] @ x))
        if c.n_shared:
            sh = w[p + "shared_down"] @ swiglu(w[p + "shared_gate_up"] @ x)
            if c.router == "softmax":
                sh = sh * torch.sigmoid(w[p + "shared_gate"] @ x)
            out = out + sh
        return out

    # ---- whole model -------------------------------------------------------------------------------
    def forward(self, tokens, st: RefState, return_hidden: bool = False):
        c, w = self.cfg, self.w
        logits, taps = [], []
        head = w["embed"] if c.tie_embeddings else w["lm_head"]
        for t in list(tokens):
            tap = []
            if c.layers:
                x = (self._token_parallel if c.parallel else self._token_conv if c.layer_norm else self._token_out_norm)(int(t), st, tap)
                st.pos += 1
                if c.parallel or c.layer_norm:
                    y = head @ F.layer_norm(x, x.shape, w["final_norm"], w.get("final_norm_bias"), c.eps) * c.logit_scale
                else:
                    y = head @ rmsnorm(x, w["final_norm"], c.eps, False) * c.logit_scale
                logits.append(c.logit_softcap * torch.tanh(y / c.logit_softcap) if c.logit_softcap else y)
                taps.append(tap)
                continue
            x = w["embed"][int(t)].clone()
            for i, kind in enumerate(c.layer_kinds):
                h = rmsnorm(x, w[f"l{i}.input_norm"], c.eps)
                if kind == "gdn":
                    x = x + self._gdn(i, h, st)
                elif kind == "attn":
                    x = x + self._attn(i, h, st)
                else:
                    x = x + self._mla(i, h, st)
                x = x + self._ffn(i, rmsnorm(x, w[f"l{i}.post_norm"], c.eps))
                if i in c.tap_layers:
                    tap.append(x.clone())
            st.pos += 1
            logits.append(head @ rmsnorm(x, w["final_norm"], c.eps))
            taps.append(tap)
        out = torch.stack(logits, 0)
        return (out, taps) if return_hidden else out

    @torch.no_grad()
    def generate(self, prompt, n_new: int) -> List[int]:
        st = self.new_state()
        lg = self.forward(prompt, st)
        out = []
        tok = int(lg[-1].argmax())
        for _ in range(n_new):
            out.append(tok)
            lg = self.forward([tok], st)
            tok = int(lg[-1].argmax())
        return out
