"""Mixers of the models whose layers are listed one by one, beside latent attention (`ops/latent.py`): grouped-query attention with
rotated and then normed queries and keys, values that may be the projected keys, and a sink ("gqa"), and the gated delta rule with
one decay per key channel ("cdelta"). `TorchMixers` states each op in plain PyTorch for the fp32 CPU engine, `CudaMixers` runs the
kernels of `csrc/gqa.cu`, `csrc/cdelta.cu` and `csrc/cdelta_chunk.cu` and the shared attention kernels; both have the same signatures
and work on the same caches and states.

Sizes are those of `models/weights.py` (`GqaDims`, `DeltaDims`).
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

UNIT_EPS = 1e-6       # inside the root of the delta rule's unit queries and keys


class TorchMixers:
    def gqa_prep(self, proj, d, bias, inv_freq, row_slot, row_pos, block_table, k_cache, v_cache, kv_block, eps):
        """Biases, rotation and norm of a step's queries and keys; keys and values into their pages. Returns q [T, heads, hp]."""
        T = proj.shape[0]
        p = proj.float() if bias is None else proj.float() + bias
        q = p[:, :d.heads * d.dim].reshape(T, d.heads, d.dim)
        k = p[:, d.heads * d.dim:(d.heads + d.kv_heads) * d.dim].reshape(T, d.kv_heads, d.dim)
        v = p[:, d.v_off:d.v_off + d.kv_heads * d.dim].reshape(T, d.kv_heads, d.dim)
        ang = row_pos.double()[:, None] * inv_freq[None, :]
        c, s = ang.cos().float()[:, None], ang.sin().float()[:, None]

        def turn(x):
            a, b = x[..., 0:d.rot_dims:2], x[..., 1:d.rot_dims:2]
            x = torch.cat([torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2), x[..., d.rot_dims:]], -1)
            return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) if d.qk_norm else x
        pad = lambda x: F.pad(x, (0, d.hp - d.dim))
        page, off = block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block
        k_cache[page, off] = pad(turn(k)).to(k_cache.dtype)
        v_cache[page, off] = pad(v).to(v_cache.dtype)
        return pad(turn(q)).to(self.dtype)

    def gqa_attention(self, q, d, k_cache, v_cache, sink, group, row_slot, row_kvlen, segs, block_table, kv_block, nsplit, out):
        """Causal attention of the rows of `group` over the cache; q, out [T, heads, hp], row tables of all T rows."""
        own = [h // (d.heads // d.kv_heads) for h in range(d.heads)]
        for r in range(group.row_lo, group.row_hi):
            n, s = int(row_kvlen[r]), int(row_slot[r])
            pages = block_table[s, :(n + kv_block - 1) // kv_block].long()
            k = k_cache[pages].flatten(0, 1)[:n, own].float()
            v = v_cache[pages].flatten(0, 1)[:n, own].float()
            sc = torch.einsum("hd,jhd->hj", q[r].float(), k) * d.scale
            if sink is not None:
                sc = torch.cat([sc, sink[:, None]], 1)
            out[r] = torch.einsum("hj,jhd->hd", torch.softmax(sc, -1)[:, :n], v).to(out.dtype)
        return out

    def cdelta(self, proj, d, w, rec_state, conv_state, groups, seg_slot, seg_row0, seg_nrows, eps, commit=True):
        """Rows of the fused projection through the delta rule of one layer -> [T, ko]. `w`: the layer's tensors by name."""
        T, H, G, D, V, K = proj.shape[0], d.heads, d.kv_heads, d.dim, d.vdim, d.conv
        f = F.linear(proj[:, :d.ra].float(), w["decay_up"].float()) + w["dt_bias"]
        g = torch.exp(-w["A_log"].exp()[None, :, None] * F.softplus(f, threshold=80.0).view(T, H, D))
        gate = torch.sigmoid(F.linear(proj[:, d.ra:d.q_off].float(), w["gate_up_lr"].float())).view(T, H, V)
        beta = torch.sigmoid(proj[:, d.b_off:d.b_off + H].float())
        own = [h // (H // G) for h in range(H)]
        unit = lambda x: x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)
        y = torch.zeros(T, d.ko, dtype=torch.float32, device=proj.device)
        for s in range(len(seg_slot)):
            n, r0, slot = int(seg_nrows[s]), int(seg_row0[s]), int(seg_slot[s])
            if n <= 0:
                continue
            x = torch.cat([conv_state[slot].float(), proj[r0:r0 + n, d.q_off:d.b_off].float()])
            c = F.silu((x.unfold(0, K, 1) * w["conv"][None]).sum(-1))
            q = unit(c[:, :G * D].reshape(n, G, D))[:, own] * D ** -0.5
            k = unit(c[:, G * D:2 * G * D].reshape(n, G, D))[:, own]
            v = c[:, 2 * G * D:].reshape(n, H, V)
            S = rec_state[slot].clone()
            o = torch.empty(n, H, V, dtype=torch.float32, device=proj.device)
            for t in range(n):
                S = S * g[r0 + t][:, :, None]
                u = beta[r0 + t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None, :]
                o[t] = torch.einsum("hdv,hd->hv", S, q[t])
            o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w["gnorm_w"] * gate[r0:r0 + n]
            y[r0:r0 + n, :H * V] = o.flatten(1)
            if commit:
                rec_state[slot] = S
                conv_state[slot] = x[n:].to(conv_state.dtype)
        return y.to(self.dtype)
