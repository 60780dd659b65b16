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

LOWRANK_ROWS = 4      # up to this many rows the low-rank products are one SIMT launch, beyond two of the row or GEMM kernels
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


class CudaMixers:
    def gqa_prep(self, proj, d, bias, inv_freq, row_slot, row_pos, block_table, k_cache, v_cache, kv_block, eps):
        q = self.empty(proj.shape[0], d.heads, d.hp, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.gqa_prep(q, k_cache, v_cache, proj, bias, inv_freq, row_slot, row_pos, block_table, kv_block, d.dim, d.rot_dims, d.v_off,
                        d.qk_norm, eps, self.status_word)
        return q

    def gqa_attention(self, q, d, k_cache, v_cache, sink, group, row_slot, row_kvlen, segs, block_table, kv_block, nsplit, out):
        """Prompt groups go to the tcgen05 flash kernel (softmax weights as value + remainder); the others are split over their keys on
        the mma.sync kernel. 32-bit runs, heads wider than 256 and pages off the 64 grid take the CUDA-core kernel. `nsplit` bounds the
        key splits; what is left of it is what fills the GPU."""
        a, b = group.row_lo, group.row_hi
        tc = self.dtype == torch.bfloat16 and d.hp in (64, 128, 256)
        if group.prompt and tc and kv_block % 64 == 0:
            self.launches += 1
            flat = q.view(q.shape[0], -1)
            rc = self.C.attn_prefill_tc(out, flat, k_cache, v_cache, flat, segs[0], segs[1], segs[2], segs[3], block_table, kv_block,
                                        group.max_rows, d.heads, d.kv_heads, d.hp, False, self.status_word, scale=d.scale, exact_p=True, sink=sink)
            assert rc == 0, "prompt attention: shape outside the tensor-core kernel"
            return out
        mma = tc and d.heads // d.kv_heads <= 64
        per_group = max(1, 64 // max(1, d.heads // d.kv_heads))
        ctas = (group.seg_hi - group.seg_lo) * -(-group.max_rows // per_group) * d.kv_heads if mma else (b - a) * d.heads
        nsplit = max(1, min(nsplit, (4 if mma else 8) * self.sm_count // max(1, ctas)))
        o_part = self.empty((b - a) * d.heads * nsplit * d.hp, dtype=torch.float32, device=self.device)
        ml_part = self.empty((b - a) * d.heads * nsplit * 2, dtype=torch.float32, device=self.device)
        self.launches += 2 if mma or nsplit > 1 else 1
        self.C.gqa_attn(out[a:b], o_part, ml_part, q[a:b], k_cache, v_cache, sink, segs[0], segs[1], segs[2], group.max_rows, row_slot[a:b],
                        row_kvlen[a:b], block_table, kv_block, a, nsplit, d.scale, not mma, self.status_word)
        return out

    def cdelta(self, proj, d, w, rec_state, conv_state, groups, seg_slot, seg_row0, seg_nrows, eps, commit=True):
        """A few rows: both low-rank products in one launch, then one launch per group for the whole mixer. Prompt groups: two GEMMs,
        the chunked scan, the gated norm. Sizes beyond the fused kernels (heads wider than 128) run conv, recurrence and norm apart."""
        T = proj.shape[0]
        sizes = [d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.q_off]
        na = d.heads * d.dim
        if T <= LOWRANK_ROWS:
            up = self.empty(T, na + d.heads * d.vdim, dtype=torch.float32, device=self.device)
            self.launches += 1
            self.C.cd_lowrank(up, proj, w["decay_up"], w["gate_up_lr"])
            decay, gate = up[:, :na], up[:, na:]
        else:
            decay = self.linear(proj[:, :d.ra], w["decay_up"], out_f32=True)
            gate = self.linear(proj[:, d.ra:d.q_off], w["gate_up_lr"], out_f32=True)
        out = self.empty(T, d.ko, dtype=self.dtype, device=self.device)
        par = (w["conv"], w["A_log"], w["dt_bias"])
        y = qkv = None
        for g in groups:
            segs = tuple(t[g.seg_lo:g.seg_hi] for t in (seg_slot, seg_row0, seg_nrows))
            a, b = g.row_lo, g.row_hi
            fused = max(d.dim, d.vdim) <= 128 and not (g.prompt and commit)
            if fused:
                self.launches += 1
                self.C.cd_step(out, rec_state, conv_state, proj, decay, gate, *par, w["gnorm_w"], *segs, sizes, eps, commit)
            else:
                if y is None:
                    y = self.empty(T, d.heads, d.vdim, dtype=torch.float32, device=self.device)
                if g.prompt and commit and d.dim <= 128:
                    nb = self.C.cd_chunk_scratch_bytes(T, g.seg_hi - g.seg_lo, d.heads, d.dim)
                    self.launches += 2
                    self.C.cd_chunk(y, rec_state, self.scratch("cd_chunk", nb // 4, torch.float32), conv_state, proj, decay, *par, *segs,
                                    g.max_rows, sizes)
                else:
                    if qkv is None:
                        qkv = self.empty(T, d.channels, dtype=self.dtype, device=self.device)
                    self.launches += 2
                    self.C.cd_rec(y, rec_state, qkv, conv_state, proj, decay, *par, *segs, g.max_rows, sizes, commit)
                self.launches += 1
                self.C.gated_norm_sigmoid(out[a:b], y[a:b], gate[a:b], w["gnorm_w"], eps)
            if commit and not (fused and d.heads == d.kv_heads):
                self.launches += 1
                self.C.cd_tail(rec_state, conv_state, proj, w["conv"], *segs, sizes)
        return out
