"""Mixers of the models whose layers are listed one by one, beside latent attention (`ops/latent.py`): grouped-query attention ("gqa")
with rotated queries and keys, normed per head after the rotation or over the whole row before it, values that may be the projected
keys, a sink, softcapped scores, sliding windows or chunks, one softmax map per head or the difference of two, gated outputs; and the
gated delta rule with one decay per key channel ("cdelta"). Routed feed-forwards are here too. `TorchMixers` states each op in plain PyTorch for the fp32 CPU engine, `CudaMixers` runs the
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
    def gqa_prep(self, proj, d, bias, inv_freq, row_slot, row_pos, block_table, k_cache, v_cache, kv_block, eps, norms=None):
        """Biases, norms over whole rows (`norms`: their weights for q and k), rotation and norms per head of a step's queries and keys;
        keys and values into their pages (a layer with another one's keys projects queries only). Returns q [T, maps * heads, hp]."""
        T, M, own = proj.shape[0], d.maps, d.source < 0
        p = proj.float() if bias is None else proj.float() + bias[:proj.shape[1]]
        nq, nk = d.heads * M * d.dim, d.kv_heads * M * d.dim
        q, k = p[:, :nq], p[:, nq:nq + nk] if own else None
        if d.row_norm:
            q, k = (None if x is None else x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w for x, w in zip((q, k), norms))
        q = q.reshape(T, d.heads * M, d.dim)
        ang = row_pos.double()[:, None] * inv_freq[None, :]
        c, s = ang.cos().float()[:, None], ang.sin().float()[:, None]

        def turn(x):
            if d.rot_half:
                a, b = x[..., :d.rot_dims // 2], x[..., d.rot_dims // 2:d.rot_dims]
                x = torch.cat([a * c - b * s, b * c + a * s, x[..., d.rot_dims:]], -1)
            else:
                a, b = x[..., 0:d.rot_dims:2], x[..., 1:d.rot_dims:2]
                x = torch.cat([torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2), x[..., d.rot_dims:]], -1)
            return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) if d.qk_norm else x
        pad = lambda x: F.pad(x, (0, d.hp - x.shape[-1]))
        if own:
            v = p[:, d.v_off:d.v_off + d.kv_heads * d.vw].reshape(T, d.kv_heads, d.vw)
            page, off = block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block
            k_cache[page, off] = pad(turn(k.reshape(T, d.kv_heads * M, d.dim)).reshape(T, d.kv_heads, M * d.dim)).to(k_cache.dtype)
            v_cache[page, off] = pad(v).to(v_cache.dtype)
        q = turn(q)
        if M == 2:                                                    # the other map's columns of a query are zeros
            q = torch.stack([F.pad(q[:, 0::2], (0, d.dim)), F.pad(q[:, 1::2], (d.dim, 0))], 2).flatten(1, 2)
        return pad(q).to(self.dtype)

    def pool_keys(self, d, k_cache, v_cache, pooled, seg_slot, seg_pos0, seg_nrows, max_rows, block_table, kv_block):
        """Means of the cached keys and values of every block of `pool` positions whose last one is in the step. A mean lies in the page of
        the block's last position, at that position's number of whole blocks in the page."""
        P = d.pool
        for s in range(len(seg_slot)):
            p0, n, slot = int(seg_pos0[s]), int(seg_nrows[s]), int(seg_slot[s])
            for e in range((p0 + P) // P * P - 1, p0 + n, P):
                at = torch.arange(e - P + 1, e + 1)
                page, off = block_table[slot, at // kv_block].long(), at % kv_block
                for cache, means in zip((k_cache, v_cache), pooled):
                    means[int(page[-1]), e % kv_block // P] = cache[page, off].float().mean(0).to(means.dtype)

    def gqa_attention(self, q, d, k_cache, v_cache, sink, group, row_slot, row_kvlen, segs, block_table, kv_block, nsplit, out, lam=None,
                      gate=None, eps=0.0, pooled=None):
        """Causal attention of the rows of `group` over what the layer's mask leaves of the cache; q [T, maps * heads, hp], out
        [T, heads, hp], row tables of all T rows. Two maps: `lam` [1] weighs the second. `gate` [T, heads * vdim]: logits of the
        outputs' sigmoid gates."""
        own = [h // (d.queries // d.kv_heads) for h in range(d.queries)]
        for r in range(group.row_lo, group.row_hi):
            n, s = int(row_kvlen[r]), int(row_slot[r])
            lo = d.first_visible(n - 1)
            pages = block_table[s, :(n + kv_block - 1) // kv_block].long()
            k = k_cache[pages].flatten(0, 1)[lo:n, own].float()
            v = v_cache[pages].flatten(0, 1)[lo:n, own].float()
            if d.pool:
                end = torch.arange(d.blocks_visible(n - 1)) * d.pool + d.pool - 1
                bp = block_table[s, end // kv_block].long()
                k, v = (torch.cat([m[bp, end % kv_block // d.pool][:, own].float(), x]) for m, x in zip(pooled, (k, v)))
            sc = torch.einsum("hd,jhd->hj", q[r].float(), k) * d.scale
            if d.softcap:
                sc = d.softcap * torch.tanh(sc / d.softcap)
            if sink is not None:
                sc = torch.cat([sc, sink[:, None]], 1)
            o = torch.einsum("hj,jhd->hd", torch.softmax(sc, -1)[:, :len(k)], v)
            if d.maps == 2:
                o = o[0::2] - lam * o[1::2]
                o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / d.vw + eps) * (1 - d.diff)
            if gate is not None:
                o[:, :d.vw] *= torch.sigmoid(gate[r].float()).view(d.heads, d.vw)
            out[r] = o.to(out.dtype)
        return out

    def expert_rows(self, h, ids, w_gu, w_down, limit=0.0, shared=None):
        """Rows of a token's experts, one per (token, pick): [T * top, width] fp32. `limit`: clamped gated units instead of swiglu; `shared` =
        (gate | up, down, limit): the expert one past the last."""
        T, K = ids.shape
        out = torch.empty(T * K, w_down.shape[1], dtype=torch.float32, device=h.device)
        for p, e in enumerate(ids.reshape(-1).tolist()):
            gu, dn, lim = (w_gu[e], w_down[e], limit) if e < w_down.shape[0] else (shared[0][0], shared[1][0], shared[2])
            a = self.glu_act(gu.float() @ h[p // K].float(), lim)
            out[p] = dn.float() @ a.to(self.dtype).float()
        return out

    @staticmethod
    def glu_act(gu, limit):
        g, u = gu.chunk(2, -1)
        if not limit:
            return F.silu(g) * u
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        return g * torch.sigmoid(1.702 * g) * (u + 1)

    def ssm(self, proj, d, w, rec_state, conv_state, groups, seg_slot, seg_row0, seg_nrows, row_slot, row_pos, eps, commit=True):
        """Rows of the projection [z | x | B | C | dt] through the state-space recurrence of one layer -> [T, ko]. `w`: the layer's tensors by
        name."""
        T, H, G, N, V = proj.shape[0], d.heads, d.groups, d.state, d.vdim
        c = self.conv_rows(proj[:, d.inner:d.dt_off], w["conv"], conv_state, row_slot, row_pos, bias=w["conv_bias"], silu=True).float()
        dt = F.softplus(proj[:, d.dt_off:d.dt_off + H].float() + w["dt_bias"], threshold=80.0)
        a = torch.exp(w["A"] * dt)
        own = [h // (H // G) for h in range(H)]
        x = c[:, :d.inner].reshape(T, H, V)
        B, C = (c[:, d.inner + j * G * N:d.inner + (j + 1) * G * N].reshape(T, G, N)[:, own] for j in (0, 1))
        y = torch.zeros(T, d.ko, dtype=torch.float32, device=proj.device)
        for s in range(len(seg_slot)):
            n, r0, slot = int(seg_nrows[s]), int(seg_row0[s]), int(seg_slot[s])
            S = rec_state[slot].clone()
            for t in range(r0, r0 + n):
                S = S * a[t][:, None, None] + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
                y[t, :d.inner] = (torch.einsum("hnv,hn->hv", S, C[t]) + w["skip"][:, None] * x[t]).flatten()
            if commit and n > 0:
                rec_state[slot] = S
        if commit:
            self.conv_tail(conv_state, proj[:, d.inner:d.dt_off], seg_slot, seg_row0, seg_nrows)
        g = (y[:, :d.inner] * F.silu(proj[:, :d.inner].float())).reshape(T, d.norm_groups, -1)
        y[:, :d.inner] = (g / torch.sqrt(g.pow(2).mean(-1, keepdim=True) + eps)).flatten(1) * w["gnorm_w"]
        return y.to(self.dtype)

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
    def gqa_prep(self, proj, d, bias, inv_freq, row_slot, row_pos, block_table, k_cache, v_cache, kv_block, eps, norms=None):
        q = self.empty(proj.shape[0], d.queries, d.hp, dtype=self.dtype, device=self.device)
        self.launches += 1
        if not d.plain:
            assert bias is None and not d.qk_norm, "row norms and two maps: no biases, no norms per head"
            caches = (k_cache, v_cache) if d.source < 0 else (None, None)
            self.C.gqa_row_prep(q, *caches, proj, *(norms or (None, None)), inv_freq, row_slot, row_pos, block_table, kv_block,
                                [d.heads, d.maps, d.dim, d.vw, d.rot_dims, d.v_off, int(d.rot_half)], eps, self.status_word)
            return q
        assert d.source < 0, "keys of another layer: row norms only"
        self.C.gqa_prep(q, k_cache, v_cache, proj, bias, inv_freq, row_slot, row_pos, block_table, kv_block, d.dim, d.rot_dims, d.v_off,
                        d.qk_norm, eps, self.status_word)
        return q

    def pool_keys(self, d, k_cache, v_cache, pooled, seg_slot, seg_pos0, seg_nrows, max_rows, block_table, kv_block):
        self.launches += 1
        self.C.pool_keys(*pooled, k_cache, v_cache, seg_slot, seg_pos0, seg_nrows, max_rows, block_table, kv_block, d.pool, self.status_word)

    def _pooled_rows(self, d, pooled, group, seg_slot, block_table, kv_block):
        """Means of the blocks that a prompt group's rows see, side by side: (keys, values, first row of every segment)."""
        count, start = group.pooled(d.window, d.pool)
        tables = torch.tensor([start[:-1], count], dtype=torch.int32).pin_memory().to(self.device, non_blocking=True)
        k, v = (self.empty(max(64, start[-1]), d.kv_heads, d.hp, dtype=self.dtype, device=self.device) for _ in "kv")
        if start[-1]:
            self.launches += 1
            self.C.pool_gather(k[:start[-1]], v[:start[-1]], *pooled, seg_slot, tables[0], tables[1], block_table, kv_block, d.pool, self.status_word)
        return k, v, tables[0]

    def gqa_attention(self, q, d, k_cache, v_cache, sink, group, row_slot, row_kvlen, segs, block_table, kv_block, nsplit, out, lam=None,
                      gate=None, eps=0.0, pooled=None):
        """Prompt groups go to the tcgen05 flash kernel (softmax weights as value + remainder); the others are split over their keys on
        the mma.sync kernels, over the warps of a CTA as well where a segment brings at most 16 (row, head) pairs per key head. 32-bit runs, heads wider than 256 and pages off the 64 grid take the CUDA-core kernel. `nsplit` bounds the
        key splits; what is left of it is what fills the GPU and what the layer's mask leaves of the keys. The difference of two maps and
        the output gate ride on the merge of the splits and on the flash kernel (a gate over single maps follows that in a pass of its own). Rows of `out` may lie apart."""
        a, b, nq = group.row_lo, group.row_hi, d.queries
        mixed = d.maps == 2 or gate is not None
        bounds = dict(window=d.window, chunk=d.chunk, softcap=d.softcap)
        mix = (lam, None if gate is None else gate[a:b], 1.0 - d.diff, d.maps, d.vw, eps)
        tc = self.dtype == torch.bfloat16 and d.hp in (64, 128, 256)
        if group.prompt and tc and kv_block % 64 == 0:
            if d.pool:
                assert not mixed and sink is None, "pooled windows: single maps without gates and sinks"
                k, v, start = self._pooled_rows(d, pooled, group, segs[0], block_table, kv_block)
                bounds.update(k_mean=k, v_mean=v, mean_start=start, pool=d.pool)
            self.launches += 1
            flat = q.view(q.shape[0], -1)
            if d.maps == 2:                                           # both maps of a head in one CTA, which joins them
                rc = self.C.attn_prefill_tc(out, flat, k_cache, v_cache, flat, segs[0], segs[1], segs[2], segs[3], block_table, kv_block,
                                            group.max_rows, nq, d.kv_heads, d.hp, False, self.status_word, scale=d.scale, exact_p=True,
                                            lam=lam, gate=gate, mix_scale=1.0 - d.diff, vdim=d.vw, eps=eps, **bounds)
                assert rc == 0, "prompt attention: shape outside the tensor-core kernel"
                return out
            rows = self.empty(q.shape[0], nq, d.hp, dtype=torch.float32, device=self.device) if mixed else out
            rc = self.C.attn_prefill_tc(rows, flat, k_cache, v_cache, flat, segs[0], segs[1], segs[2], segs[3], block_table, kv_block,
                                        group.max_rows, nq, d.kv_heads, d.hp, False, self.status_word, scale=d.scale, exact_p=True, sink=sink,
                                        **bounds)
            assert rc == 0, "prompt attention: shape outside the tensor-core kernel"
            if mixed:
                self.launches += 1
                self.C.head_mix(out[a:b], rows[a:b], *mix)
            return out
        group_heads = nq // d.kv_heads
        mma = tc and group_heads <= 64
        keys = mma and d.hp <= 128 and (1 if d.pool else group.max_rows) * group_heads <= 16 and kv_block % 64 == 0
        per_group = max(1, (16 if d.pool else 64) // max(1, group_heads))
        if d.pool:
            assert not mixed and sink is None, "pooled windows: single maps without gates and sinks"
            mma = keys
            bounds.update(k_mean=pooled[0], v_mean=pooled[1], pool=d.pool)
            seen = block_table.shape[1] * kv_block if nsplit >= 64 else nsplit * 64      # context that nsplit stands for
            nsplit = min(nsplit, -(-(d.window + group.max_rows) // 64) + 2 + -(-seen // (64 * d.pool)))
        ctas = (group.seg_hi - group.seg_lo) * -(-group.max_rows // per_group) * d.kv_heads if mma else (b - a) * nq
        nsplit = max(1, min(nsplit, ((3 if d.hp == 128 else 5) if keys else 4 if mma else 8) * self.sm_count // max(1, ctas)))
        if d.reach:
            nsplit = min(nsplit, -(-(d.reach + group.max_rows) // 64) + 1 if keys else -(-(d.reach + group.max_rows) // 32))
        o_part = self.empty((b - a) * nq * nsplit * d.hp, dtype=torch.float32, device=self.device)
        ml_part = self.empty((b - a) * nq * nsplit * 2, dtype=torch.float32, device=self.device)
        self.launches += 2 if mma or mixed or nsplit > 1 else 1
        self.C.gqa_attn(out[a:b], o_part, ml_part, q[a:b], k_cache, v_cache, sink, segs[0], segs[1], segs[2], group.max_rows, row_slot[a:b],
                        row_kvlen[a:b], block_table, kv_block, a, nsplit, d.scale, not mma, self.status_word, **bounds,
                        **(dict(zip(("lam", "gate", "mix_scale", "maps", "vdim", "eps"), mix)) if mixed else {}))
        return out

    def expert_rows(self, h, ids, w_gu, w_down, limit=0.0, shared=None):
        """One row of the expert's feed-forward per (token, pick)."""
        pairs = ids.numel()
        sgu, sdn, slim = (shared[0][0], shared[1][0], shared[2]) if shared is not None else (None, None, 0.0)
        act = self.empty(pairs, max(w_down.shape[2], 0 if sdn is None else sdn.shape[1]), dtype=self.dtype, device=self.device)
        yp = self.empty(pairs, h.shape[1], dtype=torch.float32, device=self.device)
        self.launches += 2
        self.C.expert_rows(yp, act, h, w_gu, w_down, ids, limit, sgu, sdn, slim)
        return yp

    def ssm(self, proj, d, w, rec_state, conv_state, groups, seg_slot, seg_row0, seg_nrows, row_slot, row_pos, eps, commit=True):
        """Few rows: one launch per group from the projection to the heads' outputs. Prompt groups: convolutions, then the chunked form. The
        gated norm is one launch over all rows; with one row per segment it also moves the convolution's tails on."""
        T = proj.shape[0]
        sizes = [d.heads, d.groups, d.state, d.vdim, d.conv]
        y = self.empty(T, d.inner, dtype=torch.float32, device=self.device)
        out = self.empty(T, d.ko, dtype=self.dtype, device=self.device)
        par = (w["A"], w["dt_bias"], w["skip"])
        xbc = proj[:, d.inner:d.dt_off]
        conv = None
        for g in groups:
            segs = tuple(t[g.seg_lo:g.seg_hi] for t in (seg_slot, seg_row0, seg_nrows))
            if g.prompt and commit and self.dtype == torch.bfloat16 and d.state <= 256:
                if conv is None:
                    conv = self.conv_rows(xbc, w["conv"], conv_state, row_slot, row_pos, bias=w["conv_bias"], silu=True)
                nb = self.C.ssd_chunk_scratch_bytes(T, g.seg_hi - g.seg_lo, g.max_rows, d.heads, d.state, d.vdim)
                self.launches += 3
                self.C.ssd_chunk(y, rec_state, self.scratch("ssd_chunk", nb // 4, torch.float32), conv, proj, *par, *segs, g.max_rows, sizes)
            else:
                self.launches += 1
                self.C.ssm_step(y, rec_state, conv_state, proj, w["conv"], w["conv_bias"], *par, *segs, sizes, commit)
        single = commit and d.conv > 1 and all(g.max_rows == 1 for g in groups) and seg_slot.numel() == T
        self.launches += 1
        self.C.group_norm_gated(out, y, proj, w["gnorm_w"], d.norm_groups, eps, conv_state if single else None, row_slot if single else None)
        if commit and not single:
            self.conv_tail(conv_state, xbc, seg_slot, seg_row0, seg_nrows)
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
