"""Ops of the models whose layers are listed one by one: latent attention (without positions, or with a rotated key part), norms on the
sublayers' outputs over a 32-bit residual stream, convolved operands, averages over depth, hashed bigram embeddings, softcapped logits. `TorchLatent` states each op in plain
PyTorch for the fp32 CPU engine, `CudaLatent` runs the kernels of `csrc/latent.cu` and the tcgen05 prompt attention; both have
the same signatures and work on the same paged caches.

Sizes are those of `models/weights.py:LatentDims`: padded columns hold zeros, norms divide by the true widths.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch


@dataclass
class SegGroup:
    """Consecutive segments of a step that go through attention together: rows [row_lo, row_hi), segments [seg_lo, seg_hi).
    `prompt` groups know their segments (slot, first position, rows) on the host, for what gathers their contexts."""

    seg_lo: int
    seg_hi: int
    row_lo: int
    row_hi: int
    max_rows: int
    prompt: bool = False
    segments: Optional[List[Tuple[int, int, int]]] = None
    block_table: Optional[torch.Tensor] = None
    kv_block: int = 0
    _own: Optional[torch.Tensor] = None
    _context: Dict[int, tuple] = field(default_factory=dict)

    @property
    def own(self) -> torch.Tensor:
        """Number of every segment: the slots of step-local page tables."""
        if self._own is None:
            self._own = torch.arange(len(self.segments), dtype=torch.int32, device=self.block_table.device)
        return self._own

    def context(self, window: int = 0) -> Tuple[torch.Tensor, torch.Tensor]:
        """The cache pages that rows of the group see (those from `window` positions before a segment on; 0 = all), one segment after
        another, and the step-local page table over a gathered copy of them."""
        if window in self._context:
            return self._context[window]
        kvb, pages, rows, at = self.kv_block, [], [], 0
        for s, p, n in self.segments:
            first, last = max(0, p - window + 1) // kvb if window else 0, (p + n + kvb - 1) // kvb
            pages.append(self.block_table[s, first:last])
            rows.append([at] * first + list(range(at, at + last - first)))
            at += last - first
        width = max(len(r) for r in rows)
        table = torch.tensor([r + [r[-1]] * (width - len(r)) for r in rows], dtype=torch.int32)
        dev = self.block_table.device
        out = self._context[window] = torch.cat(pages), (table.pin_memory().to(dev, non_blocking=True) if dev.type == "cuda" else table)
        return out

    def pooled(self, window: int, pool: int) -> Tuple[List[int], List[int]]:
        """Blocks of `pool` positions that rows of every segment see under `window`, and where each segment's start in one list whose
        segments begin on multiples of 64 (the last entry is its length)."""
        count = [max(0, p + n - window) // pool for _, p, n in self.segments]
        start = [0]
        for c in count:
            start.append(start[-1] + (c + 63) // 64 * 64)
        return count, start


def _prev_tokens(ids, row_slot, row_pos, block_table, tok_pages, kv_block) -> List[int]:
    """Token before every row (-1 at a sequence's start): the row before it in the step, or the cached one."""
    out = []
    for r in range(ids.numel()):
        p, s = int(row_pos[r]), int(row_slot[r])
        if p == 0:
            out.append(-1)
        elif r > 0 and int(row_slot[r - 1]) == s and int(row_pos[r - 1]) == p - 1:
            out.append(int(ids[r - 1]))
        else:
            out.append(int(tok_pages[int(block_table[s, (p - 1) // kv_block]), (p - 1) % kv_block]))
    return out


class TorchLatent:
    def embed_grams(self, table, grams, ids, row_slot, row_pos, block_table, tok_pages, kv_block, scale, buckets, mul_prev, mul_cur, out=None,
                    x=None):
        """Scaled token embedding plus the hashed bigram's row: (x fp32 [T, width], the same rows as GEMM operand). `out`: a buffer
        [T, k * width] whose k blocks of columns all take the operand. `x`: rows to write instead of new ones."""
        rows32, x = x, table[ids.long()].float() * scale
        if grams is not None:
            prev = _prev_tokens(ids, row_slot, row_pos, block_table, tok_pages, kv_block)
            rows = [buckets if p < 0 else (p * mul_prev + int(t) * mul_cur) % buckets for p, t in zip(prev, ids)]
            x = x + grams[torch.tensor(rows, dtype=torch.long, device=x.device)].float()
            tok_pages[block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block] = ids.to(tok_pages.dtype)
        if out is not None:
            for j in range(0, out.shape[1], x.shape[1]):
                out[:, j:j + x.shape[1]] = x.to(self.dtype)
        if rows32 is not None:
            x = rows32.copy_(x)
        return x, x.to(self.dtype)

    @staticmethod
    def _rms(x, w, width, eps):
        xf = x.float()
        return xf / torch.sqrt(xf.pow(2).sum(-1, keepdim=True) / width + eps) * w

    def add_normed(self, x, y, w, width, eps, bias=None, next_w=None, out=None):
        """x += rms(y + bias) * w in place (x = y + bias with w None). Returns the next GEMM operand: rms(x) * next_w, or x itself
        with next_w None; written to `out` (rows may lie apart) when given."""
        y = y.float() if bias is None else y.float() + bias
        if w is None:
            x.copy_(y)
        else:
            x += self._rms(y, w, width, eps)
        h = x if next_w is None else self._rms(x, next_w, width, eps)
        if out is not None:
            out.copy_(h)
            return out
        return h.to(self.dtype)

    def norm_rows(self, x, idx, w, width, eps, bias=None, mean=False):
        """rms(x) * w; with a bias, or with `mean`, the layer norm (x - mean) / deviation * w (+ bias)."""
        x = x if idx is None else x[idx.long()]
        return (self._layer_norm(x, w, bias, width, eps) if mean or bias is not None else self._rms(x, w, width, eps)).to(self.dtype)

    @staticmethod
    def _layer_norm(x, w, b, width, eps):
        d = x[..., :width] - x[..., :width].mean(-1, keepdim=True)
        h = torch.zeros_like(x)
        h[..., :width] = d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w[:width] + (0.0 if b is None else b[:width])
        return h

    def add_conv_normed(self, x_in, x, y, w, width, eps, next_w, pairs=None, average=None, conv=None, row_slot=None, row_pos=None, single=False,
                        commit=True):
        """x = x_in + layer norm of f, times w, where f = y + the weighted expert rows `pairs` (y may be None, and with f missing x stays);
        `average` = (results [layers + 1, T, W], place, weights): x is stored as the result at that place and then becomes the weighted sum
        of the results up to it. Returns h, the layer norm of x times next_w (None with next_w None); with `conv` = (weights [taps, W],
        inputs of every slot before the step [slots, taps - 1, W]) h + its causal convolution, as (operand, h)."""
        f = None if y is None else y.float()
        if pairs is not None:
            p = (pairs[0].view(x.shape[0], -1, x.shape[1]).float() * pairs[1][:, :, None]).sum(1)
            f = p if f is None else f + p
        if f is not None:
            x.copy_(x_in + self._layer_norm(f, w, None, width, eps))
        if average is not None:
            xs, j, dwa = average
            xs[j] = x
            x.copy_(torch.einsum("j,jtw->tw", dwa, xs[:j + 1]))
        if next_w is None:
            return None, None
        h = self._layer_norm(x if f is not None else x_in, next_w, None, width, eps).to(self.dtype)
        if conv is None:
            return h, h
        out = self.conv_rows(h, conv[0], conv[1], row_slot, row_pos, residual=True)
        if single and commit:
            for r in range(h.shape[0]):
                conv[1][int(row_slot[r])] = torch.cat([conv[1][int(row_slot[r])][1:], h[r:r + 1].to(conv[1].dtype)])
        return out, h

    def conv_rows(self, x, w, tails, row_slot, row_pos, bias=None, silu=False, residual=False):
        """Causal convolution per channel of a step's rows: x [T, C], w [taps, C] (the last tap meets the row itself), what lies before a
        segment out of `tails` [slots, taps - 1, C]."""
        taps, T = w.shape[0], x.shape[0]
        out = torch.empty(T, x.shape[1], dtype=torch.float32, device=x.device)
        for r in range(T):
            s, n = int(row_slot[r]), 1
            while n < taps and r - n >= 0 and int(row_slot[r - n]) == s and int(row_pos[r - n]) == int(row_pos[r]) - n:
                n += 1
            rows = x[r - n + 1:r + 1].float()
            if n < taps:
                rows = torch.cat([tails[s][n - 1:].float(), rows])
            out[r] = (rows * w).sum(0)
        if bias is not None:
            out = out + bias
        if silu:
            out = torch.nn.functional.silu(out)
        if residual:
            out = out + x.float()
        return out.to(self.dtype)

    def conv_tail(self, tails, x, seg_slot, seg_row0, seg_nrows):
        """The last taps - 1 inputs of every segment's sequence become its slot's tail."""
        K = tails.shape[1]
        for s in range(len(seg_slot)):
            n, r0, slot = int(seg_nrows[s]), int(seg_row0[s]), int(seg_slot[s])
            if n > 0:
                tails[slot] = torch.cat([tails[slot], x[r0:r0 + n].to(tails.dtype)])[n:n + K]

    def add_layer_norm(self, x, y, width, eps, next_w=None, next_b=None, pairs=None):
        """x += y in place, with `pairs` = (rows [T * top, width], weights [T, top]) also the weighted sum of a token's rows. Returns the
        next GEMM operand, the layer norm of x (None with next_w None)."""
        x += y.float()
        if pairs is not None:
            x += (pairs[0].view(x.shape[0], -1, x.shape[1]).float() * pairs[1][:, :, None]).sum(1)
        return None if next_w is None else self._layer_norm(x, next_w, next_b, width, eps).to(self.dtype)

    def latent_prep(self, proj, d, q_norm, kv_norm, row_slot, row_pos, block_table, cache, kv_block, eps):
        """Both latents of a token from the fused projection: returns the normalised query latent, writes the normalised key /
        value latent into its page (`kv_norm` None: the layer reads another layer's)."""
        if kv_norm is not None:
            c = self._rms(proj[:, d.qr:], kv_norm, d.kv_rank, eps)
            cache[block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block] = c.to(cache.dtype)
        return self._rms(proj[:, :d.qr], q_norm, d.q_rank, eps).to(self.dtype)

    def latent_rot_prep(self, proj, d, kv_norm, inv_freq, row_slot, row_pos, block_table, cache, kv_block, eps):
        """From the projection [q heads | latent | key part]: queries with their last `rot` columns rotated (pairs (0, 1), (2, 3), ...) to
        [T, heads, hp], normed latent and rotated key part into the token's cache row."""
        T = proj.shape[0]
        ang = row_pos.double()[:, None] * inv_freq[None, :]
        c, s = ang.cos().float(), ang.sin().float()

        def turn(x, c, s):
            a, b = x[..., 0::2], x[..., 1::2]
            return torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2)
        nq, kd = d.heads * (d.dim + d.rot), d.dim + d.rot
        pq, pc, pk = proj[:, :nq].float().reshape(T, d.heads, kd), proj[:, nq:nq + d.kv_rank], proj[:, nq + d.kv_rank:nq + d.kv_rank + d.rot].float()
        q = torch.zeros(T, d.heads, d.hp, dtype=torch.float32, device=proj.device)
        q[..., :d.dim], q[..., d.dim:kd] = pq[..., :d.dim], turn(pq[..., d.dim:], c[:, None], s[:, None])
        row = torch.zeros(T, d.lat, dtype=torch.float32, device=proj.device)
        row[:, :d.kv_rank] = self._rms(pc, kv_norm[:d.kv_rank], d.kv_rank, eps)
        row[:, d.kv_rank:d.kv_rank + d.rot] = turn(pk, c, s)
        cache[block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block] = row.to(cache.dtype)
        return q.to(self.dtype)

    def latent_attention(self, qabs, cache, group, row_slot, row_kvlen, segs, block_table, kv_block, scale, nsplit=1, vlat=0, window=0):
        """Every head attends the cached rows (the last `window` ones, 0 = all): qabs [rows, heads, lat] of the group's rows -> their
        first `vlat` columns [rows, heads, vlat] (0: all of them)."""
        vlat = vlat or qabs.shape[2]
        out = torch.zeros(*qabs.shape[:2], vlat, dtype=torch.float32, device=qabs.device)
        for r in range(qabs.shape[0]):
            n, s = int(row_kvlen[r]), int(row_slot[r])
            lo = max(0, n - window) if window else 0
            keys = cache[block_table[s, :(n + kv_block - 1) // kv_block].long()].reshape(-1, qabs.shape[2])[lo:n].float()
            out[r] = torch.softmax((qabs[r].float() @ keys.t()) * scale, -1) @ keys[:, :vlat]
        return out.to(self.dtype)

    def softcap(self, logits, cap):
        return cap * torch.tanh(logits / cap)


class CudaLatent:
    def embed_grams(self, table, grams, ids, row_slot, row_pos, block_table, tok_pages, kv_block, scale, buckets, mul_prev, mul_cur, out=None,
                    x=None):
        own, x = x, x if x is not None else self.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=self.device)
        xb = out if out is not None else None if self.dtype == torch.float32 or own is not None else self.empty(*x.shape, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.embed_grams(x, xb, table, grams, ids, row_slot, row_pos, block_table, kv_block, tok_pages, scale, buckets, mul_prev, mul_cur,
                           self.status_word)
        return x, (x if xb is None else xb)

    def add_normed(self, x, y, w, width, eps, bias=None, next_w=None, out=None):
        xb = out
        if out is None and (self.dtype != torch.float32 or next_w is not None):
            xb = self.empty(*x.shape, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.add_normed(x, xb, y, w, width, eps, bias, next_w)
        return x if xb is None else xb

    def norm_rows(self, x, idx, w, width, eps, bias=None, mean=False):
        out = self.empty(x.shape[0] if idx is None else idx.numel(), x.shape[1], dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.norm_rows(out, x, idx, w, bias, width, eps, mean)
        return out

    def add_conv_normed(self, x_in, x, y, w, width, eps, next_w, pairs=None, average=None, conv=None, row_slot=None, row_pos=None, single=False,
                        commit=True):
        """One pass over the rows; the convolution rides on it where every segment is one row (`single`), else it is a pass of its own."""
        rows, f32 = x.shape, self.dtype == torch.float32
        fused = conv is not None and single
        h = out = None
        if next_w is not None and not (fused and commit):
            h = self.empty(*rows, dtype=self.dtype, device=self.device)
        if fused:
            out = self.empty(*rows, dtype=self.dtype, device=self.device)
        xs, place, dwa = average or (None, 0, None)
        self.launches += 1
        self.C.add_conv_normed(x_in, x, y, *(pairs or (None, None)), w, xs, place, dwa, next_w, h, out, *(conv if fused else (None, None)),
                               row_slot if fused else None, commit, width, eps, f32)
        if conv is not None and not fused:
            out = self.conv_rows(h, conv[0], conv[1], row_slot, row_pos, residual=True)
        return (h if conv is None else out), h

    def conv_rows(self, x, w, tails, row_slot, row_pos, bias=None, silu=False, residual=False):
        out = self.empty(*x.shape, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.conv_rows(out, x, w, tails, row_slot, row_pos, bias, silu, residual)
        return out

    def conv_tail(self, tails, x, seg_slot, seg_row0, seg_nrows):
        self.launches += 1
        self.C.conv_tail(tails, x, seg_slot, seg_row0, seg_nrows)

    def latent_rot_prep(self, proj, d, kv_norm, inv_freq, row_slot, row_pos, block_table, cache, kv_block, eps):
        q = self.empty(proj.shape[0], d.heads, d.hp, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.latent_rot_prep(q, cache, proj, kv_norm, inv_freq, row_slot, row_pos, block_table, kv_block, d.dim, d.rot, d.kv_rank, eps,
                               self.status_word)
        return q

    def add_layer_norm(self, x, y, width, eps, next_w=None, next_b=None, pairs=None):
        xb = None if next_w is None else self.empty(*x.shape, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.add_layer_norm(x, xb, y, *(pairs or (None, None)), next_w, next_b, width, eps)
        return xb

    def latent_prep(self, proj, d, q_norm, kv_norm, row_slot, row_pos, block_table, cache, kv_block, eps):
        cq = self.empty(proj.shape[0], d.qr, dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.latent_prep(cq, cache, proj, q_norm, kv_norm, row_slot, row_pos, block_table, kv_block, d.q_rank, d.kv_rank, eps,
                           self.status_word)
        return cq

    def latent_attention(self, qabs, cache, group, row_slot, row_kvlen, segs, block_table, kv_block, scale, nsplit=1, vlat=0, window=0):
        """Rows of one slot form a segment (`segs` = slots, first rows, row counts), so its rows and heads share every pass over
        the latents on the tensor cores; fp32 and cache rows wider than 576 take the CUDA-core kernel. `nsplit` bounds the key
        splits; what is left of it is what fills the GPU and what the window leaves of the keys."""
        rows, heads, lat = qabs.shape
        vlat = vlat or lat
        mma = qabs.dtype == torch.bfloat16 and (lat <= 512 or (lat == 576 and vlat == 512)) and kv_block % 64 == 0
        tile = 64 if lat <= 512 else 32
        ctas = rows * heads if not mma else max(1, (group.seg_hi - group.seg_lo) * ((group.max_rows * heads + tile - 1) // tile))
        per_sm = 8 if not mma else 2 if lat <= 192 else 1          # CTAs; a tile of wide latents fills an SM's shared memory
        nsplit = max(1, min(nsplit, per_sm * self.sm_count // ctas))
        if window:
            nsplit = min(nsplit, -(-(window + group.max_rows) // 64) + 1)
        out = self.empty(rows, heads, vlat, dtype=qabs.dtype, device=self.device)
        o_part = ml_part = None
        if nsplit > 1:
            o_part = self.empty(rows * heads * nsplit * vlat, dtype=torch.float32, device=self.device)
            ml_part = self.empty(rows * heads * nsplit * 2, dtype=torch.float32, device=self.device)
        self.launches += 1 if nsplit == 1 else 2
        if mma and self.C.latent_mma(out, o_part, ml_part, qabs, cache, segs[0], segs[1], segs[2], group.max_rows, row_kvlen,
                                     block_table, kv_block, group.row_lo, nsplit, scale, self.status_word, window) == 0:
            return out
        self.C.latent_attn(out, o_part, ml_part, qabs, cache, row_slot, row_kvlen, block_table, kv_block, nsplit, scale, self.status_word, window)
        return out

    def latent_rows(self, cache, group, kv_block, window=0):
        """The cached latents that the group's rows see, segment after segment: [pages * kv_block, lat]."""
        self.launches += 1
        return cache.index_select(0, group.context(window)[0]).view(-1, cache.shape[-1])

    def latent_attention_prompt(self, q, lat_rows, kv_up, d, group, segs, kv_block, out):
        """Prompt segments in the expanded form: one GEMM turns the context's latents into the keys and values of every head
        (side by side, at the padded head widths), the tcgen05 flash kernel attends them; softmax weights go into its PV product
        as value + remainder. q [T, heads * hp], out [T, heads * vp]: the group's rows of all T."""
        kv = self.linear(lat_rows, kv_up)
        k = kv[:, :d.heads * d.hp].view(-1, kv_block, d.heads, d.hp)
        v = kv[:, d.heads * d.hp:].view(-1, kv_block, d.heads, d.vp)
        self.launches += 1
        rc = self.C.attn_prefill_tc(out, q, k, v, q, group.own, segs[1], segs[2], segs[3], group.context(d.window)[1], kv_block,
                                    group.max_rows, d.heads, d.heads, d.hp, False, self.status_word, scale=d.scale, exact_p=True, window=d.window)
        assert rc == 0, "prompt attention: shape outside the tensor-core kernel"
        return out

    def softcap(self, logits, cap):
        self.launches += 1
        self.C.softcap(logits, cap)
        return logits

    def glu(self, x, w, limit):
        """Clamped gated units of x w^T, w = [gate rows | up rows], more rows than the row kernels take."""
        M, N = x.shape[0], w.shape[0] // 2
        y = self.empty(M, N, dtype=self.dtype, device=self.device)
        assert self.dtype == torch.bfloat16 and N % 8 == 0 and M > 64, "glu: prompt rows in bf16"
        self.launches += 1
        self.C.gemm_glu(y, x, w, limit, 1, None, None, self.status_word)
        return y

    def silu_mul_f32(self, gu, out=None):
        y = out if out is not None else self.empty(gu.shape[0], gu.shape[1] // 2, dtype=torch.float32, device=self.device)
        self.launches += 1
        self.C.silu_mul_f32(y, gu)
        return y

    def linear_f32(self, x, w, act=None, out=None):
        """y = x W^T in 32 bits; 3-d operands: one product per head."""
        y = out if out is not None else self.empty(*x.shape[:-1], w.shape[-2], dtype=torch.float32, device=self.device)
        self.launches += 1
        self.C.gemm_f32(y, x, w, ACTS[act])
        return y


ACTS: Dict[Optional[str], int] = {None: 0, "relu2": 1}


def relu2(x):
    return torch.relu(x).square()


TORCH_ACTS = {None: lambda x: x, "relu2": relu2}


def seg_groups(segments: Optional[List[Tuple[int, int, int]]], n_seg: int, n_rows: int, max_rows: int, flash_min: int, block_table,
               kv_block: int, device) -> List[SegGroup]:
    """Cut a step into runs of prompt segments (more than `flash_min` rows) and runs of the others. `segments`: host view
    (slot, first position, rows) of an eager step, None inside a graph, whose launches must not depend on it."""
    if segments is None:
        return [SegGroup(0, n_seg, 0, n_rows, max_rows)]
    out: List[SegGroup] = []
    row = 0
    for i, (_, _, n) in enumerate(segments):
        prompt = n > flash_min
        if out and out[-1].prompt == prompt:
            g = out[-1]
            g.seg_hi, g.row_hi, g.max_rows = i + 1, row + n, max(g.max_rows, n)
        else:
            out.append(SegGroup(i, i + 1, row, row + n, n, prompt))
        row += n
    for g in out:
        if g.prompt:
            g.segments, g.block_table, g.kv_block = segments[g.seg_lo:g.seg_hi], block_table, kv_block
    return out
