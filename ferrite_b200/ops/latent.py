"""Ops of the models whose layers are listed one by one: position-free latent attention, norms on the sublayers'
outputs over a 32-bit residual stream, hashed bigram embeddings, softcapped logits. `TorchLatent` states each op in plain
PyTorch for the fp32 CPU engine, `CudaLatent` runs the kernels of `csrc/latent.cu` and the tcgen05 prompt attention; both have
the same signatures and work on the same paged caches.

Sizes are those of `models/weights.py:LatentDims`: padded columns hold zeros, norms divide by the true widths.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch


@dataclass
class SegGroup:
    """Consecutive segments of a step that go through attention together: rows [row_lo, row_hi), segments [seg_lo, seg_hi).
    `prompt` groups carry what the expanded form reads: the cache pages their contexts lie in, one segment after another, and
    the step-local page table over the gathered copy."""

    seg_lo: int
    seg_hi: int
    row_lo: int
    row_hi: int
    max_rows: int
    prompt: bool = False
    pages: Optional[torch.Tensor] = None
    table: Optional[torch.Tensor] = None
    own: Optional[torch.Tensor] = None


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
    def embed_grams(self, table, grams, ids, row_slot, row_pos, block_table, tok_pages, kv_block, scale, buckets, mul_prev, mul_cur, out=None):
        """Scaled token embedding plus the hashed bigram's row: (x fp32 [T, width], the same rows as GEMM operand). `out`: a buffer
        [T, k * width] whose k blocks of columns all take the operand."""
        x = table[ids.long()].float() * scale
        if grams is not None:
            prev = _prev_tokens(ids, row_slot, row_pos, block_table, tok_pages, kv_block)
            rows = [buckets if p < 0 else (p * mul_prev + int(t) * mul_cur) % buckets for p, t in zip(prev, ids)]
            x = x + grams[torch.tensor(rows, dtype=torch.long, device=x.device)].float()
            tok_pages[block_table[row_slot.long(), row_pos.long() // kv_block].long(), row_pos.long() % kv_block] = ids.to(tok_pages.dtype)
        if out is not None:
            for j in range(0, out.shape[1], x.shape[1]):
                out[:, j:j + x.shape[1]] = x.to(self.dtype)
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

    def norm_rows(self, x, idx, w, width, eps, bias=None):
        """rms(x) * w; with a bias the layer norm (x - mean) / deviation * w + bias."""
        x = x if idx is None else x[idx.long()]
        return (self._rms(x, w, width, eps) if bias is None else self._layer_norm(x, w, bias, width, eps)).to(self.dtype)

    @staticmethod
    def _layer_norm(x, w, b, width, eps):
        d = x[..., :width] - x[..., :width].mean(-1, keepdim=True)
        h = torch.zeros_like(x)
        h[..., :width] = d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w[:width] + b[:width]
        return h

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

    def latent_attention(self, qabs, cache, group, row_slot, row_kvlen, segs, block_table, kv_block, scale, nsplit=1):
        """Every head attends the cached latents: qabs [rows, heads, lat] of the group's rows -> [rows, heads, lat]."""
        out = torch.zeros(qabs.shape, dtype=torch.float32, device=qabs.device)
        for r in range(qabs.shape[0]):
            n, s = int(row_kvlen[r]), int(row_slot[r])
            keys = cache[block_table[s, :(n + kv_block - 1) // kv_block].long()].reshape(-1, qabs.shape[2])[:n].float()
            out[r] = torch.softmax((qabs[r].float() @ keys.t()) * scale, -1) @ keys
        return out.to(self.dtype)

    def softcap(self, logits, cap):
        return cap * torch.tanh(logits / cap)


class CudaLatent:
    def embed_grams(self, table, grams, ids, row_slot, row_pos, block_table, tok_pages, kv_block, scale, buckets, mul_prev, mul_cur, out=None):
        x = self.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=self.device)
        xb = out if out is not None else None if self.dtype == torch.float32 else self.empty(*x.shape, dtype=self.dtype, device=self.device)
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

    def norm_rows(self, x, idx, w, width, eps, bias=None):
        out = self.empty(x.shape[0] if idx is None else idx.numel(), x.shape[1], dtype=self.dtype, device=self.device)
        self.launches += 1
        self.C.norm_rows(out, x, idx, w, bias, width, eps)
        return out

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

    def latent_attention(self, qabs, cache, group, row_slot, row_kvlen, segs, block_table, kv_block, scale, nsplit=1):
        """Rows of one slot form a segment (`segs` = slots, first rows, row counts), so its rows and heads share every pass over
        the latents on the tensor cores; fp32 and latents wider than 512 take the CUDA-core kernel. `nsplit` bounds the key
        splits; what is left of it is what fills the GPU."""
        rows, heads, lat = qabs.shape
        mma = qabs.dtype == torch.bfloat16 and lat <= 512
        ctas = rows * heads if not mma else max(1, (group.seg_hi - group.seg_lo) * ((group.max_rows * heads + 63) // 64))
        per_sm = 8 if not mma else 2 if lat <= 192 else 1          # CTAs; a tile of wide latents fills an SM's shared memory
        nsplit = max(1, min(nsplit, per_sm * self.sm_count // ctas))
        out = self.empty(rows, heads, lat, dtype=qabs.dtype, device=self.device)
        o_part = ml_part = None
        if nsplit > 1:
            o_part = self.empty(rows * heads * nsplit * lat, dtype=torch.float32, device=self.device)
            ml_part = self.empty(rows * heads * nsplit * 2, dtype=torch.float32, device=self.device)
        self.launches += 1 if nsplit == 1 else 2
        if mma and self.C.latent_mma(out, o_part, ml_part, qabs, cache, segs[0], segs[1], segs[2], group.max_rows, row_kvlen,
                                     block_table, kv_block, group.row_lo, nsplit, scale, self.status_word) == 0:
            return out
        self.C.latent_attn(out, o_part, ml_part, qabs, cache, row_slot, row_kvlen, block_table, kv_block, nsplit, scale, self.status_word)
        return out

    def latent_rows(self, cache, group, kv_block):
        """The group's cached latents, segment after segment: [pages * kv_block, lat]."""
        self.launches += 1
        return cache.index_select(0, group.pages).view(-1, cache.shape[-1])

    def latent_attention_prompt(self, q, lat_rows, kv_up, d, group, segs, kv_block, out):
        """Prompt segments in the expanded form: one GEMM turns the context's latents into the keys and values of every head
        (side by side, at the padded head width), the tcgen05 flash kernel attends them; softmax weights go into its PV product
        as value + remainder. q, out [T, heads * hp]: the group's rows of all T."""
        kv = self.linear(lat_rows, kv_up).view(-1, kv_block, 2, d.heads, d.hp)
        self.launches += 1
        rc = self.C.attn_prefill_tc(out, q, kv[:, :, 0], kv[:, :, 1], q, group.own, segs[1], segs[2], segs[3], group.table, kv_block,
                                    group.max_rows, d.heads, d.heads, d.hp, False, self.status_word, scale=d.scale, exact_p=True)
        assert rc == 0, "prompt attention: shape outside the tensor-core kernel"
        return out

    def softcap(self, logits, cap):
        self.launches += 1
        self.C.softcap(logits, cap)
        return logits

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
               kv_block: int, device, gather: bool = True) -> List[SegGroup]:
    """Cut a step into runs of prompt segments (more than `flash_min` rows) and runs of the others. `segments`: host view
    (slot, first position, rows) of an eager step, None inside a graph, whose launches must not depend on it. `gather`: prompt groups
    carry the page lists of the expanded latent form."""
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
        if not g.prompt or not gather:
            continue
        counts = [(p + n + kv_block - 1) // kv_block for _, p, n in segments[g.seg_lo:g.seg_hi]]
        g.pages = torch.cat([block_table[s, :nb] for (s, _, _), nb in zip(segments[g.seg_lo:g.seg_hi], counts)])
        first = [sum(counts[:j]) for j in range(len(counts))]
        table = torch.tensor([[f + min(j, nb - 1) for j in range(max(counts))] for f, nb in zip(first, counts)], dtype=torch.int32)
        g.table = table.pin_memory().to(device, non_blocking=True)
        g.own = torch.arange(len(counts), dtype=torch.int32, device=device)
    return out
