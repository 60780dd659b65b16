"""Designs of listed layers, each beside the framework's closest other model of the same width, heads and parameter count, with
random weights: Zototar (latent attention without positions) beside the dense MLA model, Dofunex (delta rules with a decay per
channel, every fourth layer attention) beside the dense Gated DeltaNet hybrid, Rakizen (parallel blocks, windows and chunks, two maps in every
fourth layer) beside the sequential grouped-query attention model, dense or routed, Pironex (latent attention, pooled windows, state-space layers,
routed feed-forwards with a shared expert) beside the routed Gated DeltaNet hybrid.

`models()` measures prefill and decode throughput through the engine (CUDA graphs for decode steps), `kernels()`, `kernels_dofunex()`,
`kernels_rakizen()` and `kernels_pironex()` time every kernel of the first beside the kernel that does the same job for the second and give both as
fractions of their rooflines. They print nothing and return plain dictionaries; `bench.py --design ...` and `microbench
latent|cdelta|parallel|pooled` print them.
"""
from __future__ import annotations

import statistics
from dataclasses import replace
from typing import Dict, List

import torch

from ..config import EngineConfig, ModelConfig, dofunex, pironex, rakizen, zototar
from .microbench import Timer, graph_time, peaks, rnd

SIZES = {       # name: width, heads, query latent, feed-forward width, layers
    "2k": (2048, 16, 768, 8192, 16),
    "4k": (4096, 32, 1536, 16384, 8),
    "7k": (7168, 128, 1536, 27648, 4),
}
KV_RANK, DIM, ROPE, VOCAB = 512, 128, 64, 65536


def pair(size: str):
    """(Zototar model, dense MLA model) of one size: the feed-forward of the second has three matrices instead of two."""
    w, h, qr, ff, n = SIZES[size]
    a = zototar(w, n, h, qr, KV_RANK, ff, VOCAB, DIM, DIM, name=f"zototar-{size}")
    b = ModelConfig(name=f"mla-{size}", hidden=w, inter=(2 * ff // 3 + 127) // 128 * 128, n_layers=n, head_dim=DIM + ROPE, n_q=h,
                    n_kv=h, rotary_dim=ROPE, rope_theta=1e4, attn_gate=False, vocab=VOCAB, tie_embeddings=False, kv_lora=KV_RANK,
                    q_lora=qr, rope_head_dim=ROPE, nope_head_dim=DIM, v_head_dim=DIM)
    return a, b


def pair_dofunex(size: str):
    """(Dofunex model, dense hybrid of Gated DeltaNet and gated attention layers) of one size, every fourth layer attention; the
    feed-forward of the second makes up for its wider gates."""
    w, h, kv, ff, n = SIZES_DOFUNEX[size]
    a = dofunex(w, n, h, kv, ff, VOCAB, name=f"dofunex-{size}")
    kw = dict(name=f"hybrid-{size}", hidden=w, n_layers=n, full_attn_every=4, head_dim=DIM, n_q=h, n_kv=kv, rotary_dim=DIM, lin_k_heads=h,
              lin_v_heads=h, lin_dk=DIM, lin_dv=DIM, vocab=VOCAB, tie_embeddings=False)
    spare = a.param_count() - ModelConfig(inter=0, **kw).param_count()
    return a, ModelConfig(inter=max(256, round(spare / (3 * w * n) / 256) * 256), **kw)


def pair_rakizen(size: str):
    """(Rakizen model, sequential model of grouped-query attention layers) of one size, equal in width, heads, feed-forward and, by the dense
    width, parameters; routed feed-forwards in every layer of both or in none."""
    w, h, kv, ff, n, experts, top, groups, keep = SIZES_RAKIZEN[size]
    routed = dict(experts=experts, top=top, groups=groups, keep=keep, expert_ff=ff) if experts else {}
    a = rakizen(w, n, h, kv, ff, VOCAB, moe_every=1, name=f"rakizen-{size}", **routed)
    kw = dict(name=f"gqa-{size}", hidden=w, n_layers=n, full_attn_every=1, head_dim=DIM, n_q=h, n_kv=kv, rotary_dim=DIM, attn_gate=False, vocab=VOCAB,
              tie_embeddings=False)
    if experts:
        return a, ModelConfig(inter=ff, n_experts=experts, top_k=top, expert_inter=ff, router="sigmoid_group", n_groups=groups, topk_groups=keep,
                              route_scale=2.0, **kw)
    spare = a.param_count() - ModelConfig(inter=0, **kw).param_count()
    return a, ModelConfig(inter=max(256, round(spare / (3 * w * n) / 128) * 128), **kw)


def pair_pironex(size: str):
    """(Pironex model, routed hybrid of Gated DeltaNet and gated attention layers) of one size: equal width, heads, layers, experts and shared
    expert; every second layer of the hybrid is attention, as every second of the other reads keys."""
    w, h, kv, n, experts, top, ff = SIZES_PIRONEX[size]
    a = pironex(w, n, h, kv, VOCAB, dim=DIM, experts=experts, top=top, expert_ff=ff, shared_ff=ff, name=f"pironex-{size}")
    b = ModelConfig(name=f"hybrid-moe-{size}", hidden=w, inter=ff, n_layers=n, full_attn_every=2, head_dim=DIM, n_q=h, n_kv=kv, rotary_dim=DIM // 2,
                    lin_k_heads=h, lin_v_heads=h, lin_dk=DIM, lin_dv=DIM, vocab=VOCAB, tie_embeddings=True, n_experts=experts, top_k=top,
                    expert_inter=ff, n_shared=1, router="softmax")
    return a, b


SIZES_PIRONEX = {       # name: width, heads, key / value heads, layers, experts, per token, their width
    "1k": (1024, 8, 2, 16, 32, 4, 512),
    "2k": (2048, 16, 4, 12, 64, 6, 1024),
    "4k": (4096, 32, 8, 8, 32, 4, 1536),
}
SIZES_RAKIZEN = {       # name: width, heads, key / value heads, (expert's) feed-forward width, layers, experts, per token, groups, kept groups
    "2k": (2048, 16, 4, 6144, 16, 0, 0, 1, 1),
    "4k": (4096, 32, 8, 12288, 8, 0, 0, 1, 1),
    "2k-moe": (2048, 16, 4, 1024, 12, 64, 6, 8, 4),
}
SIZES_DOFUNEX = {       # name: width, heads, key / value heads of the attention layers, feed-forward width, layers
    "2k": (2048, 16, 4, 6144, 16),
    "4k": (4096, 32, 8, 11008, 8),
    "5k": (5120, 40, 8, 17408, 8),
}
DESIGNS = {"zototar": (pair, "mla_dense", "dense MLA model of equal width, heads, latent and parameter count", "2k,4k,7k"),
           "rakizen": (pair_rakizen, "gqa_sequential", "sequential grouped-query attention model of equal width, heads and parameter count (routed "
                       "feed-forwards in the moe size)", "2k,4k,2k-moe"),
           "pironex": (pair_pironex, "hybrid_moe", "routed Gated DeltaNet hybrid of equal width, heads, layers and experts", "1k,2k,4k"),
           "dofunex": (pair_dofunex, "hybrid_dense", "dense Gated DeltaNet hybrid of equal width, heads and parameter count", "2k,4k,5k")}


def run_model(cfg: ModelConfig, ctx: int, prompts: List[int], streams: List[int], steps: int, warmup: int, dev) -> Dict:
    from ..engine.engine import Engine
    from ..engine.executor import Segment
    n = max(streams)
    eng = Engine(cfg, None, EngineConfig(n_slots=n, max_ctx=max(max(prompts), ctx + steps * 8 + 128), prefill_chunk=2048), device=str(dev))
    g = torch.Generator().manual_seed(0)
    toks = lambda k: torch.randint(0, cfg.vocab, (k,), generator=g).tolist()
    out: Dict = {"params": cfg.param_count(), "cache_bytes_per_token": eng.ex.kv_block_bytes() // eng.ecfg.kv_block}
    for p in prompts:
        ids, times = toks(p), []
        for rep in range(5):
            eng.reset_slot(0)
            torch.cuda.synchronize(dev)
            e0, e1 = torch.cuda.Event(True), torch.cuda.Event(True)
            e0.record()
            eng.prefill(0, ids)
            e1.record()
            torch.cuda.synchronize(dev)
            times.append(e0.elapsed_time(e1))
        out[f"prefill_{p}_tok_s"] = round(p / statistics.median(times[2:]) * 1e3, 1)
    ids = toks(ctx)
    for s in range(n):
        eng.reset_slot(s)
        eng.prefill(s, ids)
    for m in streams:
        def step():
            eng.forward([Segment(s, eng.slot_len[s], [ids[s]], "last") for s in range(m)])
        for _ in range(max(3, warmup)):
            step()
        torch.cuda.synchronize(dev)
        e0, e1 = torch.cuda.Event(True), torch.cuda.Event(True)
        e0.record()
        for _ in range(steps):
            step()
        e1.record()
        torch.cuda.synchronize(dev)
        ms = e0.elapsed_time(e1) / steps
        out[f"decode_{m}_tok_s"], out[f"decode_{m}_ms"] = round(m / ms * 1e3, 1), round(ms, 4)
    eng.check()
    del eng
    torch.cuda.empty_cache()
    return out


def models(sizes: List[str], steps: int, warmup: int, dev, ctx: int = 2048, design: str = "zototar") -> Dict:
    out = {}
    of, other = DESIGNS[design][:2]
    for size in sizes:
        a, b = of(size)
        ra = run_model(a, ctx, [2048, 8192], [1, 4, 16], steps, warmup, dev)
        rb = run_model(b, ctx, [2048, 8192], [1, 4, 16], steps, warmup, dev)
        out[size] = {design: ra, other: rb, "ratio": {k: round(ra[k] / rb[k], 3) for k in ra if k.endswith("tok_s")}}
    return out


class _Rows:
    """Collects {kernel, like, ms, like_ms, frac, like_frac}: times in a CUDA graph of calls over buffers that together exceed L2."""

    def __init__(self, dev):
        self.t, self.rows = Timer(dev, 3, 20, flush=False), []
        self.hbm, self.tf, _ = peaks()

    def timed(self, fn, nbytes: float, flops: float, bufs: int):
        reps = max(4, min(40, int(-(-(400 << 20) // max(1, nbytes)))), bufs)
        ms = graph_time(self.t, lambda: [fn(j % bufs) for j in range(reps)], reps)
        return ms, max(nbytes / (self.hbm * 1e6), flops / (self.tf * 1e9)) / ms

    def add(self, name, new, like_name, like):
        (ms, fr), (lms, lfr) = self.timed(*new), self.timed(*like)
        self.rows.append({"kernel": name, "ms": round(ms, 5), "frac": round(fr, 4), "like": like_name, "like_ms": round(lms, 5),
                          "like_frac": round(lfr, 4)})


def kernels(dev, heads: int = 32, width: int = 4096, ctx: int = 4096, prompt: int = 2048) -> List[Dict]:
    """Zototar's kernels beside those of the dense MLA model."""
    from ..models.weights import LatentDims
    from ..ops.cuda_ops import CudaOps
    from ..ops.latent import SegGroup, seg_groups
    ops, acc = CudaOps(dev), _Rows(dev)
    t, hbm, tf, rows, add = acc.t, acc.hbm, acc.tf, acc.rows, acc.add
    L, R, D, QR, kvb = KV_RANK, ROPE, DIM, 1536, 64

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    inv = torch.rand(R // 2, device=dev)
    for m in (1, 4, 16):
        nb = ctx // kvb
        bufs = max(1, min(8, (400 << 20) // (m * ctx * L * 2)))
        c0, c1 = [rnd(m * nb, kvb, L) for _ in range(bufs)], [rnd(m * nb, kvb, L + R) for _ in range(bufs)]
        bt, slot = torch.arange(m * nb, dtype=torch.int32, device=dev).view(m, nb), torch.arange(m, dtype=torch.int32, device=dev)
        kvlen, ones = torch.full((m,), ctx, dtype=torch.int32, device=dev), torch.ones(m, dtype=torch.int32, device=dev)
        q0, q1 = rnd(m, heads, L), rnd(m, heads, L + R)
        grp = SegGroup(0, m, 0, m, 1)
        add(f"latent_mma + merge, {m} rows, {heads} heads, {ctx} keys",
            (lambda j: ops.latent_attention(q0, c0[j], grp, slot, kvlen, (slot, slot, ones), bt, kvb, 0.088, 64), m * ctx * L * 2.0,
             4.0 * m * heads * ctx * L, bufs), "mla_attn + combine",
            (lambda j: ops.mla_attention(q1, c1[j], slot, kvlen, bt, kvb, heads, L, R, 0.07, nsplit=64), m * ctx * (L + R) * 2.0,
             2.0 * m * heads * ctx * (2 * L + R), bufs))
        del c0, c1
    for m in (1, 16, prompt):
        bufs = max(1, min(8, (400 << 20) // (m * width * 4)))
        x0, y0 = [rnd(m, width, dtype=torch.float32) for _ in range(bufs)], [rnd(m, width, dtype=torch.float32) for _ in range(bufs)]
        xb, yb = [rnd(m, width) for _ in range(bufs)], [rnd(m, width) for _ in range(bufs)]
        w32, w16 = torch.ones(width, device=dev), rnd(width)
        add(f"add_normed, {m} rows", (lambda j: ops.add_normed(x0[j], y0[j], w32, width, 1e-6), m * width * 14.0, 0.0, bufs),
            "rmsnorm + residual", (lambda j: ops.rmsnorm(xb[j], w16, 1e-6, True, res=yb[j]), m * width * 8.0, 0.0, bufs))
        add(f"norm_rows, {m} rows", (lambda j: ops.norm_rows(x0[j], None, w32, width, 1e-6), m * width * 6.0, 0.0, bufs),
            "rmsnorm", (lambda j: ops.rmsnorm(xb[j], w16, 1e-6, True), m * width * 4.0, 0.0, bufs))
        nb = max(1, m // kvb)
        slot = torch.zeros(m, dtype=torch.int32, device=dev) if m > kvb else torch.arange(m, dtype=torch.int32, device=dev)
        pos = torch.arange(m, dtype=torch.int32, device=dev) if m > kvb else torch.zeros(m, dtype=torch.int32, device=dev)
        bt = torch.arange((1 if m > kvb else m) * nb, dtype=torch.int32, device=dev).view(-1, nb)
        d = LatentDims(heads, QR, L, QR, L, D, 0.088, 0)
        pb = 8 if m > kvb else 32
        proj = [rnd(m, QR + L, dtype=torch.float32) for _ in range(pb)]
        cl = torch.zeros(m * kvb if m <= kvb else m, L, dtype=torch.bfloat16, device=dev).view(-1, kvb, L)
        cm = torch.zeros(cl.shape[0], kvb, L + R, dtype=torch.bfloat16, device=dev)
        kva, qq, qa, qn, kn = [rnd(m, L + R) for _ in range(pb)], rnd(m, heads * (D + R)), [rnd(m, QR) for _ in range(pb)], rnd(QR), rnd(L)

        def mla_norms(j):
            ops.rmsnorm(qa[j], qn, 1e-6, True)
            ops.mla_prep(qq, kva[j], kn, None, inv, slot, pos, bt, cm, kvb, heads, D, L, R, 1e-6, absorb=False)
        add(f"latent_prep, {m} rows", (lambda j: ops.latent_prep(proj[j], d, w32[:QR], w32[:L], slot, pos, bt, cl, kvb, 1e-6),
                                       m * (QR + L) * 6.0, 0.0, pb),
            "rmsnorm + mla_prep", (mla_norms, m * (QR * 4.0 + (L + R) * 4.0 + heads * R * 4.0), 0.0, pb))
        tab, gr = rnd(VOCAB, width), rnd(65522, width)
        tok = [torch.randint(0, VOCAB, (m,), device=dev).to(torch.int32) for _ in range(8)]
        tp = torch.zeros(cl.shape[0], kvb, dtype=torch.int32, device=dev)
        add(f"embed_grams, {m} rows", (lambda j: ops.embed_grams(tab, gr, tok[j], slot, pos, bt, tp, kvb, 64.0, 65521, 31, 7),
                                       m * width * 10.0, 0.0, 8), "embed", (lambda j: ops.embed(tab, tok[j]), m * width * 4.0, 0.0, 8))
        del tab, gr, x0, y0, xb, yb
    for m in (1, 16):
        z = [rnd(m, 129280, dtype=torch.float32) for _ in range(8)]
        add(f"softcap, {m} rows of 129280", (lambda j: ops.softcap(z[j], 30.0), m * 129280 * 8.0, 0.0, 8), "argmax",
            (lambda j: ops.argmax(z[j]), m * 129280 * 4.0, 0.0, 8))
    ff, inter = 4 * width, (8 * width // 3 + 127) // 128 * 128
    for m in (1, 4, 16, prompt):
        x, xw = rnd(m, width), m * width * 2.0
        up, gu = [rnd(ff, width, scale=0.02) for _ in range(4)], [rnd(2 * inter, width, scale=0.02) for _ in range(4)]
        add(f"linear + relu^2, {m} rows, {width} -> {ff}", (lambda j: ops.linear(x, up[j], act="relu2"), ff * width * 2.0 + xw + m * ff * 2.0,
                                                            2.0 * m * ff * width, 4), "linear + SwiGLU",
            (lambda j: ops.linear(x, gu[j], swiglu=True), inter * width * 4.0 + xw + m * inter * 2.0, 4.0 * m * inter * width, 4))
        wo = [rnd(width, heads * D, scale=0.02) for _ in range(8)]
        o, res = rnd(m, heads * D), rnd(m, width)
        add(f"linear, fp32 sums, {m} rows, {heads * D} -> {width}",
            (lambda j: ops.linear(o, wo[j], out_f32=True), width * heads * D * 2.0 + m * (heads * D * 2.0 + width * 4.0),
             2.0 * m * width * heads * D, 8), "linear + residual",
            (lambda j: ops.linear(o, wo[j], res=res), width * heads * D * 2.0 + m * (heads * D * 2.0 + width * 4.0), 2.0 * m * width * heads * D, 8))
        del up, gu, wo
    # prompt attention: expansion GEMM and flash kernel of one whole prompt
    T, nb = prompt, prompt // kvb
    perm = torch.randperm(nb, device=dev).to(torch.int32).view(1, nb)
    c0, c1 = rnd(nb, kvb, L), rnd(nb, kvb, L + R)
    kv_up, kv_b = rnd(2 * heads * D, L, scale=L ** -0.5), rnd(2 * heads * D, L, scale=L ** -0.5)
    q0, q1, qabs = rnd(T, heads * D), rnd(T, heads * (D + R)), rnd(T, heads, L + R)
    (grp,) = seg_groups([(0, 0, T)], 1, T, T, 32, perm, kvb, dev)
    s0 = (i32([0]), i32([0]), i32([T]), i32([0]))
    d = LatentDims(heads, QR, L, QR, L, D, 0.088, 0)
    out = torch.empty_like(q0)
    work = 2.0 * T * L * 2 * heads * D
    tri = T * (T + 1) / 2.0
    torch.cuda.synchronize(dev)
    ms = t.run(lambda: ops.latent_attention_prompt(q0, ops.latent_rows(c0, grp, kvb), kv_up, d, grp, s0, kvb, out))
    lms = t.run(lambda: ops.mla_attention_prefill(q1, qabs, c1, kv_b, [(0, 0, T)], s0[1], s0[2], s0[3], perm, kvb, heads, D, D, L, R))
    fl, lfl = work + tri * heads * 4 * D, work + tri * heads * 2 * (2 * D + R)
    rows.append({"kernel": f"prompt attention (gather, expansion GEMM, flash with 16-bit weight remainders), {T} rows", "ms": round(ms, 5),
                 "frac": round(fl / (tf * 1e9) / ms, 3), "like": "mla prompt attention (gather, GEMM, packing, flash)",
                 "like_ms": round(lms, 5), "like_frac": round(lfl / (tf * 1e9) / lms, 3)})
    kv = ops.linear(ops.latent_rows(c0, grp, kvb), kv_up).view(-1, kvb, 2, heads, D)

    def flash(exact):
        return lambda j: ops.C.attn_prefill_tc(out, q0, kv[:, :, 0], kv[:, :, 1], q0, grp.own, s0[1], s0[2], s0[3], grp.context()[1], kvb, T, heads,
                                               heads, D, False, ops.status_word, scale=0.088, exact_p=exact)
    add(f"flash, softmax weights as value + remainder, {T} rows, {heads} heads of {D}", (flash(True), 0.0, tri * heads * 4 * D, 1),
        "flash, bf16 softmax weights", (flash(False), 0.0, tri * heads * 4 * D, 1))
    assert ops.status() == 0
    return rows


def kernels_dofunex(dev, heads: int = 32, kv_heads: int = 8, width: int = 4096, ctx: int = 4096, prompt: int = 2048) -> List[Dict]:
    """Dofunex's kernels beside those of the dense hybrid (heads of 128 columns, four taps, ranks of 128)."""
    from ..models.weights import DeltaDims, GqaDims
    from ..ops.cuda_ops import CudaOps
    from ..ops.latent import SegGroup
    from ..ops.mixers import LOWRANK_ROWS
    ops, acc = CudaOps(dev), _Rows(dev)
    add = acc.add
    D, kvb, K, R, H, G = DIM, 64, 4, 128, heads, kv_heads
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    f32 = lambda *s: torch.randn(*s, device=dev)
    inv, inv64 = torch.rand(D // 2, device=dev), torch.rand(D // 2, device=dev, dtype=torch.float64)
    gd, sink = GqaDims(H, G, D, D, D ** -0.5, D, H * D, True), f32(H)
    nw = rnd(D)
    # rows between the products
    for m in (1, 16, prompt):
        bufs = max(1, min(8, (400 << 20) // (m * width * 4)))
        x0, y0 = [f32(m, width) for _ in range(bufs)], [f32(m, width) for _ in range(bufs)]
        xb, yb = [rnd(m, width) for _ in range(bufs)], [rnd(m, width) for _ in range(bufs)]
        w32, w16 = torch.ones(width, device=dev), rnd(width)
        add(f"add_normed (bias, norm of y, add, next norm), {m} rows", (lambda j: ops.add_normed(x0[j], y0[j], w32, width, 1e-6, bias=w32, next_w=w32),
                                                                          m * width * 14.0, 0.0, bufs),
            "rmsnorm + residual", (lambda j: ops.rmsnorm(xb[j], w16, 1e-6, True, res=yb[j]), m * width * 8.0, 0.0, bufs))
        # attention: projection to operands
        nb = max(1, m // kvb)
        many = m > kvb
        slot = torch.zeros(m, dtype=torch.int32, device=dev) if many else torch.arange(m, dtype=torch.int32, device=dev)
        pos = torch.arange(m, dtype=torch.int32, device=dev) if many else torch.zeros(m, dtype=torch.int32, device=dev)
        bt = torch.arange((1 if many else m) * nb, dtype=torch.int32, device=dev).view(-1, nb)
        kc, vc = rnd(bt.numel(), kvb, G, D), rnd(bt.numel(), kvb, G, D)
        pb = 8 if many else 32
        proj, bias = [f32(m, (H + G) * D) for _ in range(pb)], f32((H + G) * D)
        pq = [rnd(m, (2 * H + 2 * G) * D) for _ in range(pb)]
        add(f"gqa_prep, {m} rows, {H} / {G} heads", (lambda j: ops.gqa_prep(proj[j], gd, bias, inv64, slot, pos, bt, kc, vc, kvb, 1e-6),
                                                      m * D * ((H + G) * 4.0 + (H + 2 * G) * 2.0), 0.0, pb),
            "attn_prep", (lambda j: ops.attn_prep(pq[j], nw, nw, inv, slot, pos, bt, kc, vc, kvb, H, G, D, D, True, 1e-6),
                          m * D * (H + 2 * G) * 4.0, 0.0, pb))
        del x0, y0, xb, yb, proj, pq
    for m in (1, 4, 16):
        nb = ctx // kvb
        bufs = max(1, min(8, (400 << 20) // (m * ctx * G * D * 4)))
        kc, vc = [rnd(m * nb, kvb, G, D) for _ in range(bufs)], [rnd(m * nb, kvb, G, D) for _ in range(bufs)]
        bt, slot = torch.arange(m * nb, dtype=torch.int32, device=dev).view(m, nb), torch.arange(m, dtype=torch.int32, device=dev)
        kvlen, ones = torch.full((m,), ctx, dtype=torch.int32, device=dev), torch.ones(m, dtype=torch.int32, device=dev)
        q, out, pj = rnd(m, H, D), rnd(m, H, D), rnd(m, 2 * H * D)
        grp = SegGroup(0, m, 0, m, 1)
        work = (m * ctx * G * D * 4.0, 4.0 * m * H * ctx * D, bufs)
        add(f"decode attention + merge with sink, weights as value + remainder, {m} rows, {ctx} keys",
            (lambda j: ops.gqa_attention(q, gd, kc[j], vc[j], sink, grp, slot, kvlen, (slot, slot, ones), bt, kvb, 64, out), *work), "attention + combine",
            (lambda j: ops.attention(q, pj, kc[j], vc[j], slot, kvlen, bt, kvb, H, G, D, True, nsplit=64, segs=(slot, slot, ones, 1)), *work))
        del kc, vc
    T, nb = prompt, prompt // kvb
    perm = torch.randperm(nb, device=dev).to(torch.int32).view(1, nb)
    kc, vc, q, out, pj = rnd(nb, kvb, G, D), rnd(nb, kvb, G, D), rnd(T, H, D), rnd(T, H, D), rnd(T, 2 * H * D)
    s0 = (i32([0]), i32([0]), i32([T]), i32([0]))
    rslot, rlen = torch.zeros(T, dtype=torch.int32, device=dev), torch.arange(1, T + 1, dtype=torch.int32, device=dev)
    grp = SegGroup(0, 1, 0, T, T, True)
    work = (0.0, T * (T + 1) / 2.0 * H * 4 * D, 1)
    add(f"prompt attention with sink, weights as value + remainder, {T} rows",
        (lambda j: ops.gqa_attention(q, gd, kc, vc, sink, grp, rslot, rlen, s0, perm, kvb, 1, out), *work), "prompt attention, bf16 weights",
        (lambda j: ops.attention_prefill(q, pj, kc, vc, *s0, perm, kvb, H, G, D, True, T), *work))
    # delta rule
    d = DeltaDims(H, H, D, D, K, R, R, H * D)
    sizes = [H, H, D, D, K, d.q_off]
    w = dict(decay_up=rnd(H * D, R, scale=R ** -0.5), gate_up_lr=rnd(H * D, R, scale=R ** -0.5), conv=f32(d.channels, K), A_log=f32(H),
             dt_bias=f32(H * D) - 3, gnorm_w=f32(D))
    cw, A, dtb, gw = rnd(3 * H * D, K), f32(H), f32(H), rnd(D)
    for m in (1, 4, 16):
        bufs = max(2, min(64, (400 << 20) // (m * H * D * D * 4)))
        rec, tail = [f32(m, H, D, D) for _ in range(bufs)], [rnd(m, K - 1, d.channels) for _ in range(bufs)]
        proj, pg = rnd(m, d.b_off + H), rnd(m, 4 * H * D + 2 * H)
        up = f32(m, 2 * H * D)
        slot, ones, out = torch.arange(m, dtype=torch.int32, device=dev), torch.ones(m, dtype=torch.int32, device=dev), rnd(m, H * D)
        state = m * H * D * D * 8.0
        add(f"cd_step, {m} rows, {H} heads", (lambda j: ops.C.cd_step(out, rec[j], tail[j], proj, up[:, :H * D], up[:, H * D:], w["conv"], w["A_log"],
                                                                       w["dt_bias"], w["gnorm_w"], slot, slot, ones, sizes, 1e-6, True),
                                               state + m * H * D * 24.0, 0.0, bufs), "gdn_step",
            (lambda j: ops.gdn_step(pg, cw, rec[j], tail[j], A, dtb, gw, slot, slot, ones, H, H, D, D, 1e-6), state + m * H * D * 20.0, 0.0, bufs))
        ups = [(rnd(H * D, R), rnd(H * D, R)) for _ in range(32)]
        wo = [rnd(2 * H * D, R) for _ in range(32)]
        xr = rnd(m, R)

        def low_rank(j):
            if m <= LOWRANK_ROWS:
                ops.C.cd_lowrank(up, proj, *ups[j])
            else:
                ops.linear(proj[:, :R], ups[j][0], out_f32=True)
                ops.linear(proj[:, R:2 * R], ups[j][1], out_f32=True)
        work = (H * D * R * 4.0 + m * H * D * 8.0, 4.0 * m * H * D * R, 32)
        add(f"low-rank products, {m} rows", (low_rank, *work), "linear of the same bytes", (lambda j: ops.linear(xr, wo[j], out_f32=True), *work))
        del rec, tail
    rec, tail = f32(1, H, D, D), rnd(1, K - 1, d.channels)
    proj, pg = rnd(T, d.b_off + H), rnd(T, 4 * H * D + 2 * H)
    decay = f32(T, H * D)
    scratch = ops.scratch("cd_chunk", ops.C.cd_chunk_scratch_bytes(T, 1, H, D) // 4, torch.float32)
    y, gate = f32(T, H, D), f32(T, H * D)
    # 64-row chunks: the Gram products, the solve and the five products with the state, per head
    fl = T / 64 * H * (4 * 64 * 64 * D + 64 * 64 * 64 / 3 + 6 * 64 * D * D + 4 * 64 * 64 * D)
    one = (i32([0]), i32([0]), i32([T]))
    add(f"cd_chunk (prep + scan), {T} rows, {H} heads",
        (lambda j: ops.C.cd_chunk(y, rec, scratch, tail, proj, decay, w["conv"], w["A_log"], w["dt_bias"], *one, T, sizes), T * H * D * 14.0, fl, 1),
        "gdn_conv + gdn_chunk",
        (lambda j: ops.gdn_rec(ops.gdn_conv(pg, cw, tail, *one, 3 * H * D, T), pg, rec, tail, A, dtb, *one, H, H, D, D, 1e-6, chunked=True, max_rows=T),
         T * H * D * 10.0, fl, 1))
    gout = rnd(T, H * D)
    add(f"gated head norm, {T} rows", (lambda j: ops.C.gated_norm_sigmoid(gout, y, gate, w["gnorm_w"], 1e-6), T * H * D * 10.0, 0.0, 1), "gated_norm",
        (lambda j: ops.gated_norm(y.view(T, H * D), pg, 3 * H * D, gw, H, D, 1e-6), T * H * D * 8.0, 0.0, 1))
    assert ops.status() == 0
    return acc.rows


def kernels_rakizen(dev, heads: int = 32, kv_heads: int = 8, width: int = 4096, ctx: int = 4096, prompt: int = 2048, size: int = 1024) -> List[Dict]:
    """Rakizen's kernels beside those of the sequential grouped-query attention model (heads of 128 columns; two maps of 64 over values of 128
    in half the heads). Bounded rows see `size` keys; the like kernel of few rows gets a cache of that many."""
    from ..models.weights import GqaDims
    from ..ops.cuda_ops import CudaOps
    from ..ops.latent import SegGroup
    ops, acc = CudaOps(dev), _Rows(dev)
    add = acc.add
    D, kvb, H, G = DIM, 64, heads, kv_heads
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    f32 = lambda *s: torch.randn(*s, device=dev)
    inv, inv64 = torch.rand(D // 2, device=dev), torch.rand(D // 2, device=dev, dtype=torch.float64)
    one = GqaDims(H, G, D, D, D ** -0.5, D, (H + G) * D, False, D, 1, True, 30.0, size)
    two = GqaDims(H // 2, G // 2, D // 2, D, (D // 2) ** -0.5, 0, (H + G) * D // 2, False, D, 2, False, 30.0, 0, size, 0.5, (H + G) * D // 2 + G * D // 2)
    nw, lam = rnd(D), torch.full((1,), 0.7, device=dev)
    for m in (1, 16, prompt):
        bufs = max(1, min(8, (400 << 20) // (m * width * 4)))
        x0, y0 = [f32(m, width) for _ in range(bufs)], [f32(m, width) for _ in range(bufs)]
        xb, yb = [rnd(m, width) for _ in range(bufs)], [rnd(m, width) for _ in range(bufs)]
        w32, w16 = torch.ones(width, device=dev), rnd(width)
        add(f"add_layer_norm (add, next norm), {m} rows", (lambda j: ops.add_layer_norm(x0[j], y0[j], width, 1e-6, w32, w32), m * width * 14.0, 0.0, bufs),
            "rmsnorm + residual", (lambda j: ops.rmsnorm(xb[j], w16, 1e-6, True, res=yb[j]), m * width * 8.0, 0.0, bufs))
        nb, many = max(1, m // kvb), m > kvb
        slot = torch.zeros(m, dtype=torch.int32, device=dev) if many else torch.arange(m, dtype=torch.int32, device=dev)
        pos = torch.arange(m, dtype=torch.int32, device=dev) if many else torch.zeros(m, dtype=torch.int32, device=dev)
        bt = torch.arange((1 if many else m) * nb, dtype=torch.int32, device=dev).view(-1, nb)
        kc, vc = rnd(bt.numel(), kvb, G, D), rnd(bt.numel(), kvb, G, D)
        kc2, vc2 = rnd(bt.numel(), kvb, G // 2, D), rnd(bt.numel(), kvb, G // 2, D)
        pb = 8 if many else 32
        proj, norms = [f32(m, (H + 2 * G) * D) for _ in range(pb)], (f32(H * D), f32(G * D))
        pq = [rnd(m, (H + 2 * G) * D) for _ in range(pb)]
        like = ("attn_prep", (lambda j: ops.attn_prep(pq[j], nw, nw, inv, slot, pos, bt, kc, vc, kvb, H, G, D, D, False, 1e-6),
                              m * D * (H + 2 * G) * 4.0, 0.0, pb))
        add(f"gqa_row_prep, row norms and rotation, {m} rows, {H} / {G} heads",
            (lambda j: ops.gqa_prep(proj[j], one, None, inv64, slot, pos, bt, kc, vc, kvb, 1e-6, norms=norms), m * D * (H + 2 * G) * 6.0, 0.0, pb), *like)
        half = D * (H // 2 + G)                              # projected columns: H / 2 heads of two maps of D / 2, G / 2 keys and values of D
        add(f"gqa_row_prep, two maps, {m} rows, {H // 2} / {G // 2} heads",
            (lambda j: ops.gqa_prep(proj[j], two, None, inv64[:0], slot, pos, bt, kc2, vc2, kvb, 1e-6), m * (half * 4.0 + D * (H + G) * 2.0), 0.0, pb), *like)
        rows, gate, o = f32(m, H, D), f32(m, H // 2 * D), rnd(m, H // 2, D)
        if many:
            add(f"head_mix (difference, norm, gate), {m} rows", (lambda j: ops.C.head_mix(o, rows, lam, gate, 0.4, 2, D, 1e-6), m * H * D * 7.0, 0.0, 1),
                "gated_norm", (lambda j: ops.gated_norm(rows.view(m, H * D), pq[0], 0, nw, H, D, 1e-6), m * H * D * 8.0, 0.0, 1))
        del x0, y0, xb, yb, proj, pq, rows
    for m in (1, 4, 16):
        nb, nbl = ctx // kvb, size // kvb
        bufs = max(1, min(32, (400 << 20) // (m * size * G * D * 4)))
        kc, vc = [rnd(m * nb, kvb, G, D) for _ in range(min(bufs, 8))], [rnd(m * nb, kvb, G, D) for _ in range(min(bufs, 8))]
        kl, vl = [rnd(m * nbl, kvb, G, D) for _ in range(bufs)], [rnd(m * nbl, kvb, G, D) for _ in range(bufs)]
        bt, slot = torch.arange(m * nb, dtype=torch.int32, device=dev).view(m, nb), torch.arange(m, dtype=torch.int32, device=dev)
        btl = torch.arange(m * nbl, dtype=torch.int32, device=dev).view(m, nbl)
        kvlen, lenl, ones = (torch.full((m,), v, dtype=torch.int32, device=dev) for v in (ctx, size, 1))
        q, out, out2, pj, gate = rnd(m, H, D), rnd(m, H, D), rnd(m, H // 2, D), rnd(m, H * D), f32(m, H // 2 * D)
        grp = SegGroup(0, m, 0, m, 1)
        work = (m * size * G * D * 4.0, 4.0 * m * H * size * D, bufs)
        like = ("attention + combine", (lambda j: ops.attention(q, pj, kl[j], vl[j], slot, lenl, btl, kvb, H, G, D, False, nsplit=16,
                                                                segs=(slot, slot, ones, 1)), *work))
        nk = len(kc)
        add(f"decode attention + merge, softcap, window of {size}, {m} rows",
            (lambda j: ops.gqa_attention(q, one, kc[j % nk], vc[j % nk], None, grp, slot, kvlen, (slot, slot, ones), bt, kvb, 64, out), work[0], work[1], nk), *like)
        c2, v2 = [c.view(-1, kvb, G // 2, D) for c in kc], [c.view(-1, kvb, G // 2, D) for c in vc]
        work2 = (m * size * G // 2 * D * 4.0, m * H * size * D * 3.0, nk)
        add(f"decode attention + merge, two maps, gate, chunk of {size}, {m} rows",
            (lambda j: ops.gqa_attention(q, two, c2[j % nk], v2[j % nk], None, grp, slot, kvlen, (slot, slot, ones), bt, kvb, 64, out2, lam=lam, gate=gate,
                                         eps=1e-6), *work2), *like)
        del kc, vc, kl, vl, c2, v2
    T, nb = prompt, prompt // kvb
    perm = torch.randperm(nb, device=dev).to(torch.int32).view(1, nb)
    kc, vc, q, out, pj = rnd(nb, kvb, G, D), rnd(nb, kvb, G, D), rnd(T, H, D), rnd(T, H, D), rnd(T, H * D)
    k2, v2, o2, gate = rnd(nb, kvb, G // 2, D), rnd(nb, kvb, G // 2, D), rnd(T, H // 2, D), f32(T, H // 2 * D)
    s0 = (i32([0]), i32([0]), i32([T]), i32([0]))
    rslot, rlen = torch.zeros(T, dtype=torch.int32, device=dev), torch.arange(1, T + 1, dtype=torch.int32, device=dev)
    grp = SegGroup(0, 1, 0, T, T, True)
    like = ("prompt attention, bf16 weights", (lambda j: ops.attention_prefill(q, pj, kc, vc, *s0, perm, kvb, H, G, D, False, T), 0.0,
                                               T * (T + 1) / 2.0 * H * 4 * D, 1))
    # rows see the keys of their chunk as rows of separate prompts of that length see theirs
    n = T // size
    parts = (torch.arange(n, dtype=torch.int32, device=dev), torch.arange(0, T, size, dtype=torch.int32, device=dev), i32([size] * n), i32([0] * n))
    like_chunks = (f"prompt attention, bf16 weights, {n} prompts of {size}",
                   (lambda j: ops.attention_prefill(q, pj, kc, vc, *parts, perm.view(n, -1), kvb, H, G, D, False, size), 0.0,
                    n * size * (size + 1) / 2.0 * H * 4 * D, 1))
    for sz in (size, T):
        one, two = replace(one, window=sz), replace(two, chunk=sz)
        seen1, seen2 = sum(min(t + 1, sz) for t in range(T)), sum(t % sz + 1 for t in range(T))
        add(f"prompt attention, softcap, window of {sz}, {T} rows",
            (lambda j: ops.gqa_attention(q, one, kc, vc, None, grp, rslot, rlen, s0, perm, kvb, 1, out), 0.0, seen1 * H * 4.0 * D, 1), *like)
        add(f"prompt attention, two maps, difference, gate, chunk of {sz}, {T} rows",
            (lambda j: ops.gqa_attention(q, two, k2, v2, None, grp, rslot, rlen, s0, perm, kvb, 1, o2, lam=lam, gate=gate, eps=1e-6), 0.0,
             seen2 * H * 3.0 * D, 1), *(like if sz == T else like_chunks))
    del kc, vc, k2, v2
    # products: both output projections at once, beside the two of the sequential model; in_proj with fp32 sums
    ff = 3 * width
    for m in (1, 4, 16, prompt):
        both, o, a, res = rnd(m, H * D + ff), rnd(m, H * D), rnd(m, ff), rnd(m, width)
        wj = [rnd(width, H * D + ff, scale=0.02) for _ in range(4)]
        wo, wd = [rnd(width, H * D, scale=0.02) for _ in range(4)], [rnd(width, ff, scale=0.02) for _ in range(4)]
        work = (width * (H * D + ff) * 2.0 + m * ((H * D + ff) * 2.0 + width * 4.0), 2.0 * m * width * (H * D + ff), 4)
        add(f"joint output projection, fp32 sums, {m} rows, {H * D} + {ff} -> {width}", (lambda j: ops.linear(both, wj[j], out_f32=True), *work),
            "two linears + residual", (lambda j: ops.linear(a, wd[j], res=ops.linear(o, wo[j], res=res)), *work))
        del wj, wo, wd
        wi, x = [rnd((H + 2 * G) * D, width, scale=0.02) for _ in range(8)], rnd(m, width)
        n = (H + 2 * G) * D
        add(f"input projection, fp32 sums, {m} rows, {width} -> {n}",
            (lambda j: ops.linear(x, wi[j], out_f32=True), n * width * 2.0 + m * (width * 2.0 + n * 4.0), 2.0 * m * n * width, 8), "linear, norm in front",
            (lambda j: ops.linear(x, wi[j], norm_w=res[0], eps=1e-6), n * width * 2.0 + m * (width * 2.0 + n * 2.0), 2.0 * m * n * width, 8))
        del wi
    # routed feed-forward: 64 experts of 1024, six per token, four of eight groups
    E, K, F, W = 64, 6, 1024, 2048
    gu, dn = rnd(E, 2 * F, W, scale=0.02), rnd(E, W, F, scale=0.02)
    for m in (1, 4, 16):
        h, x, y, res = rnd(m, W), f32(m, W), f32(m, W), rnd(m, W)
        picks = [ops.moe_route(f32(m, E), None, 1, K, 8, 4, 2.0) for _ in range(16)]
        used = sum(len(set(ids.reshape(-1).tolist())) for ids, _ in picks) / 16
        w32 = torch.ones(W, device=dev)
        work = (used * 3.0 * F * W * 2, 6.0 * m * K * F * W, 16)
        add(f"expert rows + add_layer_norm, {m} rows",
            (lambda j: ops.add_layer_norm(x, y, W, 1e-6, w32, w32, (ops.expert_rows(h, picks[j][0], gu, dn), picks[j][1])), *work),
            "moe_experts (pairs, combine)", (lambda j: ops.moe_experts(h, *picks[j], gu, dn, 0, E, None, None, res), *work))
    from ..parallel.ep import ExpertParallel
    h, y, res = rnd(T, W), f32(T, W), rnd(T, W)
    ids, wts = ops.moe_route(f32(T, E), None, 1, K, 8, 4, 2.0)
    ep = ExpertParallel(None, torch.device(dev), E, W, T * K, status=ops.status_word)
    work = (E * 3.0 * F * W * 2, 6.0 * T * K * F * W, 1)
    add(f"grouped experts added in fp32, {T} rows", (lambda j: ep.moe(ops, h, ids, wts, gu, dn, acc=y), *work), "grouped experts + residual",
        (lambda j: ep.moe(ops, h, ids, wts, gu, dn, res=res), *work))
    for grp_n, keep in ((8, 4), (16, 5)):
        z, zl = f32(T, 48 if grp_n == 16 else E), f32(T, E)
        n = z.shape[1]
        add(f"router, {n} experts, {keep} of {grp_n} groups, {T} rows", (lambda j: ops.moe_route(z, None, 1, K, grp_n, keep, 2.0), T * (n + 2 * K) * 4.0, 0.0, 1),
            "router, 4 of 8 groups", (lambda j: ops.moe_route(zl, None, 1, K, 8, 4, 2.0), T * (E + 2 * K) * 4.0, 0.0, 1))
    assert ops.status() == 0
    return acc.rows


def kernels_pironex(dev, heads: int = 16, kv_heads: int = 4, width: int = 2048, ctx: int = 4096, prompt: int = 2048, size: int = 1024,
                    pool: int = 16) -> List[Dict]:
    """Pironex's kernels beside those of the routed Gated DeltaNet hybrid and, for its latent attention, of the MLA model. Bounded rows see `size`
    keys and the means before them; the like kernel of few rows gets a cache of as many keys."""
    from ..models.weights import GqaDims, LatentDims, SsmDims
    from ..ops.cuda_ops import CudaOps
    from ..ops.latent import SegGroup
    from ..parallel.ep import ExpertParallel
    ops, acc = CudaOps(dev), _Rows(dev)
    add = acc.add
    D, L, R, kvb, H, G, W, T = DIM, KV_RANK, ROPE, 64, heads, kv_heads, width, prompt
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    f32 = lambda *s: torch.randn(*s, device=dev)
    full = lambda m, v: torch.full((m,), v, dtype=torch.int32, device=dev)
    inv, inv64 = torch.rand(D // 2, device=dev), torch.rand(D // 2, device=dev, dtype=torch.float64)
    att = GqaDims(H, G, D, D, D ** -0.5, D // 2, (H + G) * D, False, D, row_norm=True, softcap=50.0, window=size, rot_half=True, pool=pool)
    lat = LatentDims(H, 0, L, 0, L + R, D + R, (D + R) ** -0.5, 0, D, L, D, R, size)
    E, K, F = 64, 6, 1024
    for m in (1, 16, T):
        many, n = m > 64, 3
        slot = torch.zeros(m, dtype=torch.int32, device=dev) if many else torch.arange(m, dtype=torch.int32, device=dev)
        pos = torch.arange(m, dtype=torch.int32, device=dev) if many else torch.zeros(m, dtype=torch.int32, device=dev)
        bufs = max(1, min(8, (400 << 20) // (m * W * 4)))
        x, y = [f32(m, W) for _ in range(bufs)], [f32(m, W) for _ in range(bufs)]
        xb, yb = [rnd(m, W) for _ in range(bufs)], [rnd(m, W) for _ in range(bufs)]
        w32, w16, cw, tails = torch.ones(W, device=dev), rnd(W), f32(4, W), rnd(64, n, W)
        place, xs = 8, [f32(10, m, W) for _ in range(max(1, bufs // 4))]
        dwa, one = torch.rand(place + 1, device=dev), dict(conv=(cw, tails), row_slot=slot, row_pos=pos, single=not many)
        like = ("rmsnorm + residual", (lambda j: ops.rmsnorm(xb[j], w16, 1e-6, True, res=yb[j]), m * W * 8.0, 0.0, bufs))
        conv_bytes = m * W * (4.0 if many else 14.0)               # the convolution's own pass, or the tails of every row
        add(f"seam: norm of y, add, norm, convolution, {m} rows", (lambda j: ops.add_conv_normed(x[j], x[j], y[j], w32, W, 1e-6, w32, **one),
                                                                  m * W * 14.0 + conv_bytes, 0.0, bufs), *like)
        add(f"seam with an average over {place + 1} results, {m} rows",
            (lambda j: ops.add_conv_normed(x[j], x[j], y[j], w32, W, 1e-6, w32, average=(xs[j % len(xs)], place, dwa), **one),
             m * W * (14.0 + 4.0 * place + 4.0) + conv_bytes, 0.0, bufs), *like)
        nb = max(1, m // kvb)
        bt = torch.arange((1 if many else m) * nb, dtype=torch.int32, device=dev).view(-1, nb)
        kc, vc, pb = rnd(bt.numel(), kvb, G, D), rnd(bt.numel(), kvb, G, D), 8 if many else 32
        means = tuple(rnd(bt.numel(), kvb // pool, G, D) for _ in "kv")
        proj, norms, pq = [f32(m, (H + 2 * G) * D) for _ in range(pb)], (f32(H * D), f32(G * D)), [rnd(m, (2 * H + 2 * G) * D) for _ in range(pb)]
        nw, segs = rnd(D), (i32([0]), i32([0]), i32([m])) if many else (slot, slot * 0, full(m, 1))

        def prep(j):
            ops.gqa_prep(proj[j], att, None, inv64, slot, pos, bt, kc, vc, kvb, 1e-6, norms=norms)
            ops.pool_keys(att, kc, vc, means, *segs, m if many else 1, bt, kvb)
        attn_prep = ("attn_prep", (lambda j: ops.attn_prep(pq[j], nw, nw, inv, slot, pos, bt, kc, vc, kvb, H, G, D, D // 2, True, 1e-6),
                                   m * D * (H + 2 * G) * 4.0, 0.0, pb))
        add(f"gqa_row_prep + pool_keys, {m} rows, {H} / {G} heads", (prep, m * D * ((H + 2 * G) * 6.0 + (4.0 * G if many else 0.0)), 0.0, pb), *attn_prep)
        pl, cl, kn = [f32(m, H * (D + R) + L + R) for _ in range(pb)], rnd(bt.numel(), kvb, L + R), torch.ones(L + R, device=dev)
        qq, kva, k16, inv_r = rnd(m, H * (D + R)), [rnd(m, L + R) for _ in range(pb)], rnd(L), torch.rand(R // 2, device=dev)
        add(f"latent_rot_prep, {m} rows", (lambda j: ops.latent_rot_prep(pl[j], lat, kn, inv64[:R // 2], slot, pos, bt, cl, kvb, 1e-6),
                                           m * (H * (D + R) + L + R) * 6.0, 0.0, pb),
            "mla_prep", (lambda j: ops.mla_prep(qq, kva[j], k16, None, inv_r, slot, pos, bt, cl, kvb, H, D, L, R, 1e-6, absorb=False),
                         m * ((L + R) * 4.0 + H * R * 4.0), 0.0, pb))
        del x, y, xb, yb, xs, proj, pq, pl
    blocks = (ctx - size) // pool
    for m in (1, 4, 16):
        nb, seen = ctx // kvb, (size + blocks + kvb - 1) // kvb * kvb
        nbl = seen // kvb
        bufs = max(1, min(32, (400 << 20) // (m * seen * G * D * 4)))
        nk = min(bufs, 8)
        kc, vc = [rnd(m * nb, kvb, G, D) for _ in range(nk)], [rnd(m * nb, kvb, G, D) for _ in range(nk)]
        means = [tuple(rnd(m * nb, kvb // pool, G, D) for _ in "kv") for _ in range(nk)]
        kl, vl = [rnd(m * nbl, kvb, G, D) for _ in range(bufs)], [rnd(m * nbl, kvb, G, D) for _ in range(bufs)]
        slot, ones, full_len, like_len = torch.arange(m, dtype=torch.int32, device=dev), full(m, 1), full(m, ctx), full(m, seen)
        bt, btl = torch.arange(m * nb, dtype=torch.int32, device=dev).view(m, nb), torch.arange(m * nbl, dtype=torch.int32, device=dev).view(m, nbl)
        q, out, pj, grp = rnd(m, H, D), rnd(m, H, D), rnd(m, 2 * H * D), SegGroup(0, m, 0, m, 1)
        work = (m * (size + blocks) * G * D * 4.0, 4.0 * m * H * (size + blocks) * D)
        add(f"decode attention + merge, window of {size} and {blocks} means, {m} rows",
            (lambda j: ops.gqa_attention(q, att, kc[j], vc[j], None, grp, slot, full_len, (slot, slot, ones), bt, kvb, 64, out, pooled=means[j]), *work, nk),
            f"attention + combine, {seen} keys",
            (lambda j: ops.attention(q, pj, kl[j], vl[j], slot, like_len, btl, kvb, H, G, D, True, nsplit=32, segs=(slot, slot, ones, 1)), *work, bufs))
        del kc, vc, means, kl, vl
        nbl = size // kvb
        bufs = max(1, min(16, (400 << 20) // (m * ctx * (L + R) * 2)))
        c0, c1 = [rnd(m * nb, kvb, L + R) for _ in range(bufs)], [rnd(m * nbl, kvb, L + R) for _ in range(2 * bufs)]
        btl = torch.arange(m * nbl, dtype=torch.int32, device=dev).view(m, nbl)
        qa, short = rnd(m, H, L + R), full(m, size)
        work = (m * size * (L + R) * 2.0, 2.0 * m * H * size * (2 * L + R))
        add(f"latent_mma + merge, window of {size} in {ctx}, {m} rows",
            (lambda j: ops.latent_attention(qa, c0[j], grp, slot, full_len, (slot, slot, ones), bt, kvb, 0.07, 64, vlat=L, window=size), *work, bufs),
            f"mla_attn + combine, {size} keys", (lambda j: ops.mla_attention(qa, c1[j], slot, short, btl, kvb, H, L, R, 0.07, nsplit=16), *work, 2 * bufs))
        del c0, c1
    # prompt attention
    nb = T // kvb
    perm = torch.randperm(nb, device=dev).to(torch.int32).view(1, nb)
    s0, rslot, rlen = (i32([0]), i32([0]), i32([T]), i32([0])), torch.zeros(T, dtype=torch.int32, device=dev), torch.arange(1, T + 1, dtype=torch.int32, device=dev)
    kc, vc, q, out, pj = rnd(nb, kvb, G, D), rnd(nb, kvb, G, D), rnd(T, H, D), rnd(T, H, D), rnd(T, 2 * H * D)
    grp = SegGroup(0, 1, 0, T, T, True)
    grp.segments, grp.block_table, grp.kv_block = [(0, 0, T)], perm, kvb
    start, rows = i32([0]), (T - size) // pool
    km, vm = rnd(max(64, (rows + 63) // 64 * 64), G, D), rnd(max(64, (rows + 63) // 64 * 64), G, D)
    seen = sum(min(t + 1, size) + max(0, t + 1 - size) // pool for t in range(T))
    like = ("prompt attention, bf16 weights", (lambda j: ops.attention_prefill(q, pj, kc, vc, *s0, perm, kvb, H, G, D, True, T), 0.0,
                                               T * (T + 1) / 2.0 * H * 4 * D, 1))
    add(f"prompt attention, softcap, window of {size} and means, {T} rows",
        (lambda j: ops.C.attn_prefill_tc(out, q.view(T, -1), kc, vc, q.view(T, -1), s0[0], s0[1], s0[2], s0[3], perm, kvb, T, H, G, D, False,
                                         ops.status_word, scale=D ** -0.5, exact_p=True, window=size, softcap=50.0, k_mean=km, v_mean=vm,
                                         mean_start=start, pool=pool), 0.0, seen * H * 4.0 * D, 1), *like)
    c0, kv_up, kv_b = rnd(nb, kvb, L + R), rnd(H * (2 * D + R), L + R, scale=L ** -0.5), rnd(2 * H * D, L, scale=L ** -0.5)
    q1, ol, qabs = rnd(T, H * (D + R)), rnd(T, H * D), rnd(T, H, L + R)
    lat_seen, lat_all = sum(min(t + 1, size) for t in range(T)), T * (T + 1) / 2.0
    up0, up1 = 2.0 * T * (L * 2 * D) * H, 2.0 * T * L * 2 * H * D
    add(f"latent prompt attention (gather, expansion, flash), window of {size}, {T} rows",
        (lambda j: ops.latent_attention_prompt(q1, ops.latent_rows(c0, grp, kvb, size), kv_up, lat, grp, s0, kvb, ol), 0.0,
         up0 + lat_seen * H * 2.0 * (2 * D + R), 1), "mla prompt attention (gather, GEMM, packing, flash)",
        (lambda j: ops.mla_attention_prefill(q1, qabs, c0, kv_b, [(0, 0, T)], s0[1], s0[2], s0[3], perm, kvb, H, D, D, L, R), 0.0,
         up1 + lat_all * H * 2.0 * (2 * D + R), 1))
    # recurrences: 2 W / 64 heads of 64 with a state of 128, beside W / 128 heads of 128 x 128
    SH, SV, SN = 2 * W // 64, 64, 128
    d = SsmDims(SH, 1, SN, SV, 4, 1, SH * SV)
    w = dict(conv=f32(4, d.channels), conv_bias=f32(d.channels), A=-torch.rand(SH, device=dev), dt_bias=f32(SH) - 2, skip=f32(SH), gnorm_w=f32(d.inner))
    cw, A, dtb, gw = rnd(3 * H * D, 4), f32(H), f32(H), rnd(D)
    ld = (d.dt_off + SH + 7) // 8 * 8
    for m in (1, 4, 16):
        bufs = max(2, min(64, (400 << 20) // (m * SH * SN * SV * 4)))
        rec, tail, rec2, tail2 = ([f32(m, SH, SN, SV) for _ in range(bufs)], [rnd(m, 3, d.channels) for _ in range(bufs)],
                                  [f32(m, H, D, D) for _ in range(2 * bufs)], [rnd(m, 3, 3 * H * D) for _ in range(2 * bufs)])
        proj, pg, slot, ones = rnd(m, ld), rnd(m, 4 * H * D + 2 * H), torch.arange(m, dtype=torch.int32, device=dev), full(m, 1)
        grp1 = [SegGroup(0, m, 0, m, 1)]
        add(f"ssm_step + gated norm, {m} rows, {SH} heads of {SN} x {SV}",
            (lambda j: ops.ssm(proj, d, w, rec[j], tail[j], grp1, slot, slot, ones, slot, slot, 1e-6), m * (SH * SN * SV * 8.0 + ld * 8.0), 0.0, bufs),
            f"gdn_step, {H} heads of {D} x {D}",
            (lambda j: ops.gdn_step(pg, cw, rec2[j], tail2[j], A, dtb, gw, slot, slot, ones, H, H, D, D, 1e-6), m * (H * D * D * 8.0 + H * D * 20.0), 0.0, 2 * bufs))
        del rec, rec2
    rec, tail, rec2, tail2 = f32(1, SH, SN, SV), rnd(1, 3, d.channels), f32(1, H, D, D), rnd(1, 3, 3 * H * D)
    proj, pg, pos = rnd(T, ld), rnd(T, 4 * H * D + 2 * H), rlen - 1
    # per 64-row chunk and head: C B^T, its product with x, C with the state, and the chunk's state
    fl = T / 64 * SH * (2.0 * 64 * 64 * SN + 2 * 64 * 64 * SV + 4 * 64 * SN * SV)
    fl2 = T / 64 * H * (4 * 64 * 64 * D + 64 * 64 * 64 / 3 + 6 * 64 * D * D + 4 * 64 * 64 * D)
    one, grp1 = (i32([0]), i32([0]), i32([T])), [SegGroup(0, 1, 0, T, T, True)]
    gdn = (lambda: ops.gdn_rec(ops.gdn_conv(pg, cw, tail2, *one, 3 * H * D, T), pg, rec2, tail2, A, dtb, *one, H, H, D, D, 1e-6, chunked=True, max_rows=T))
    add(f"state-space layer (convolutions, three chunk kernels, gated norm, tail), {T} rows",
        (lambda j: ops.ssm(proj, d, w, rec, tail, grp1, *one, rslot, pos, 1e-6), T * (ld * 2.0 + d.inner * 2.0), fl, 1),
        "gdn_conv + gdn_chunk + gated_norm", (lambda j: ops.gated_norm(gdn(), pg, 3 * H * D, gw, H, D, 1e-6), T * H * D * 10.0, fl2, 1))
    xbc = proj[:, d.inner:d.dt_off]
    add(f"conv_rows, {T} rows of {d.channels}",
        (lambda j: ops.conv_rows(xbc, w["conv"], tail, rslot, pos, bias=w["conv_bias"], silu=True), T * d.channels * 4.0, 0.0, 1), "gdn_conv",
        (lambda j: ops.gdn_conv(pg, cw, tail2, *one, 3 * H * D, T), T * 3 * H * D * 4.0, 0.0, 1))
    ys, conv = f32(T, d.inner), ops.conv_rows(xbc, w["conv"], tail, rslot, pos, bias=w["conv_bias"], silu=True)
    scratch = ops.scratch("ssd_chunk", ops.C.ssd_chunk_scratch_bytes(T, 1, T, SH, SN, SV) // 4, torch.float32)
    sizes = [SH, 1, SN, SV, 4]
    qkv = ops.gdn_conv(pg, cw, tail2, *one, 3 * H * D, T)
    add(f"ssd_chunk (states, scan, outputs), {T} rows", (lambda j: ops.C.ssd_chunk(ys, rec, scratch, conv, proj, w["A"], w["dt_bias"], w["skip"], *one, T, sizes),
                                                       T * d.channels * 2.0 + T * d.inner * 4.0, fl, 1), "gdn_chunk",
        (lambda j: ops.gdn_rec(qkv, pg, rec2, tail2, A, dtb, *one, H, H, D, D, 1e-6, chunked=True, max_rows=T), T * H * D * 10.0, fl2, 1))
    yg, go = f32(T, H * D), rnd(T, d.ko)
    add(f"gated norm of whole rows, {T} rows of {d.inner}", (lambda j: ops.C.group_norm_gated(go, ys, proj, w["gnorm_w"], 1, 1e-6, None, None),
                                                            T * d.inner * 8.0, 0.0, 1), "gated_norm",
        (lambda j: ops.gated_norm(yg, pg, 3 * H * D, gw, H, D, 1e-6), T * H * D * 8.0, 0.0, 1))
    # routed feed-forward with a shared expert
    gu, dn = rnd(E + 1, 2 * F, W, scale=0.02), rnd(E + 1, W, F, scale=0.02)
    sh = (rnd(1, 2 * F, W, scale=0.02), rnd(1, W, F, scale=0.02), 7.0)
    for m in (1, 4, 16):
        h, x, res, w32 = rnd(m, W), f32(m, W), rnd(m, W), torch.ones(W, device=dev)
        z = [f32(m, E + 8) for _ in range(16)]
        picks = [ops.moe_route(v, None, 2, K, 1, 1, 1.0, n_exp=E, shared_col=E, shared_id=E) for v in z]
        used = sum(len(set(ids.reshape(-1).tolist())) for ids, _ in picks) / 16
        work = (used * 3.0 * F * W * 2, 6.0 * m * (K + 1) * F * W, 16)
        add(f"expert rows, shared one included, + seam, {m} rows",
            (lambda j: ops.add_conv_normed(x, x, None, w32, W, 1e-6, w32, pairs=(ops.expert_rows(h, picks[j][0], gu[:E], dn[:E], 7.0, sh), picks[j][1])), *work),
            "moe_experts (pairs, combine)", (lambda j: ops.moe_experts(h, *picks[j], gu, dn, 0, E + 1, None, None, res), *work))
        add(f"router by logits, {E} experts, {m} rows", (lambda j: ops.moe_route(z[j], None, 2, K, 1, 1, 1.0, n_exp=E, shared_col=E, shared_id=E),
                                                        m * (E + 2 * K) * 4.0, 0.0, 16), "router, softmax",
            (lambda j: ops.moe_route(z[j], None, 0, K, 1, 1, 1.0, n_exp=E, shared_col=E, shared_id=E), m * (E + 2 * K) * 4.0, 0.0, 16))
    h, y, res, z = rnd(T, W), f32(T, W), rnd(T, W), f32(T, E + 8)
    ids, wts = ops.moe_route(z, None, 2, K, 1, 1, 1.0, n_exp=E)
    ep = ExpertParallel(None, torch.device(dev), E, W, T * K, status=ops.status_word)
    work = ((E + 1) * 3.0 * F * W * 2, 6.0 * T * (K + 1) * F * W, 1)
    add(f"clamped experts and shared expert, {T} rows",
        (lambda j: ep.moe(ops, h, ids, wts, gu[:E], dn[:E], ops.linear(ops.glu(h, sh[0][0], 7.0), sh[1][0]), z[:, E], acc=y, add=False, limit=7.0), *work),
        "swiglu experts and shared expert",
        (lambda j: ep.moe(ops, h, ids, wts, gu[:E], dn[:E], ops.linear(ops.linear(h, sh[0][0], swiglu=True), sh[1][0]), z[:, E], res=res), *work))
    assert ops.status() == 0
    return acc.rows
