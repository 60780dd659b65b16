"""Small Dofunex models for the tests: configurations off and on the kernels' tile grid, seeded weights whose attention is sharp enough
that a key, a sink or a turn left out shows in the logits, decays from almost none to total. Drivers come from `zototar_cases`."""
import torch

from zototar_cases import engine, error, run_cuts, tokens, write  # noqa: F401


def attn(heads, kv_heads, dim, ff, gain=3.0, rot=None, base=700.0, scaling=(3.0, 1.0, 5.0, 96)):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=gain * dim ** -0.5)
    r = dim if rot is None else rot
    if r:
        m["rot"] = dict(base=base, dims=r)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m, "mlp": ff and {"kind": "dense", "ff": ff}}


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
            "mlp": ff and {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, loop=None, mult=1.0, scale=1.0, eps=1e-5):
    c = {"architecture": "Dofunex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
         "logit_scale": scale}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # everything on the 64 grid, heads shared and not, a loop in the middle
    "grid": config(128, 200, [attn(4, 2, 64, 192), delta(2, 2, 64, 64, 4, 128), delta(4, 2, 128, 128, 2, None), attn(2, 1, 128, 128)], (1, 3, 2),
                   mult=0.8),
    # nothing on it: unequal layers, part of a head rotated, group sizes of 1, 2, 3, five taps, a loop of three passes
    "ragged": config(100, 211, [attn(6, 2, 40, 90, rot=24, scaling=None), delta(6, 3, 24, 40, 3, 70), attn(5, 5, 20, None, base=1e4), delta(3, 1, 72, 20, 5, 50)],
                     (1, 4, 3), mult=0.55, scale=1.7),
    # delta rules only, one tap, no loop
    "bare": config(64, 96, [delta(1, 1, 16, 24, 1, 48), delta(2, 1, 32, 8, 2, None)], eps=1e-3),
    # attention without positions between rotated layers, loop over everything
    "round": config(72, 130, [attn(3, 3, 24, 40, rot=0), attn(4, 1, 32, None, rot=8, scaling=(16.0, 2.0, 2.5, 40))], (0, 2, 3), mult=0.6, scale=0.25),
    # odd widths throughout
    "odd": config(70, 101, [delta(3, 3, 13, 27, 2, 51), attn(3, 1, 21, 35, rot=10), delta(5, 1, 65, 3, 4, None)], (1, 2, 2), mult=0.9),
    # heads wider than the tensor-core and fused kernels take
    "broad": config(96, 120, [attn(2, 1, 272, 64), delta(2, 2, 160, 136, 4, 64), delta(1, 1, 40, 264, 3, None)], (2, 3, 2)),
}


def weights(cfg, seed=0, ranks=(20, 28)):
    """Checkpoint tensors (bf16); `ranks`: of the decay and the gate projections."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    u = lambda lo, hi, *s: lo + (hi - lo) * torch.rand(*s, generator=g)
    W, w = cfg["width"], {}
    mat = lambda n, k, f=1.0: r(n, k) * (f * k ** -0.5)
    nrm = lambda n: 1.0 + 0.3 * r(n)
    w["embed"] = r(cfg["vocab"], W)
    if cfg.get("loop"):
        w["loop.in"], w["loop.step"] = mat(W, 2 * W), 0.4 * r(cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        x, H, G, D, V = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = nrm(W), nrm(W)
        if l["type"] == "attention":
            w[x + "q"], w[x + "q.b"], w[x + "k"], w[x + "k.b"] = mat(H * D, W), 0.3 * r(H * D), mat(G * D, W), 0.3 * r(G * D)
            w[x + "sink"] = u(0.0, 6.0, H)
            w[x + "o"], w[x + "o.b"] = mat(W, H * D), 0.3 * r(W)
        else:
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[x + n], w[x + n + ".conv"] = mat(rows, W), r(rows, m["conv"]) * m["conv"] ** -0.5
            # queries near their keys: the first read of a head is sign(q k) v after its norm, and at right angles 16-bit operands
            # would pick the sign
            w[x + "q"], w[x + "q.conv"] = 0.6 * w[x + "q"] + 0.8 * w[x + "k"], 0.3 * w[x + "q.conv"] + 0.9 * w[x + "k.conv"]
            w[x + "b"], w[x + "norm"] = mat(H, W, 2.0), nrm(V)
            w[x + "A_log"], w[x + "dt_bias"] = u(-3.0, 3.5, H), u(-7.0, 2.0, H * D)
            w[x + "a1"], w[x + "a2"] = mat(ranks[0], W), mat(H * D, ranks[0], 2.0)
            w[x + "g1"], w[x + "g2"] = mat(ranks[1], W), mat(H * V, ranks[1])
            w[x + "o"] = mat(W, H * V)
        if l["mlp"]:
            F = l["mlp"]["ff"]
            w[p + "norm2"], w[p + "norm2b"] = nrm(W), nrm(W)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(F, W), mat(F, W), mat(W, F)
    w["final.norm"], w["head"] = nrm(W), mat(cfg["vocab"], W, 3.0)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
