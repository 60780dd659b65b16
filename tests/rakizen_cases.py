"""Small Rakizen models for the tests: configurations off and on the kernels' tile grid, seeded weights whose attention is sharp enough
that a key, a map, a gate or an expert left out shows in the logits. Drivers come from `zototar_cases`."""
import torch

from zototar_cases import engine, error, run_cuts, tokens, write  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, groups, keep, ff, scale=1.3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}


def window(heads, kv_heads, dim, vdim, size, mlp, rot=None, base=900.0, gain=2.0, cap=15.0):
    r = dim if rot is None else rot
    return {"type": "attention_2", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=gain * dim ** -0.5, softcap=cap,
                                                             mask={"size": size}, rot={"base": base, "dims": r})}


def chunks(heads, kv_heads, dim, vdim, size, mlp, diff=0.4, gain=2.0, cap=25.0):
    return {"type": "attention", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=gain * dim ** -0.5, softcap=cap,
                                                           mask={"size": size}, diff=diff)}


def config(width, vocab, layers, loop=None, eps=1e-5):
    c = {"architecture": "Rakizen", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # everything on the 64 grid, a loop in the middle
    "grid": config(128, 192, [window(4, 2, 64, 64, 48, dense(192)), chunks(2, 1, 32, 64, 80, moe(8, 2, 4, 2, 64)), window(2, 2, 128, 128, 100, dense(64)),
                              chunks(4, 2, 64, 128, 64, dense(128), diff=0.7)], (1, 3, 2)),
    # nothing on it: unequal layers, key and value widths that differ both ways, group sizes of 1, 2, 3, routers of 12 and 10 experts
    "ragged": config(100, 211, [window(6, 2, 40, 24, 17, dense(90), rot=24), chunks(3, 1, 20, 44, 33, moe(12, 3, 3, 2, 22)),
                                window(5, 5, 20, 36, 70, None, base=1e4), chunks(4, 2, 12, 9, 90, moe(10, 4, 5, 3, 30, scale=0.7))], (0, 4, 2)),
    # one layer, one head, a window of a few tokens, no feed-forward, no loop
    "bare": config(64, 96, [window(1, 1, 24, 40, 5, None, rot=2)], eps=1e-3),
    # odd widths, one expert per token, no groups to speak of
    "odd": config(70, 101, [chunks(3, 3, 13, 27, 19, dense(51)), window(2, 1, 21, 7, 64, moe(3, 1, 1, 1, 35), rot=10)], (1, 2, 3)),
    # heads wider than the tensor-core kernels take
    "broad": config(96, 120, [window(2, 1, 272, 40, 30, dense(64)), chunks(1, 1, 140, 264, 50, None)]),
    # masks at and beside the pages, no rotation, many small groups of experts; a window of one token: every row sees itself only
    "edges": config(72, 130, [window(4, 1, 32, 32, 64, moe(48, 6, 16, 5, 20), rot=0), chunks(2, 2, 24, 16, 65, dense(40)), window(3, 3, 16, 16, 1, None),
                              chunks(3, 1, 16, 32, 128, moe(6, 2, 3, 3, 24))], (3, 4, 2)),
}


def weights(cfg, seed=0):
    """Checkpoint tensors (bf16)."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    W, w = cfg["width"], {}
    mat = lambda n, k, f=1.0: r(n, k) * (f * k ** -0.5)
    nrm = lambda n: 1.0 + 0.3 * r(n)
    w["embed"] = r(cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        x, H, G, D, V = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1.b"] = nrm(W), 0.3 * r(W)
        M = 2 if l["type"] == "attention" else 1
        w[x + "q"], w[x + "k"], w[x + "v"], w[x + "o"] = mat(H * M * D, W), mat(G * M * D, W), mat(G * V, W), mat(W, H * V)
        if M == 2:
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[x + n] = 0.5 * r(D) * D ** -0.25
            w[x + "g"] = mat(H * V, W)
        else:
            w[x + "q.norm"], w[x + "k.norm"] = nrm(H * D), nrm(G * D)
        f = l["mlp"]
        if f and f["kind"] == "dense":
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(f["ff"], W), mat(f["ff"], W), mat(W, f["ff"])
        elif f:
            w[p + "mlp.router"], F = mat(f["router"]["experts"], W, 2.0), f["expert"]["ff"]
            for e in range(f["router"]["experts"]):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = mat(F, W), mat(F, W), mat(W, F)
    w["final.norm"], w["final.norm.b"], w["head"] = nrm(W), 0.3 * r(W), mat(cfg["vocab"], W, 3.0)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def errors(got, want):
    """Relative error of every position: rms over the vocabulary, mean off."""
    d, w = got.double() - want.double(), want.double()
    d, w = d - d.mean(-1, keepdim=True), w - w.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
