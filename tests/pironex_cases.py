"""Small Pironex models for the tests: configurations off and on the kernels' tile grid, seeded weights whose attention is sharp enough that a
key, a block, a tap, an expert or a state left out shows in the logits. Drivers come from `zototar_cases`."""
import torch

from rakizen_cases import errors  # noqa: F401
from zototar_cases import engine, error, run_cuts, tokens, write  # noqa: F401


def moe(experts, top, ff, limit=1.2, shared=None, shared_limit=0.9):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    return f


def pooled(heads, kv_heads, dim, vdim, size, pool, mlp, rot=None, base=700.0, gain=2.0, cap=12.0, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=gain * dim ** -0.5, softcap=cap, mask={"size": size, "pool": pool},
             rot={"base": base, "dims": dim if rot is None else rot})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(heads, dim, rot, vdim, kv_rank, size, mlp, base=300.0, gain=2.0):
    return {"type": "latent_attention", "mlp": mlp, "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank,
                                                                 scale=gain * (dim + rot) ** -0.5, mask={"size": size}, rot={"base": base, "dims": rot})}


def mamba(heads, vdim, state, groups, mlp, norm_groups=1, conv=4):
    return {"type": "mamba2", "mlp": mlp, "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv)}


def config(width, vocab, layers, taps=4, scale=3.0, eps=1e-5):
    return {"architecture": "Pironex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": scale}}


CASES = {
    # everything on the 64 grid; the fourth layer reads the keys and the means of the second
    "grid": config(128, 160, [latent(2, 64, 64, 128, 64, 48, moe(8, 2, 64, shared=64)), pooled(4, 2, 64, 64, 48, 8, moe(8, 2, 64, shared=64)),
                              mamba(4, 32, 32, 1, moe(4, 2, 128, shared=64)), pooled(4, 2, 64, 64, 48, 8, moe(8, 2, 64, shared=64), kv_from=1)]),
    # nothing on it: unequal layers, means of other blocks over another layer's keys, layers without a feed-forward or a shared expert
    "ragged": config(100, 131, [mamba(6, 20, 24, 3, moe(6, 3, 30), norm_groups=4, conv=3), pooled(6, 2, 40, 24, 17, 5, moe(5, 2, 22, shared=50), rot=24),
                                latent(3, 20, 12, 36, 50, 33, None), pooled(4, 2, 40, 24, 31, 7, moe(6, 1, 26, shared=18), rot=24, cap=None, kv_from=1),
                                mamba(4, 36, 12, 2, None, norm_groups=2, conv=2)], taps=3),
    # one layer, one head, a window of one token and blocks of one
    "bare": config(64, 96, [pooled(1, 1, 24, 40, 1, 1, moe(3, 1, 20), rot=2)], taps=2, eps=1e-3),
    # odd widths of keys, values and states
    "odd": config(70, 101, [latent(3, 13, 6, 11, 31, 9, moe(4, 2, 19, shared=23)), mamba(3, 9, 7, 3, moe(7, 4, 13, shared=13)),
                            pooled(3, 3, 21, 7, 20, 3, moe(3, 2, 35), rot=10)], taps=5),
    # sizes beyond the tensor-core kernels
    "broad": config(96, 120, [pooled(2, 1, 272, 40, 30, 6, moe(4, 2, 32, shared=32)), latent(2, 24, 16, 264, 600, 50, None),
                              mamba(2, 24, 264, 1, moe(4, 2, 32))]),
    # wide latents beside a rotated key part: keys of 192 and values of 128 columns, states wider than a tile
    "wide": config(128, 120, [latent(3, 128, 64, 128, 512, 70, moe(4, 2, 64, shared=128)), mamba(3, 72, 136, 1, moe(4, 2, 32), norm_groups=3),
                              pooled(4, 1, 128, 96, 65, 10, moe(4, 2, 64, shared=32), rot=64), latent(2, 16, 8, 136, 200, 64, None)]),
    # masks at and beside the pages, blocks of a page, beside a page and longer than one; many heads on one key head; no rotation
    "edges": config(72, 130, [pooled(4, 1, 32, 32, 64, 64, moe(12, 5, 20, shared=20), rot=0), pooled(18, 1, 16, 16, 65, 63, moe(4, 2, 24), rot=8),
                              latent(2, 16, 16, 16, 48, 128, moe(4, 3, 16, shared=40)), pooled(3, 3, 16, 16, 10, 70, None, kv_from=None),
                              pooled(3, 3, 16, 16, 63, 16, moe(4, 2, 16), kv_from=3)]),
}


def weights(cfg, seed=0):
    """Checkpoint tensors (bf16)."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    W, w, taps = cfg["width"], {}, cfg["canon"]["taps"]
    mat = lambda n, k, f=1.0: r(n, k) * (f * k ** -0.5)
    nrm = lambda n: 1.0 + 0.3 * r(n)
    w["embed"] = r(cfg["vocab"], W) * W ** -0.5 * 3.0
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        x, H, V = p + "mix.", m["heads"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"], w[p + "canon1"] = nrm(W), nrm(W), 0.6 * r(W, taps) * taps ** -0.5
        w[p + "dwa"] = torch.cat([0.3 * r(i + 1), torch.ones(1)])
        w[x + "o"] = mat(W, H * V)
        if l["type"] == "attention":
            D, G = m["dim"], m["kv_heads"]
            w[x + "q"], w[x + "q.norm"] = mat(H * D, W), nrm(H * D)
            if m.get("kv_from") is None:
                w[x + "k"], w[x + "v"], w[x + "k.norm"] = mat(G * D, W), mat(G * V, W), nrm(G * D)
        elif l["type"] == "latent_attention":
            D, R, L = m["dim"], m["rot_dim"], m["kv_rank"]
            w[x + "q"], w[x + "dkv"], w[x + "dkv.norm"] = mat(H * (D + R), W), mat(L + R, W), nrm(L)
            w[x + "uk"], w[x + "uv"] = mat(H * D, L), mat(H * V, L)
        else:
            N, G = m["state"], m["groups"]
            C = H * V + 2 * G * N
            w[x + "in"], w[x + "conv"], w[x + "conv.b"] = mat(H * V + C + H, W), r(C, m["conv"]) * m["conv"] ** -0.5, 0.2 * r(C)
            w[x + "dt_bias"], w[x + "A_log"], w[x + "D"] = -3.0 + 1.5 * r(H), 0.7 * r(H), r(H)
            w[x + "norm"] = nrm(H * V)
        f = l["mlp"]
        if f:
            w[p + "norm2"], w[p + "norm2b"], w[p + "canon2"] = nrm(W), nrm(W), 0.6 * r(W, taps) * taps ** -0.5
            w[p + "mlp.router"], F = mat(f["router"]["experts"], W, 2.0), f["expert"]["ff"]
            for e in range(f["router"]["experts"]):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = mat(F, W), mat(F, W), mat(W, F)
            if f.get("shared"):
                S, s = f["shared"]["ff"], p + "mlp.shared."
                w[s + "gate"], w[s + "up"], w[s + "down"], w[s + "sg"] = mat(S, W), mat(S, W), mat(W, S), mat(1, W)
    w["final.norm"] = nrm(W)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
