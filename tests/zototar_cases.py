"""Small Zototar models for the tests: configurations off and on the kernels' tile grid, seeded weights whose attention is
sharp enough that a key left out or added shows in the logits, and drivers that run sequences through an engine step by step."""
import json

import torch

from ferrite_b200.config import EngineConfig, ModelConfig
from ferrite_b200.engine.engine import Engine
from ferrite_b200.engine.executor import Segment
from ferrite_b200.formats.loader import load_model_weights
from ferrite_b200.formats.safetensors_io import save_file


def layer(heads, dim, vdim, q_rank, kv_rank, ff, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=dim ** -0.5 if scale is None else scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, scale=3.0, bigram=(101, 13, 7), cap=20.0, eps=1e-5):
    c = {"architecture": "Zototar", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
         "embedding": {"scale": scale}, "logit_softcap": cap}
    if bigram:
        c["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return c


CASES = {
    # everything on the 64 grid
    "grid": config(128, 192, [layer(4, 64, 64, 128, 64, 256), layer(4, 64, 64, 64, 64, 192, kv_from=0), layer(2, 128, 128, 64, 128, 128)]),
    # nothing on it: odd vocabulary, unequal layers, one without a feed-forward, latents shared over a distance and twice
    "ragged": config(100, 211, [layer(3, 20, 36, 28, 44, 90, scale=0.31), layer(1, 72, 8, 52, 84, None), layer(5, 12, 28, 36, 44, 50, kv_from=0),
                                layer(2, 40, 24, 20, 84, 70, kv_from=1, scale=0.1), layer(7, 16, 16, 44, 44, 34, kv_from=0)], scale=7.5),
    # no bigram table, no softcap, one layer of one head
    "bare": config(64, 96, [layer(1, 24, 40, 16, 24, 48)], scale=1.0, bigram=None, cap=None, eps=1e-3),
    # latents wider than the tensor-core decode kernel takes, heads at the widest the prompt kernel takes
    "wide": config(192, 130, [layer(2, 200, 136, 72, 576, 96), layer(3, 136, 250, 96, 576, 160, kv_from=0)], bigram=(7, 1000003, 998244353)),
    # heads wider than the prompt kernel takes
    "broad": config(96, 120, [layer(2, 272, 300, 64, 160, 64)]),
}


def weights(cfg, seed=0, gain=4.0):
    """Checkpoint tensors (bf16). `gain` scales the query up-projections: scores of a standard deviation around it, so that a few
    keys carry each row."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    W, w = cfg["width"], {}
    mat = lambda n, k, f=1.0: r(n, k) * (f * k ** -0.5)
    nrm = lambda n: 1.0 + 0.3 * r(n)
    w["embed"] = r(cfg["vocab"], W) / cfg["embedding"]["scale"]
    if cfg["embedding"].get("bigram"):
        w["bigram"] = 0.7 * r(cfg["embedding"]["bigram"]["buckets"] + 1, W)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        w[p + "norm1"] = nrm(W)
        w[p + "mix.dq"], w[p + "mix.dq.norm"] = mat(m["q_rank"], W), nrm(m["q_rank"])
        w[p + "mix.uq"] = mat(m["heads"] * m["dim"], m["q_rank"], gain / (m["scale"] * m["dim"] ** 0.5))
        if m.get("kv_from") is None:
            w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = mat(m["kv_rank"], W), nrm(m["kv_rank"])
        w[p + "mix.uk"] = mat(m["heads"] * m["dim"], m["kv_rank"])
        w[p + "mix.uv"] = mat(m["heads"] * m["vdim"], m["kv_rank"])
        w[p + "mix.o"] = mat(W, m["heads"] * m["vdim"])
        if l["mlp"]:
            w[p + "norm2"] = nrm(W)
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(l["mlp"]["ff"], W), mat(W, l["mlp"]["ff"])
    w["final.norm"], w["head"] = nrm(W), mat(cfg["vocab"], W, 3.0)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write(cfg, w, path):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(path / "model.safetensors"))
    return str(path)


def engine(path, device="cpu", compute="fp32", slots=4, max_ctx=512, pool=0, **kw):
    cfg = ModelConfig.from_hf(f"{path}/config.json")
    ecfg = EngineConfig(n_slots=slots, max_ctx=max_ctx, kv_pool_tokens=pool, compute_dtype=compute, **kw)
    return Engine(cfg, load_model_weights(path, cfg), ecfg, device=device)


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cuts(eng, ids, cuts, slot=0):
    """Logits of every position, the sequence fed in portions (the last size repeats)."""
    eng.reset_slot(slot)
    out, at, k = [], 0, 0
    while at < len(ids):
        n = min(cuts[min(k, len(cuts) - 1)], len(ids) - at)
        lg, _, _ = eng.forward([Segment(slot, at, ids[at:at + n], "all")], greedy=False)
        out.append(lg.float().cpu().clone())
        at, k = at + n, k + 1
    eng.reset_slot(slot)
    return torch.cat(out)


def error(got, want):
    """Largest relative error of a position: rms over the vocabulary, mean off."""
    d, w = got.double() - want.double(), want.double()
    d, w = d - d.mean(-1, keepdim=True), w - w.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()).max())
