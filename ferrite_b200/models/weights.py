"""Weight naming, seeded random initialisation and tensor-parallel slicing.

Layout choices that differ from the reference's per-projection tensors (`crates/fe-model/src/model.rs:406-460`):
projections that share an input are stored fused, so a decode step issues one weight-streaming kernel per input:

* GDN  `in_proj`  rows = [q | k | v | z | b | a]            (`gdn_in_dim` x hidden)
* attn `in_proj`  rows = [per q head: q, gate] | k | v      (`attn_in_dim` x hidden)
* MLP  `gate_up`  rows = [gate | up]                        (2*inter x hidden)

RMSNorm weights are stored zero-centred (effective weight 1 + w), the GDN gated-norm weight as used
(reference convention, the design notes of `crates/fe-xe`, lines 56-57).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List

import torch

from ..config import ModelConfig
from ..formats.packed import cat_rows

Weights = Dict[str, torch.Tensor]


def listed_weight_shapes(cfg: ModelConfig, i: int) -> Dict[str, tuple]:
    """A layer of a model that lists its layers (`LayerSpec`): norms on the sublayers' outputs and, with `pre_norm`, inputs."""
    l, h, p = cfg.layers[i], cfg.hidden, f"l{i}."
    out: Dict[str, tuple] = {p + "pre_norm": (h,)} if cfg.pre_norm else {}
    if cfg.parallel:
        out[p + "pre_norm_bias"] = (h,)
    if cfg.out_norm:
        out[p + "mix_norm"] = (h,)
    if l.mixer == "latent":
        if l.q_rank:
            out.update({p + "q_a": (l.q_rank, h), p + "q_a_norm": (l.q_rank,), p + "q_b": (l.heads * l.dim, l.q_rank)})
        else:
            out[p + "q"] = (l.heads * (l.dim + l.rot_dims), h)
        if l.kv_from is None:
            out[p + "kv_a"] = (l.kv_rank + l.rot_dims, h)
            out[p + "kv_a_norm"] = (l.kv_rank,)
        out[p + "k_b"] = (l.heads * l.dim, l.kv_rank)
        out[p + "v_b"] = (l.heads * l.vdim, l.kv_rank)
        out[p + "out_proj"] = (h, l.heads * l.vdim)
    elif l.mixer == "gqa":
        kd, own = l.maps * l.dim, l.kv_from is None
        for n, heads, d in (("q", l.heads, kd),) + ((("k", l.kv_heads, kd),) if own else ()) + ((("v", l.kv_heads, l.vdim),) if own and not l.key_values else ()):
            out[p + n] = (heads * d, h)
            if l.bias:
                out[p + n + "_bias"] = (heads * d,)
        if l.sink:
            out[p + "sink"] = (l.heads,)
        if l.row_norm:
            out.update({p + "q_norm": (l.heads * kd,), **({p + "k_norm": (l.kv_heads * kd,)} if own else {})})
        if l.maps == 2:
            out.update({p + n: (l.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        if l.out_gate:
            out[p + "g"] = (l.heads * l.vdim, h)
        out[p + "out_proj"] = (h, l.heads * l.vdim)
        if l.bias:
            out[p + "out_bias"] = (h,)
    elif l.mixer == "ssm":
        nv, ch = l.heads * l.vdim, l.heads * l.vdim + 2 * l.kv_heads * l.dim
        out.update({p + "in": (nv + ch + l.heads, h), p + "xbc_conv": (ch, l.conv), p + "xbc_bias": (ch,), p + "A_log": (l.heads,), p + "dt_bias": (l.heads,),
                    p + "skip": (l.heads,), p + "gnorm_w": (nv,), p + "out_proj": (h, nv)})
    else:
        nk, nv = l.kv_heads * l.dim, l.heads * l.vdim
        for n, rows in (("q", nk), ("k", nk), ("v", nv)):
            out[p + n] = (rows, h)
            out[p + n + "_conv"] = (rows, l.conv)
        out.update({p + "b": (l.heads, h), p + "A_log": (l.heads,), p + "dt_bias": (l.heads * l.dim,), p + "gnorm_w": (l.vdim,),
                    p + "a1": (l.decay_rank, h), p + "a2": (l.heads * l.dim, l.decay_rank), p + "g1": (l.gate_rank, h),
                    p + "g2": (nv, l.gate_rank), p + "out_proj": (h, nv)})
    if cfg.canon:
        out[p + "mix_canon"] = (h, cfg.canon)
        if l.ff:
            out[p + "ffn_canon"] = (h, cfg.canon)
    if cfg.depth_average:
        out[p + "dwa"] = (i + 2,)
    if l.ff and not cfg.parallel:
        if cfg.pre_norm:
            out[p + "ffn_pre_norm"] = (h,)
        out[p + "ffn_norm"] = (h,)
    if l.experts:
        out.update({p + "router": (l.experts, h), p + "experts_gate_up": (l.experts, 2 * l.ff, h), p + "experts_down": (l.experts, h, l.ff)})
        if l.shared_ff:
            out.update({p + "shared_gate": (1, h), p + "shared_gate_up": (1, 2 * l.shared_ff, h), p + "shared_down": (1, h, l.shared_ff)})
    elif l.ff:
        if l.act == "swiglu":
            out[p + "gate"] = (l.ff, h)
        out.update({p + "up": (l.ff, h), p + "down": (h, l.ff)})
    return out


def layer_weight_shapes(cfg: ModelConfig, i: int) -> Dict[str, tuple]:
    h = cfg.hidden
    p = f"l{i}."
    if cfg.layers:
        return listed_weight_shapes(cfg, i)
    out: Dict[str, tuple] = {p + "input_norm": (h,), p + "post_norm": (h,)}
    kind = cfg.layer_kinds[i]
    if kind == "gdn":
        out[p + "in_proj"] = (cfg.gdn_in_dim, h)
        out[p + "conv_w"] = (cfg.conv_dim, cfg.conv_k)
        out[p + "A_log"] = (cfg.lin_v_heads,)
        out[p + "dt_bias"] = (cfg.lin_v_heads,)
        out[p + "gnorm_w"] = (cfg.lin_dv,)
        out[p + "out_proj"] = (h, cfg.lin_v_heads * cfg.lin_dv)
    elif kind == "attn":
        out[p + "in_proj"] = (cfg.attn_in_dim, h)
        out[p + "q_norm"] = (cfg.head_dim,)
        out[p + "k_norm"] = (cfg.head_dim,)
        out[p + "out_proj"] = (h, cfg.n_q * cfg.head_dim)
    else:  # mla
        qd = cfg.nope_head_dim + cfg.rope_head_dim
        out[p + "q_a"] = (cfg.q_lora, h)
        out[p + "q_a_norm"] = (cfg.q_lora,)
        out[p + "q_b"] = (cfg.n_q * qd, cfg.q_lora)
        out[p + "kv_a"] = (cfg.kv_lora + cfg.rope_head_dim, h)
        out[p + "kv_a_norm"] = (cfg.kv_lora,)
        out[p + "kv_b"] = (cfg.n_q * (cfg.nope_head_dim + cfg.v_head_dim), cfg.kv_lora)
        out[p + "out_proj"] = (h, cfg.n_q * cfg.v_head_dim)
    if cfg.is_moe(i):
        e, ei = cfg.n_experts, cfg.expert_inter
        out[p + "router"] = (e, h)
        if cfg.router == "sigmoid_group":
            out[p + "router_bias"] = (e,)
        out[p + "experts_gate_up"] = (e, 2 * ei, h)
        out[p + "experts_down"] = (e, h, ei)
        if cfg.n_shared:
            out[p + "shared_gate_up"] = (2 * ei * cfg.n_shared, h)
            out[p + "shared_down"] = (h, ei * cfg.n_shared)
            out[p + "shared_gate"] = (1, h)
    else:
        inter = cfg.dense_inter if (cfg.n_experts > 0 and cfg.dense_inter) else cfg.inter
        out[p + "gate_up"] = (2 * inter, h)
        out[p + "down"] = (h, inter)
    return out


def weight_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    out: Dict[str, tuple] = {"embed": (cfg.vocab, cfg.hidden), "final_norm": (cfg.hidden,)}
    if not cfg.tie_embeddings:
        out["lm_head"] = (cfg.vocab, cfg.hidden)
    if cfg.gram_buckets:
        out["bigram"] = (cfg.gram_buckets + 1, cfg.hidden)
    if cfg.parallel:
        out["final_norm_bias"] = (cfg.hidden,)
    if cfg.loop and cfg.loop_input:
        out["loop_in"] = (cfg.hidden, 2 * cfg.hidden)
        out["loop_step"] = (cfg.loop[2], cfg.hidden)
    for i in range(cfg.n_layers):
        out.update(layer_weight_shapes(cfg, i))
    return out


_F32_NAMES = ("A_log", "dt_bias", "router_bias")
_F32_LISTED = ("norm", "gnorm_w", "_bias", "sink", "_conv", "_canon", "dwa", "skip", "loop_step", "lq1", "lk1", "lq2", "lk2")     # ... of models of listed layers


def keeps_f32(cfg: ModelConfig, name: str) -> bool:
    """Small tensors that enter 32-bit arithmetic and stay in 32 bits whatever the engine computes in."""
    return name.endswith(_F32_NAMES) or (bool(cfg.layers) and name.endswith(_F32_LISTED))


def init_weights(cfg: ModelConfig, seed: int = 0, dtype=torch.float32, device="cpu", std: float = 0.02, post=None) -> Weights:
    """Seeded N(0, std) weights for every tensor of the architecture. The GDN gated-norm weight is drawn
    around one (it multiplies directly); all other norm weights are zero-centred offsets. `post(name, tensor)` may
    replace a tensor as soon as it is drawn (a quantised engine packs the big ones at once, so a model that only fits
    packed never exists unpacked)."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    w: Weights = {}
    for name, shape in weight_shapes(cfg).items():
        t = torch.randn(shape, generator=g, device=device, dtype=torch.float32) * std
        if name.endswith("gnorm_w") or (cfg.layers and name.endswith("norm")):
            t = t + 1.0
        if cfg.layers and name.endswith(("_conv", "_canon")):
            t = t / std * shape[1] ** -0.5
        if name.endswith("dwa"):
            t[-1] += 1.0
        t = t if keeps_f32(cfg, name) else t.to(dtype)
        w[name] = post(name, t) if post is not None else t
    return w


# ---- tensor-parallel slicing ---------------------------------------------------------------------------

def _rows(t: torch.Tensor, lo: int, hi: int) -> torch.Tensor:
    return t[lo:hi]


_BY_ROWS = ("q", "k", "v", "q_bias", "k_bias", "v_bias", "sink", "q_conv", "k_conv", "v_conv", "b", "A_log", "dt_bias", "a2", "g2", "gate", "up")


def _shard_listed(base: str, t: torch.Tensor, rank: int, world: int) -> torch.Tensor:
    """gqa / cdelta layers and their feed-forwards: heads (rows of what makes them, columns of what reads them) divide evenly."""
    if base in _BY_ROWS:
        per = t.shape[0] // world
        return t[rank * per:(rank + 1) * per].contiguous()
    if base in ("out_proj", "down"):
        per = t.shape[1] // world
        return t[:, rank * per:(rank + 1) * per].contiguous()
    return t


def shard_weights(cfg: ModelConfig, w: Weights, rank: int, world: int) -> Weights:
    """Slice whole-model weights for one tensor-parallel rank. Column-parallel projections keep whole heads
    (KV heads are replicated when world > n_kv), row-parallel ones keep the matching input columns; norms,
    embeddings and the router are replicated, `lm_head` is split by vocabulary rows. Split table modelled
    on the reference's (`TP2.md:36-50`, `crates/fe-exl3/src/tp.rs`). Packed quantised linears (`formats/packed.py`)
    are cut the same way as dense ones: row and column slices move code and scale bytes, nothing is re-quantised."""
    if world == 1:
        return dict(w)
    out: Weights = {}
    h = cfg.hidden
    for name, t in w.items():
        base = name.split(".")[-1]
        li = int(name[1:name.index(".")]) if name.startswith("l") and "." in name else -1
        kind = cfg.layer_kinds[li] if li >= 0 else ""
        if kind in ("gqa", "cdelta"):
            out[name] = _shard_listed(base, t, rank, world)
        elif name == "lm_head":
            per = (cfg.vocab + world - 1) // world
            out[name] = t[rank * per:min(cfg.vocab, (rank + 1) * per)].contiguous()
        elif base == "in_proj" and kind == "gdn":
            nk, nv, dk, dv = cfg.lin_k_heads, cfg.lin_v_heads, cfg.lin_dk, cfg.lin_dv
            nkr, nvr = nk // world, nv // world
            o = 0
            parts = []
            for n_heads, per_rank, d in ((nk, nkr, dk), (nk, nkr, dk), (nv, nvr, dv), (nv, nvr, dv)):
                parts.append(t[o + rank * per_rank * d:o + (rank + 1) * per_rank * d])
                o += n_heads * d
            for _ in range(2):  # b, a
                parts.append(t[o + rank * nvr:o + (rank + 1) * nvr])
                o += nv
            out[name] = cat_rows(parts)
        elif base == "conv_w":
            nk, nv, dk, dv = cfg.lin_k_heads, cfg.lin_v_heads, cfg.lin_dk, cfg.lin_dv
            nkr, nvr = nk // world, nv // world
            o = 0
            parts = []
            for n_heads, per_rank, d in ((nk, nkr, dk), (nk, nkr, dk), (nv, nvr, dv)):
                parts.append(t[o + rank * per_rank * d:o + (rank + 1) * per_rank * d])
                o += n_heads * d
            out[name] = cat_rows(parts)
        elif base in ("A_log", "dt_bias"):
            nvr = cfg.lin_v_heads // world
            out[name] = t[rank * nvr:(rank + 1) * nvr].contiguous()
        elif base == "in_proj" and kind == "attn":
            hd = cfg.head_dim
            qw = hd * (2 if cfg.attn_gate else 1)
            nqr = cfg.n_q // world
            nkvr = max(1, cfg.n_kv // world)
            kv_first = (rank * cfg.n_kv) // world if cfg.n_kv >= world else (rank * cfg.n_kv) // world
            q = t[rank * nqr * qw:(rank + 1) * nqr * qw]
            ko = cfg.n_q * qw
            vo = ko + cfg.n_kv * hd
            k = t[ko + kv_first * hd:ko + (kv_first + nkvr) * hd]
            v = t[vo + kv_first * hd:vo + (kv_first + nkvr) * hd]
            out[name] = cat_rows([q, k, v])
        elif base == "out_proj":
            if kind == "gdn":
                per = cfg.lin_v_heads // world * cfg.lin_dv
            elif kind == "attn":
                per = cfg.n_q // world * cfg.head_dim
            elif kind == "latent":
                per = t.shape[1] // world
            else:
                per = cfg.n_q // world * cfg.v_head_dim
            out[name] = t[:, rank * per:(rank + 1) * per].contiguous()
        elif base in ("gate_up", "shared_gate_up"):
            inter = t.shape[0] // 2
            per = inter // world
            out[name] = cat_rows([t[rank * per:(rank + 1) * per], t[inter + rank * per:inter + (rank + 1) * per]])
        elif base in ("down", "shared_down"):
            per = t.shape[1] // world
            out[name] = t[:, rank * per:(rank + 1) * per].contiguous()
        elif base in ("experts_gate_up", "experts_down"):
            # expert parallel: whole experts per rank
            per = cfg.n_experts // world
            out[name] = t[rank * per:(rank + 1) * per].contiguous()
        elif base in ("k_b", "v_b", "up"):
            per = t.shape[0] // world
            out[name] = t[rank * per:(rank + 1) * per].contiguous()
        elif base == "q_b":
            per = t.shape[0] // world
            out[name] = t[rank * per:(rank + 1) * per].contiguous()
        elif base == "kv_b":
            per = t.shape[0] // world
            out[name] = t[rank * per:(rank + 1) * per].contiguous()
        else:
            out[name] = t
    return out


# ---- kernel layout of latent-attention layers ------------------------------------------------------------------------

def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentDims:
    """Sizes of one latent-attention layer as its kernels see them. Every dimension is padded with zeros to the tile grid
    of the GEMMs (64 columns) and the head width to one the tensor-core prompt kernel takes (64 / 128 / 256; wider heads
    go up in steps of 64 and keep to the latent form). Norms divide by the true sizes."""

    heads: int
    q_rank: int
    kv_rank: int
    qr: int           # padded q_rank
    lat: int          # padded kv_rank + rot = cache row: the latent, then the rotated key part
    hp: int           # padded head width of the keys (unrotated part, then rotated part)
    scale: float
    source: int       # layer whose cache holds the latents
    vp: int = 0       # ... of the values
    vlat: int = 0     # columns of a cache row that the few-row kernel gathers as values (kv_rank at least)
    dim: int = 0      # unrotated width of a key
    rot: int = 0      # rotated width
    window: int = 0   # a row sees itself and the window - 1 positions before it, 0 = all of them

    def __post_init__(self):
        object.__setattr__(self, "vp", self.vp or self.hp)
        object.__setattr__(self, "vlat", self.vlat or self.lat)


def latent_dims(cfg: ModelConfig, i: int) -> LatentDims:
    l = cfg.layers[i]
    kd = l.dim + l.rot_dims
    # 192 / 128 are one form of the prompt kernel, else it takes keys and values of one width
    hp, vp = (192, 128) if 128 < kd <= 192 and l.vdim <= 128 else 2 * (head_width(max(kd, l.vdim)),)
    lat, vlat = round_up(l.kv_rank + l.rot_dims, 64), round_up(l.kv_rank, 64)
    return LatentDims(l.heads, l.q_rank, l.kv_rank, round_up(l.q_rank, 64), lat, hp, l.scale, i if l.kv_from is None else l.kv_from, vp,
                      vlat if lat == 576 else lat, l.dim, l.rot_dims, l.window)


def _pad(t: torch.Tensor, *shape: int) -> torch.Tensor:
    if tuple(t.shape) == shape:
        return t.contiguous()
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


@dataclass(frozen=True)
class GqaDims:
    """Sizes of one grouped-query attention layer as its kernels see them. Cache rows and attention operands have heads of `hp`
    columns, zeros beyond the true widths: 64 / 128 / 256 are what the tensor-core kernels take, wider heads run on the CUDA cores.
    With two maps a cached key row holds both maps' keys side by side and every head brings two queries, each with zeros in the other
    map's columns: differential attention is grouped-query attention over `maps * heads` queries, and values are read once for both."""

    heads: int
    kv_heads: int
    dim: int
    hp: int
    scale: float
    rot_dims: int
    v_off: int        # column of the projection where the values start (the keys' column when they are the values)
    qk_norm: bool
    vdim: int = 0     # value width, 0 = dim
    maps: int = 1
    row_norm: bool = False
    softcap: float = 0.0
    window: int = 0
    chunk: int = 0
    diff: float = 0.0
    gate_off: int = -1      # column of the projection where the output gates start, -1 = none
    router_off: int = -1    # ... and the router's logits
    rot_half: bool = False  # rotated pairs are (i, i + rot_dims / 2)
    pool: int = 0           # blocks of this many positions before the window are seen as their means
    source: int = -1        # layer whose cache holds keys and values, -1 = the layer itself

    @property
    def vw(self) -> int:
        return self.vdim or self.dim

    @property
    def queries(self) -> int:
        """Query heads of the attention kernels."""
        return self.maps * self.heads

    @property
    def plain(self) -> bool:
        """No mechanism beyond what a causal grouped-query attention over one key and value width has."""
        return self.maps == 1 and not self.row_norm and self.vw == self.dim and not self.rot_half

    @property
    def reach(self) -> int:
        """Keys that a row can see, 0 = no bound."""
        return 0 if self.pool else self.window or self.chunk

    def first_visible(self, pos: int) -> int:
        return max(0, pos - self.window + 1) if self.window else pos - pos % self.chunk if self.chunk else 0

    def blocks_visible(self, pos: int) -> int:
        """Pooled blocks that the row at `pos` sees: those that end before its window."""
        return max(0, pos - self.window + 1) // self.pool if self.pool else 0


def head_width(d: int) -> int:
    return next((w for w in (64, 128, 256) if d <= w), round_up(d, 64))


def gqa_dims(cfg: ModelConfig, i: int) -> GqaDims:
    l = cfg.layers[i]
    kd = l.maps * l.dim
    assert l.dim == l.vdim or not l.key_values, "values that are the keys have their width"
    v_off = (l.heads + (0 if l.key_values else l.kv_heads)) * kd
    g_off = v_off + l.kv_heads * l.vdim
    r_off = g_off + (l.heads * l.vdim if l.out_gate else 0)
    return GqaDims(l.heads, l.kv_heads, l.dim, head_width(max(kd, l.vdim)), l.scale, l.rot_dims, v_off, l.qk_norm, l.vdim, l.maps,
                   l.row_norm, l.softcap, l.window, l.chunk, l.diff, g_off if l.out_gate else -1, r_off if l.experts and cfg.parallel else -1,
                   l.rot_half, l.pool, -1 if l.kv_from is None else l.kv_from)


def rope_frequencies(l) -> torch.Tensor:
    """Angle per position of every rotated pair of a gqa layer. With `rot_scaling` wavelengths beyond original / low are stretched
    by `factor`, those below original / high stay, the ones between are blended."""
    f = l.rot_base ** (-torch.arange(0, l.rot_dims, 2, dtype=torch.float64) / max(1, l.rot_dims))
    s = l.rot_scaling
    if s:
        turns = s["original"] * f / (2 * math.pi)                            # of the pair over the original context
        if s["high"] != s["low"]:
            t = ((turns - s["low"]) / (s["high"] - s["low"])).clamp(0, 1)
        else:
            t = (turns >= s["low"]).double()
        f = (1 - t) * f / s["factor"] + t * f
    return f


@dataclass(frozen=True)
class DeltaDims:
    """Sizes of one channel-delta layer as its kernels see them: columns of the fused projection [a1 | g1 | q | k | v | b]
    (the two low-rank inputs first, so that they are aligned operands of their own) and the padded width of the mixer's output."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    ra: int           # padded decay rank
    rg: int           # padded gate rank
    ko: int           # padded heads * vdim

    @property
    def q_off(self) -> int:
        return self.ra + self.rg

    @property
    def channels(self) -> int:
        """Columns that pass the short convolutions: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def b_off(self) -> int:
        return self.q_off + self.channels


def delta_dims(cfg: ModelConfig, i: int) -> DeltaDims:
    l = cfg.layers[i]
    return DeltaDims(l.heads, l.kv_heads, l.dim, l.vdim, l.conv, round_up(l.decay_rank, 64), round_up(l.gate_rank, 64),
                     round_up(l.heads * l.vdim, 64))


@dataclass(frozen=True)
class SsmDims:
    """Sizes of one state-space layer as its kernels see them: columns of the projection [z | x | B | C | dt]; the state of a head is
    [state][vdim]."""

    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int
    ko: int           # padded heads * vdim

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Columns that pass the short convolution: x | B | C."""
        return self.inner + 2 * self.groups * self.state

    @property
    def dt_off(self) -> int:
        return self.inner + self.channels


def ssm_dims(cfg: ModelConfig, i: int) -> SsmDims:
    l = cfg.layers[i]
    return SsmDims(l.heads, l.kv_heads, l.dim, l.vdim, l.conv, l.norm_groups, round_up(l.heads * l.vdim, 64))


def _pack_latent(cfg: ModelConfig, w: Weights, i: int, W: int, out: Weights) -> None:
    """* in_proj  rows = [q_a | kv_a]           one product for both latents of a token; without a query latent [q | kv_a] at true widths
    * q_b      [heads * hp, qr]              per head zero-padded rows, so queries come out at the padded width
    * kv_up    [heads * (hp + vp), lat]      key rows of every head, then value rows: expands latents for prompt rows. The rotated part
                                             of a cache row passes to every head's keys through ones
    * k_abs    [heads, lat, hp]              W_uk^T per head (and the same ones): folds the key projection into a decode row's query
    * v_up     [heads, vp, vlat]             W_uv per head: latent-space outputs to values
    * out_proj [width, heads * vp]"""
    l, p, d = cfg.layers[i], f"l{i}.", latent_dims(cfg, i)
    if l.q_rank:
        parts = [_pad(w[p + "q_a"], d.qr, W)]
        out[p + "q_a_norm"] = _pad(w[p + "q_a_norm"].float(), d.qr)
        q_b = _pad(w[p + "q_b"].view(l.heads, l.dim, l.q_rank), l.heads, d.hp, d.qr)
        out[p + "q_b"] = q_b.view(l.heads * d.hp, d.qr)
    else:
        parts = [_pad(w[p + "q"], w[p + "q"].shape[0], W)]
        out[p + "inv_freq"] = rope_frequencies(l).to(w[p + "q"].device)
    if l.kv_from is None:
        parts.append(_pad(w[p + "kv_a"], d.lat if l.q_rank else l.kv_rank + l.rot_dims, W))
        out[p + "kv_a_norm"] = _pad(w[p + "kv_a_norm"].float(), d.lat)
    rows = torch.cat(parts)
    out[p + "in_proj"] = _pad(rows, round_up(rows.shape[0], 8), W)
    k = _pad(w[p + "k_b"].view(l.heads, l.dim, l.kv_rank), l.heads, d.hp, d.lat)
    for j in range(l.rot_dims):
        k[:, l.dim + j, l.kv_rank + j] = 1.0
    v = _pad(w[p + "v_b"].view(l.heads, l.vdim, l.kv_rank), l.heads, d.vp, d.lat)
    out[p + "kv_up"] = torch.cat([k.view(-1, d.lat), v.view(-1, d.lat)])
    out[p + "k_abs"] = k.transpose(1, 2).contiguous()
    out[p + "v_up"] = out[p + "kv_up"][l.heads * d.hp:].view(l.heads, d.vp, d.lat)[..., :d.vlat].contiguous()
    o = _pad(w[p + "out_proj"].view(cfg.hidden, l.heads, l.vdim), W, l.heads, d.vp)
    out[p + "out_proj"] = o.view(W, l.heads * d.vp)


def _pack_gqa(cfg: ModelConfig, w: Weights, i: int, W: int, out: Weights) -> None:
    """* in_proj  rows = [q | k (| v) (| output gates) (| router)] of all heads at their true width; in_bias the same
    * out_proj [width, heads * hp]; in a parallel block with a dense feed-forward [width, heads * hp + ff]: both sublayers end in one
      product over their joined operands
    * lam      [1] weight of the second map"""
    l, p, d = cfg.layers[i], f"l{i}.", gqa_dims(cfg, i)
    names = ("q",) if l.kv_from is not None else ("q", "k") if l.key_values else ("q", "k", "v")
    rows = torch.cat([w[p + n] for n in names] + ([w[p + "g"]] if l.out_gate else []) + ([w[p + "router"]] if l.experts and cfg.parallel else []))
    out[p + "in_proj"] = _pad(rows, round_up(rows.shape[0], 8), W)
    if l.bias:
        out[p + "in_bias"] = _pad(torch.cat([w[p + n + "_bias"].float() for n in names]), round_up(rows.shape[0], 8))
        out[p + "out_bias"] = _pad(w[p + "out_bias"].float(), W)
    if l.sink:
        out[p + "sink"] = w[p + "sink"].float().contiguous()
    if l.row_norm:
        for n in ("q_norm", "k_norm") if l.kv_from is None else ("q_norm",):
            out[p + n] = w[p + n].float().contiguous()
    if l.maps == 2:
        dot = lambda a, b: torch.exp((w[p + a].float() * w[p + b].float()).sum())
        out[p + "lam"] = (dot("lq1", "lk1") - dot("lq2", "lk2") + l.diff).view(1)
    out[p + "out_proj"] = _pad(w[p + "out_proj"].view(cfg.hidden, l.heads, l.vdim), W, l.heads, d.hp).view(W, -1)
    if cfg.parallel and l.ff and not l.experts:
        out[p + "out_proj"] = torch.cat([out[p + "out_proj"], _pad(w[p + "down"], W, round_up(l.ff, 64))], 1)
    out[p + "inv_freq"] = rope_frequencies(l).to(rows.device)


def _pack_cdelta(cfg: ModelConfig, w: Weights, i: int, W: int, out: Weights) -> None:
    """* in_proj  rows = [a1 | g1 | q | k | v | b] (see `DeltaDims`)
    * conv     [channels, taps], decay_up [heads * dim, ra], gate_up_lr [heads * vdim, rg]
    * out_proj [width, ko]"""
    l, p, d = cfg.layers[i], f"l{i}.", delta_dims(cfg, i)
    rows = torch.cat([_pad(w[p + "a1"], d.ra, cfg.hidden), _pad(w[p + "g1"], d.rg, cfg.hidden)] + [w[p + n] for n in ("q", "k", "v", "b")])
    out[p + "in_proj"] = _pad(rows, round_up(rows.shape[0], 8), W)
    out[p + "conv"] = torch.cat([w[p + n + "_conv"].float() for n in ("q", "k", "v")]).contiguous()
    out[p + "decay_up"] = _pad(w[p + "a2"], l.heads * l.dim, d.ra)
    out[p + "gate_up_lr"] = _pad(w[p + "g2"], l.heads * l.vdim, d.rg)
    for n in ("A_log", "dt_bias", "gnorm_w"):
        out[p + n] = w[p + n].float().contiguous()
    out[p + "out_proj"] = _pad(w[p + "out_proj"], W, d.ko)


def _pack_ssm(cfg: ModelConfig, w: Weights, i: int, W: int, out: Weights) -> None:
    """* in_proj  rows = [z | x | B | C | dt]
    * conv     [taps, channels], conv_bias; A [heads] = -exp(A_log)
    * out_proj [width, ko]"""
    l, p, d = cfg.layers[i], f"l{i}.", ssm_dims(cfg, i)
    out[p + "in_proj"] = _pad(w[p + "in"], round_up(w[p + "in"].shape[0], 8), W)
    out[p + "conv"] = w[p + "xbc_conv"].float().t().contiguous()
    out[p + "conv_bias"] = w[p + "xbc_bias"].float().contiguous()
    out[p + "A"] = -torch.exp(w[p + "A_log"].float())
    for n in ("dt_bias", "skip", "gnorm_w"):
        out[p + n] = w[p + n].float().contiguous()
    out[p + "out_proj"] = _pad(w[p + "out_proj"], W, d.ko)


def _pack_experts(cfg: ModelConfig, w: Weights, p: str, l, W: int, out: Weights) -> None:
    """* experts_gate_up [experts, 2 F, width], experts_down [experts, width, F]; shared_gate_up, shared_down the same of the shared expert
    * router  rows = [router | shared expert's gate], unless the router rides on another product"""
    def stack(name, n, ff):
        F = round_up(ff, 64)
        gu = _pad(w[f"{p}{name}_gate_up"].view(n, 2, ff, cfg.hidden), n, 2, F, W)
        out[f"{p}{name}_gate_up"] = gu.view(n, 2 * F, W)
        out[f"{p}{name}_down"] = _pad(w[f"{p}{name}_down"], n, W, F)
    stack("experts", l.experts, l.ff)
    if l.shared_ff:
        stack("shared", 1, l.shared_ff)
    if not cfg.parallel:
        rows = torch.cat([w[p + "router"]] + ([w[p + "shared_gate"]] if l.shared_ff else []))
        out[p + "router"] = _pad(rows, round_up(rows.shape[0], 8), W)


_PACK = {"latent": _pack_latent, "gqa": _pack_gqa, "cdelta": _pack_cdelta, "ssm": _pack_ssm}


def pack_listed(cfg: ModelConfig, w: Weights) -> Weights:
    """Engine weights of a model of listed layers in the kernels' layout (see `LatentDims`, `GqaDims`, `DeltaDims`): sizes padded
    with zeros, projections that share an input joined, norm weights in 32 bits with the residual's and the logits' multipliers in
    them."""
    W = round_up(cfg.hidden, 64)
    vec = lambda n, f=1.0: _pad(w[n].float() * f, W)
    out: Weights = {"embed": _pad(w["embed"], cfg.vocab, W), "final_norm": vec("final_norm", cfg.logit_scale)}
    out["lm_head"] = out["embed"] if cfg.tie_embeddings else _pad(w["lm_head"], w["lm_head"].shape[0], W)
    if cfg.gram_buckets:
        out["bigram"] = _pad(w["bigram"], cfg.gram_buckets + 1, W)
    if cfg.parallel:
        out["final_norm_bias"] = vec("final_norm_bias", cfg.logit_scale)
    if cfg.loop and cfg.loop_input:
        out["loop_in"] = _pad(w["loop_in"].view(cfg.hidden, 2, cfg.hidden), W, 2, W).view(W, 2 * W)
        out["loop_step"] = _pad(w["loop_step"].float(), cfg.loop[2], W)
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        _PACK[l.mixer](cfg, w, i, W, out)
        if cfg.pre_norm:
            out[p + "pre_norm"] = vec(p + "pre_norm")
        if cfg.parallel:
            out[p + "pre_norm_bias"] = vec(p + "pre_norm_bias")
            if l.experts:
                _pack_experts(cfg, w, p, l, W, out)
            elif l.ff:
                out[p + "gate_up"] = torch.cat([_pad(w[p + n], round_up(l.ff, 64), W) for n in ("gate", "up")])
            continue
        out[p + "mix_norm"] = vec(p + "mix_norm", cfg.residual_mult)
        for n in (("mix_canon", "ffn_canon") if l.ff else ("mix_canon",)) if cfg.canon else ():
            out[p + n] = _pad(w[p + n].float().t(), cfg.canon, W)                          # [taps, width]
        if cfg.depth_average:
            out[p + "dwa"] = w[p + "dwa"].float().contiguous()
        if l.ff:
            F = round_up(l.ff, 64)
            if l.experts:
                _pack_experts(cfg, w, p, l, W, out)
            else:
                up = _pad(w[p + "up"], F, W)
                if l.act == "swiglu":
                    out[p + "gate_up"] = torch.cat([_pad(w[p + "gate"], F, W), up])
                else:
                    out[p + "up"] = up
                out[p + "down"] = _pad(w[p + "down"], W, F)
            out[p + "ffn_norm"] = vec(p + "ffn_norm", cfg.residual_mult)
            if cfg.pre_norm:
                out[p + "ffn_pre_norm"] = vec(p + "ffn_pre_norm")
    return out
