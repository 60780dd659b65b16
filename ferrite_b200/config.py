"""Typed configuration: model shapes, engine options and operator-tier site settings.

The reference keeps three tiers (operator env `FERRITE_*`, server flags, engine env knobs `FE_*`;
`scripts/serve.sh:14-43`, `crates/fe-model/src/config.rs:6-107`, `crates/fe-model/src/sched.rs:14-48`).
Here one set of dataclasses is filled from file + env + CLI, and model dimensions are run-time values
instead of recompiled kernel crates (`kernels/k-core/src/dims.rs`).
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, Optional


@dataclass
class LayerSpec:
    """One layer of a model that lists its layers one by one (`ModelConfig.layers`): the mixer, its sizes and the
    feed-forward behind it. Layers of one model may differ in all of them."""

    # "latent": attention over a cached low-rank latent, without positions or with one rotated key part beside the latent. "gqa":
    # grouped-query attention over cached keys and values. "cdelta": gated delta rule with one decay per key channel (recurrent state,
    # no cache). "ssm": state-space duality (Mamba-2): a state per head with one decay, inputs convolved
    mixer: str = "latent"
    heads: int = 1
    dim: int = 0                    # query / key width of a head (latent with rotation: its unrotated part; ssm: width of the state)
    vdim: int = 0                   # value width of a head
    q_rank: int = 0                 # the queries come out of a normalised latent of this width (0: straight out of the input)
    kv_rank: int = 0                # width of the cached latent
    scale: float = 1.0              # scores are (q . k) * scale
    kv_from: Optional[int] = None   # use the latents (gqa: keys and values) that this (earlier) layer caches instead of own ones
    ff: int = 0                     # feed-forward width, 0 = the layer has none
    # its activation; "swiglu": silu(gate) * up; "clamped_glu": with g = min(gate, limit) and u = up clamped to +- limit,
    # g * sigmoid(1.702 g) * (u + 1)
    act: str = "relu2"
    limit: float = 0.0
    experts: int = 0                # the feed-forward is a mixture of this many experts (swiglu or clamped_glu) of width `ff` ...
    top: int = 0                    # ... of which a token takes the `top` best (sigmoid scores) ...
    groups: int = 1                 # ... among the best `keep_groups` of `groups` groups of neighbours ...
    keep_groups: int = 1
    route_scale: float = 1.0        # ... weighted by their share of the chosen scores times this
    router: str = "sigmoid"         # "softmax": the largest logits, weighted by the softmax over the chosen ones (no groups)
    shared_ff: int = 0              # width of an expert that every token takes as well, times the sigmoid of a product; 0 = none
    shared_limit: float = 0.0       # ... and its limit
    kv_heads: int = 0               # gqa, cdelta, ssm: key / value (cdelta: query / key; ssm: input / output) heads, each serving heads / kv_heads heads
    bias: bool = False              # gqa: biases on the query, key and output projections
    sink: bool = False              # gqa: a learned number per head in every softmax denominator
    key_values: bool = False        # gqa: the values are the projected keys, before rotation and norm
    qk_norm: bool = False           # gqa: queries and keys divided by their root mean square after the rotation
    row_norm: bool = False          # gqa: RMS norms with weights over a whole row of queries and of keys, before the rotation
    softcap: float = 0.0            # gqa: scores <- cap * tanh(scores / cap), 0 = off
    window: int = 0                 # gqa, latent: a row sees itself and the window - 1 positions before it, 0 = all of them
    pool: int = 0                   # gqa, window: blocks of this many positions that lie before the window are seen as their mean key and value
    chunk: int = 0                  # gqa: a row sees the positions of its own chunk of this many, counted from 0
    maps: int = 1                   # gqa: 2 = differential: two softmax maps per head over shared values, their weighted difference
    diff: float = 0.0               # gqa, two maps: constant of the difference's weight; 1 - diff scales its normed rows
    out_gate: bool = False          # gqa: the heads' outputs are multiplied by the sigmoid of a projection of the mixer's input
    rot_dims: int = 0               # gqa: rotated columns of a head, pairs (0, 1), (2, 3), ...; latent: width of the rotated part
    rot_half: bool = False          # gqa: pairs (i, i + rot_dims / 2) instead
    rot_base: float = 1e4
    rot_scaling: Optional[dict] = None   # long wavelengths stretched: factor, low, high, original
    conv: int = 0                   # cdelta, ssm: taps of the short convolutions
    norm_groups: int = 1            # ssm: equal parts of the gated output with an RMS norm each
    decay_rank: int = 0             # cdelta: width between the two decay projections (0: the checkpoint says)
    gate_rank: int = 0              # cdelta: ... and between the two output gate projections

    @property
    def cached(self) -> bool:
        """The layer keeps rows of its own in the page pool."""
        return self.mixer not in ("cdelta", "ssm") and self.kv_from is None


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer. Looped layers run several times with the same weights; every run has its own cache or state."""

    index: int                      # place in the order of execution: names the run's cache or state
    layer: int                      # whose weights
    enter: Optional[int] = None     # this run opens pass number `enter` of the loop


@dataclass
class ModelConfig:
    """Dense hybrid decoder (Gated DeltaNet + gated GQA attention), optionally with MoE FFN or MLA attention."""

    name: str = "tiny-hybrid"
    hidden: int = 256
    inter: int = 768
    n_layers: int = 4
    # layer i is full attention when (i % full_attn_every) == full_attn_every - 1, else Gated DeltaNet
    full_attn_every: int = 4
    head_dim: int = 64
    n_q: int = 4
    n_kv: int = 2
    rotary_dim: int = 64
    rope_theta: float = 1e6
    attn_gate: bool = True          # q_proj carries a per-head sigmoid output gate
    lin_k_heads: int = 4
    lin_v_heads: int = 4
    lin_dk: int = 64
    lin_dv: int = 64
    conv_k: int = 4
    eps: float = 1e-6
    vocab: int = 4096
    tie_embeddings: bool = True
    eos: int = 0
    # ---- MoE FFN (0 experts = dense SwiGLU) ----
    n_experts: int = 0
    top_k: int = 0
    expert_inter: int = 0
    n_shared: int = 0
    router: str = "softmax"         # "softmax" (top-k, renormalised) | "sigmoid_group" (grouped top-k with bias)
    n_groups: int = 1
    topk_groups: int = 1
    route_scale: float = 1.0
    first_dense: int = 0            # leading layers that keep a dense FFN
    dense_inter: int = 0
    # ---- MLA attention (kv_lora > 0 switches every layer to MLA; no GDN layers) ----
    kv_lora: int = 0
    q_lora: int = 0
    rope_head_dim: int = 0
    nope_head_dim: int = 0
    v_head_dim: int = 0
    # ---- layers listed one by one (they replace the pattern fields above) ----
    layers: List[LayerSpec] = field(default_factory=list)
    out_norm: bool = False          # x + norm(f(x)): norms on the sublayers' outputs, a 32-bit residual stream, plain norm weights
    pre_norm: bool = False          # ... and norms on the sublayers' inputs as well: x + norm(f(norm(x)))
    layer_norm: bool = False        # ... and these norms take the mean off (weights, no biases)
    canon: int = 0                  # what a sublayer reads is h + causal convolution of h with this many taps per channel, 0 = h
    depth_average: bool = False     # after a layer, x becomes a weighted sum of the embedding output and all layers' results so far
    parallel: bool = False          # x + (mixer(norm(x)) + f(norm(x))): one layer norm (with bias) ahead of both sublayers, none behind
    residual_mult: float = 1.0      # x + residual_mult * norm(f(..))
    loop: Optional[List[int]] = None     # [start, stop, times]: layers start .. stop - 1 run `times` times in a row
    loop_input: bool = True         # a pass of the loop opens with a product of [x | embedding] and a bias per pass
    logit_scale: float = 1.0
    embed_scale: float = 1.0
    gram_buckets: int = 0           # hashed bigram embedding: rows of the table besides the one for a sequence's first token
    gram_mul_prev: int = 0
    gram_mul_cur: int = 0
    logit_softcap: float = 0.0      # logits <- cap * tanh(logits / cap), 0 = off
    # ---- drafter taps ----
    tap_layers: List[int] = field(default_factory=list)

    # derived -----------------------------------------------------------------------------------
    def is_attn(self, i: int) -> bool:
        if self.kv_lora > 0:
            return True
        return (i % self.full_attn_every) == self.full_attn_every - 1

    @property
    def layer_kinds(self) -> List[str]:
        if self.layers:
            return [l.mixer for l in self.layers]
        if self.kv_lora > 0:
            return ["mla"] * self.n_layers
        return ["attn" if self.is_attn(i) else "gdn" for i in range(self.n_layers)]

    @property
    def layer_runs(self) -> List[LayerRun]:
        """Layers in the order they run."""
        n = self.n_layers
        if not self.loop:
            return [LayerRun(i, i) for i in range(n)]
        a, b, times = self.loop
        order = [(i, None) for i in range(a)]
        for t in range(times):
            order += [(i, t if i == a else None) for i in range(a, b)]
        order += [(i, None) for i in range(b, n)]
        return [LayerRun(r, i, t) for r, (i, t) in enumerate(order)]

    @property
    def n_attn(self) -> int:
        if self.layers:
            return sum(1 for r in self.layer_runs if self.layers[r.layer].cached)
        return sum(1 for k in self.layer_kinds if k != "gdn")

    @property
    def n_gdn(self) -> int:
        return self.n_layers - self.n_attn

    @property
    def conv_dim(self) -> int:
        return 2 * self.lin_k_heads * self.lin_dk + self.lin_v_heads * self.lin_dv

    @property
    def gdn_in_dim(self) -> int:
        """Rows of the fused GDN input projection: qkv | z | b | a."""
        return self.conv_dim + self.lin_v_heads * self.lin_dv + 2 * self.lin_v_heads

    @property
    def attn_q_dim(self) -> int:
        return self.n_q * self.head_dim * (2 if self.attn_gate else 1)

    @property
    def attn_in_dim(self) -> int:
        """Rows of the fused attention input projection: per head [q|gate], then k, then v."""
        return self.attn_q_dim + 2 * self.n_kv * self.head_dim

    def is_moe(self, i: int) -> bool:
        return self.n_experts > 0 and i >= self.first_dense

    def param_count(self) -> int:
        h = self.hidden
        n = self.vocab * h * (1 if self.tie_embeddings else 2)
        if self.layers:
            n += (self.gram_buckets + 1) * h if self.gram_buckets else 0
            n += 2 * h * h if self.loop and self.loop_input else 0
            for l in self.layers:
                if l.mixer == "gqa":
                    own = l.kv_heads if l.kv_from is None else 0
                    n += h * (l.maps * l.dim * (l.heads + own) + l.vdim * ((2 if l.out_gate else 1) * l.heads + (0 if l.key_values else own)))
                elif l.mixer == "cdelta":
                    n += h * (2 * l.kv_heads * l.dim + 2 * l.heads * l.vdim + l.heads) + (2 * l.kv_heads * l.dim + l.heads * l.vdim) * l.conv
                    n += l.decay_rank * (h + l.heads * l.dim) + l.gate_rank * (h + l.heads * l.vdim)
                elif l.mixer == "ssm":
                    n += h * (3 * l.heads * l.vdim + 2 * l.kv_heads * l.dim + l.heads) + (l.heads * l.vdim + 2 * l.kv_heads * l.dim) * l.conv
                else:
                    qd = l.heads * (l.dim + l.rot_dims)
                    n += (h * l.q_rank + l.q_rank * qd if l.q_rank else h * qd) + l.heads * (l.dim + l.vdim) * l.kv_rank + l.heads * l.vdim * h
                    n += h * (l.kv_rank + l.rot_dims) if l.kv_from is None else 0
                n += h * self.canon * (2 if l.ff else 1)
                if l.experts:
                    n += l.experts * (h + 3 * h * l.ff) + (h * (3 * l.shared_ff + 1) if l.shared_ff else 0)
                else:
                    n += (3 if l.act == "swiglu" else 2) * h * l.ff
            return n
        for i, kind in enumerate(self.layer_kinds):
            if kind == "gdn":
                n += h * self.gdn_in_dim + self.lin_v_heads * self.lin_dv * h + self.conv_dim * self.conv_k
            elif kind == "attn":
                n += h * self.attn_in_dim + self.n_q * self.head_dim * h
            else:
                qd = self.n_q * (self.nope_head_dim + self.rope_head_dim)
                n += h * self.q_lora + self.q_lora * qd + h * (self.kv_lora + self.rope_head_dim)
                n += self.kv_lora * self.n_q * (self.nope_head_dim + self.v_head_dim) + self.n_q * self.v_head_dim * h
            if self.is_moe(i):
                n += (self.n_experts + self.n_shared) * 3 * h * self.expert_inter + self.n_experts * h
            else:
                n += 3 * h * (self.dense_inter if (self.n_experts > 0 and self.dense_inter) else self.inter)
        return n

    def shard(self, world: int) -> "ModelConfig":
        """Per-rank shapes of a `world`-way tensor-parallel split (reference `Config::shard`,
        `crates/fe-model/src/config.rs:80`): whole heads and FFN columns per rank; KV heads are
        replicated when there are fewer of them than ranks."""
        c = dataclasses.replace(self)
        if world == 1:
            return c
        if self.layers:
            if self.parallel or self.canon or any(l.row_norm or l.mixer == "ssm" for l in self.layers):
                raise ValueError("models of parallel blocks, convolved inputs or norms that span all heads run on one rank")
            assert all(l.heads % world == 0 and l.kv_heads % world == 0 and l.ff % world == 0 for l in self.layers), \
                f"heads and feed-forward widths must divide over {world} ranks"
            c.layers = [dataclasses.replace(l, heads=l.heads // world, kv_heads=l.kv_heads // world, ff=l.ff // world) for l in self.layers]
            return c
        assert self.n_q % world == 0 and self.inter % world == 0
        c.n_q = self.n_q // world
        c.n_kv = max(1, self.n_kv // world)
        if self.kv_lora == 0:
            assert self.lin_k_heads % world == 0 and self.lin_v_heads % world == 0
            c.lin_k_heads = self.lin_k_heads // world
            c.lin_v_heads = self.lin_v_heads // world
        c.inter = self.inter // world
        if self.dense_inter:
            c.dense_inter = self.dense_inter // world
        return c

    def to_json(self) -> str:
        return json.dumps(dataclasses.asdict(self), indent=1)

    @staticmethod
    def from_hf(path: str | os.PathLike) -> "ModelConfig":
        """Read a Hugging Face `config.json` (the `text_config` block when present), the way the
        reference does in `crates/fe-model/src/config.rs:44-78`. A file that names its `architecture` is read by that
        architecture's entry in `ARCHITECTURES`."""
        v = json.loads(Path(path).read_text())
        if "architecture" in v:
            arch = v["architecture"]
            if arch not in ARCHITECTURES:
                raise ValueError(f"unknown architecture {arch!r}: known are {', '.join(sorted(ARCHITECTURES))}")
            return ARCHITECTURES[arch](v)
        t = v.get("text_config", v)
        rp = t.get("rope_parameters") or {}
        head_dim = int(t["head_dim"])
        prf = float(rp.get("partial_rotary_factor", t.get("partial_rotary_factor", 0.25)))
        lt = t.get("layer_types")
        every = 4
        if lt:
            idx = [i for i, x in enumerate(lt) if x == "full_attention"]
            every = (idx[0] + 1) if idx else len(lt) + 1
        return ModelConfig(
            name=str(v.get("model_type", "hf")),
            hidden=int(t["hidden_size"]), inter=int(t["intermediate_size"]), n_layers=int(t["num_hidden_layers"]),
            full_attn_every=every, head_dim=head_dim, n_q=int(t["num_attention_heads"]),
            n_kv=int(t["num_key_value_heads"]), rotary_dim=int(head_dim * prf),
            rope_theta=float(rp.get("rope_theta", t.get("rope_theta", 1e7))),
            lin_k_heads=int(t.get("linear_num_key_heads", 16)), lin_v_heads=int(t.get("linear_num_value_heads", 16)),
            lin_dk=int(t.get("linear_key_head_dim", 128)), lin_dv=int(t.get("linear_value_head_dim", 128)),
            conv_k=int(t.get("linear_conv_kernel_dim", 4)), eps=float(t.get("rms_norm_eps", 1e-6)),
            vocab=int(t["vocab_size"]), tie_embeddings=bool(v.get("tie_word_embeddings", False)),
            eos=int(t.get("eos_token_id", 0) if not isinstance(t.get("eos_token_id"), list) else t["eos_token_id"][0]),
        )


# ---- architectures by the name their config.json carries ------------------------------------------------------------

def zototar_config(v: dict) -> ModelConfig:
    """A Zototar config.json: position-free latent attention (latents optionally shared between layers), norms on the
    sublayers' outputs, squared-relu feed-forwards, a hashed bigram embedding beside the token's, softcapped logits."""
    layers: List[LayerSpec] = []
    for i, e in enumerate(v["layers"]):
        if e["type"] != "latent_attention":
            raise ValueError(f"layer {i}: mixer type {e['type']!r} is not latent_attention")
        m, ff = e["mixer"], e.get("mlp")
        if ff and ff["kind"] != "dense":
            raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not dense")
        src = m.get("kv_from")
        if src is not None and (not 0 <= src < i or layers[src].kv_from is not None or layers[src].kv_rank != int(m["kv_rank"])):
            raise ValueError(f"layer {i}: kv_from {src} must name an earlier layer with latents of its own and the same kv_rank")
        layers.append(LayerSpec(mixer="latent", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                kv_from=None if src is None else int(src), ff=int(ff["ff"]) if ff else 0))
    emb = v["embedding"]
    gram = emb.get("bigram") or {}
    return ModelConfig(
        name="zototar", hidden=int(v["width"]), inter=max([l.ff for l in layers] + [0]), n_layers=len(layers),
        n_q=layers[0].heads, n_kv=1, head_dim=layers[0].dim, eps=float(v["norm"]["eps"]), vocab=int(v["vocab"]),
        attn_gate=False, tie_embeddings=False, layers=layers, out_norm=True, embed_scale=float(emb.get("scale", 1.0)),
        gram_buckets=int(gram.get("buckets", 0)), gram_mul_prev=int(gram.get("mul_prev", 0)),
        gram_mul_cur=int(gram.get("mul_cur", 0)), logit_softcap=float(v.get("logit_softcap") or 0.0))


def dofunex_config(v: dict) -> ModelConfig:
    """A Dofunex config.json: grouped-query attention whose values are the projected keys (interleaved rotation, normed queries and
    keys, a sink) and gated delta rules with a decay per channel, norms before and after every sublayer, looped layers."""
    layers: List[LayerSpec] = []
    for i, e in enumerate(v["layers"]):
        kind, m, ff = e["type"], e["mixer"], e.get("mlp")
        if kind not in ("attention", "channel_delta"):
            raise ValueError(f"layer {i}: mixer type {kind!r} is neither attention nor channel_delta")
        if ff and ff["kind"] != "dense":
            raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not dense")
        kw = dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                  ff=int(ff["ff"]) if ff else 0, act="swiglu")
        if kw["heads"] % kw["kv_heads"]:
            raise ValueError(f"layer {i}: {kw['heads']} heads do not divide over {kw['kv_heads']} key heads")
        if kind == "attention":
            if kw["dim"] != kw["vdim"]:
                raise ValueError(f"layer {i}: the values are the keys, so vdim {kw['vdim']} must be dim {kw['dim']}")
            rot = m.get("rot") or {}
            s = rot.get("scaling")
            layers.append(LayerSpec(mixer="gqa", scale=float(m["scale"]), bias=True, sink=True, key_values=True, qk_norm=True,
                                    rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1e4)),
                                    rot_scaling={k: float(s[k]) for k in ("factor", "low", "high", "original")} if s else None, **kw))
        else:
            layers.append(LayerSpec(mixer="cdelta", conv=int(m["conv"]), **kw))
    lp = v.get("loop")
    if lp and not 0 <= lp["start"] < lp["stop"] <= len(layers):
        raise ValueError(f"loop {lp['start']} .. {lp['stop']} lies outside the {len(layers)} layers")
    return ModelConfig(
        name="dofunex", hidden=int(v["width"]), inter=max([l.ff for l in layers] + [0]), n_layers=len(layers), n_q=layers[0].heads,
        n_kv=layers[0].kv_heads, head_dim=layers[0].dim, eps=float(v["norm"]["eps"]), vocab=int(v["vocab"]), attn_gate=False,
        tie_embeddings=False, layers=layers, out_norm=True, pre_norm=True, residual_mult=float(v.get("residual_mult", 1.0)),
        loop=[int(lp[k]) for k in ("start", "stop", "times")] if lp else None, logit_scale=float(v.get("logit_scale", 1.0)))


def rakizen_config(v: dict) -> ModelConfig:
    """A Rakizen config.json: parallel blocks under one layer norm; "attention" takes the difference of two softmax maps over chunks of
    the sequence, with gated outputs and no positions, "attention_2" normed and rotated queries and keys under a sliding window, both
    with softcapped scores; dense or routed swiglu feed-forwards; layers may loop, with a cache per pass."""
    layers: List[LayerSpec] = []
    for i, e in enumerate(v["layers"]):
        kind, m, ff = e["type"], e["mixer"], e.get("mlp")
        if kind not in ("attention", "attention_2"):
            raise ValueError(f"layer {i}: mixer type {kind!r} is neither attention nor attention_2")
        size, cap = int(m["mask"]["size"]), float(m.get("softcap") or 0.0)
        if size < 1 or cap < 0:
            raise ValueError(f"layer {i}: mask size {size} or softcap {cap} out of range")
        kw = dict(mixer="gqa", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                  scale=float(m["scale"]), softcap=cap, act="swiglu")
        if kw["heads"] % kw["kv_heads"]:
            raise ValueError(f"layer {i}: {kw['heads']} heads do not divide over {kw['kv_heads']} key heads")
        if kind == "attention":
            kw.update(chunk=size, maps=2, diff=float(m["diff"]), out_gate=True)
        else:
            rot = m.get("rot") or {}
            kw.update(window=size, row_norm=True, rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1e4)))
            if kw["rot_dims"] % 2 or kw["rot_dims"] > kw["dim"]:
                raise ValueError(f"layer {i}: {kw['rot_dims']} rotated dimensions of {kw['dim']}")
        if ff and ff["kind"] == "dense":
            kw["ff"] = int(ff["ff"])
        elif ff and ff["kind"] == "moe":
            r = ff["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            kw.update(ff=int(ff["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), groups=int(g["count"]),
                      keep_groups=int(g["keep"]), route_scale=float(r.get("scale", 1.0)))
            if kw["experts"] % kw["groups"] or not 1 <= kw["keep_groups"] <= kw["groups"]:
                raise ValueError(f"layer {i}: {kw['experts']} experts in {kw['groups']} groups, of which {kw['keep_groups']} are kept")
            if not 1 <= kw["top"] <= kw["experts"] // kw["groups"] * kw["keep_groups"]:
                raise ValueError(f"layer {i}: {kw['top']} experts per token cannot come out of {kw['keep_groups']} groups")
        elif ff:
            raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is neither dense nor moe")
        layers.append(LayerSpec(**kw))
    lp = v.get("loop")
    if lp and not (0 <= lp["start"] <= lp["stop"] <= len(layers) and lp["times"] >= 1):
        raise ValueError(f"loop {lp['start']} .. {lp['stop']}, {lp['times']} times, over {len(layers)} layers")
    return ModelConfig(
        name="rakizen", hidden=int(v["width"]), inter=max([l.ff for l in layers] + [0]), n_layers=len(layers), n_q=layers[0].heads,
        n_kv=layers[0].kv_heads, head_dim=layers[0].dim, eps=float(v["norm"]["eps"]), vocab=int(v["vocab"]), attn_gate=False,
        tie_embeddings=False, layers=layers, pre_norm=True, parallel=True,
        loop=[int(lp[k]) for k in ("start", "stop", "times")] if lp else None, loop_input=False)


def pironex_config(v: dict) -> ModelConfig:
    """A Pironex config.json: layer norms on both sides of every sublayer, convolved inputs, a learned average over depth; "attention" over a
    window and the means of the blocks before it (keys optionally another layer's), "latent_attention" with a rotated key part under a
    window, "mamba2"; routed feed-forwards of clamped gated units with a shared expert; logits over the embedding table."""
    layers: List[LayerSpec] = []
    for i, e in enumerate(v["layers"]):
        kind, m, ff = e["type"], e["mixer"], e.get("mlp")
        kw = dict(heads=int(m["heads"]), vdim=int(m["vdim"]))
        if kind in ("attention", "latent_attention"):
            rot, mask = m.get("rot") or {}, m["mask"]
            kw.update(dim=int(m["dim"]), scale=float(m["scale"]), window=int(mask["size"]), rot_dims=int(rot.get("dims", 0)),
                      rot_base=float(rot.get("base", 1e4)))
            if kw["window"] < 1 or kw["rot_dims"] % 2:
                raise ValueError(f"layer {i}: mask size {kw['window']} or {kw['rot_dims']} rotated dimensions out of range")
        if kind == "attention":
            kw.update(mixer="gqa", kv_heads=int(m["kv_heads"]), row_norm=True, rot_half=True, softcap=float(m.get("softcap") or 0.0),
                      pool=int(mask.get("pool") or 0))
            src = m.get("kv_from")
            if kw["heads"] % kw["kv_heads"]:
                raise ValueError(f"layer {i}: {kw['heads']} heads do not divide over {kw['kv_heads']} key heads")
            if kw["rot_dims"] > kw["dim"] or kw["softcap"] < 0 or kw["pool"] < 0:
                raise ValueError(f"layer {i}: {kw['rot_dims']} rotated dimensions of {kw['dim']}, softcap or pool out of range")
            if src is not None:
                o = layers[int(src)] if 0 <= int(src) < i else None
                if o is None or o.mixer != "gqa" or o.kv_from is not None or (o.kv_heads, o.dim, o.vdim) != (kw["kv_heads"], kw["dim"], kw["vdim"]):
                    raise ValueError(f"layer {i}: kv_from {src} must name an earlier attention layer with keys of its own and the same key heads and widths")
                kw["kv_from"] = int(src)
        elif kind == "latent_attention":
            kw.update(mixer="latent", kv_rank=int(m["kv_rank"]))
            if kw["rot_dims"] != int(m["rot_dim"]):
                raise ValueError(f"layer {i}: the rotated part has rot_dim {m['rot_dim']} dimensions, not {kw['rot_dims']}")
        elif kind == "mamba2":
            kw.update(mixer="ssm", dim=int(m["state"]), kv_heads=int(m["groups"]), conv=int(m["conv"]), norm_groups=int(m["norm_groups"]))
            if kw["heads"] % kw["kv_heads"] or kw["heads"] * kw["vdim"] % kw["norm_groups"]:
                raise ValueError(f"layer {i}: {kw['heads']} heads over {kw['kv_heads']} groups, {kw['norm_groups']} norm groups")
        else:
            raise ValueError(f"layer {i}: mixer type {kind!r} is none of attention, latent_attention, mamba2")
        if ff:
            if ff["kind"] != "moe":
                raise ValueError(f"layer {i}: feed-forward kind {ff['kind']!r} is not moe")
            r, sh = ff["router"], ff.get("shared")
            kw.update(ff=int(ff["expert"]["ff"]), limit=float(ff["expert"]["limit"]), act="clamped_glu", router="softmax", experts=int(r["experts"]),
                      top=int(r["top"]))
            if not 1 <= kw["top"] <= kw["experts"]:
                raise ValueError(f"layer {i}: {kw['top']} of {kw['experts']} experts per token")
            if sh:
                kw.update(shared_ff=int(sh["ff"]), shared_limit=float(sh["limit"]))
        layers.append(LayerSpec(**kw))
    return ModelConfig(
        name="pironex", hidden=int(v["width"]), inter=max([l.ff for l in layers] + [0]), n_layers=len(layers), n_q=layers[0].heads,
        n_kv=max(1, layers[0].kv_heads), head_dim=layers[0].dim, eps=float(v["norm"]["eps"]), vocab=int(v["vocab"]), attn_gate=False,
        tie_embeddings=True, layers=layers, out_norm=True, pre_norm=True, layer_norm=True, canon=int((v.get("canon") or {}).get("taps", 0)),
        depth_average=True, embed_scale=float((v.get("embedding") or {}).get("scale", 1.0)))


ARCHITECTURES = {"Zototar": zototar_config, "Dofunex": dofunex_config, "Rakizen": rakizen_config, "Pironex": pironex_config}


# ---- presets: the five benchmark configurations ----------------------------------------------------

def tiny_hybrid() -> ModelConfig:
    """4 layers (3 GDN + 1 GQA), hidden 256, vocab 4096, tied embeddings: the fp32 CPU plumbing model and oracle."""
    return ModelConfig()


def hybrid_27b() -> ModelConfig:
    """27B-class dense hybrid: 64 layers 3:1 GDN:GQA, hidden 5120, FFN 17408, vocab 151936."""
    return ModelConfig(
        name="hybrid-27b", hidden=5120, inter=17408, n_layers=64, full_attn_every=4, head_dim=256, n_q=24, n_kv=4,
        rotary_dim=64, rope_theta=1e7, lin_k_heads=16, lin_v_heads=16, lin_dk=128, lin_dv=128, vocab=151936,
        tie_embeddings=False, tap_layers=[15, 31, 47],
    )


def drafter_block() -> ModelConfig:
    """5-layer block drafter conditioned on tapped target hidden states (reference `crates/fe-dflash/src/lib.rs:1-66`)."""
    return ModelConfig(
        name="block-drafter", hidden=5120, inter=17408, n_layers=5, full_attn_every=1, head_dim=128, n_q=32, n_kv=8,
        rotary_dim=128, rope_theta=1e7, attn_gate=False, vocab=151936, tie_embeddings=False,
    )


def moe_80b() -> ModelConfig:
    """80B-A3B-class hybrid MoE: 48 layers 3:1, hidden 2048, 512 experts (FFN 512) top-10 + 1 shared."""
    return ModelConfig(
        name="moe-80b-a3b", hidden=2048, inter=512, n_layers=48, full_attn_every=4, head_dim=256, n_q=16, n_kv=2,
        rotary_dim=64, rope_theta=1e7, lin_k_heads=16, lin_v_heads=32, lin_dk=128, lin_dv=128, vocab=151936,
        tie_embeddings=False, n_experts=512, top_k=10, expert_inter=512, n_shared=1, router="softmax",
    )


def mla_671b() -> ModelConfig:
    """671B-class MLA MoE: 61 layers (3 dense), hidden 7168, 256 experts (FFN 2048) sigmoid top-8 in 4 of 8 groups."""
    return ModelConfig(
        name="mla-671b", hidden=7168, inter=18432, n_layers=61, head_dim=192, n_q=128, n_kv=128, rotary_dim=64,
        rope_theta=1e4, attn_gate=False, vocab=129280, tie_embeddings=False, n_experts=256, top_k=8,
        expert_inter=2048, n_shared=1, router="sigmoid_group", n_groups=8, topk_groups=4, route_scale=2.5,
        first_dense=3, dense_inter=18432, kv_lora=512, q_lora=1536, rope_head_dim=64, nope_head_dim=128,
        v_head_dim=128,
    )


def tiny_mla(moe: bool = True) -> ModelConfig:
    """3-layer MLA model (latent 64 + rope 64) with the grouped-sigmoid MoE and a leading dense layer: the plumbing
    model of the 671B-class family."""
    kw = dict(n_experts=16, top_k=4, expert_inter=64, n_shared=1, router="sigmoid_group", n_groups=4, topk_groups=2,
              route_scale=2.5, first_dense=1, dense_inter=512) if moe else {}
    return ModelConfig(name="tiny-mla", hidden=256, inter=512, n_layers=3, head_dim=96, n_q=4, n_kv=4, rotary_dim=64,
                       vocab=1024, tie_embeddings=True, kv_lora=64, q_lora=128, rope_head_dim=64, nope_head_dim=32,
                       v_head_dim=32, **kw)


def zototar(width: int, n_layers: int, heads: int, q_rank: int, kv_rank: int, ff: int, vocab: int, dim: int = 128,
            vdim: int = 128, buckets: int = 65521, name: str = "zototar") -> ModelConfig:
    """A Zototar model of uniform layers in which every second layer shares the latents of the one before it."""
    layers = [LayerSpec(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=dim ** -0.5,
                        kv_from=None if i % 2 == 0 else i - 1, ff=ff) for i in range(n_layers)]
    return ModelConfig(name=name, hidden=width, inter=ff, n_layers=n_layers, n_q=heads, n_kv=1, head_dim=dim, eps=1e-6,
                       vocab=vocab, attn_gate=False, tie_embeddings=False, layers=layers, out_norm=True,
                       embed_scale=width ** 0.5, gram_buckets=buckets, gram_mul_prev=31, gram_mul_cur=7, logit_softcap=30.0)


def tiny_zototar() -> ModelConfig:
    """5-layer plumbing model of the latent-attention family: unequal layers, sizes off the kernels' tile grid."""
    c = zototar(200, 5, 4, 72, 80, 224, 300, dim=40, vdim=24, buckets=97, name="tiny-zototar")
    c.layers[2] = dataclasses.replace(c.layers[2], heads=6, dim=16, vdim=48, q_rank=56, kv_rank=136, scale=0.3, ff=0)
    c.layers[3] = dataclasses.replace(c.layers[3], kv_from=0, heads=2)
    c.layers[4] = dataclasses.replace(c.layers[4], kv_from=2, kv_rank=136, ff=104)
    return c


def zototar_7b() -> ModelConfig:
    """7B-class latent-attention model: 32 layers of width 4096, 32 heads of 128, latents of 512, FFN 16384."""
    return zototar(4096, 32, 32, 1536, 512, 16384, 129280, name="zototar-7b")


def dofunex(width: int, n_layers: int, heads: int, kv_heads: int, ff: int, vocab: int, dim: int = 128, every: int = 4,
            rank: int = 128, loop: Optional[List[int]] = None, name: str = "dofunex") -> ModelConfig:
    """A Dofunex model of equal layers, every `every`-th one attention, the others delta rules with `heads` heads of `dim`."""
    scaling = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192.0}
    attn = LayerSpec(mixer="gqa", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, ff=ff, act="swiglu", bias=True,
                     sink=True, key_values=True, qk_norm=True, rot_dims=dim, rot_base=5e5, rot_scaling=scaling)
    delta = LayerSpec(mixer="cdelta", heads=heads, kv_heads=heads, dim=dim, vdim=dim, ff=ff, act="swiglu", conv=4, decay_rank=rank,
                      gate_rank=rank)
    layers = [dataclasses.replace(attn if i % every == every - 1 else delta) for i in range(n_layers)]
    return ModelConfig(name=name, hidden=width, inter=ff, n_layers=n_layers, n_q=heads, n_kv=kv_heads, head_dim=dim, eps=1e-6, vocab=vocab,
                       attn_gate=False, tie_embeddings=False, layers=layers, out_norm=True, pre_norm=True, loop=loop)


def tiny_dofunex() -> ModelConfig:
    """4-layer plumbing model of the channel-delta family: unequal layers, sizes off the kernels' tile grid, two layers looped."""
    c = dofunex(136, 4, 4, 2, 168, 300, dim=40, every=2, rank=20, loop=[1, 3, 3], name="tiny-dofunex")
    c.residual_mult, c.logit_scale = 0.6, 1.5
    c.layers[0] = dataclasses.replace(c.layers[0], dim=24, vdim=56, kv_heads=2, conv=3, ff=0)
    c.layers[3] = dataclasses.replace(c.layers[3], heads=6, kv_heads=6, rot_dims=16, rot_scaling=None, ff=72)
    return c


def dofunex_7b() -> ModelConfig:
    """7B-class channel-delta model: 32 layers of width 4096 (every fourth attention), 32 heads of 128, FFN 11008."""
    return dofunex(4096, 32, 32, 8, 11008, 129280, name="dofunex-7b")


def rakizen(width: int, n_layers: int, heads: int, kv_heads: int, ff: int, vocab: int, dim: int = 128, window: int = 1024,
            chunk: int = 2048, experts: int = 0, top: int = 0, groups: int = 1, keep: int = 1, expert_ff: int = 0, every: int = 4, moe_every: int = 2,
            loop: Optional[List[int]] = None, name: str = "rakizen") -> ModelConfig:
    """A Rakizen model in which every `every`-th layer takes the difference of two maps (half the heads, twice the value width), the
    others a window; with `experts`, every `moe_every`-th layer has a routed feed-forward."""
    common = dict(mixer="gqa", act="swiglu", softcap=30.0)
    win = LayerSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, window=window, row_norm=True, rot_dims=dim,
                    rot_base=5e5, ff=ff, **common)
    two = LayerSpec(heads=heads // 2, kv_heads=max(1, kv_heads // 2), dim=dim // 2, vdim=dim, scale=(dim // 2) ** -0.5, chunk=chunk, maps=2,
                    diff=0.5, out_gate=True, ff=ff, **common)
    moe = dict(ff=expert_ff, experts=experts, top=top, groups=groups, keep_groups=keep, route_scale=2.0) if experts else {}
    layers = [dataclasses.replace(two if i % every == every - 1 else win, **(moe if i % moe_every == moe_every - 1 else {})) for i in range(n_layers)]
    return ModelConfig(name=name, hidden=width, inter=ff, n_layers=n_layers, n_q=heads, n_kv=kv_heads, head_dim=dim, eps=1e-6, vocab=vocab,
                       attn_gate=False, tie_embeddings=False, layers=layers, pre_norm=True, parallel=True, loop=loop, loop_input=False)


def tiny_rakizen() -> ModelConfig:
    """4-layer plumbing model of the parallel-block family: unequal layers, sizes off the kernels' tile grid, two layers looped."""
    c = rakizen(136, 4, 4, 2, 104, 300, dim=40, window=24, chunk=56, experts=6, top=2, groups=3, keep=2, expert_ff=44, every=2, loop=[1, 3, 2],
                name="tiny-rakizen")
    c.layers[0] = dataclasses.replace(c.layers[0], dim=24, vdim=56, kv_heads=1, rot_dims=10, rot_base=500.0)
    c.layers[2] = dataclasses.replace(c.layers[2], heads=6, kv_heads=3, ff=0)
    return c


def rakizen_7b() -> ModelConfig:
    """7B-class parallel-block model: 32 layers of width 4096, 32 heads of 128, dense feed-forwards of 12288."""
    return rakizen(4096, 32, 32, 8, 12288, 129280, name="rakizen-7b")


def pironex(width: int, n_layers: int, heads: int, kv_heads: int, vocab: int, dim: int = 128, kv_rank: int = 512, rot_dim: int = 64,
            state: int = 128, groups: int = 1, ssm_heads: int = 0, ssm_vdim: int = 64, window: int = 1024, pool: int = 16, experts: int = 64,
            top: int = 6, expert_ff: int = 1024, shared_ff: int = 1024, name: str = "pironex") -> ModelConfig:
    """A Pironex model that repeats latent attention, pooled attention (every second one with the keys of the one before it), and two
    state-space layers."""
    ff = dict(ff=expert_ff, act="clamped_glu", limit=7.0, experts=experts, top=top, router="softmax", shared_ff=shared_ff, shared_limit=7.0)
    lat = LayerSpec(mixer="latent", heads=heads, dim=dim, vdim=dim, kv_rank=kv_rank, rot_dims=rot_dim, rot_base=1e4, window=window,
                    scale=(dim + rot_dim) ** -0.5, **ff)
    att = LayerSpec(mixer="gqa", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, row_norm=True, rot_half=True, rot_dims=dim // 2,
                    rot_base=1e6, softcap=50.0, window=window, pool=pool, **ff)
    ssm = LayerSpec(mixer="ssm", heads=ssm_heads or 2 * width // ssm_vdim, vdim=ssm_vdim, dim=state, kv_heads=groups, conv=4, norm_groups=groups, **ff)
    layers = [dataclasses.replace((lat, att, ssm, ssm)[i % 4]) for i in range(n_layers)]
    for i in range(5, n_layers, 8):
        layers[i].kv_from = i - 4
    return ModelConfig(name=name, hidden=width, inter=expert_ff, n_layers=n_layers, n_q=heads, n_kv=kv_heads, head_dim=dim, eps=1e-5, vocab=vocab,
                       attn_gate=False, tie_embeddings=True, layers=layers, out_norm=True, pre_norm=True, layer_norm=True, canon=4, depth_average=True,
                       embed_scale=width ** 0.5)


def tiny_pironex() -> ModelConfig:
    """6-layer plumbing model of the pooled-attention / state-space family: unequal layers, sizes off the kernels' tile grid."""
    c = pironex(136, 6, 4, 2, 300, dim=40, kv_rank=72, rot_dim=20, state=24, groups=2, ssm_heads=4, ssm_vdim=36, window=24, pool=5, experts=6, top=2,
                expert_ff=44, shared_ff=60, name="tiny-pironex")
    c.layers[3] = dataclasses.replace(c.layers[3], heads=6, kv_heads=3, vdim=20, dim=40, conv=3, norm_groups=4, ff=0, experts=0, top=0, shared_ff=0)
    c.layers[4] = dataclasses.replace(c.layers[4], heads=3, dim=24, vdim=56, kv_rank=136, rot_dims=8, window=70)
    c.layers[5] = dataclasses.replace(c.layers[5], pool=7, window=31, softcap=0.0)
    return c


def pironex_moe() -> ModelConfig:
    """24-layer Pironex model of width 2048, 64 experts of 1024 with 6 per token and a shared one."""
    return pironex(2048, 24, 16, 4, 129280, name="pironex-moe")


PRESETS = {
    "tiny-pironex": tiny_pironex, "pironex-moe": pironex_moe,
    "tiny-rakizen": tiny_rakizen, "rakizen-7b": rakizen_7b,
    "tiny-dofunex": tiny_dofunex, "dofunex-7b": dofunex_7b,
    "tiny-zototar": tiny_zototar, "zototar-7b": zototar_7b,
    "tiny": tiny_hybrid, "tiny-mla": tiny_mla, "27b": hybrid_27b, "drafter": drafter_block, "moe80b": moe_80b, "mla671b": mla_671b,
}


def scaled(cfg: ModelConfig, n_layers: int) -> ModelConfig:
    """Same architecture with fewer layers (for tests that need real widths but little memory)."""
    c = dataclasses.replace(cfg)
    c.n_layers = n_layers
    c.layers = list(cfg.layers[:n_layers])
    if cfg.loop:
        a, b = cfg.loop[0], min(cfg.loop[1], n_layers)
        c.loop = [a, b, cfg.loop[2]] if a < b else None
    c.tap_layers = [t for t in cfg.tap_layers if t < n_layers]
    return c


@dataclass
class EngineConfig:
    """Engine-tier options (reference `LoadOpts::from_env` `crates/fe-model/src/model.rs:585-597`,
    `SchedOptions` `crates/fe-model/src/sched.rs:14-48`)."""

    n_slots: int = 4
    max_ctx: int = 4096
    kv_block: int = 64                 # tokens per KV page
    kv_pool_tokens: int = 0            # tokens the page pool holds over all slots (0 = max_ctx for every slot)
    compute_dtype: str = "bf16"        # "bf16" | "fp32": activations, weights, cache and products in 32 bits (models of listed layers)
    kv_dtype: str = "bf16"             # "bf16" | "fp8"
    weight_dtype: str = "bf16"         # "bf16" | "nvfp4" | "nvfp4-w4a4" | "nvfp4-a16" | "fp8-block" (e4m3, 128 x 128 blocks) | "exl3[-bits]"
    prefill_chunk: int = 2048          # rows per prompt forward (reference FERRITE_CHUNK)
    prompt_align: int = 32             # chunk cuts land on this grid (reference PROMPT_ALIGN)
    max_step_rows: int = 4096
    decode_rows_max: int = 64          # rows routed to the small-M (GEMV) kernels
    attn_splits: int = 0               # 0 = pick from context length
    use_graphs: bool = True
    fused_layers: Optional[bool] = None   # plain decode rows: one persistent kernel per layer (None = when tensor parallel)
    # "bf16" | "fp8" (e4m3, one scale per (token, kv head)) | "int6" | "int4" (integer codes, one scale per 32 elements);
    # "fp8h" / "int6h" / "int4h": the same with keys stored in a Walsh-Hadamard rotated basis
    kv_dtype: str = "bf16"
    seq_parallel: bool = True          # TP prompts: row-sharded residual stream, all-gather/reduce-scatter fused into the GEMMs
    graph_max: int = 128               # LRU size of the CUDA-graph cache (reference GRAPH_MAX)
    spec_depth: int = 0
    park_gb: float = 0.0
    park_host: bool = False
    finite_check: bool = True
    step_timeout_s: float = 120.0
    seed: int = 0

    @staticmethod
    def from_env(**over) -> "EngineConfig":
        e = os.environ
        c = EngineConfig()
        def geti(name, cur):
            return int(e[name]) if name in e and e[name] != "" else cur
        c.n_slots = geti("FERRITE_SLOTS", c.n_slots)
        c.max_ctx = geti("FERRITE_CTX", c.max_ctx)
        c.kv_pool_tokens = geti("FERRITE_KV_TOKENS", c.kv_pool_tokens)
        c.compute_dtype = e.get("FERRITE_COMPUTE", "") or c.compute_dtype
        c.prefill_chunk = geti("FERRITE_CHUNK", c.prefill_chunk)
        c.spec_depth = geti("FE_SPEC", c.spec_depth)
        c.graph_max = geti("FE_GRAPH_MAX", c.graph_max)
        if "FE_KVQ" in e:
            c.kv_dtype = "fp8" if e["FE_KVQ"] not in ("", "0") else "bf16"
        if "FERRITE_WEIGHTS" in e:
            c.weight_dtype = e["FERRITE_WEIGHTS"]
        if "FE_PARK_GB" in e:
            c.park_gb = float(e["FE_PARK_GB"])
        c.park_host = e.get("FE_PARK_HOST", "0") not in ("", "0")
        c.use_graphs = e.get("FE_NO_GRAPHS", "0") in ("", "0")
        c.seq_parallel = e.get("FE_NO_SEQ_PARALLEL", "0") in ("", "0")
        c.kv_dtype = e.get("FE_KV_DTYPE", c.kv_dtype)
        c.step_timeout_s = float(e.get("FE_STEP_TIMEOUT", c.step_timeout_s))
        for k, v in over.items():
            if v is not None:
                setattr(c, k, v)
        return c


@dataclass
class SiteConfig:
    """Operator tier: the `FERRITE_*` names of `tools/site.sh:1-40` / `crates/fe-site`."""

    models_dir: str = ""
    state_dir: str = ""
    host: str = "127.0.0.1"
    port: int = 8080
    served_model_name: str = "ferrite"
    max_concurrent: int = 16

    @staticmethod
    def from_env() -> "SiteConfig":
        e = os.environ
        return SiteConfig(
            models_dir=e.get("FERRITE_MODELS", ""), state_dir=e.get("FERRITE_STATE", ""),
            host=e.get("FERRITE_HOST", "127.0.0.1"), port=int(e.get("FERRITE_PORT", "8080")),
            served_model_name=e.get("FERRITE_NAME", "ferrite"),
            max_concurrent=int(e.get("FERRITE_MAX_CONCURRENT", "16")),
        )
