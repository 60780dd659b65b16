"""The Dofunex design on the fp32 CPU engine against a plain statement of it (`plain_dofunex.py`): configuration and checkpoint
reading, each mechanism, prompts, decoding, portions, batches, reused pages and slots, speculation, the scheduler and two ranks."""
import copy
import io
import json
import math
import sys

import pytest
import torch

import plain_dofunex as plain
from dofunex_cases import CASES, engine, error, run_cuts, tokens, weights, write
from ferrite_b200.config import EngineConfig, ModelConfig, dofunex_7b, scaled, tiny_dofunex
from ferrite_b200.engine.engine import Engine
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.formats.loader import load_model_weights
from ferrite_b200.models.ref import RefModel
from ferrite_b200.models.weights import DeltaDims, GqaDims, gqa_dims, init_weights, pack_listed, rope_frequencies, weight_shapes
from ferrite_b200.ops.torch_ops import TorchOps

LIM = 6e-5          # fp32 rounding through up to eleven layer runs


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """The models are tiny: threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, directory), written once."""
    root = tmp_path_factory.mktemp("dofunex")
    out = {}
    for j, (name, cfg) in enumerate(CASES.items()):
        w = weights(cfg, seed=j)
        out[name] = (cfg, w, write(cfg, w, root / name))
    return out


# ---- reading --------------------------------------------------------------------------------------------------------

def test_configuration_is_read_and_refused(tmp_path):
    p = tmp_path / "config.json"

    def read(c):
        p.write_text(json.dumps(c))
        return ModelConfig.from_hf(str(p))
    c = read(CASES["ragged"])
    assert c.layer_kinds == ["gqa", "cdelta", "gqa", "cdelta"] and c.loop == [1, 4, 3] and c.n_attn == 1 + 3
    assert [l.rot_dims for l in c.layers] == [24, 0, 20, 0] and c.layers[0].rot_scaling is None and c.layers[2].rot_scaling["high"] == 5.0
    assert [(l.conv, l.ff) for l in c.layers] == [(0, 90), (3, 70), (0, 0), (5, 50)]
    assert (c.residual_mult, c.logit_scale, c.pre_norm, c.out_norm) == (0.55, 1.7, True, True)
    b = read(CASES["bare"])
    assert b.loop is None and b.n_attn == 0 and b.eps == 1e-3
    for change, what in (((lambda c: c.update(architecture="Dofunix")), "architecture"),
                         ((lambda c: c["layers"][1].update(type="conv")), "type"),
                         ((lambda c: c["layers"][0]["mlp"].update(kind="routed")), "kind"),
                         ((lambda c: c["layers"][0]["mixer"].update(vdim=24)), "vdim"),
                         ((lambda c: c["layers"][0]["mixer"].update(kv_heads=4)), "heads"),
                         ((lambda c: c["loop"].update(stop=5)), "loop")):
        bad = copy.deepcopy(CASES["ragged"])
        change(bad)
        with pytest.raises(ValueError, match=what):
            read(bad)


def test_order_of_layer_runs():
    for name, cfg in CASES.items():
        lp = cfg.get("loop")
        c = ModelConfig(n_layers=len(cfg["layers"]), loop=[lp["start"], lp["stop"], lp["times"]] if lp else None)
        assert [(r.layer, r.enter) for r in c.layer_runs] == plain.order(cfg), name
        assert [r.index for r in c.layer_runs] == list(range(len(c.layer_runs)))
    assert [r.layer for r in ModelConfig(n_layers=5, loop=[1, 3, 2]).layer_runs] == [0, 1, 2, 1, 2, 3, 4]
    assert scaled(dofunex_7b(), 2).loop is None and scaled(tiny_dofunex(), 2).loop == [1, 2, 3]


def test_checkpoint_shapes_are_checked_and_ranks_come_from_it(tmp_path):
    cfg = CASES["bare"]
    w = weights(cfg, ranks=(12, 36))
    d = write(cfg, w, tmp_path / "good")
    c = ModelConfig.from_hf(d + "/config.json")
    load_model_weights(d, c)
    assert [(l.decay_rank, l.gate_rank) for l in c.layers] == [(12, 36)] * 2
    for change, what in (((lambda w: w.pop("l0.mix.a2")), "l0.mix.a2"),
                         ((lambda w: w.update({"l1.mix.g2": w["l1.mix.g2"][:, :-1]})), "l1.mix.g2"),
                         ((lambda w: w.update({"l0.norm1b": w["l0.norm1b"][:-1]})), "l0.norm1b")):
        bad = dict(w)
        change(bad)
        d = write(cfg, bad, tmp_path / what.replace(".", "_"))
        with pytest.raises((KeyError, ValueError), match=what):
            load_model_weights(d, ModelConfig.from_hf(d + "/config.json"))


def test_kernel_layout_pads_with_zeros():
    cfg = tiny_dofunex()
    w = init_weights(cfg, seed=3)
    pk = pack_listed(cfg, w)
    W = 192
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        assert pk[p + "in_proj"].shape[0] % 8 == 0 and pk[p + "in_proj"].shape[1] == W and float(pk[p + "in_proj"][:, cfg.hidden:].abs().sum()) == 0
        assert torch.equal(pk[p + "mix_norm"][:cfg.hidden], w[p + "mix_norm"].float() * 0.6)
        if l.mixer == "gqa":
            d = gqa_dims(cfg, i)
            o = pk[p + "out_proj"].view(W, l.heads, d.hp)
            assert d.hp == 64 and torch.equal(o[:cfg.hidden, :, :l.dim].reshape(cfg.hidden, -1), w[p + "out_proj"])
            assert float(o[:, :, l.dim:].abs().sum()) == 0
    assert torch.equal(pk["final_norm"][:cfg.hidden], w["final_norm"].float() * 1.5) and pk["loop_in"].shape == (W, 2 * W)
    assert torch.equal(pk["loop_in"][:cfg.hidden, W:W + cfg.hidden], w["loop_in"][:, cfg.hidden:])
    assert cfg.param_count() == pytest.approx(sum(v.numel() for k, v in w.items() if v.dim() == 2 and "step" not in k), rel=1e-6)


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def rnd(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


def i32(v):
    return torch.tensor(v, dtype=torch.int32)


def test_frequencies_by_hand():
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 2 * math.pi * 10}}
    f = plain.frequencies(rot)
    # 10 f turns over the original context: 10, 3.16, 1, 0.316: kept, kept, on the lower edge (f / factor), below it
    assert torch.allclose(f, torch.tensor([1.0, 100 ** -0.25, 0.025, 100 ** -0.75 / 4], dtype=torch.float64))
    rot["scaling"]["high"] = 5.0                                     # 3.16 turns now lie between: s = 2.16 / 4
    s = (10 * 100 ** -0.25 - 1) / 4
    assert float(plain.frequencies(rot)[1]) == pytest.approx((1 - s) * 100 ** -0.25 / 4 + s * 100 ** -0.25)
    from ferrite_b200.config import LayerSpec
    for rt in (rot, {"base": 5e5, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 700}}, {"base": 1e4, "dims": 6}):
        l = LayerSpec(rot_dims=rt["dims"], rot_base=rt["base"], rot_scaling=rt.get("scaling"))
        assert torch.allclose(rope_frequencies(l), plain.frequencies(rt), rtol=1e-12)


def prep_case(heads, kvh, dim, rot, hp=64, n=9, kvb=4, qk_norm=True, v_off=None, seed=1):
    """Rows 0 .. n - 1 of one sequence through the op -> (q, cached k, cached v, projection, bias, frequencies)."""
    d = GqaDims(heads, kvh, dim, hp, 0.3, rot, heads * dim if v_off is None else v_off, qk_norm)
    cols = max((heads + kvh) * dim, d.v_off + kvh * dim)
    proj, bias = rnd(n, cols, seed=seed), rnd(cols, seed=seed + 1)
    freq = plain.frequencies({"base": 50.0, "dims": rot}) if rot else torch.zeros(0, dtype=torch.float64)
    kc, vc = torch.full((4, kvb, kvh, hp), 9.0), torch.full((4, kvb, kvh, hp), 9.0)
    bt = i32([[0, 1, 2, 3], [2, 0, 3, 1]])
    q = TorchOps("cpu").gqa_prep(proj, d, bias, freq, i32([1] * n), i32(list(range(n))), bt, kc, vc, kvb, 1e-4)
    rows = lambda c: torch.stack([c[int(bt[1, t // kvb]), t % kvb] for t in range(n)])
    return q, rows(kc), rows(vc), proj + bias, freq


@pytest.mark.parametrize("heads,kvh,dim,rot", [(4, 2, 12, 12), (3, 1, 10, 4), (2, 2, 8, 0), (6, 3, 64, 64)])
def test_rotation_norm_and_values_from_keys(heads, kvh, dim, rot):
    q, k, v, p, f = prep_case(heads, kvh, dim, rot)
    n = p.shape[0]
    pq, pk = p[:, :heads * dim].reshape(n, heads, dim), p[:, heads * dim:].reshape(n, kvh, dim)
    assert torch.allclose(q[..., :dim], plain.rms(plain.rotate(pq, f), 1e-4), atol=1e-5)
    assert torch.allclose(k[..., :dim], plain.rms(plain.rotate(pk, f), 1e-4), atol=1e-5)
    assert torch.equal(v[..., :dim], pk)                             # as projected, before rotation and norm
    for t in (q, k, v):
        assert float(t[..., dim:].abs().sum()) == 0


def test_values_of_their_own_and_no_norm():
    """The op's options that this design does not use: separate values, rotation without a norm."""
    q, k, v, p, f = prep_case(2, 2, 8, 8, qk_norm=False, v_off=32)
    assert torch.allclose(v[..., :8], p[:, 32:].reshape(-1, 2, 8)) and torch.allclose(q[..., :8], plain.rotate(p[:, :16].reshape(-1, 2, 8), f), atol=1e-5)


@pytest.mark.parametrize("at", [0, 3, 4, 7, 8, 9, 10])
def test_one_key_stands_out(at):
    """A key that every query points at: its value is returned when it is at or before the row, not one position later."""
    from ferrite_b200.ops.latent import SegGroup
    ops, kvb, D, bt = TorchOps("cpu"), 4, 16, i32([[2, 0, 1]])
    kc, vc = torch.zeros(3, kvb, 2, D), torch.zeros(3, kvb, 2, D)
    k, v = rnd(12, 2, D) * 0.1, rnd(12, 2, D, seed=1)
    k[at] = 1.0
    for t in range(12):
        kc[int(bt[0, t // kvb]), t % kvb], vc[int(bt[0, t // kvb]), t % kvb] = k[t], v[t]
    d = GqaDims(4, 2, D, D, 3.0, 0, 0, True)
    for kvlen in (at, at + 1, 11):
        if kvlen == 0:
            continue
        o = ops.gqa_attention(torch.ones(1, 4, D), d, kc, vc, torch.tensor([0.0, 1, 2, 3]), SegGroup(0, 1, 0, 1, 1), i32([0]), i32([kvlen]), None, bt,
                              kvb, 1, torch.empty(1, 4, D))
        assert torch.allclose(o[0], v[at, [0, 0, 1, 1]], atol=1e-4) == (kvlen > at)


def test_sink_joins_the_denominator_once_and_unscaled():
    s = plain.sink_softmax(torch.zeros(2, 3, 3), torch.tensor([0.0, math.log(4.0)]))
    assert torch.allclose(s[0, :, 0], torch.tensor([1 / 2, 1 / 3, 1 / 4])) and torch.allclose(s[1].sum(-1), torch.tensor([1 / 5, 2 / 6, 3 / 7]))
    assert float(s[:, 0, 1:].sum()) == 0
    from ferrite_b200.ops.latent import SegGroup
    kc = vc = torch.ones(1, 4, 1, 8)
    o = TorchOps("cpu").gqa_attention(torch.zeros(1, 2, 8), GqaDims(2, 1, 8, 8, 7.0, 0, 0, True), kc, vc, torch.tensor([0.0, math.log(4.0)]),
                                      SegGroup(0, 1, 0, 1, 1), i32([0]), i32([3]), None, i32([[0]]), 4, 1, torch.empty(1, 2, 8))
    assert torch.allclose(o[0, :, 0], torch.tensor([3 / 4, 3 / 7]))


def test_norms_around_a_sublayer_bias_and_entry_of_a_pass():
    ops = TorchOps("cpu")
    x, y, w, w2, b = rnd(5, 12), rnd(5, 12, seed=1) * 3, rnd(12, seed=2), rnd(12, seed=3), rnd(12, seed=4)
    want = x + plain.rms_norm(y + b, w, 1e-3)
    xx, buf = x.clone(), torch.zeros(5, 24)
    h = ops.add_normed(xx, y, w, 12, 1e-3, bias=b, next_w=w2)
    assert torch.allclose(xx, want) and torch.allclose(h, plain.rms_norm(want, w2, 1e-3))
    ops.add_normed(xx, y, None, 12, 1e-3, bias=b, out=buf[:, 12:])
    assert torch.allclose(xx, y + b) and torch.allclose(buf[:, 12:], y + b) and float(buf[:, :12].abs().sum()) == 0


def delta_case(H, G, D, V, K, n, seed=0, decays=(-6.0, 3.0)):
    """One layer's tensors under the plain names and the op's, and projected rows for n tokens."""
    ra, rg, W = 8, 8, 16
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    w = {n: r(rows, W) * W ** -0.5 for n, rows in (("q", G * D), ("k", G * D), ("v", H * V), ("b", H), ("a1", ra), ("g1", rg))}
    w.update({n + ".conv": r(rows, K) for n, rows in (("q", G * D), ("k", G * D), ("v", H * V))})
    w.update(a2=r(H * D, ra), g2=r(H * V, rg), norm=r(V), A_log=torch.linspace(-4, 3, H),
             dt_bias=torch.rand(H * D, generator=g) * (decays[1] - decays[0]) + decays[0], o=torch.eye(H * V))
    d = DeltaDims(H, G, D, V, K, ra, rg, H * V)
    h = r(n, W)
    proj = h @ torch.cat([w[x] for x in ("a1", "g1", "q", "k", "v", "b")]).t()
    op = dict(decay_up=w["a2"], gate_up_lr=w["g2"], conv=torch.cat([w[x + ".conv"] for x in "qkv"]), A_log=w["A_log"], dt_bias=w["dt_bias"],
              gnorm_w=w["norm"])
    m = dict(heads=H, kv_heads=G, dim=D, vdim=V)
    return d, op, proj, plain.channel_delta(m, {k: v.double() for k, v in w.items()}, "", h.double(), 1e-5)


@pytest.mark.parametrize("H,G,D,V,K", [(2, 2, 8, 6, 4), (6, 2, 5, 9, 3), (1, 1, 16, 4, 1), (4, 2, 12, 8, 6)])
def test_delta_rule_across_steps_slots_and_batches(H, G, D, V, K):
    """State and convolution inputs carried over cuts of any size, two sequences in one batch, slots used again."""
    ops = TorchOps("cpu")
    d, op, pa, want_a = delta_case(H, G, D, V, K, 23)
    _, _, _, _ = d, op, pa, want_a
    rec, tail = torch.zeros(3, H, D, V), torch.zeros(3, K - 1, d.channels)
    order = ((2, 0, 3), (2, 3, 4), (0, 0, 10), (2, 4, 9), (2, 9, 23), (0, 10, 23))            # (slot, rows from, to)
    got = {0: [], 2: []}
    for s, lo, hi in order:
        got[s].append(ops.cdelta(pa[lo:hi], d, op, rec, tail, [], i32([s]), i32([0]), i32([hi - lo]), 1e-5))
    for s in got:
        assert torch.allclose(torch.cat(got[s]).double(), want_a, atol=2e-5, rtol=1e-4)
    assert float(rec[1].abs().sum()) == 0
    rec[2], tail[2] = 0, 0
    before = rec[0].clone()
    y = ops.cdelta(torch.cat([pa[:4], pa[:7]]), d, op, rec, tail, [], i32([2, 1]), i32([0, 4]), i32([4, 7]), 1e-5, commit=False)
    assert torch.allclose(y.double(), torch.cat([want_a[:4], want_a[:7]]), atol=2e-5, rtol=1e-4)
    assert torch.equal(rec[0], before) and float(rec[1:].abs().sum() + tail[1:].abs().sum()) == 0


def test_read_out_sees_the_write_and_decay_comes_first():
    one = torch.ones(1, 1, 1)
    k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]])
    g = torch.tensor([[[0.5, 0.25]], [[0.5, 0.25]]])
    o = plain.delta_scan(k, k, torch.tensor([[[4.0]], [[10.0]]]), torch.tensor([[0.5], [0.5]]), g)
    assert o[:, 0, 0].tolist() == [2.0, 1.0 + 0.5 * (10.0 - 1.0)] and float(one) == 1.0
    assert torch.allclose(plain.short_conv(torch.arange(1.0, 4)[:, None], torch.tensor([[2.0, 10.0]])), torch.tensor([[10.0], [22.0], [34.0]]))
    assert torch.allclose(plain.unit(torch.tensor([[3.0, 4.0]])), torch.tensor([[0.6, 0.8]]))


# ---- whole models ------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", list(CASES))
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [63, 2, 1, 64, 3, 65, 2]], ids=["whole", "single", "pairs", "mixed"])
def test_sequence_in_portions(models, name, cuts):
    cfg, w, d = models[name]
    ids = tokens(cfg, 150 if cuts[0] > 2 else 70, 11)
    want, _ = plain.forward(cfg, w, ids)
    assert error(run_cuts(engine(d), ids, cuts), want) < LIM


def test_every_part_shows_in_the_logits(models):
    """The power of the comparisons: a token far back, a sink, a turn, a decay, a tap, a pass left out moves the last logits by far
    more than the tolerance."""
    cfg, w, d = models["ragged"]
    ids = tokens(cfg, 150, 11)
    base = plain.forward(cfg, w, ids)[0][-1:]
    for t in range(0, 6):
        assert error(plain.forward(cfg, w, ids[:t] + [(ids[t] + 1) % cfg["vocab"]] + ids[t + 1:])[0][-1:], base) > 20 * LIM
    for name in ("l0.mix.sink", "l2.mix.sink", "l0.mix.k.b", "l2.mix.o.b", "l1.mix.dt_bias", "l3.mix.A_log", "l1.mix.b", "loop.step", "l3.mix.g2"):
        assert error(plain.forward(cfg, dict(w, **{name: w[name] * 0.9}), ids)[0][-1:], base) > 50 * LIM, name
    for name in ("l1.mix.q.conv", "l3.mix.v.conv"):
        cut = w[name].clone()
        cut[:, 0] = 0                                                # the oldest tap
        assert error(plain.forward(cfg, dict(w, **{name: cut}), ids)[0][-1:], base) > 50 * LIM, name
    for change in (lambda c: c["loop"].update(times=2), lambda c: c["layers"][0]["mixer"]["rot"].update(base=705.0),
                   lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(low=1.1), lambda c: c.update(residual_mult=0.551)):
        other = copy.deepcopy(cfg)
        change(other)
        assert error(plain.forward(other, w, ids)[0][-1:], base) > 20 * LIM


def test_residual_rows_after_every_layer(models):
    cfg, w, d = models["grid"]
    cfg = dict(copy.deepcopy(cfg), loop=None)
    eng = engine(write(cfg, {k: v for k, v in w.items() if not k.startswith("loop")}, __import__("pathlib").Path(d).parent / "flat"))
    eng.cfg.tap_layers[:] = range(len(cfg["layers"]))
    ids = tokens(cfg, 40, 12)
    eng.forward([Segment(0, 0, ids, "none")])
    _, after = plain.forward(cfg, w, ids)
    assert len(eng.taps) == len(cfg["layers"])
    for got, want in zip(eng.taps, after):
        assert float((got.double() - want).abs().max()) < 1e-4 * float(want.abs().max())


def test_unequal_requests_together_and_reused_pages_and_slots(models):
    """Portions of some requests beside single tokens of others, in a pool that only holds what is live: requests end, their
    pages and slots (and the states in them) go to the next ones, one request pauses for some steps."""
    cfg, w, d = models["ragged"]
    eng = engine(d, max_ctx=256, pool=448)
    lens = {"a": 150, "b": 70, "c": 3, "d": 130, "e": 65, "f": 1}
    seqs = {k: tokens(cfg, n, 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: plain.forward(cfg, w, s)[0] for k, s in seqs.items()}
    slot, at, got, used = {}, {k: 0 for k in seqs}, {k: [] for k in seqs}, []
    free = [0, 1, 2, 3]
    steps = [dict(a=64, b=2), dict(a=1, b=60, c=3), dict(a=63, d=1), dict(b=8, d=64), dict(a=2, d=2), dict(a=20, d=63, f=1), dict(e=64), dict(e=1)]
    for st in steps:
        segs = []
        for k, n in st.items():
            if k not in slot:
                slot[k] = free.pop(0)
            segs.append((k, Segment(slot[k], at[k], seqs[k][at[k]:at[k] + n], "all")))
        lg, _, _ = eng.forward([s for _, s in segs], greedy=False)
        r = 0
        for k, s in segs:
            got[k].append(lg[r:r + len(s.tokens)].clone())
            r += len(s.tokens)
            at[k] += len(s.tokens)
            if at[k] == lens[k]:
                used.append(list(eng.ex.slot_blocks[slot[k]]))
                eng.reset_slot(slot[k])
                free.append(slot.pop(k))
    assert eng.ex.pool.n_free == eng.ex.pool.n_blocks == 7
    assert any(set(used[-1]) & set(u) for u in used[:-1])                         # pages did go round
    for k in seqs:
        assert error(torch.cat(got[k]), want[k]) < LIM, k


def test_rejected_rows_leave_no_trace(models):
    """Verify rows that are not kept: caches, recurrent states and convolution inputs follow the last kept one."""
    for name in ("grid", "ragged", "broad"):
        cfg, w, d = models[name]
        ids = tokens(cfg, 90, 6)
        want, _ = plain.forward(cfg, w, ids)
        eng = engine(d)
        eng.forward([Segment(0, 0, ids[:62], "none")])
        wrong = [(t + 1) % cfg["vocab"] for t in ids[64:69]]
        lg, _, _ = eng.forward([Segment(0, 62, ids[62:64] + wrong, "all")], commit=False, greedy=False)
        assert error(lg[:2], want[62:64]) < LIM
        eng.commit_verified([2])
        lg, _, _ = eng.forward([Segment(0, eng.slot_len[0], ids[64:], "all")], greedy=False)
        assert error(lg, want[64:]) < LIM


def test_snapshots_and_forks_carry_unequal_states(models):
    cfg, w, d = models["ragged"]
    ids = tokens(cfg, 60, 8)
    want, _ = plain.forward(cfg, w, ids)
    eng = engine(d)
    eng.forward([Segment(0, 0, ids[:40], "none")])
    snap = eng.ex.state_save(0)
    eng.ex.copy_slot(0, 2, 40)
    eng.forward([Segment(0, 40, ids[:9], "none")])                                # moves slot 0 away from the snapshot
    eng.slot_len[2] = 40
    lg, _, _ = eng.forward([Segment(2, 40, ids[40:], "all")], greedy=False)
    assert error(lg, want[40:]) < LIM
    eng.ex.state_restore(0, snap)
    lg, _, _ = eng.forward([Segment(0, 40, ids[40:], "all")], greedy=False)
    assert error(lg, want[40:]) < LIM


@pytest.mark.parametrize("name", ["grid", "round"])
def test_greedy_generation_and_scheduler(models, name):
    """Engine.generate, and the scheduler with more requests than slots, copy-drafted verify rows, a shared prefix resumed from
    the prompt cache, forks, parking and a page pool below slots x context."""
    cfg, w, d = models[name]
    prompts = [tokens(cfg, n, 30 + n) for n in (5, 70, 33, 1)]
    prompts.append(prompts[1] + tokens(cfg, 9, 77))
    prompts.append((tokens(cfg, 6, 78) * 6)[:34])
    want = [plain.greedy(cfg, w, p, 6) for p in prompts]
    eng = engine(d, slots=1, max_ctx=128)
    assert eng.generate(prompts[1], 6) == want[1]
    for spec, pool in ((0, 0), (0, 320), (4, 0), (3, 384)):
        eng = engine(d, slots=3, max_ctx=192, pool=pool, prefill_chunk=32)
        sched = Scheduler(eng, SchedOptions(spec=spec, arrival_ms=0, share_min=32))
        out = generate(sched, prompts, Sampling(max_tokens=6), snapshots=[[64] if len(p) > 64 else [] for p in prompts])
        assert out == want, (spec, pool)
        again = generate(sched, [prompts[4]], Sampling(max_tokens=6), snapshots=[[64]])      # from a kept or parked prefix
        assert again[0] == want[4]
        held = sum(len(b) for b in eng.ex.slot_blocks) + sum(len(e.blocks) for e in sched.park.entries.values())
        assert held + eng.ex.pool.n_free == eng.ex.pool.n_blocks


def test_long_decode_over_page_borders(models):
    cfg, w, d = models["ragged"]
    ids = tokens(cfg, 135, 9)
    want, _ = plain.forward(cfg, w, ids)
    assert error(run_cuts(engine(d), ids, [3, 1]), want) < LIM


def test_every_run_of_a_layer_has_its_own_cache_or_state():
    cfg = tiny_dofunex()
    eng = Engine(cfg, None, EngineConfig(n_slots=2, max_ctx=64), device="cpu")
    kinds = [cfg.layer_kinds[r.layer] for r in cfg.layer_runs]
    assert kinds == ["cdelta"] + ["gqa", "cdelta"] * 3 + ["gqa"]
    assert sorted(eng.ex.k_cache) == [r for r, k in enumerate(kinds) if k == "gqa"] and sorted(eng.ex.rec_state) == [0, 2, 4, 6]
    assert eng.ex.kv_block_bytes() == 64 * 4 * sum(2 * t.shape[2] * t.shape[3] for t in eng.ex.k_cache.values())
    assert set(weight_shapes(cfg)) == set(init_weights(cfg))


def test_reference_model_agrees():
    cfg = tiny_dofunex()
    w = init_weights(cfg, seed=4, std=0.1)
    ids = torch.randint(0, cfg.vocab, (20,), generator=torch.Generator().manual_seed(1)).tolist()
    ref = RefModel(cfg, w)
    want = ref.forward(ids, ref.new_state())
    eng = Engine(cfg, w, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    lg, _, _ = eng.forward([Segment(0, 0, ids, "all")], greedy=False)
    assert error(lg, want) < LIM


def test_trace_replay(models, tmp_path, monkeypatch, capsys):
    from ferrite_b200.tools.trace_run import main
    cfg, w, d = models["ragged"]
    a, b = tokens(cfg, 80, 40), tokens(cfg, 70, 41)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [65, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": []}, {"id": "y", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[5:], "want": []}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[67:], "want": [0, 12]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert main(["--model", d, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "256", "--device", "cpu"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = plain.forward(cfg, w, a)[0], plain.forward(cfg, w, b)[0]
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert error(read(0), wa[[65, 0]]) < LIM and error(read(1), wb[[4]]) < LIM and error(read(3), wa[[67, 79]]) < LIM
    assert not (tmp_path / "2.f32").exists()


def test_command_line_generates(models, capsys):
    from ferrite_b200.cli import main
    cfg, w, d = models["bare"]
    ids = tokens(cfg, 12, 3)
    assert main(["generate", "--model", d, "--device", "cpu", "--ids", ",".join(map(str, ids)), "--max-tokens", "5"]) == 0
    out = [json.loads(l) for l in capsys.readouterr().out.splitlines() if l.startswith("{")][-1]
    assert out["ids"] == plain.greedy(cfg, w, ids, 5)


# ---- two ranks ----------------------------------------------------------------------------------------------------------

def test_two_ranks_equal_one():
    import torch.multiprocessing as mp

    from test_tp_cpu import _free_port, _worker, gather
    cfg = tiny_dofunex()
    prompt = torch.randint(0, cfg.vocab, (70,), generator=torch.Generator().manual_seed(6)).tolist()
    eng = Engine(cfg, init_weights(cfg, seed=0), EngineConfig(n_slots=1, max_ctx=128), device="cpu")
    want, wp, _ = eng.forward([Segment(0, 0, prompt, "all")])
    want2, _, _ = eng.forward([Segment(0, len(prompt), [int(wp[0][-1])], "last")])
    ctx = mp.get_context("spawn")
    q, port = ctx.Queue(), _free_port()
    procs = [ctx.Process(target=_worker, args=(r, 2, port, prompt, q, "tiny-dofunex")) for r in range(2)]
    for p in procs:
        p.start()
    outs = gather(q, 2)
    for p in procs:
        p.join(timeout=60)
    for rank, logits, ids, l2 in outs:
        assert error(logits, want) < LIM and error(l2, want2) < LIM and ids.tolist() == wp[0].tolist()
    assert torch.equal(outs[0][1], outs[1][1]) and torch.equal(outs[0][3], outs[1][3])
