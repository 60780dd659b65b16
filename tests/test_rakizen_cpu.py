"""The Rakizen design on the fp32 CPU engine against a plain statement of it (`plain_rakizen.py`): configuration and checkpoint reading,
each mechanism, prompts, decoding, portions, batches, reused pages and slots, speculation, the scheduler."""
import copy
import io
import json
import math
import sys

import pytest
import torch

import plain_rakizen as plain
from rakizen_cases import CASES, config, dense, engine, error, run_cuts, tokens, weights, window, write
from ferrite_b200.config import EngineConfig, ModelConfig, rakizen, rakizen_7b, tiny_rakizen
from ferrite_b200.engine.engine import Engine
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.formats.loader import load_model_weights
from ferrite_b200.models.ref import RefModel
from ferrite_b200.models.weights import GqaDims, gqa_dims, init_weights, pack_listed, weight_shapes
from ferrite_b200.ops.latent import SegGroup
from ferrite_b200.ops.torch_ops import TorchOps

LIM = 6e-5          # fp32 rounding through up to eight layer runs


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """The models are tiny: threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, directory, 150 token ids, their plain logits), made once."""
    root = tmp_path_factory.mktemp("rakizen")
    out = {}
    for j, (name, cfg) in enumerate(CASES.items()):
        w, ids = weights(cfg, seed=j), tokens(cfg, 150, 11)
        out[name] = (cfg, w, write(cfg, w, root / name), ids, plain.forward(cfg, w, ids)[0])
    return out


def rnd(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


def i32(v):
    return torch.tensor(v, dtype=torch.int32)


# ---- reading --------------------------------------------------------------------------------------------------------

def test_configuration_is_read_and_refused(tmp_path):
    p = tmp_path / "config.json"

    def read(c):
        p.write_text(json.dumps(c))
        return ModelConfig.from_hf(str(p))
    c = read(CASES["ragged"])
    assert [(l.window, l.chunk, l.maps, l.out_gate, l.row_norm) for l in c.layers] == [(17, 0, 1, False, True), (0, 33, 2, True, False),
                                                                                      (70, 0, 1, False, True), (0, 90, 2, True, False)]
    assert [(l.ff, l.experts, l.top, l.groups, l.keep_groups) for l in c.layers] == [(90, 0, 0, 1, 1), (22, 12, 3, 3, 2), (0, 0, 0, 1, 1), (30, 10, 4, 5, 3)]
    assert [l.rot_dims for l in c.layers] == [24, 0, 20, 0] and c.layers[3].route_scale == 0.7 and c.layers[1].diff == 0.4
    assert c.parallel and c.pre_norm and not c.out_norm and not c.loop_input and c.n_attn == 8 and len(c.layer_runs) == 8
    assert [r.layer for r in c.layer_runs] == plain.order(CASES["ragged"])
    assert read(dict(CASES["bare"], loop=None)).loop is None
    free = copy.deepcopy(CASES["bare"])
    free["layers"][0]["mixer"]["softcap"] = None
    assert read(free).layers[0].softcap == 0.0
    for change, what in (((lambda c: c.update(architecture="Rakizan")), "architecture"),
                         ((lambda c: c["layers"][1].update(type="conv")), "type"),
                         ((lambda c: c["layers"][0]["mlp"].update(kind="routed")), "kind"),
                         ((lambda c: c["layers"][0]["mixer"].update(kv_heads=4)), "heads"),
                         ((lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)), "mask"),
                         ((lambda c: c["layers"][1]["mixer"].update(softcap=-1.0)), "softcap"),
                         ((lambda c: c["layers"][0]["mixer"]["rot"].update(dims=42)), "rotated"),
                         ((lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5)), "groups"),
                         ((lambda c: c["layers"][1]["mlp"]["router"].update(top=9)), "experts per token"),
                         ((lambda c: c["loop"].update(stop=5)), "loop")):
        bad = copy.deepcopy(CASES["ragged"])
        change(bad)
        with pytest.raises(ValueError, match=what):
            read(bad)


def test_checkpoint_shapes_are_checked(tmp_path):
    cfg = CASES["ragged"]
    w = weights(cfg)
    for change, what in (((lambda w: w.pop("l1.mlp.e7.up")), "l1.mlp.e7.up"),
                         ((lambda w: w.update({"l3.mlp.e0.down": w["l3.mlp.e0.down"][:, :-1]})), "l3.mlp.e0.down"),
                         ((lambda w: w.pop("final.norm.b")), "final.norm.b"),
                         ((lambda w: w.update({"l1.mix.lk2": w["l1.mix.lk2"][:-1]})), "l1.mix.lk2"),
                         ((lambda w: w.update({"l0.mix.q.norm": w["l0.mix.q.norm"][:40]})), "l0.mix.q.norm")):
        bad = dict(w)
        change(bad)
        d = write(cfg, bad, tmp_path / what.replace(".", "_"))
        with pytest.raises((KeyError, ValueError), match=what):
            load_model_weights(d, ModelConfig.from_hf(d + "/config.json"))


def test_kernel_layout():
    cfg = tiny_rakizen()
    w = init_weights(cfg, seed=3)
    pk, W = pack_listed(cfg, w), 192
    for i, l in enumerate(cfg.layers):
        p, d = f"l{i}.", gqa_dims(cfg, i)
        ip = pk[p + "in_proj"]
        assert ip.shape[0] % 8 == 0 and ip.shape[1] == W and float(ip[:, cfg.hidden:].abs().sum()) == 0
        assert torch.equal(ip[d.v_off:d.v_off + l.kv_heads * l.vdim, :cfg.hidden], w[p + "v"])
        if l.maps == 2:
            assert torch.equal(ip[d.gate_off:d.gate_off + l.heads * l.vdim, :cfg.hidden], w[p + "g"])
            lam = plain.difference_weight(*(w[p + n].double() for n in ("lq1", "lk1", "lq2", "lk2")), l.diff)
            assert float(pk[p + "lam"]) == pytest.approx(float(lam), rel=1e-6)
        if l.experts:
            assert torch.equal(ip[d.router_off:d.router_off + l.experts, :cfg.hidden], w[p + "router"])
            gu = pk[p + "experts_gate_up"].view(l.experts, 2, 64, W)
            assert torch.equal(gu[:, :, :l.ff, :cfg.hidden].reshape(l.experts, 2 * l.ff, -1), w[p + "experts_gate_up"]) and float(gu[:, :, l.ff:].abs().sum()) == 0
        elif l.ff:                                                   # both output projections in one
            o = pk[p + "out_proj"]
            assert o.shape == (W, l.heads * d.hp + 128) and torch.equal(o[:cfg.hidden, l.heads * d.hp:][:, :l.ff], w[p + "down"])
    assert cfg.param_count() == sum(v.numel() for v in w.values() if v.dim() > 1) and set(weight_shapes(cfg)) == set(w)
    assert 6.5e9 < rakizen_7b().param_count() < 9e9
    with pytest.raises(ValueError, match="one rank"):
        cfg.shard(2)


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def test_layer_norm_by_hand():
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]])
    h = plain.layer_norm(x, torch.tensor([1.0, 2.0, 1.0, 1.0]), torch.tensor([0.0, 0.5, 0.0, 0.0]), 4.0)      # mean 4, variance 5, root 3
    assert torch.allclose(h, torch.tensor([[-1.0, -2 / 3 + 0.5, 1 / 3, 1.0]]))
    ops = TorchOps("cpu")
    x, y, w, b = rnd(5, 16), rnd(5, 16, seed=1) + 3, rnd(16, seed=2), rnd(16, seed=3)
    for t in (x, y, w, b):
        t[..., 13:] = 0
    yp, wts = rnd(10, 16, seed=4), rnd(5, 2, seed=5).abs()
    yp[:, 13:] = 0
    for pairs, extra in ((None, 0), ((yp, wts), (yp.view(5, 2, 16) * wts[:, :, None]).sum(1))):
        xx = x.clone()
        h = ops.add_layer_norm(xx, y, 13, 1e-3, w, b, pairs)
        assert torch.allclose(xx, x + y + extra, atol=1e-6)
        assert torch.allclose(h[:, :13], plain.layer_norm(xx[:, :13], w[:13], b[:13], 1e-3), atol=1e-5) and float(h[:, 13:].abs().sum()) == 0
    assert ops.add_layer_norm(x.clone(), y, 13, 1e-3) is None
    got = ops.norm_rows(x, i32([4, 0]), w, 13, 1e-3, bias=b)
    assert torch.allclose(got[:, :13], plain.layer_norm(x[[4, 0], :13], w[:13], b[:13], 1e-3), atol=1e-5)


def dims(H, G, D, V, hp, M=1, scale=0.3, rot=0, **kw):
    v_off = (H + G) * M * D
    return GqaDims(H, G, D, hp, scale, rot, v_off, False, V, M, M == 1, **kw)


@pytest.mark.parametrize("H,G,D,V,rot,M,hp", [(4, 2, 12, 20, 12, 1, 64), (3, 1, 10, 6, 4, 1, 64), (2, 2, 8, 8, 0, 2, 64), (3, 3, 13, 27, 0, 2, 64), (4, 1, 64, 64, 64, 1, 64)])
def test_queries_keys_and_values(H, G, D, V, rot, M, hp):
    d, n, kvb = dims(H, G, D, V, hp, M, rot=rot), 9, 4
    proj = rnd(n, d.v_off + G * V + 3)
    norms = (rnd(H * D, seed=1), rnd(G * D, seed=2)) if M == 1 else None
    kc, vc, bt = torch.full((4, kvb, G, hp), 9.0), torch.full((4, kvb, G, hp), 9.0), i32([[0, 1, 2, 3], [2, 0, 3, 1]])
    freq = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    q = TorchOps("cpu").gqa_prep(proj, d, None, freq, i32([1] * n), i32(list(range(n))), bt, kc, vc, kvb, 1e-4, norms=norms)
    rows = lambda c: torch.stack([c[int(bt[1, t // kvb]), t % kvb] for t in range(n)])
    pq, pk, pv = proj[:, :H * M * D], proj[:, H * M * D:d.v_off], proj[:, d.v_off:d.v_off + G * V]
    if M == 1:
        pq, pk = plain.rms(pq, 1e-4) * norms[0], plain.rms(pk, 1e-4) * norms[1]
    pq, pk = (plain.rotate(x.reshape(n, -1, D), 50.0, rot) if rot else x.reshape(n, -1, D) for x in (pq, pk))
    assert torch.equal(rows(vc)[..., :V], pv.view(n, G, V)) and float(rows(vc)[..., V:].abs().sum()) == 0
    assert torch.allclose(rows(kc)[..., :M * D], pk.reshape(n, G, M * D), atol=1e-5) and float(rows(kc)[..., M * D:].abs().sum()) == 0
    assert q.shape == (n, H * M, hp)
    for m in range(M):                                               # a query meets its own map's keys only
        assert torch.allclose(q[:, m::M, m * D:(m + 1) * D], pq[:, m::M], atol=1e-5)
        assert float(q[:, m::M].abs().sum()) == pytest.approx(float(q[:, m::M, m * D:(m + 1) * D].abs().sum()))


@pytest.mark.parametrize("size", [1, 2, 3, 4, 5, 8, 11, 40])
@pytest.mark.parametrize("kind", ["window", "chunk"])
def test_masks_in_pages(kind, size):
    """Every row against every key it may see, pages of four keys."""
    n, kvb, H, G, D = 23, 4, 4, 2, 8
    mask = (plain.window_mask if kind == "window" else plain.chunk_mask)(n, size)
    d = dims(H, G, D, D, D, scale=2.0, softcap=3.0, **{kind: size})
    k, v, q = rnd(n, G, D), rnd(n, G, D, seed=1), rnd(n, H, D, seed=2)
    kc, vc, bt = torch.zeros(6, kvb, G, D), torch.zeros(6, kvb, G, D), i32([[5, 0, 3, 1, 4, 2]])
    for t in range(n):
        kc[int(bt[0, t // kvb]), t % kvb], vc[int(bt[0, t // kvb]), t % kvb] = k[t], v[t]
    out = TorchOps("cpu").gqa_attention(q, d, kc, vc, None, SegGroup(0, 1, 0, n, n), i32([0] * n), i32(list(range(1, n + 1))), None, bt, kvb, 1,
                                        torch.empty(n, H, D))
    assert torch.allclose(out, plain.attend(q, k, v, mask, 2.0, 3.0), atol=1e-5)
    assert [d.first_visible(i) for i in range(n)] == [int(mask[i].nonzero()[0]) for i in range(n)]


@pytest.mark.parametrize("at", [0, 3, 4, 7, 8, 9, 10])
def test_one_key_stands_out(at):
    """A key that every query points at: seen from its own row on while it is inside the window or the chunk, not one row longer."""
    n, kvb, D = 24, 4, 16
    k, v = 0.1 * rnd(n, 1, D), rnd(n, 1, D, seed=1)
    k[at] = 1.0
    kc, vc, bt = torch.zeros(6, kvb, 1, D), torch.zeros(6, kvb, 1, D), i32([[5, 0, 3, 1, 4, 2]])
    for t in range(n):
        kc[int(bt[0, t // kvb]), t % kvb], vc[int(bt[0, t // kvb]), t % kvb] = k[t], v[t]
    for kind, size, last in (("window", 6, at + 5), ("chunk", 5, at // 5 * 5 + 4)):
        d = dims(2, 1, D, D, D, scale=3.0, softcap=30.0, **{kind: size})
        o = TorchOps("cpu").gqa_attention(torch.ones(n, 2, D), d, kc, vc, None, SegGroup(0, 1, 0, n, n), i32([0] * n), i32(list(range(1, n + 1))), None,
                                          bt, kvb, 1, torch.empty(n, 2, D))
        hit = ((o - v[at]).abs().amax((1, 2)) < 1e-4).tolist()
        assert hit == [at <= t <= last for t in range(n)], (kind, hit)


def test_softcap_difference_and_gate_by_hand():
    assert float(plain.capped(torch.tensor(2.0), 4.0)) == pytest.approx(4.0 * math.tanh(0.5))
    a1, a2 = torch.tensor([[[3.0, 4.0]]]), torch.tensor([[[0.0, 8.0]]])
    assert torch.allclose(plain.difference(a1, a2, 0.5, 0.25, 0.0), torch.tensor([[[3.0, 0.0]]]) / math.sqrt(4.5) * 0.75)
    assert float(plain.difference_weight(*(torch.tensor([x]) for x in (1.0, math.log(3.0), 1.0, 0.0)), 0.5)) == pytest.approx(3.0 - 1.0 + 0.5)
    # two maps over one head: map 1 sees key 0 alone, map 2 both keys alike
    kc, vc = torch.zeros(1, 4, 1, 8), torch.zeros(1, 4, 1, 8)
    kc[0, 0, 0, 0], vc[0, 0, 0, :2], vc[0, 1, 0, :2] = 1.0, torch.tensor([4.0, 0.0]), torch.tensor([0.0, 2.0])
    q = torch.zeros(1, 2, 8)
    q[0, 0, 0] = 1.0
    d = dims(1, 1, 4, 2, 8, 2, scale=100.0, softcap=50.0, chunk=4, diff=0.2)
    gate, lam = torch.tensor([[0.0, math.log(3.0)]]), torch.tensor([0.5])
    o = TorchOps("cpu").gqa_attention(q, d, kc, vc, None, SegGroup(0, 1, 0, 1, 1), i32([0]), i32([2]), None, i32([[0]]), 4, 1, torch.empty(1, 1, 8),
                                      lam=lam, gate=gate, eps=0.0)
    want = torch.tensor([4.0 - 0.5 * 2.0, 0.0 - 0.5 * 1.0])
    want = want / want.pow(2).mean().sqrt() * 0.8 * torch.tensor([0.5, 0.75])
    assert torch.allclose(o[0, 0, :2], want, atol=1e-5) and float(o[0, 0, 2:].abs().sum()) == 0


@pytest.mark.parametrize("experts,top,groups,keep", [(8, 2, 4, 2), (12, 3, 3, 2), (10, 4, 5, 3), (6, 6, 1, 1), (48, 6, 16, 5), (5, 2, 5, 3), (7, 1, 1, 1)])
def test_routing(experts, top, groups, keep):
    z = rnd(40, experts, seed=experts)
    ids, wts = TorchOps("cpu").moe_route(z, None, 1, top, groups, keep, 1.7)
    for t in range(40):
        want = plain.route(z[t].double(), top, groups, keep, 1.7)
        assert ids[t].tolist() == [e for e, _ in want] and torch.allclose(wts[t].double(), torch.tensor([g for _, g in want], dtype=torch.float64), rtol=1e-5)


def test_a_group_wins_by_its_two_best_not_its_best():
    z = torch.tensor([3.0, -9.0, -9.0, 1.0, 1.0, -9.0])               # the best expert sits in the weaker group
    assert [e for e, _ in plain.route(z, 2, 2, 1, 1.0)] == [3, 4] and [e for e, _ in plain.route(z, 2, 2, 2, 1.0)] == [0, 3]


# ---- whole models ------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", list(CASES))
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [63, 2, 1, 64, 3, 65, 2]], ids=["whole", "single", "pairs", "mixed"])
def test_sequence_in_portions(models, name, cuts):
    cfg, w, d, ids, want = models[name]
    n = 150 if cuts[0] > 2 else 100
    assert error(run_cuts(engine(d), ids[:n], cuts), want[:n]) < LIM


def test_every_part_shows_in_the_logits(models):
    """The power of the comparisons: a weight, a constant, a mask's edge moved by one token moves the logits by far more than the tolerance."""
    cfg, w, d, ids, _ = models["ragged"]
    ids = ids[:100]
    base = plain.forward(cfg, w, ids)[0]
    for name in ("l0.mix.q.norm", "l2.mix.k.norm", "l1.mix.lq1", "l3.mix.lk2", "l1.mix.g", "l0.norm1.b", "final.norm.b", "l3.mlp.router", "l1.mlp.e5.up"):
        assert error(plain.forward(cfg, dict(w, **{name: w[name] * 0.9}), ids)[0], base) > 20 * LIM, name
    for change in (lambda c: c["loop"].update(times=1), lambda c: c["layers"][0]["mixer"]["rot"].update(base=930.0),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(size=18), lambda c: c["layers"][1]["mixer"]["mask"].update(size=34),
                   lambda c: c["layers"][2]["mixer"]["mask"].update(size=71), lambda c: c["layers"][3]["mixer"]["mask"].update(size=89),
                   lambda c: c["layers"][0]["mixer"].update(softcap=12.0), lambda c: c["layers"][3]["mixer"].update(softcap=18.0),
                   lambda c: c["layers"][1]["mixer"].update(diff=0.41), lambda c: c["layers"][1]["mlp"]["router"].update(scale=1.32),
                   lambda c: c["layers"][3]["mlp"]["router"]["groups"].update(keep=4), lambda c: c["layers"][3]["mlp"]["router"].update(top=3),
                   lambda c: c["norm"].update(eps=2e-3)):
        other = copy.deepcopy(cfg)
        change(other)
        assert error(plain.forward(other, w, ids)[0], base) > 20 * LIM


def test_residual_rows_after_every_layer(models):
    cfg, w, d, ids, _ = models["grid"]
    cfg = dict(copy.deepcopy(cfg), loop=None)
    eng = engine(write(cfg, w, __import__("pathlib").Path(d).parent / "flat"))
    eng.cfg.tap_layers[:] = range(len(cfg["layers"]))
    eng.forward([Segment(0, 0, ids[:40], "none")])
    _, after = plain.forward(cfg, w, ids[:40])
    assert len(eng.taps) == len(cfg["layers"])
    for got, want in zip(eng.taps, after):
        assert float((got.double() - want).abs().max()) < 1e-4 * float(want.abs().max())


def test_unequal_requests_together_and_reused_pages_and_slots(models):
    """Portions of some requests beside single tokens of others, in a pool that only holds what is live: requests end, their pages and
    slots go to the next ones, one request pauses for some steps."""
    cfg, w, d, _, _ = models["ragged"]
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


def test_rejected_rows_and_forks_leave_no_trace(models):
    for name in ("grid", "ragged"):
        cfg, w, d, ids, want = models[name]
        eng = engine(d)
        eng.forward([Segment(0, 0, ids[:62], "none")])
        wrong = [(t + 1) % cfg["vocab"] for t in ids[64:69]]
        lg, _, _ = eng.forward([Segment(0, 62, ids[62:64] + wrong, "all")], commit=False, greedy=False)
        assert error(lg[:2], want[62:64]) < LIM
        eng.commit_verified([2])
        eng.ex.copy_slot(0, 2, 64)
        eng.forward([Segment(0, 64, ids[:9], "none")])                            # moves slot 0 away from its copy
        lg, _, _ = eng.forward([Segment(2, 64, ids[64:90], "all")], greedy=False)
        assert error(lg, want[64:90]) < LIM


def test_greedy_generation_and_scheduler(models):
    """Engine.generate, and the scheduler with more requests than slots, copy-drafted verify rows, a shared prefix resumed from the prompt
    cache, parking and a page pool below slots x context."""
    cfg, w, d, _, _ = models["edges"]
    prompts = [tokens(cfg, n, 30 + n) for n in (5, 70, 33, 1)]
    prompts.append(prompts[1] + tokens(cfg, 9, 77))
    prompts.append((tokens(cfg, 6, 78) * 6)[:34])
    want = [plain.greedy(cfg, w, p, 5) for p in prompts]
    eng = engine(d, slots=1, max_ctx=128)
    assert eng.generate(prompts[1], 5) == want[1]
    for spec, pool in ((0, 0), (0, 320), (4, 384)):
        eng = engine(d, slots=3, max_ctx=192, pool=pool, prefill_chunk=32)
        sched = Scheduler(eng, SchedOptions(spec=spec, arrival_ms=0, share_min=32))
        out = generate(sched, prompts, Sampling(max_tokens=5), snapshots=[[64] if len(p) > 64 else [] for p in prompts])
        assert out == want, (spec, pool)
        again = generate(sched, [prompts[4]], Sampling(max_tokens=5), snapshots=[[64]])      # from a kept or parked prefix
        assert again[0] == want[4]
        held = sum(len(b) for b in eng.ex.slot_blocks) + sum(len(e.blocks) for e in sched.park.entries.values())
        assert held + eng.ex.pool.n_free == eng.ex.pool.n_blocks


def test_long_decode_over_windows_chunks_and_pages(models):
    cfg, w, d, ids, want = models["ragged"]
    assert error(run_cuts(engine(d), ids, [3, 1]), want) < LIM


def test_every_run_of_a_layer_has_its_own_cache():
    cfg = tiny_rakizen()
    eng = Engine(cfg, None, EngineConfig(n_slots=2, max_ctx=64), device="cpu")
    assert [r.layer for r in cfg.layer_runs] == [0, 1, 2, 1, 2, 3] and sorted(eng.ex.k_cache) == list(range(6))
    assert eng.ex.kv_block_bytes() == 64 * 4 * sum(2 * t.shape[2] * t.shape[3] for t in eng.ex.k_cache.values())


def test_expert_counters(monkeypatch, tmp_path):
    monkeypatch.setenv("FE_EXPERT_HEAT", str(tmp_path / "heat.json"))
    cfg = tiny_rakizen()
    eng = Engine(cfg, None, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    eng.forward([Segment(0, 0, list(range(10)), "none")])
    heat = eng.expert_heat()
    assert {i: sum(v) for i, v in heat.items()} == {1: 2 * 10 * 2, 3: 10 * 2} and all(len(v) == 7 for v in heat.values())


def test_index_checks_cover_the_ops(monkeypatch):
    monkeypatch.setenv("FB_DEBUG_BOUNDS", "1")
    eng = Engine(tiny_rakizen(), None, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    eng.forward([Segment(0, 0, list(range(10)), "last")])
    assert {"embed_grams", "gqa_prep", "gqa_attention", "expert_rows"} <= set(eng.bounds.checked)
    with pytest.raises(IndexError, match="experts of the layer"):
        eng.ex.ops.expert_rows(torch.zeros(1, 192), i32([[6]]), torch.zeros(6, 128, 192), torch.zeros(6, 192, 64))


def test_reference_model_agrees():
    cfg = tiny_rakizen()
    w = init_weights(cfg, seed=4, std=0.1)
    ids = torch.randint(0, cfg.vocab, (70,), generator=torch.Generator().manual_seed(1)).tolist()
    ref = RefModel(cfg, w)
    want = ref.forward(ids, ref.new_state())
    eng = Engine(cfg, w, EngineConfig(n_slots=1, max_ctx=128), device="cpu")
    lg, _, _ = eng.forward([Segment(0, 0, ids, "all")], greedy=False)
    assert error(lg, want) < LIM
    c = rakizen(64, 2, 4, 2, 96, 50, dim=16, window=9, chunk=8, every=2)
    assert [l.maps for l in c.layers] == [1, 2] and Engine(c, None, EngineConfig(n_slots=1, max_ctx=64), device="cpu").generate(list(range(20)), 3)


def test_trace_replay(models, tmp_path, monkeypatch, capsys):
    from ferrite_b200.tools.trace_run import main
    cfg, w, d, a, wa = models["ragged"]
    a, b = a[:80], tokens(cfg, 70, 41)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [65, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": []}, {"id": "y", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[5:], "want": []}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[67:], "want": [0, 12]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    assert main(["--model", d, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "256", "--device", "cpu"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wb = plain.forward(cfg, w, b)[0]
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert error(read(0), wa[[65, 0]]) < LIM and error(read(1), wb[[4]]) < LIM and error(read(3), wa[[67, 79]]) < LIM
    assert not (tmp_path / "2.f32").exists()


def test_command_line_generates(models, capsys):
    from ferrite_b200.cli import main
    cfg, w, d, _, _ = models["bare"]
    ids = tokens(cfg, 12, 3)
    assert main(["generate", "--model", d, "--device", "cpu", "--ids", ",".join(map(str, ids)), "--max-tokens", "5"]) == 0
    out = [json.loads(l) for l in capsys.readouterr().out.splitlines() if l.startswith("{")][-1]
    assert out["ids"] == plain.greedy(cfg, w, ids, 5)


def test_a_window_and_a_chunk_of_one_page_differ(tmp_path):
    """The two masks agree up to the first edge and nowhere behind it."""
    cfg = config(64, 90, [window(2, 1, 16, 16, 64, dense(32), rot=0)])
    w = weights(cfg, seed=5)
    ids = tokens(cfg, 130, 1)
    got = run_cuts(engine(write(cfg, w, tmp_path / "m")), ids, [130])
    free = copy.deepcopy(cfg)
    free["layers"][0]["mixer"]["mask"]["size"] = 1000
    all_keys = plain.forward(free, w, ids)[0]
    assert error(got[:64], all_keys[:64]) < LIM and error(got[64:], all_keys[64:]) > 100 * LIM
