"""The kernels and the engine of the Dofunex design on the GPU, in bf16 and in fp32, against plain statements of the same arithmetic:
every kernel alone (sizes on and off its tiles, keys at page borders and just inside and outside what a row sees, decays from none
to total), then whole models in prompts, portions, decoding, mixed batches and through the scheduler."""
import copy
import math

import pytest
import torch

import plain_dofunex as plain
from dofunex_cases import CASES, attn, config, delta, engine, error, run_cuts, tokens, weights, write
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.models.weights import DeltaDims, GqaDims
from ferrite_b200.ops.latent import SegGroup
from ferrite_b200.ops.torch_ops import TorchOps

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
LIM = {"fp32": 1e-4, "bf16": 8e-2}


@pytest.fixture(scope="module")
def cops(ext):
    from ferrite_b200.ops.cuda_ops import CudaOps
    return {BF: CudaOps(DEV), F32: CudaOps(DEV, F32)}


def gen(seed):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return lambda *s, sc=1.0, dt=F32: (torch.randn(*s, generator=g, device=DEV) * sc).to(dt)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


up = lambda n, m: (n + m - 1) // m * m


# ---- rows ---------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("width", [64, 320, 4096, 13312])
def test_residual_add_with_bias_and_next_norm(cops, dt, width):
    ops, r = cops[dt], gen(width)
    true, tol = width - 5, 1e-5 if dt == F32 else 3e-2
    x, w, w2, b = r(9, width), r(width), r(width), r(width)
    for t in (x, w, w2, b):
        t[..., true:] = 0
    xd = lambda t: t[..., :true].double()
    for y in (r(9, width, sc=4.0), r(9, width + 16)[:, :width]) + ((r(9, width, dt=BF),) if dt == BF else ()):
        y[:, true:] = 0
        for bias in (None, b):
            yd = xd(y) + (0 if bias is None else xd(b))
            want = xd(x) + plain.rms_norm(yd, xd(w), 1e-5)
            for nw in (None, w2):
                x1, buf = x.clone(), torch.full((9, 2 * width), 7.0, dtype=dt, device=DEV)
                h = ops.add_normed(x1, y, w, true, 1e-5, bias=bias, next_w=nw)
                ref = want if nw is None else plain.rms_norm(want, xd(w2), 1e-5)
                assert torch.allclose(xd(x1), want, atol=3e-5, rtol=1e-5) and torch.allclose(xd(h), ref, atol=tol, rtol=tol)
                assert float(h[:, true:].float().abs().sum()) == 0
                x2 = x.clone()
                ops.add_normed(x2, y, None, true, 1e-5, bias=bias, next_w=nw, out=buf[:, width:])
                ref = yd if nw is None else plain.rms_norm(yd, xd(w2), 1e-5)
                assert torch.allclose(xd(x2), yd, atol=1e-5) and torch.allclose(xd(buf[:, width:]), ref, atol=tol, rtol=tol)
                assert bool((buf[:, :width] == 7.0).all())
    table, tok = r(50, width, dt=dt), i32([3, 49, 0])
    buf = torch.zeros(3, 2 * width, dtype=dt, device=DEV)
    x, xb = ops.embed_grams(table, None, tok, i32([0] * 3), i32([0, 1, 2]), i32([[0]]), None, 64, 1.0, 0, 0, 0, out=buf)
    assert torch.equal(x, table[tok.long()].float()) and torch.equal(buf, torch.cat([table[tok.long()]] * 2, 1)) and xb is buf
    assert ops.status() == 0


def test_fp32_swiglu(cops):
    ops, r = cops[F32], gen(5)
    x, w = r(7, 128), r(2 * 64, 128)
    assert torch.allclose(ops.linear(x, w, swiglu=True), plain.silu(x @ w[:64].t()) * (x @ w[64:].t()), atol=1e-3, rtol=1e-4)


# ---- attention ------------------------------------------------------------------------------------------------------------

def head(d):
    return next((h for h in (64, 128, 256) if d <= h), up(d, 64))


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("heads,kvh,dim,rot", [(4, 2, 64, 64), (5, 1, 40, 16), (3, 3, 128, 128), (9, 3, 100, 36), (2, 1, 256, 128), (2, 2, 272, 272), (1, 1, 18, 0),
                                               (40, 8, 128, 128), (2, 1, 900, 64)])
def test_queries_keys_and_values(cops, dt, heads, kvh, dim, rot):
    ops, tops, r, kvb = cops[dt], TorchOps(DEV, F32), gen(dim), 64
    for key_values, norm, with_bias in ((True, True, True), (False, True, False), (True, False, True)):
        d = GqaDims(heads, kvh, dim, head(dim), 0.3, rot, (heads + (0 if key_values else kvh)) * dim, norm)
        cols = (heads + (1 if key_values else 2) * kvh) * dim
        proj, bias = r(8, up(cols, 8) + 8, sc=2.0)[:, :cols], r(cols) if with_bias else None
        freq = plain.frequencies({"base": 3e4, "dims": rot}).to(DEV) if rot else torch.zeros(0, dtype=torch.float64, device=DEV)
        bt = torch.full((2, 1 << 14), -1, dtype=torch.int32, device=DEV)
        pos = i32([62, 63, 64, 0, 1, 127, 128, 1000003])                              # page borders, a position past what fp32 angles hold
        slot = i32([0, 0, 0, 1, 1, 1, 1, 0])
        bt[0, :2], bt[1, :3], bt[0, 1000003 // kvb] = i32([3, 1]), i32([0, 2, 4]), 5
        caches = [torch.full((6, kvb, kvh, d.hp), 5.0, dtype=t, device=DEV) for t in (dt, dt, F32, F32)]
        q = ops.gqa_prep(proj, d, bias, freq, slot, pos, bt, caches[0], caches[1], kvb, 1e-4)
        want = tops.gqa_prep(proj, d, bias, freq, slot, pos, bt, caches[2], caches[3], kvb, 1e-4)
        tol = 2e-5 if dt == F32 else 4e-2
        assert torch.allclose(q.float(), want, atol=tol, rtol=tol)
        for a, b in zip(caches[:2], caches[2:]):
            assert torch.allclose(a.float(), b, atol=tol, rtol=tol) and int((a != 5.0).flatten(2).any(-1).sum()) == 8
    assert ops.status() == 0


def paged(kvh, hp, lens, dt, seed, kvb=64):
    r = gen(seed)
    nb = [(n + kvb - 1) // kvb for n in lens]
    perm = torch.randperm(sum(nb) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
    bt = torch.full((len(lens), max(nb)), -1, dtype=torch.int32)
    k = 0
    for s, n in enumerate(nb):
        for j in range(n):
            bt[s, j] = perm[k]
            k += 1
    return r(sum(nb) + 2, kvb, kvh, hp, dt=dt), r(sum(nb) + 2, kvb, kvh, hp, dt=dt), bt.to(DEV)


def attend_case(ops, dt, heads, kvh, hp, segs, nsplit, scale, seed, sink=None, prompt=False, plant=None, lead=0):
    """segs: (rows, context length after the segment), the first `lead` of them outside the group. Returns (kernel's rows, plain rows)."""
    kvb, r = 64, gen(seed + 1)
    kc, vc, bt = paged(kvh, hp, [n for _, n in segs], dt, seed)
    slot = i32([s for s, (m, _) in enumerate(segs) for _ in range(m)])
    kvlen = i32([n - m + j + 1 for m, n in segs for j in range(m)])
    row0 = [sum(m for m, _ in segs[:s]) for s in range(len(segs))]
    q = r(slot.numel(), heads, hp, dt=dt)
    if plant is not None:
        plant(q, kc, vc, bt, kvb)
    d = GqaDims(heads, kvh, hp, hp, scale, 0, 0, True)
    tables = [i32(list(range(len(segs)))), i32(row0), i32([m for m, _ in segs]), i32([n - m for m, n in segs])]
    a = sum(m for m, _ in segs[:lead])
    g = SegGroup(lead, len(segs), a, slot.numel(), max(m for m, _ in segs[lead:]), prompt)
    out = torch.full_like(q, 7.0)
    ops.gqa_attention(q, d, kc, vc, sink, g, slot, kvlen, tuple(t[lead:] for t in tables), bt, kvb, nsplit, out)
    want = TorchOps(DEV, F32).gqa_attention(q, d, kc, vc, sink, g, slot, kvlen, None, bt, kvb, 1, torch.full(q.shape, 7.0, device=DEV))
    assert ops.status() == 0 and bool((out[:a] == 7.0).all())
    return out.float(), want


TOL = {F32: dict(atol=2e-5, rtol=1e-4), BF: dict(atol=2e-2, rtol=1e-2)}


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("heads,kvh,hp", [(1, 1, 64), (8, 2, 64), (6, 2, 128), (5, 1, 128), (32, 8, 128), (4, 4, 256), (16, 1, 256), (3, 1, 320), (70, 1, 64), (2, 2, 1024)])
def test_few_rows_attention_sizes(cops, dt, heads, kvh, hp):
    sink = gen(hp)(heads, sc=2.0)
    for nsplit in (1, 3, 64):
        segs = [(1, 1), (1, 63), (1, 64), (1, 65), (1, 400)]
        got, want = attend_case(cops[dt], dt, heads, kvh, hp, segs, nsplit, 2.0 * hp ** -0.5, hp + heads, sink)
        assert torch.allclose(got, want, **TOL[dt]), (nsplit, (got - want).abs().max())
    segs = [(5, 9), (7, 130), (2, 2), (1, 321), (30, 96), (3, 66)]
    for s, lead in ((sink, 0), (None, 2)):
        got, want = attend_case(cops[dt], dt, heads, kvh, hp, segs, 8, 2.0 * hp ** -0.5, hp + heads, s, lead=lead)
        assert torch.allclose(got, want, **TOL[dt])


@pytest.mark.parametrize("dt,prompt", [(BF, False), (BF, True), (F32, False)])
@pytest.mark.parametrize("at", [0, 1, 63, 64, 127, 128, 198, 199])
def test_one_key_stands_out(cops, dt, prompt, at):
    """One key that all queries point at among hundreds: rows at or after it return its value, rows before it do not see it."""
    def plant(q, kc, vc, bt, kvb):
        q.fill_(1.0)
        vc.mul_(0.1)
        page = int(bt[0, at // kvb])
        kc[page, at % kvb], vc[page, at % kvb] = 8.0, 2.0
    sink = torch.tensor([0.0, 1.0, 3.0, 300.0], device=DEV)                            # the last one outweighs any key
    got, want = attend_case(cops[dt], dt, 4, 2, 64, [(200, 200)], 4, 0.3, at, sink, prompt, plant)
    hit = (got[:, :3] - 2.0).abs().amax((1, 2)) < 2e-2
    assert bool(hit[at:].all()) and not bool(hit[:at].any())
    assert torch.allclose(got, want, **TOL[dt]) and float(got[:, 3].abs().max()) < 1e-6


@pytest.mark.parametrize("heads,kvh,hp", [(4, 2, 64), (3, 1, 128), (2, 2, 256), (10, 2, 128)])
def test_prompt_attention(cops, heads, kvh, hp):
    sink = gen(hp)(heads, sc=2.0)
    for segs, lead, s in (([(200, 200)], 0, sink), ([(1, 90), (40, 40), (130, 400), (64, 128)], 1, sink), ([(33, 97)], 0, None)):
        got, want = attend_case(cops[BF], BF, heads, kvh, hp, segs, 1, 2.0 * hp ** -0.5, hp + heads, s, True, lead=lead)
        assert torch.allclose(got, want, **TOL[BF]), (got - want).abs().max()


@pytest.mark.parametrize("prompt", [False, True])
def test_softmax_weights_keep_more_than_16_bit_operands(cops, prompt):
    """Two keys whose large values nearly cancel: softmax weights rounded to bf16 would be off by 2^-9 of them."""
    def plant(q, kc, vc, bt, kvb):
        q.zero_(); kc.zero_(); vc.zero_()
        q[..., 0] = 1.0
        page = int(bt[0, 0])
        kc[page, 0, :, 0], vc[page, 0, :, 1], vc[page, 1, :, 1] = 0.3, 64.0, -86.0
        kc[page, 2:, :, 0] = -60.0
    got, _ = attend_case(cops[BF], BF, 1, 1, 64, [(40, 40)], 1, 1.0, 3, None, prompt, plant)
    p = torch.softmax(torch.tensor([float(torch.tensor(0.3).to(BF)), 0.0], dtype=torch.float64), 0)
    want = float(p[0] * 64.0 - p[1] * 86.0)
    assert float((got[1:, 0, 1].double() - want).abs().max()) < 64 * 2.0 ** -12 and abs(want) < 0.5


# ---- delta rule -------------------------------------------------------------------------------------------------------------

def delta_layer(dt, H, G, D, V, K, n, seed, decays, ra=20, rg=28):
    r = gen(seed)
    d = DeltaDims(H, G, D, V, K, up(ra, 64), up(rg, 64), up(H * V, 64))
    cols = d.b_off + H
    proj = r(n, up(cols, 8), sc=1.0)
    proj[:, ra:d.ra], proj[:, d.ra + rg:d.q_off] = 0, 0
    w = dict(decay_up=torch.zeros(H * D, d.ra, device=DEV), gate_up_lr=torch.zeros(H * V, d.rg, device=DEV), conv=r(d.channels, K, sc=K ** -0.5),
             A_log=torch.linspace(-3, 4, H, device=DEV), gnorm_w=1 + 0.3 * r(V),
             dt_bias=torch.rand(H * D, device=DEV, generator=torch.Generator(DEV).manual_seed(seed)) * (decays[1] - decays[0]) + decays[0])
    w["decay_up"][:, :ra], w["gate_up_lr"][:, :rg] = r(H * D, ra, sc=1.5 * ra ** -0.5), r(H * V, rg, sc=rg ** -0.5)
    w["decay_up"], w["gate_up_lr"] = w["decay_up"].to(dt), w["gate_up_lr"].to(dt)
    return d, w, proj.to(dt)


def delta_both(ops, dt, H, G, D, V, K, segs, seed=0, decays=(-7.0, 3.0), groups=None, commit=True, fresh=False):
    """segs: (slot, rows). Runs the kernels and the plain op from one random state; returns both (rows, states, tails)."""
    n = sum(m for _, m in segs)
    d, w, proj = delta_layer(dt, H, G, D, V, K, n, seed, decays)
    r = gen(seed + 9)
    rec, tail = r(4, H, D, V, sc=0.0 if fresh else 0.5), r(4, K - 1, d.channels, sc=0.0 if fresh else 1.0, dt=dt)
    slots, rows = i32([s for s, _ in segs]), i32([m for _, m in segs])
    row0 = i32([sum(m for _, m in segs[:j]) for j in range(len(segs))])
    groups = groups or [SegGroup(0, len(segs), 0, n, max(m for _, m in segs))]
    rec1, tail1, rec2, tail2 = rec.clone(), tail.clone(), rec.clone(), tail.clone()
    got = ops.cdelta(proj, d, w, rec1, tail1, groups, slots, row0, rows, 1e-5, commit)
    f = {k: v.float() for k, v in w.items()}
    want = TorchOps(DEV, F32).cdelta(proj, d, f, rec2, tail2, groups, slots, row0, rows, 1e-5, commit)
    assert ops.status() == 0 and float(got[:, H * V:].float().abs().sum()) == 0
    return (got.float(), rec1, tail1), (want, rec2, tail2), (rec, tail)


def close(got, want, dt):
    # bf16: the convolved rows are rounded to bf16, the state stays exact to that
    tol = 3e-5 if dt == F32 else 2e-2
    e = lambda a, b: float((a.double() - b.double()).pow(2).mean().sqrt() / (b.double().pow(2).mean().sqrt() + 1e-30))
    assert e(got[0], want[0]) < tol and e(got[1], want[1]) < tol, (e(got[0], want[0]), e(got[1], want[1]))
    assert torch.equal(got[2], want[2])


SIZES = [(2, 2, 64, 64, 4), (3, 1, 24, 40, 3), (4, 2, 128, 128, 2), (6, 3, 72, 20, 5), (2, 2, 128, 64, 1), (2, 1, 48, 128, 8), (8, 8, 128, 128, 4)]
WIDE = [(2, 2, 160, 136, 4), (2, 1, 32, 300, 3), (1, 1, 512, 24, 2)]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,D,V,K", SIZES + WIDE)
def test_delta_rule_few_rows(cops, dt, H, G, D, V, K):
    for segs in ([(1, 1)], [(2, 2), (0, 1)], [(3, 5), (0, 1), (1, 9), (2, 32)]):
        got, want, _ = delta_both(cops[dt], dt, H, G, D, V, K, segs, seed=D + len(segs))
        close(got, want, dt)
        got, want, (rec, tail) = delta_both(cops[dt], dt, H, G, D, V, K, segs, seed=D, commit=False)
        close((got[0], rec, tail), (want[0], rec, tail), dt)
        assert torch.equal(got[1], rec) and torch.equal(got[2], tail)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,D,V,K", SIZES + WIDE)
def test_delta_rule_prompts(cops, dt, H, G, D, V, K):
    for segs in ([(1, 33)], [(2, 63)], [(0, 64)], [(3, 65)], [(1, 200)], [(3, 34), (0, 129), (2, 128)]):
        n = sum(m for _, m in segs)
        got, want, _ = delta_both(cops[dt], dt, H, G, D, V, K, segs, seed=n, groups=[SegGroup(0, len(segs), 0, n, max(m for _, m in segs), True)])
        close(got, want, dt)
    # prompt segments between decoded rows
    groups = [SegGroup(0, 1, 0, 1, 1), SegGroup(1, 2, 1, 101, 100, True), SegGroup(2, 4, 101, 104, 2)]
    got, want, _ = delta_both(cops[dt], dt, H, G, D, V, K, [(1, 1), (0, 100), (3, 2), (2, 1)], seed=5, groups=groups)
    close(got, want, dt)


@pytest.mark.parametrize("decays", [(-12.0, -9.0), (2.0, 6.0), (-40.0, 6.0)], ids=["slow", "total", "both"])
@pytest.mark.parametrize("H,G,D,V,K", [(8, 8, 128, 128, 4), (4, 2, 40, 24, 2)])
def test_decays_from_none_to_total(cops, decays, H, G, D, V, K):
    """exp(A_log) reaches 54, so decays run from 1 - 1e-5 down to e^-300 per token, side by side in one head."""
    for segs, groups in (([(1, 190)], [SegGroup(0, 1, 0, 190, 190, True)]), ([(1, 31)], None)):
        got, want, _ = delta_both(cops[F32], F32, H, G, D, V, K, segs, seed=7, decays=decays, groups=groups)
        close(got, want, F32)
        assert bool(torch.isfinite(got[0]).all())


def test_wide_batches_of_prompts_take_wider_slices(cops):
    """Enough heads and segments for 32-column slices of the state."""
    got, want, _ = delta_both(cops[BF], BF, 30, 15, 64, 96, 4, [(0, 70), (1, 64), (2, 40)], seed=3, groups=[SegGroup(0, 3, 0, 174, 70, True)])
    close(got, want, BF)
    got, want, _ = delta_both(cops[F32], F32, 32, 32, 128, 128, 4, [(0, 70), (1, 64)], seed=4, groups=[SegGroup(0, 2, 0, 134, 70, True)])
    close(got, want, F32)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("T", [1, 5, 8, 33, 64])
def test_low_rank_products(cops, dt, T):
    ops, r = cops[dt], gen(T)
    for na, ra, ng, rg in ((40, 64, 24, 64), (256, 128, 384, 192), (31, 64, 2, 128)):
        proj, wa, wg = r(T, ra + rg + 24, dt=dt), r(na, ra, dt=dt), r(ng, rg, dt=dt)
        out = torch.empty(T, na + ng, device=DEV)
        ops.C.cd_lowrank(out, proj, wa, wg)
        want = torch.cat([proj[:, :ra].double() @ wa.double().t(), proj[:, ra:ra + rg].double() @ wg.double().t()], 1)
        assert float((out.double() - want).abs().max()) < 1e-4


# ---- models --------------------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("dofunex")
    out = {}
    for j, (name, cfg) in enumerate(CASES.items()):
        for compute in ("fp32", "bf16"):
            c = copy.deepcopy(cfg)
            for l in c["layers"]:                                    # sharper attention than bf16 activations can follow for fp32
                if l["type"] == "attention" and compute == "bf16":
                    l["mixer"]["scale"] /= 2
            w = weights(c, seed=j)
            ids = tokens(c, 420, 11)
            out[name, compute] = (c, w, write(c, w, root / (name + compute)), ids, plain.forward(c, w, ids)[0])
    return out


@pytest.mark.parametrize("compute", ["fp32", "bf16"])
@pytest.mark.parametrize("name", list(CASES))
@pytest.mark.parametrize("cuts", [[1000], [301, 1], [2], [63, 2, 1, 64, 33, 3, 65, 100, 2, 32]], ids=["whole", "decode", "pairs", "mixed"])
def test_sequence_in_portions(ext, models, compute, name, cuts):
    cfg, w, d, ids, want = models[name, compute]
    eng = engine(d, DEV, compute)
    err = error(run_cuts(eng, ids, cuts), want)
    eng.check()
    assert err < LIM[compute], err


@pytest.mark.parametrize("compute", ["fp32", "bf16"])
def test_portions_and_batches_agree_beyond_rounding_only(ext, models, compute):
    """Requests together (prompt portions beside decoded tokens, long segments beside short ones, a tight pool, slots and pages
    that go round) against the plain rows of each."""
    for name in CASES:
        cfg, w, d, ids, want = models[name, compute]
        eng = engine(d, DEV, compute, max_ctx=448, pool=1024)
        seqs = {"a": (ids, want)}
        for k, n in (("b", 90), ("c", 3), ("d", 200), ("e", 65), ("f", 1)):
            s = tokens(cfg, n, 250 + n)
            seqs[k] = (s, plain.forward(cfg, w, s)[0])
        slot, at, got, free = {}, {k: 0 for k in seqs}, {k: [] for k in seqs}, [0, 1, 2, 3]
        for st in (dict(a=100, b=2), dict(b=40, a=1, c=3), dict(a=50, d=1), dict(b=48, d=100, a=1), dict(a=200, d=2), dict(d=97, a=2, f=1),
                   dict(e=64, a=33), dict(a=33, e=1)):
            segs = []
            for k, n in st.items():
                if k not in slot:
                    slot[k] = free.pop(0)
                segs.append((k, Segment(slot[k], at[k], seqs[k][0][at[k]:at[k] + n], "all")))
            lg, _, _ = eng.forward([s for _, s in segs], greedy=False)
            lg, r = lg.float().cpu().clone(), 0
            for k, s in segs:
                got[k].append(lg[r:r + len(s.tokens)])
                r += len(s.tokens)
                at[k] += len(s.tokens)
                if at[k] == len(seqs[k][0]):
                    eng.reset_slot(slot[k])
                    free.append(slot.pop(k))
        eng.check()
        assert eng.ex.pool.n_free == eng.ex.pool.n_blocks
        for k in seqs:
            e = error(torch.cat(got[k]), seqs[k][1])
            assert e < LIM[compute], (name, k, e)


@pytest.mark.parametrize("compute", ["fp32", "bf16"])
def test_rejected_rows_leave_no_trace(ext, models, compute):
    """Verify rows that are not kept, in a captured step and outside one: caches, states and convolution inputs follow the last kept row."""
    for name in ("grid", "ragged", "broad"):
        cfg, w, d, ids, want = models[name, compute]
        for graphs in (True, False):
            eng = engine(d, DEV, compute, use_graphs=graphs)
            eng.forward([Segment(0, 0, ids[:62], "none")])
            pos = 62
            for keep in (2, 1, 5):
                wrong = [(t + 1) % cfg["vocab"] for t in ids[pos + keep:pos + 7]]
                lg, _, _ = eng.forward([Segment(0, pos, ids[pos:pos + keep] + wrong, "all")], commit=False, greedy=False)
                assert error(lg[:keep].cpu(), want[pos:pos + keep]) < LIM[compute]
                eng.commit_verified([keep])
                pos += keep
            lg, _, _ = eng.forward([Segment(0, pos, ids[pos:140], "all")], greedy=False)
            assert error(lg.cpu(), want[pos:140]) < LIM[compute]


def test_residual_rows_after_the_last_layer(ext, models):
    for compute, tol in (("fp32", 2e-4), ("bf16", 5e-2)):
        cfg, w, d, ids, _ = models["ragged", compute]
        _, after = plain.forward(cfg, w, ids[:50])
        eng = engine(d, DEV, compute)
        eng.cfg.tap_layers[:] = [0, 3]
        eng.forward([Segment(0, 0, ids[:50], "none")])
        for got, want in zip(eng.taps, (after[0], after[-1])):
            assert float((got.cpu().double() - want).pow(2).mean().sqrt()) < tol * float(want.pow(2).mean().sqrt())


def test_greedy_generation_and_scheduler(ext, models):
    for name in ("grid", "ragged"):
        cfg, w, d, _, _ = models[name, "fp32"]
        prompts = [tokens(cfg, n, 30 + n) for n in (5, 70, 33, 1)]
        prompts += [prompts[1] + tokens(cfg, 9, 77), (tokens(cfg, 6, 78) * 6)[:34]]
        want = [plain.greedy(cfg, w, p, 8) for p in prompts]
        assert engine(d, DEV, "fp32", slots=1, max_ctx=128).generate(prompts[1], 8) == want[1]
        for spec, pool in ((0, 0), (0, 320), (4, 0)):
            eng = engine(d, DEV, "fp32", slots=3, max_ctx=192, pool=pool, prefill_chunk=32)
            sched = Scheduler(eng, SchedOptions(spec=spec, arrival_ms=0, share_min=32))
            assert generate(sched, prompts, Sampling(max_tokens=8), snapshots=[[64] if len(p) > 64 else [] for p in prompts]) == want
            assert generate(sched, [prompts[4]], Sampling(max_tokens=8), snapshots=[[64]])[0] == want[4]
            eng.check()
        # bf16: every generated token is the plain model's choice, or one that rounding cannot tell from it
        eng = engine(d, DEV, "bf16", slots=3, max_ctx=192)
        for p, out in zip(prompts, generate(Scheduler(eng, SchedOptions(arrival_ms=0)), prompts, Sampling(max_tokens=8))):
            lg = plain.forward(cfg, w, p + out[:-1])[0][len(p) - 1:]
            gap = lg.amax(-1) - lg.gather(1, torch.tensor(out)[:, None])[:, 0]
            assert float(gap.max()) < 4 * LIM["bf16"] * float(lg.std())


def test_long_decode_and_bigger_sizes(ext, tmp_path):
    """A model at the head sizes of real ones: a prompt over several chunks, then decoding over page borders, one step at a time."""
    cfg = config(512, 300, [delta(4, 4, 128, 128, 4, 512), attn(8, 2, 128, 512, gain=1.5), delta(8, 4, 128, 128, 4, 512)], (0, 2, 2), mult=0.7)
    w = weights(cfg, seed=2, ranks=(64, 128))
    ids = tokens(cfg, 700, 4)
    want = plain.forward(cfg, w, ids)[0]
    d = write(cfg, w, tmp_path / "m")
    for compute in ("fp32", "bf16"):
        eng = engine(d, DEV, compute, max_ctx=768)
        assert error(run_cuts(eng, ids, [500, 1]), want) < LIM[compute]
        eng.check()


@pytest.mark.parametrize("fmt", ["nvfp4-a16", "nvfp4", "fp8-block"])
def test_packed_weights(ext, tmp_path, fmt):
    """Quantised projections against the plain model with the same dequantised weights."""
    cfg = config(256, 128, [attn(4, 2, 64, 512, gain=1.0), delta(4, 2, 64, 64, 4, 256)])
    w = weights(cfg, ranks=(64, 64))
    eng = engine(write(cfg, w, tmp_path / "m"), DEV, "bf16", weight_dtype=fmt)
    deq = lambda n: (lambda t: t.dense.float().cpu() if hasattr(t, "dense") else t.float().cpu())(eng.ex.w[n])
    w = dict(w, head=deq("lm_head"))
    for i in range(2):
        gu, ip = deq(f"l{i}.gate_up"), deq(f"l{i}.in_proj")
        F = cfg["layers"][i]["mlp"]["ff"]
        w.update({f"l{i}.mix.o": deq(f"l{i}.out_proj"), f"l{i}.mlp.gate": gu[:F], f"l{i}.mlp.up": gu[F:], f"l{i}.mlp.down": deq(f"l{i}.down")})
        names = (("q", 256), ("k", 128)) if i == 0 else (("a1", 64), ("g1", 64), ("q", 128), ("k", 128), ("v", 256), ("b", 4))
        o = 0
        for n, rows in names:
            w[f"l{i}.mix.{n}"] = ip[o:o + rows]
            o += rows
    ids = tokens(cfg, 90, 1)
    want = plain.forward(cfg, w, ids)[0]
    for cuts in ([90], [70, 1]):
        err = error(run_cuts(eng, ids, cuts), want)
        assert err < 0.1, (cuts, err)
    eng.check()
