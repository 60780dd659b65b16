"""The kernels and the engine of the Rakizen design on the GPU, in bf16 and in fp32, against plain statements of the same arithmetic: every
kernel alone (sizes on and off its tiles, keys at page borders and just inside and outside windows and chunks), then whole models in prompts,
portions, decoding, mixed batches and through the scheduler."""
import copy

import pytest
import torch

import plain_rakizen as plain
from rakizen_cases import CASES, chunks, config, dense, engine, error, errors, moe, run_cuts, tokens, weights, window, write
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.models.weights import GqaDims
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
head = lambda d: next((h for h in (64, 128, 256) if d <= h), up(d, 64))


# ---- rows ---------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("width", [64, 320, 4096, 13312])
def test_residual_add_and_layer_norm(cops, dt, width):
    ops, r = cops[dt], gen(width)
    tol = 1e-5 if dt == F32 else 3e-2
    for true in (width, width - 5):
        x, w, b = r(9, width) + 2, r(width), r(width)
        wts = r(9, 3).abs()
        yp = r(27, width)
        for t in (x, w, b, yp):
            t[..., true:] = 0
        xd = lambda t: t[..., :true].double()
        for y in (r(9, width, sc=4.0), r(9, width + 16)[:, :width]) + ((r(9, width, dt=BF),) if dt == BF else ()):
            y[:, true:] = 0
            for pairs in (None, (yp, wts)):
                want = xd(x) + xd(y) + (0 if pairs is None else (xd(yp).view(9, 3, true) * wts.double()[:, :, None]).sum(1))
                x1 = x.clone()
                h = ops.add_layer_norm(x1, y, true, 1e-3, w, b, pairs)
                assert h.dtype == dt and torch.allclose(xd(x1), want, atol=3e-5, rtol=1e-5) and float(x1[:, true:].abs().sum()) == 0
                assert torch.allclose(xd(h), plain.layer_norm(want, xd(w), xd(b), 1e-3), atol=tol, rtol=tol) and float(h[:, true:].float().abs().sum()) == 0
                x2 = x.clone()
                assert ops.add_layer_norm(x2, y, true, 1e-3, pairs=pairs) is None and torch.equal(x1, x2)
        idx = i32([8, 0, 3])
        for i, rows in ((None, x), (idx, x[idx.long()])):
            got = ops.norm_rows(x, i, w, true, 1e-3, bias=b)
            assert torch.allclose(xd(got), plain.layer_norm(xd(rows), xd(w), xd(b), 1e-3), atol=tol, rtol=tol) and float(got[:, true:].float().abs().sum()) == 0
    assert ops.status() == 0


def test_layer_norm_keeps_small_deviations_on_a_large_mean(cops):
    ops, r = cops[F32], gen(3)
    x = 1000.0 + r(4, 256)
    got = ops.norm_rows(x, None, torch.ones(256, device=DEV), 256, 1e-5, bias=torch.zeros(256, device=DEV))
    d = x.double() - x.double().mean(-1, keepdim=True)
    assert torch.allclose(got.double(), d / (d.pow(2).mean(-1, keepdim=True) + 1e-5).sqrt(), atol=2e-4)


# ---- attention ------------------------------------------------------------------------------------------------------------

def dims(H, G, D, V, M=1, scale=0.3, rot=0, hp=0, **kw):
    return GqaDims(H, G, D, hp or head(max(M * D, V)), scale, rot, (H + G) * M * D, False, V, M, kw.pop("row_norm", M == 1), **kw)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,D,V,M,rot", [(4, 2, 64, 64, 1, 64), (5, 1, 40, 64, 1, 16), (3, 3, 128, 80, 1, 128), (9, 3, 100, 100, 1, 36), (2, 1, 256, 128, 1, 128),
                                           (2, 2, 272, 40, 1, 272), (1, 1, 18, 33, 1, 0), (40, 8, 128, 128, 1, 128), (4, 2, 32, 64, 2, 0), (3, 1, 13, 27, 2, 0),
                                           (16, 4, 64, 128, 2, 0), (2, 2, 140, 264, 2, 0), (3, 3, 24, 16, 2, 12)])
def test_queries_keys_and_values(cops, dt, H, G, D, V, M, rot):
    ops, tops, r, kvb = cops[dt], TorchOps(DEV, F32), gen(D), 64
    for normed in (True, False) if M == 1 else (False,):
        d = dims(H, G, D, V, M, rot=rot, row_norm=normed)
        if d.plain:
            continue
        cols = d.v_off + G * V + 11
        proj = r(8, up(cols, 8) + 8, sc=2.0)[:, :cols]
        norms = (r(H * D), r(G * D)) if normed else None
        freq = torch.tensor([3e4 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=DEV)
        bt = torch.full((2, 1 << 14), -1, dtype=torch.int32, device=DEV)
        pos = i32([62, 63, 64, 0, 1, 127, 128, 1000003])                              # page borders, a position past what fp32 angles hold
        slot = i32([0, 0, 0, 1, 1, 1, 1, 0])
        bt[0, :2], bt[1, :3], bt[0, 1000003 // kvb] = i32([3, 1]), i32([0, 2, 4]), 5
        caches = [torch.full((6, kvb, G, d.hp), 5.0, dtype=t, device=DEV) for t in (dt, dt, F32, F32)]
        q = ops.gqa_prep(proj, d, None, freq, slot, pos, bt, caches[0], caches[1], kvb, 1e-4, norms=norms)
        want = tops.gqa_prep(proj, d, None, freq, slot, pos, bt, caches[2], caches[3], kvb, 1e-4, norms=norms)
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


def attend_case(ops, dt, d, segs, nsplit, seed, prompt=False, plant=None, lead=0, gated=False, lam=0.6):
    """segs: (rows, context length after the segment), the first `lead` of them outside the group. Returns (kernel's rows, plain rows)."""
    kvb, r = 64, gen(seed + 1)
    kc, vc, bt = paged(d.kv_heads, d.hp, [n for _, n in segs], dt, seed)
    kc[..., d.maps * d.dim:], vc[..., d.vw:] = 0, 0
    slot = i32([s for s, (m, _) in enumerate(segs) for _ in range(m)])
    kvlen = i32([n - m + j + 1 for m, n in segs for j in range(m)])
    row0 = [sum(m for m, _ in segs[:s]) for s in range(len(segs))]
    T = slot.numel()
    q = r(T, d.queries, d.hp, dt=dt)
    if d.maps == 2:
        q[:, 0::2, d.dim:], q[:, 1::2, :d.dim] = 0, 0
    q[..., d.maps * d.dim:] = 0
    if plant is not None:
        plant(q, kc, vc, bt, kvb)
    tables = [i32(list(range(len(segs)))), i32(row0), i32([m for m, _ in segs]), i32([n - m for m, n in segs])]
    a = sum(m for m, _ in segs[:lead])
    g = SegGroup(lead, len(segs), a, T, max(m for m, _ in segs[lead:]), prompt)
    mix = dict(lam=torch.tensor([lam], device=DEV) if d.maps == 2 else None, eps=1e-4,
               gate=r(T, d.heads * d.vw + 8, sc=2.0)[:, 3:3 + d.heads * d.vw] if gated else None) if gated or d.maps == 2 else {}
    both = torch.full((T, d.heads * d.hp + 64), 7.0, dtype=dt, device=DEV)             # rows of the output lie apart
    out = both[:, :d.heads * d.hp].unflatten(1, (d.heads, d.hp))
    ops.gqa_attention(q, d, kc, vc, None, g, slot, kvlen, tuple(t[lead:] for t in tables), bt, kvb, nsplit, out, **mix)
    want = TorchOps(DEV, F32).gqa_attention(q, d, kc, vc, None, g, slot, kvlen, None, bt, kvb, 1, torch.full(out.shape, 7.0, device=DEV), **mix)
    assert ops.status() == 0 and bool((out[:a] == 7.0).all()) and bool((both[:, d.heads * d.hp:] == 7.0).all())
    return out.float(), want


TOL = {F32: dict(atol=3e-5, rtol=1e-4), BF: dict(atol=2e-2, rtol=1e-2)}
MASKS = [dict(window=1), dict(window=40), dict(window=64), dict(window=65), dict(window=500), dict(chunk=1), dict(chunk=33), dict(chunk=64), dict(chunk=130), {}]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("mask", MASKS, ids=str)
@pytest.mark.parametrize("H,G,D,V,M,gated", [(8, 2, 64, 64, 1, False), (6, 2, 100, 128, 1, False), (3, 1, 320, 40, 1, False), (4, 2, 32, 64, 2, True), (3, 3, 64, 50, 2, False),
                                             (2, 1, 128, 256, 2, True), (1, 1, 140, 264, 2, True), (5, 1, 64, 64, 1, True)])
def test_few_rows_attention(cops, dt, mask, H, G, D, V, M, gated):
    d = dims(H, G, D, V, M, scale=2.0 * D ** -0.5, softcap=6.0, diff=0.3, **mask)
    for nsplit in (1, 3, 64):
        got, want = attend_case(cops[dt], dt, d, [(1, 1), (1, 63), (1, 64), (1, 65), (1, 400)], nsplit, D + H, gated=gated)
        assert torch.allclose(got, want, **TOL[dt]), (nsplit, (got - want).abs().max())
    got, want = attend_case(cops[dt], dt, d, [(5, 9), (7, 130), (2, 2), (1, 321), (30, 96), (3, 66)], 8, D + H, lead=2, gated=gated)
    assert torch.allclose(got, want, **TOL[dt])


@pytest.mark.parametrize("mask", MASKS, ids=str)
@pytest.mark.parametrize("H,G,D,V,M,gated", [(4, 2, 64, 64, 1, False), (3, 1, 128, 96, 1, False), (2, 2, 200, 256, 1, False), (4, 2, 32, 64, 2, True), (2, 1, 64, 128, 2, True),
                                             (2, 2, 128, 250, 2, False), (3, 1, 64, 40, 1, True)])
def test_prompt_attention(cops, mask, H, G, D, V, M, gated):
    d = dims(H, G, D, V, M, scale=2.0 * D ** -0.5, softcap=6.0, diff=0.3, **mask)
    for segs, lead in (([(200, 200)], 0), ([(1, 90), (40, 40), (130, 400), (64, 128)], 1), ([(33, 97)], 0), ([(300, 1000)], 0)):
        got, want = attend_case(cops[BF], BF, d, segs, 1, D + H, True, lead=lead, gated=gated)
        assert torch.allclose(got, want, **TOL[BF]), (segs, (got - want).abs().max())


@pytest.mark.parametrize("dt,prompt", [(BF, False), (BF, True), (F32, False)])
@pytest.mark.parametrize("at", [0, 1, 31, 32, 63, 64, 127, 128, 198, 299])
def test_one_key_stands_out(cops, dt, prompt, at):
    """One key that all queries point at among hundreds: its value comes back from its own row on while it is inside the window or the chunk."""
    def plant(q, kc, vc, bt, kvb):
        q.fill_(1.0)
        vc.mul_(0.1)
        page = int(bt[0, at // kvb])
        kc[page, at % kvb], vc[page, at % kvb] = 8.0, 2.0
    for kind, size in (("window", 1), ("window", 64), ("window", 101), ("chunk", 64), ("chunk", 77)):
        last = at + size - 1 if kind == "window" else at // size * size + size - 1
        d = dims(4, 2, 64, 64, scale=0.3, softcap=60.0, **{kind: size})
        got, want = attend_case(cops[dt], dt, d, [(300, 300)], 4, at, prompt, plant)
        hit = (got - 2.0).abs().amax((1, 2)) < 2e-2
        assert hit.tolist() == [at <= t <= last for t in range(300)], (kind, size)
        assert torch.allclose(got, want, **TOL[dt])


@pytest.mark.parametrize("dt,prompt", [(BF, False), (BF, True), (F32, False)])
@pytest.mark.parametrize("cap", [0.5, 20.0, 50.0, 1000.0])
def test_softcap_from_tiny_to_saturated_scores(cops, dt, prompt, cap):
    """Two keys per row whose scores run from far below to far above the cap: the weight of each is sigmoid(cap tanh(s / cap) - s')."""
    scores = torch.cat([torch.linspace(-3 * cap, 3 * cap, 60), cap * torch.logspace(-4, 0.5, 60)])
    n = scores.numel()

    def plant(q, kc, vc, bt, kvb):
        q.zero_(); kc.zero_(); vc.zero_()
        q[:, 0, 0] = scores.to(DEV).to(q.dtype)
        for t in range(n):
            kc[int(bt[0, t // kvb]), t % kvb, 0, 0] = 1.0 if t % 2 == 0 else 0.0
            vc[int(bt[0, t // kvb]), t % kvb, 0, 0] = 1.0 if t % 2 == 0 else 0.0
    d = dims(1, 1, 64, 64, scale=1.0, softcap=cap, window=2)
    got, _ = attend_case(cops[dt], dt, d, [(n, n)], 1, 3, prompt, plant)
    s = scores.to(dt).double()
    want = torch.sigmoid(cap * torch.tanh(s / cap))[1:]
    tol = 2e-6 * max(1.0, cap / 20) if dt == F32 else 4e-3
    assert float((got[1:, 0, 0].cpu().double() - want).abs().max()) < tol
    if dt == BF and cap <= 50:                                        # the scores themselves are good to 32 bits: odds of rare keys
        low = (want < 1e-3) & (want > 1e-30)
        assert float((got[1:, 0, 0].cpu().double()[low] / want[low] - 1).abs().max()) < 1e-2 if bool(low.any()) else True


def test_difference_keeps_32_bit_rows(cops):
    """Two maps that nearly cancel: rows rounded to 16 bits before the difference would leave noise of its own size."""
    n = 40

    def plant(q, kc, vc, bt, kvb):
        q.zero_(); kc.zero_()
        q[:, 0, 0], q[:, 1, 64] = 0.01, -0.01
        kc[..., 0] = gen(1)(*kc.shape[:3], dt=BF)
        kc[..., 64] = kc[..., 0]
        vc.copy_(1.0 + vc.float() * 0.01)
    for prompt in (False, True):
        d = dims(1, 1, 64, 128, 2, scale=1.0, softcap=30.0, chunk=1000, diff=0.3)
        got, want = attend_case(cops[BF], BF, d, [(n, n)], 1, 5, prompt, plant, lam=0.999)
        assert torch.allclose(got[4:], want[4:], atol=3e-2, rtol=3e-2), (got - want)[4:].abs().max()


# ---- experts --------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("experts,top,groups,keep", [(8, 2, 4, 2), (12, 3, 3, 2), (10, 4, 5, 3), (6, 6, 1, 1), (48, 6, 16, 5), (5, 2, 5, 3), (7, 1, 1, 1), (96, 8, 6, 2),
                                                     (64, 4, 8, 8), (256, 8, 8, 4), (40, 9, 2, 1), (320, 7, 20, 3)])
def test_routing(cops, experts, top, groups, keep):
    z = gen(experts)(50, experts + 5)[:, 2:2 + experts]
    ids, wts = cops[BF].moe_route(z, None, 1, top, groups, keep, 1.7)
    want_ids, want = TorchOps("cpu").moe_route(z.cpu(), None, 1, top, groups, keep, 1.7)
    assert torch.equal(ids.cpu(), want_ids) and torch.allclose(wts.cpu(), want, rtol=1e-5)
    for t in range(5):
        assert ids[t].tolist() == [e for e, _ in plain.route(z[t].double().cpu(), top, groups, keep, 1.7)]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("T,W,F,E,K", [(1, 128, 64, 6, 2), (9, 320, 192, 5, 3), (64, 64, 64, 16, 6), (3, 1024, 448, 4, 4)])
def test_expert_rows(cops, dt, T, W, F, E, K):
    ops, r = cops[dt], gen(W + T)
    h, gu, dn = r(T, W, dt=dt), r(E, 2 * F, W, sc=W ** -0.5, dt=dt), r(E, W, F, sc=F ** -0.5, dt=dt)
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:K] for t in range(T)]).to(torch.int32).to(DEV)
    got = ops.expert_rows(h, ids, gu, dn).double().view(T, K, W)
    for t in range(T):
        for k in range(K):
            e = int(ids[t, k])
            want = plain.gated_mlp(h[t].double(), gu[e, :F].double(), gu[e, F:].double(), dn[e].double())
            assert torch.allclose(got[t, k], want, atol=2e-5 if dt == F32 else 2e-2, rtol=1e-2)


@pytest.mark.parametrize("T,W,F,E,K", [(70, 128, 64, 6, 2), (300, 320, 192, 5, 3), (129, 64, 64, 3, 1), (1000, 192, 128, 32, 8)])
def test_experts_of_prompt_rows_are_added_in_32_bits(cops, T, W, F, E, K):
    from ferrite_b200.parallel.ep import ExpertParallel
    ops, r = cops[BF], gen(W + T)
    h, gu, dn, acc = r(T, W, dt=BF), r(E, 2 * F, W, sc=W ** -0.5, dt=BF), r(E, W, F, sc=F ** -0.5, dt=BF), r(T, W, sc=100.0)
    ids, wts = ops.moe_route(r(T, E), None, 1, K, 1, 1, 1.3)
    ep = ExpertParallel(None, torch.device(DEV), E, W, cap_rows=max(256, T * K), status=ops.status_word)
    rows = ops.expert_rows(h, ids, gu, dn).double().view(T, K, W)
    want = acc.double() + (rows * wts.double()[:, :, None]).sum(1)
    for _ in range(2):                                                # the buffers are used again
        y = acc.clone()
        ep.moe(ops, h, ids, wts, gu, dn, acc=y)
        assert ops.status() == 0 and float((y.double() - want).abs().max()) < 4e-2
    with pytest.raises(AssertionError, match="pairs"):
        ep.moe(ops, r(ep.cap_rows, W, dt=BF), ids.repeat(ep.cap_rows // T + 1, 1)[:ep.cap_rows].repeat(1, 2), wts, gu, dn, acc=y)


# ---- models --------------------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("rakizen")
    out = {}
    for j, (name, cfg) in enumerate(CASES.items()):
        w, ids = weights(cfg, seed=j), tokens(cfg, 420, 11)
        out[name] = (cfg, w, write(cfg, w, root / name), ids, plain.forward(cfg, w, ids)[0])
    return out


def close(got, want, compute, routed):
    """Routed models in bf16: a router's close call may fall the other way at a few positions (and, through the cache, disturb their
    neighbours a little)."""
    e = errors(got, want)
    if compute == "fp32" or not routed:
        assert float(e.max()) < LIM[compute], float(e.max())
    else:
        assert float(e.median()) < LIM[compute] / 2 and float(e.quantile(0.8)) < LIM[compute], (float(e.median()), float(e.quantile(0.8)))


routed = lambda cfg: any(l["mlp"] and l["mlp"]["kind"] == "moe" for l in cfg["layers"])


@pytest.mark.parametrize("compute", ["fp32", "bf16"])
@pytest.mark.parametrize("name", list(CASES))
@pytest.mark.parametrize("cuts", [[1000], [301, 1], [2], [63, 2, 1, 64, 33, 3, 65, 100, 2, 32]], ids=["whole", "decode", "pairs", "mixed"])
def test_sequence_in_portions(ext, models, compute, name, cuts):
    cfg, w, d, ids, want = models[name]
    eng = engine(d, DEV, compute)
    close(run_cuts(eng, ids, cuts), want, compute, routed(cfg))
    eng.check()


@pytest.mark.parametrize("compute", ["fp32", "bf16"])
@pytest.mark.parametrize("name", list(CASES))
def test_unequal_requests_together(ext, models, compute, name):
    """Requests together (prompt portions beside decoded tokens, long segments beside short ones, a tight pool, slots and pages that go
    round) against the plain rows of each."""
    cfg, w, d, ids, want = models[name]
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
    close(torch.cat([torch.cat(got[k]) for k in seqs]), torch.cat([seqs[k][1] for k in seqs]), compute, routed(cfg))


def test_rejected_rows_leave_no_trace(ext, models):
    """Verify rows that are not kept, in a captured step and outside one."""
    for name in ("grid", "ragged", "broad"):
        cfg, w, d, ids, want = models[name]
        for graphs in (True, False):
            eng = engine(d, DEV, "fp32", use_graphs=graphs)
            eng.forward([Segment(0, 0, ids[:62], "none")])
            pos = 62
            for keep in (2, 1, 5):
                wrong = [(t + 1) % cfg["vocab"] for t in ids[pos + keep:pos + 7]]
                lg, _, _ = eng.forward([Segment(0, pos, ids[pos:pos + keep] + wrong, "all")], commit=False, greedy=False)
                assert error(lg[:keep].cpu(), want[pos:pos + keep]) < LIM["fp32"]
                eng.commit_verified([keep])
                pos += keep
            lg, _, _ = eng.forward([Segment(0, pos, ids[pos:140], "all")], greedy=False)
            assert error(lg.cpu(), want[pos:140]) < LIM["fp32"]


def test_residual_rows_after_the_layers(ext, models):
    for compute, tol in (("fp32", 2e-4), ("bf16", 5e-2)):
        cfg, w, d, ids, _ = models["broad"]
        _, after = plain.forward(cfg, w, ids[:50])
        eng = engine(d, DEV, compute)
        eng.cfg.tap_layers[:] = [0, 1]
        eng.forward([Segment(0, 0, ids[:50], "none")])
        for got, want in zip(eng.taps, after):
            assert float((got.cpu().double() - want).pow(2).mean().sqrt()) < tol * float(want.pow(2).mean().sqrt())


def test_greedy_generation_and_scheduler(ext, models):
    for name in ("grid", "edges"):
        cfg, w, d, _, _ = models[name]
        prompts = [tokens(cfg, n, 30 + n) for n in (5, 70, 33, 1)]
        prompts += [prompts[1] + tokens(cfg, 9, 77), (tokens(cfg, 6, 78) * 6)[:34]]
        want = [plain.greedy(cfg, w, p, 6) for p in prompts]
        assert engine(d, DEV, "fp32", slots=1, max_ctx=128).generate(prompts[1], 6) == want[1]
        for spec, pool in ((0, 0), (0, 320), (4, 0)):
            eng = engine(d, DEV, "fp32", slots=3, max_ctx=192, pool=pool, prefill_chunk=32)
            sched = Scheduler(eng, SchedOptions(spec=spec, arrival_ms=0, share_min=32))
            assert generate(sched, prompts, Sampling(max_tokens=6), snapshots=[[64] if len(p) > 64 else [] for p in prompts]) == want
            assert generate(sched, [prompts[4]], Sampling(max_tokens=6), snapshots=[[64]])[0] == want[4]
            eng.check()
        eng = engine(d, DEV, "bf16", slots=3, max_ctx=192)
        outs = generate(Scheduler(eng, SchedOptions(arrival_ms=0)), prompts, Sampling(max_tokens=6))
        assert all(len(o) == 6 for o in outs)
        eng.check()


def test_long_decode_and_bigger_sizes(ext, tmp_path):
    """A model at the head sizes of real ones: a prompt over several chunks, then decoding over page, window and chunk borders."""
    cfg = config(512, 300, [window(8, 2, 128, 128, 200, dense(512), gain=1.0), chunks(4, 2, 64, 128, 256, dense(512), gain=1.0),
                            window(8, 8, 64, 64, 333, dense(320), gain=1.0), chunks(2, 1, 128, 256, 400, None, gain=1.0)], (0, 2, 2))
    w = weights(cfg, seed=2)
    ids = tokens(cfg, 700, 4)
    want = plain.forward(cfg, w, ids)[0]
    d = write(cfg, w, tmp_path / "m")
    for compute in ("fp32", "bf16"):
        eng = engine(d, DEV, compute, max_ctx=768)
        assert error(run_cuts(eng, ids, [500, 1]), want) < LIM[compute]
        eng.check()


@pytest.mark.parametrize("fmt", ["nvfp4-a16", "nvfp4", "fp8-block"])
def test_packed_weights(ext, tmp_path, fmt):
    """Quantised projections against the plain model with the same dequantised weights; routed layers' products stay in 16 bits."""
    cfg = config(256, 128, [window(4, 2, 64, 64, 50, dense(256), gain=1.0), chunks(2, 1, 32, 64, 40, moe(4, 2, 2, 2, 64), gain=1.0)])
    w = weights(cfg)
    eng = engine(write(cfg, w, tmp_path / "m"), DEV, "bf16", weight_dtype=fmt)
    deq = lambda n: (lambda t: t.dense.float().cpu() if hasattr(t, "dense") else t.float().cpu())(eng.ex.w[n])
    gu, ip, op = deq("l0.gate_up"), deq("l0.in_proj"), deq("l0.out_proj")
    w = dict(w, head=deq("lm_head"))
    w.update({"l0.mlp.gate": gu[:256], "l0.mlp.up": gu[256:], "l0.mix.q": ip[:256], "l0.mix.k": ip[256:384], "l0.mix.v": ip[384:512], "l0.mix.o": op[:, :256],
              "l0.mlp.down": op[:, 256:], "l1.mix.o": deq("l1.out_proj")})
    assert isinstance(eng.ex.w["l1.in_proj"], torch.Tensor)
    ids = tokens(cfg, 90, 1)
    want = plain.forward(cfg, w, ids)[0]
    for cuts in ([90], [70, 1]):
        e = errors(run_cuts(eng, ids, cuts), want)
        assert float(e.quantile(0.8)) < 0.1, (cuts, float(e.quantile(0.8)))
    eng.check()
