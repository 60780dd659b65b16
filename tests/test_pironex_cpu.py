"""The Pironex design on the fp32 CPU engine against a plain statement of it (`plain_pironex.py`): configuration and checkpoint reading,
each mechanism, prompts, decoding, portions, batches, reused pages and slots, speculation, the scheduler."""
import copy
import io
import json
import math
import sys

import pytest
import torch

import plain_pironex as plain
from pironex_cases import CASES, config, engine, error, moe, pooled, run_cuts, tokens, weights, write
from ferrite_b200.config import EngineConfig, ModelConfig, pironex, pironex_moe, tiny_pironex
from ferrite_b200.engine.engine import Engine
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.formats.loader import load_model_weights
from ferrite_b200.models.ref import RefModel
from ferrite_b200.models.weights import GqaDims, LatentDims, SsmDims, gqa_dims, init_weights, latent_dims, pack_listed, weight_shapes
from ferrite_b200.ops.latent import SegGroup
from ferrite_b200.ops.torch_ops import TorchOps

LIM = 6e-5          # fp32 rounding through up to five layers


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
    root = tmp_path_factory.mktemp("pironex")
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
    assert [l.mixer for l in c.layers] == ["ssm", "gqa", "latent", "gqa", "ssm"] and c.canon == 3 and c.embed_scale == 3.0
    assert [(l.window, l.pool, l.kv_from, l.softcap) for l in c.layers] == [(0, 0, None, 0.0), (17, 5, None, 12.0), (33, 0, None, 0.0), (31, 7, 1, 0.0),
                                                                           (0, 0, None, 0.0)]
    assert [(l.ff, l.experts, l.top, l.limit, l.shared_ff, l.shared_limit) for l in c.layers] == [
        (30, 6, 3, 1.2, 0, 0.0), (22, 5, 2, 1.2, 50, 0.9), (0, 0, 0, 0.0, 0, 0.0), (26, 6, 1, 1.2, 18, 0.9), (0, 0, 0, 0.0, 0, 0.0)]
    assert [(l.dim, l.kv_heads, l.norm_groups, l.conv) for l in c.layers if l.mixer == "ssm"] == [(24, 3, 4, 3), (12, 2, 2, 2)]
    assert (c.layers[2].rot_dims, c.layers[2].kv_rank, c.layers[2].q_rank) == (12, 50, 0) and c.layers[1].rot_half and not c.layers[2].rot_half
    assert c.layer_norm and c.depth_average and c.out_norm and c.pre_norm and c.tie_embeddings and not c.parallel and c.n_attn == 2
    for change, what in (((lambda c: c.update(architecture="Pironax")), "architecture"),
                         ((lambda c: c["layers"][1].update(type="conv")), "type"),
                         ((lambda c: c["layers"][0]["mlp"].update(kind="dense")), "kind"),
                         ((lambda c: c["layers"][1]["mixer"].update(kv_heads=4)), "heads"),
                         ((lambda c: c["layers"][1]["mixer"]["mask"].update(size=0)), "mask"),
                         ((lambda c: c["layers"][1]["mixer"]["mask"].update(pool=-1)), "pool"),
                         ((lambda c: c["layers"][1]["mixer"].update(softcap=-1.0)), "softcap"),
                         ((lambda c: c["layers"][1]["mixer"]["rot"].update(dims=42)), "rotated"),
                         ((lambda c: c["layers"][2]["mixer"].update(rot_dim=14)), "rot_dim"),
                         ((lambda c: c["layers"][3]["mixer"].update(kv_from=2)), "kv_from"),
                         ((lambda c: c["layers"][3]["mixer"].update(kv_from=3)), "kv_from"),
                         ((lambda c: c["layers"][3]["mixer"].update(vdim=20)), "kv_from"),
                         ((lambda c: c["layers"][0]["mixer"].update(norm_groups=7)), "norm groups"),
                         ((lambda c: c["layers"][4]["mixer"].update(groups=3)), "groups"),
                         ((lambda c: c["layers"][0]["mlp"]["router"].update(top=7)), "experts per token")):
        bad = copy.deepcopy(CASES["ragged"])
        change(bad)
        with pytest.raises(ValueError, match=what):
            read(bad)


def test_checkpoint_shapes_are_checked(tmp_path):
    cfg = CASES["ragged"]
    w = weights(cfg)
    for change, what in (((lambda w: w.pop("l1.mlp.e4.up")), "l1.mlp.e4.up"), ((lambda w: w.pop("l3.mlp.shared.sg")), "l3.mlp.shared.sg"),
                         ((lambda w: w.update({"l1.canon2": w["l1.canon2"][:, :-1]})), "l1.canon2"),
                         ((lambda w: w.update({"l2.dwa": w["l2.dwa"][:-1]})), "l2.dwa"),
                         ((lambda w: w.update({"l0.mix.in": w["l0.mix.in"][:-6]})), "l0.mix.in"),
                         ((lambda w: w.update({"l1.mix.q.norm": w["l1.mix.q.norm"][:40]})), "l1.mix.q.norm")):
        bad = dict(w)
        change(bad)
        d = write(cfg, bad, tmp_path / what.replace(".", "_"))
        with pytest.raises((KeyError, ValueError), match=what):
            load_model_weights(d, ModelConfig.from_hf(d + "/config.json"))


def test_kernel_layout():
    cfg = tiny_pironex()
    w = init_weights(cfg, seed=3)
    pk, W = pack_listed(cfg, w), 192
    assert pk["lm_head"] is pk["embed"]
    for i, l in enumerate(cfg.layers):
        p, ip = f"l{i}.", pk[f"l{i}.in_proj"]
        assert ip.shape[0] % 8 == 0 and ip.shape[1] == W and float(ip[:, cfg.hidden:].abs().sum()) == 0
        assert torch.equal(pk[p + "mix_canon"][:, :cfg.hidden].t(), w[p + "mix_canon"]) and pk[p + "dwa"].numel() == i + 2
        if l.mixer == "gqa":
            d = gqa_dims(cfg, i)
            rows = [w[p + "q"]] if l.kv_from is not None else [w[p + n] for n in "qkv"]
            assert torch.equal(ip[:sum(r.shape[0] for r in rows), :cfg.hidden], torch.cat(rows)) and (d.source, d.pool) == ((-1, 5) if i == 1 else (1, 7))
        elif l.mixer == "latent":
            d = latent_dims(cfg, i)
            assert (d.lat, d.vlat, d.hp, d.vp) == ((128, 128, 64, 64) if i == 0 else (192, 192, 64, 64))
            # the rotated columns of a cache row reach the keys of every head as they are, and no value
            row = torch.zeros(d.lat)
            row[l.kv_rank:l.kv_rank + l.rot_dims] = torch.arange(1.0, l.rot_dims + 1)
            kv = pk[p + "kv_up"] @ row
            k, v = kv[:l.heads * d.hp].view(l.heads, d.hp), kv[l.heads * d.hp:]
            assert torch.equal(k[:, l.dim:l.dim + l.rot_dims], row[l.kv_rank:l.kv_rank + l.rot_dims].expand(l.heads, -1))
            assert float(k[:, :l.dim].abs().sum()) == 0 and float(v.abs().sum()) == 0
            assert torch.equal(pk[p + "k_abs"], pk[p + "kv_up"][:l.heads * d.hp].view(l.heads, d.hp, d.lat).transpose(1, 2))
        else:
            assert torch.equal(pk[p + "conv"].t(), w[p + "xbc_conv"]) and torch.allclose(pk[p + "A"], -torch.exp(w[p + "A_log"]))
        if l.experts:
            gu = pk[p + "experts_gate_up"].view(l.experts, 2, 64, W)
            assert torch.equal(gu[:, :, :l.ff, :cfg.hidden].reshape(l.experts, 2 * l.ff, -1), w[p + "experts_gate_up"]) and float(gu[:, :, l.ff:].abs().sum()) == 0
            assert torch.equal(pk[p + "router"][:l.experts + 1, :cfg.hidden], torch.cat([w[p + "router"], w[p + "shared_gate"]]))
            assert pk[p + "shared_down"].shape == (1, W, 64)
    assert cfg.param_count() == sum(v.numel() for v in w.values() if v.dim() > 1) and set(weight_shapes(cfg)) == set(w)
    assert 9e9 < pironex_moe().param_count() < 12e9
    with pytest.raises(ValueError, match="one rank"):
        cfg.shard(2)


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def test_convolution_by_hand():
    x = torch.tensor([[1.0], [2.0], [4.0], [8.0]])
    assert plain.causal_conv(x, torch.tensor([[100.0, 10.0, 1.0]])).flatten().tolist() == [1.0, 12.0, 124.0, 248.0]
    ops, w = TorchOps("cpu"), torch.tensor([[100.0], [10.0], [1.0]])
    tails = torch.tensor([[[0.0], [0.0]], [[3.0], [5.0]]])
    slot, pos = i32([1, 1, 0, 0]), i32([7, 8, 0, 1])                        # two segments in one step: the tail is each slot's own
    got = ops.conv_rows(x, w, tails, slot, pos)
    assert got.flatten().tolist() == [300 + 50 + 1, 500 + 10 + 2, 4.0, 48.0]
    assert torch.equal(ops.conv_rows(x, w, tails, slot, pos, residual=True), got + x)
    b = torch.tensor([0.5])
    assert torch.allclose(ops.conv_rows(0.001 * x, w, 0.001 * tails, slot, pos, bias=b, silu=True), plain.silu(0.001 * got + b))
    for keep, want in ((0, [3.0, 5.0]), (1, [5.0, 1.0]), (2, [1.0, 2.0])):
        t = tails.clone()
        ops.conv_tail(t, x, i32([1, 0]), i32([0, 2]), i32([keep, 1]))
        assert t[1].flatten().tolist() == want and t[0].flatten().tolist() == [0.0, 4.0]


def test_seam_between_sublayers():
    """Residual sum of the normed output, the average over depth, the next norm and its convolution."""
    ops, T, W, width, eps = TorchOps("cpu"), 5, 16, 13, 1e-3
    x_in, y, w, nw, dwa = rnd(T, W), rnd(T, W, seed=1) + 2, rnd(W, seed=2), rnd(W, seed=3), torch.tensor([0.2, -0.7, 1.1])
    cw, tails, yp, wts = rnd(4, W, seed=4), rnd(3, 3, W, seed=5), rnd(2 * T, W, seed=6), rnd(T, 2, seed=7).abs()
    for t in (x_in, y, w, nw, cw, tails, yp):
        t[..., width:] = 0
    slot, pos, cut = i32([0, 2, 2, 2, 1]), i32([3, 9, 10, 11, 0]), slice(0, width)
    for pairs, add in ((None, 0), ((yp, wts), (yp.view(T, 2, W) * wts[:, :, None]).sum(1))):
        xs, x = torch.zeros(3, T, W), torch.empty(T, W)
        xs[:2] = rnd(2, T, W, seed=8)
        xs[..., width:] = 0
        got, h = ops.add_conv_normed(x_in, x, y, w, width, eps, nw, pairs=pairs, average=(xs, 2, dwa), conv=(cw, tails), row_slot=slot, row_pos=pos)
        res = x_in[:, cut] + plain.layer_norm((y + add)[:, cut], w[cut], eps)
        assert torch.allclose(xs[2, :, cut], res, atol=1e-5)
        mean = plain.depth_average([xs[0, :, cut], xs[1, :, cut], res], dwa)
        assert torch.allclose(x[:, cut], mean, atol=1e-5) and float(x[:, width:].abs().sum()) == 0
        hh = plain.layer_norm(mean, nw[cut], eps)
        assert torch.allclose(h[:, cut], hh, atol=1e-4)
        for rows, s in (([0], 0), ([1, 2, 3], 2), ([4], 1)):
            seq = torch.cat([tails[s][:, cut], hh[rows]])
            assert torch.allclose(got[rows, cut], plain.input_conv(seq, cw[:, cut].t())[3:], atol=1e-4)
    assert torch.equal(ops.norm_rows(x, i32([2]), nw, width, eps, mean=True)[:, cut], ops._layer_norm(x[2:3], nw, None, width, eps)[:, cut])


@pytest.mark.parametrize("H,G,D,V,rot,hp", [(4, 2, 12, 20, 12, 64), (3, 1, 10, 6, 4, 64), (2, 2, 13, 9, 10, 64), (4, 1, 64, 64, 0, 64)])
def test_queries_and_keys_rotate_halves(H, G, D, V, rot, hp):
    n, kvb, v_off = 9, 4, (H + G) * D
    freq = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    proj, norms = rnd(n, v_off + G * V + 3), (rnd(H * D, seed=1), rnd(G * D, seed=2))
    kc, vc, bt = torch.full((4, kvb, G, hp), 9.0), torch.full((4, kvb, G, hp), 9.0), i32([[0, 1, 2, 3], [2, 0, 3, 1]])
    for source in (-1, 0):
        d = GqaDims(H, G, D, hp, 0.3, rot, v_off, False, V, row_norm=True, rot_half=True, source=source)
        args = (d, None, freq, i32([1] * n), i32(list(range(n))), bt, kc, vc, kvb, 1e-4)
        q = TorchOps("cpu").gqa_prep(proj if source < 0 else proj[:, :H * D], *args, norms=norms if source < 0 else (norms[0], None))
        want = plain.rotate_half((plain.rms(proj[:, :H * D], 1e-4) * norms[0]).view(n, H, D), 50.0, rot)
        assert torch.allclose(q[..., :D], want, atol=1e-5) and float(q[..., D:].abs().sum()) == 0
    rows = lambda c: torch.stack([c[int(bt[1, t // kvb]), t % kvb] for t in range(n)])
    k = plain.rotate_half((plain.rms(proj[:, H * D:v_off], 1e-4) * norms[1]).view(n, G, D), 50.0, rot)
    assert torch.allclose(rows(kc)[..., :D], k, atol=1e-5) and torch.equal(rows(vc)[..., :V], proj[:, v_off:v_off + G * V].view(n, G, V))


@pytest.mark.parametrize("size,pool", [(1, 1), (1, 3), (3, 4), (4, 4), (5, 3), (8, 8), (7, 9), (11, 2), (40, 4)])
def test_windows_and_blocks_in_pages(size, pool):
    """Every row against every key and mean it may see, pages of four keys; the means written in portions of the sequence."""
    n, kvb, H, G, D = 31, 4, 4, 2, 8
    d = GqaDims(H, G, D, D, 2.0, 0, 0, False, D, row_norm=True, softcap=3.0, window=size, pool=pool)
    k, v, q = rnd(n, G, D), rnd(n, G, D, seed=1), rnd(n, H, D, seed=2)
    pages, bt = [5, 0, 3, 1, 4, 2, 7, 6], i32([[5, 0, 3, 1, 4, 2, 7, 6]])
    kc, vc = torch.zeros(8, kvb, G, D), torch.zeros(8, kvb, G, D)
    for t in range(n):
        kc[pages[t // kvb], t % kvb], vc[pages[t // kvb], t % kvb] = k[t], v[t]
    ops = TorchOps("cpu")
    for cuts in ([31], [1] * 31, [2, 9, 1, 19]):
        means, at = tuple(torch.zeros(8, -(-kvb // pool), G, D) for _ in "kv"), 0
        for c in cuts:
            ops.pool_keys(d, kc, vc, means, i32([0]), i32([at]), i32([c]), c, bt, kvb)
            at += c
        out = ops.gqa_attention(q, d, kc, vc, None, SegGroup(0, 1, 0, n, n), i32([0] * n), i32(list(range(1, n + 1))), None, bt, kvb, 1,
                                torch.empty(n, H, D), pooled=means)
        assert torch.allclose(out, plain.pooled_attention(q, k, v, size, pool, 2.0, 3.0), atol=1e-5)
    assert [d.blocks_visible(i) for i in range(n)] == plain.block_mask(n, size, pool).sum(1).tolist()
    assert [d.first_visible(i) for i in range(n)] == [int(plain.window_mask(n, size)[i].nonzero()[0]) for i in range(n)]


@pytest.mark.parametrize("at", [0, 3, 4, 7, 8, 11])
def test_one_key_stands_out(at):
    """A key that every query points at: seen as itself while it is in the window, then not at all until its block has left it, then as a share
    of the block's mean."""
    n, kvb, D, size, pool = 40, 4, 16, 6, 4
    k, v = 0.05 * rnd(n, 1, D), rnd(n, 1, D, seed=1)
    k[at] = 4.0
    kc, vc, bt = torch.zeros(10, kvb, 1, D), torch.zeros(10, kvb, 1, D), i32([[5, 0, 3, 1, 4, 2, 9, 8, 7, 6]])
    for t in range(n):
        kc[int(bt[0, t // kvb]), t % kvb], vc[int(bt[0, t // kvb]), t % kvb] = k[t], v[t]
    d = GqaDims(2, 1, D, D, 3.0, 0, 0, False, D, row_norm=True, softcap=60.0, window=size, pool=pool)
    ops, means = TorchOps("cpu"), tuple(torch.zeros(10, 1, 1, D) for _ in "kv")
    ops.pool_keys(d, kc, vc, means, i32([0]), i32([0]), i32([n]), n, bt, kvb)
    o = ops.gqa_attention(torch.ones(n, 2, D), d, kc, vc, None, SegGroup(0, 1, 0, n, n), i32([0] * n), i32(list(range(1, n + 1))), None, bt, kvb, 1,
                          torch.empty(n, 2, D), pooled=means)
    itself = ((o - v[at]).abs().amax((1, 2)) < 1e-4).tolist()
    block = v[at // pool * pool:at // pool * pool + pool].mean(0)
    mean = ((o - block).abs().amax((1, 2)) < 1e-4).tolist()
    assert itself == [at <= t <= at + size - 1 for t in range(n)]
    assert mean == [t >= at // pool * pool + pool - 1 + size for t in range(n)]


@pytest.mark.parametrize("size", [1, 3, 4, 5, 9, 30])
def test_latent_rows_and_windows(size):
    n, kvb, H, D, R, L, V = 17, 4, 3, 5, 6, 10, 7
    d = LatentDims(H, 0, L, 0, 16, 16, 0.7, 0, 16, 16, D, R, size)
    proj, norm, base = rnd(n, H * (D + R) + L + R), rnd(L, seed=1), 40.0
    freq = torch.tensor([base ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64)
    cache, bt = torch.full((5, kvb, 16), 9.0), i32([[4, 0, 3, 1, 2]])
    ops = TorchOps("cpu")
    q = ops.latent_rot_prep(proj, d, norm, freq, i32([0] * n), i32(list(range(n))), bt, cache, kvb, 1e-4)
    rows = torch.stack([cache[int(bt[0, t // kvb]), t % kvb] for t in range(n)])
    pq = proj[:, :H * (D + R)].view(n, H, D + R)
    assert torch.equal(q[..., :D], pq[..., :D]) and torch.allclose(q[..., D:D + R], plain.rotate_pairs(pq[..., D:], base, R), atol=1e-5)
    c, kr = plain.rms(proj[:, H * (D + R):-R], 1e-4) * norm, plain.rotate_pairs(proj[:, None, -R:], base, R)[:, 0]
    assert torch.allclose(rows[:, :L], c, atol=1e-5) and torch.allclose(rows[:, L:L + R], kr, atol=1e-5) and float(rows[:, L + R:].abs().sum()) == 0
    out = ops.latent_attention(q[..., :16], cache, SegGroup(0, 1, 0, n, n), i32([0] * n), i32(list(range(1, n + 1))), None, bt, kvb, 0.7, vlat=12, window=size)
    sc = torch.einsum("ihd,jd->hij", q[..., :16], rows) * 0.7
    want = torch.softmax(sc.masked_fill(~plain.window_mask(n, size), -math.inf), -1) @ rows[:, :12]
    assert out.shape == (n, H, 12) and torch.allclose(out, want.transpose(0, 1), atol=1e-5)


@pytest.mark.parametrize("H,G,N,V,K,parts", [(4, 2, 6, 5, 4, 2), (3, 3, 7, 9, 2, 1), (2, 1, 8, 8, 3, 4)])
def test_state_space_rows(H, G, N, V, K, parts):
    """Portions of two sequences in one batch against the recurrence over whole sequences."""
    d = SsmDims(H, G, N, V, K, parts, 64)
    n, inner, ch = 19, H * V, H * V + 2 * G * N
    w = dict(conv=rnd(K, ch, seed=1), conv_bias=rnd(ch, seed=2), A=-torch.exp(rnd(H, seed=3)), dt_bias=rnd(H, seed=4) - 1, skip=rnd(H, seed=5),
             gnorm_w=rnd(inner, seed=6))
    seqs = [rnd(n, inner + ch + H, seed=7), rnd(n, inner + ch + H, seed=8)]

    def whole(p):
        c = plain.silu(plain.causal_conv(p[:, inner:inner + ch], w["conv"].t()) + w["conv_bias"])
        x, B, C = c[:, :inner].view(n, H, V), c[:, inner:inner + G * N].view(n, G, N), c[:, inner + G * N:].view(n, G, N)
        y = plain.ssm(x, B, C, torch.log1p(torch.exp(p[:, inner + ch:] + w["dt_bias"])), torch.log(-w["A"]), w["skip"])
        return plain.group_norm_gated(y.reshape(n, inner), p[:, :inner], w["gnorm_w"], parts, 1e-4)
    want = [whole(p) for p in seqs]
    ops, rec, tail, at, got = TorchOps("cpu"), torch.zeros(3, H, N, V), torch.zeros(3, K - 1, ch), [0, 0], [[], []]
    for a, b in ((1, 2), (7, 1), (2, 9), (9, 7)):
        proj = torch.cat([seqs[0][at[0]:at[0] + a], seqs[1][at[1]:at[1] + b]])
        slot, pos = i32([2] * a + [0] * b), i32(list(range(at[0], at[0] + a)) + list(range(at[1], at[1] + b)))
        args = (i32([2, 0]), i32([0, a]), i32([a, b]), slot, pos, 1e-4)
        dry = ops.ssm(proj, d, w, rec, tail, None, *args, commit=False)
        y = ops.ssm(proj, d, w, rec, tail, None, *args)
        assert torch.equal(dry, y) and float(y[:, inner:].abs().sum()) == 0
        got[0].append(y[:a, :inner]), got[1].append(y[a:, :inner])
        at[0], at[1] = at[0] + a, at[1] + b
    for g, x in zip(got, want):
        assert torch.allclose(torch.cat(g), x, atol=2e-4)
    assert float(rec[1].abs().sum()) == 0


def test_experts_by_hand():
    z = torch.tensor([0.0, 2.0, -1.0, 2.0 + math.log(3.0)])
    assert [e for e, _ in plain.route(z, 2)] == [3, 1] and [float(g) for _, g in plain.route(z, 2)] == pytest.approx([0.75, 0.25])
    ids, wts = TorchOps("cpu").moe_route(torch.cat([z, torch.tensor([0.0])])[None], None, 2, 2, 1, 1, 1.0, n_exp=4, shared_col=4, shared_id=4)
    assert ids.tolist() == [[3, 1, 4]] and wts[0].tolist() == pytest.approx([0.75, 0.25, 0.5])
    g, u = torch.tensor([3.0, -4.0, 0.5]), torch.tensor([5.0, -5.0, 0.25])
    want = [1.0 / (1.0 + math.exp(-1.702)) * 2.0, -4.0 / (1.0 + math.exp(1.702 * 4.0)) * 0.0, 0.5 / (1.0 + math.exp(-0.851)) * 1.25]
    assert plain.clamped_glu(g, u, 1.0).tolist() == pytest.approx(want)
    ops, E, F, S, W = TorchOps("cpu"), 3, 4, 6, 8
    gu, dn, sgu, sdn, h = rnd(E, 2 * F, W), rnd(E, W, F, seed=1), rnd(1, 2 * S, W, seed=2), rnd(1, W, S, seed=3), rnd(2, W, seed=4)
    got = ops.expert_rows(h, i32([[1, 3], [3, 0]]), gu, dn, 0.8, (sgu, sdn, 0.3))
    one = lambda t, e: plain.expert(h[t], gu[e, :F], gu[e, F:], dn[e], 0.8) if e < E else plain.expert(h[t], sgu[0, :S], sgu[0, S:], sdn[0], 0.3)
    assert torch.allclose(got, torch.stack([one(0, 1), one(0, 3), one(1, 3), one(1, 0)]), atol=1e-5)


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
    for name in ("l1.mix.q.norm", "l1.mix.k.norm", "l2.mix.dkv.norm", "l2.mix.uv", "l0.mix.conv.b", "l0.mix.D", "l4.mix.A_log", "l4.mix.norm", "l0.canon1",
                 "l1.canon2", "l2.norm1b", "l4.dwa", "l0.dwa", "l3.mlp.router", "l1.mlp.e3.up", "l1.mlp.shared.sg", "l3.mlp.shared.down", "final.norm"):
        every_other = torch.ones_like(w[name])
        every_other.view(-1)[::2] = 0.8                                           # (the norms take a common factor out again)
        assert error(plain.forward(cfg, dict(w, **{name: w[name] * every_other}), ids)[0], base) > 20 * LIM, name
    for change in (lambda c: c["layers"][1]["mixer"]["rot"].update(base=730.0), lambda c: c["layers"][2]["mixer"]["rot"].update(base=310.0),
                   lambda c: c["layers"][1]["mixer"]["mask"].update(size=18), lambda c: c["layers"][1]["mixer"]["mask"].update(pool=6),
                   lambda c: c["layers"][3]["mixer"]["mask"].update(size=30), lambda c: c["layers"][3]["mixer"]["mask"].update(pool=5),
                   lambda c: c["layers"][2]["mixer"]["mask"].update(size=34), lambda c: c["layers"][1]["mixer"].update(softcap=10.0),
                   lambda c: c["layers"][0]["mlp"]["expert"].update(limit=1.1), lambda c: c["layers"][1]["mlp"]["shared"].update(limit=0.8),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=2), lambda c: c["layers"][0]["mixer"].update(norm_groups=2),
                   lambda c: c["embedding"].update(scale=2.8), lambda c: c["norm"].update(eps=2e-3)):
        other = copy.deepcopy(cfg)
        change(other)
        assert error(plain.forward(other, w, ids)[0], base) > 20 * LIM


def test_residual_rows_after_every_layer(models):
    cfg, w, d, ids, _ = models["grid"]
    eng = engine(d)
    eng.cfg.tap_layers[:] = range(len(cfg["layers"]))
    eng.forward([Segment(0, 0, ids[:40], "none")])
    _, after = plain.forward(cfg, w, ids[:40])
    assert len(eng.taps) == len(cfg["layers"])
    for got, want in zip(eng.taps, after):
        assert float((got.double() - want).abs().max()) < 1e-4 * float(want.abs().max())


STEPS = [dict(a=64, b=2), dict(a=1, b=60, c=3), dict(a=63, d=1), dict(b=8, d=64), dict(a=2, d=2), dict(a=20, d=63, f=1), dict(e=64), dict(e=1)]
LENS = {"a": 150, "b": 70, "c": 3, "d": 130, "e": 65, "f": 1}


def test_unequal_requests_together_and_reused_pages_and_slots(models):
    """Portions of some requests beside single tokens of others, in a pool that only holds what is live: requests end, their pages, means and
    slots go to the next ones, one request pauses for some steps."""
    for name in ("ragged", "edges"):
        cfg, w, d, _, _ = models[name]
        eng = engine(d, max_ctx=256, pool=448)
        seqs = {k: tokens(cfg, n, 20 + i) for i, (k, n) in enumerate(LENS.items())}
        want = {k: plain.forward(cfg, w, s)[0] for k, s in seqs.items()}
        slot, at, got, used, free = {}, {k: 0 for k in seqs}, {k: [] for k in seqs}, [], [0, 1, 2, 3]
        for st in STEPS:
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
                if at[k] == LENS[k]:
                    used.append(list(eng.ex.slot_blocks[slot[k]]))
                    eng.reset_slot(slot[k])
                    free.append(slot.pop(k))
        assert eng.ex.pool.n_free == eng.ex.pool.n_blocks == 7
        assert any(set(used[-1]) & set(u) for u in used[:-1])                     # pages did go round
        for k in seqs:
            assert error(torch.cat(got[k]), want[k]) < LIM, (name, k)


def test_rejected_rows_and_forks_leave_no_trace(models):
    """Verify rows whose end is rejected (a block of means ends in it), then a fork of the slot."""
    for name in ("grid", "ragged", "edges"):
        cfg, w, d, ids, want = models[name]
        eng = engine(d)
        eng.forward([Segment(0, 0, ids[:62], "none")])
        wrong = [(t + 1) % cfg["vocab"] for t in ids[64:69]]
        for keep in (0, 2):
            lg, _, _ = eng.forward([Segment(0, 62, ids[62:64] + wrong, "all")], commit=False, greedy=False)
            assert error(lg[:2], want[62:64]) < LIM
            eng.commit_verified([keep])
        eng.ex.copy_slot(0, 2, 64)
        eng.forward([Segment(0, 64, ids[:9], "none")])                            # moves slot 0 away from its copy
        lg, _, _ = eng.forward([Segment(2, 64, ids[64:120], "all")], greedy=False)
        assert error(lg, want[64:120]) < LIM


def test_snapshots_hold_every_state(models):
    cfg, w, d, ids, want = models["ragged"]
    eng = engine(d)
    eng.forward([Segment(1, 0, ids[:40], "none")])
    snap = eng.ex.state_save(1)
    eng.forward([Segment(1, 40, ids[100:110], "none")])
    eng.ex.state_restore(1, snap)
    lg, _, _ = eng.forward([Segment(1, 40, ids[40:90], "all")], greedy=False)
    assert error(lg, want[40:90]) < LIM


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


def test_long_decode_over_windows_blocks_and_pages(models):
    cfg, w, d, ids, want = models["ragged"]
    assert error(run_cuts(engine(d), ids, [3, 1]), want) < LIM


def test_sizes_of_caches_and_states():
    cfg = tiny_pironex()
    eng = Engine(cfg, None, EngineConfig(n_slots=2, max_ctx=64), device="cpu")
    ex = eng.ex
    assert sorted(ex.k_cache) == [0, 1, 4] and sorted(ex.pools) == [(1, 5), (1, 7)] and sorted(ex.rec_state) == [2, 3]
    assert ex.conv_state["canon"].shape == (2, 11, 3, 192) and len(ex.canon_at) == 11          # five layers of two sublayers, one of one
    pages = list(ex.k_cache.values()) + [t for i, t in ex.v_cache.items()] + [t for m in ex.pools.values() for t in m]
    assert ex.kv_block_bytes() == sum(t[0].numel() * 4 for t in pages)


def test_expert_counters(monkeypatch, tmp_path):
    monkeypatch.setenv("FE_EXPERT_HEAT", str(tmp_path / "heat.json"))
    cfg = tiny_pironex()
    eng = Engine(cfg, None, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    eng.forward([Segment(0, 0, list(range(10)), "none")])
    heat = eng.expert_heat()
    assert sorted(heat) == [0, 1, 2, 4, 5] and all(len(v) == 7 and sum(v[:6]) == 20 and v[6] == 10 for v in heat.values())


def test_index_checks_cover_the_ops(monkeypatch):
    monkeypatch.setenv("FB_DEBUG_BOUNDS", "1")
    eng = Engine(tiny_pironex(), None, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    eng.forward([Segment(0, 0, list(range(10)), "last")])
    assert {"embed_grams", "gqa_prep", "gqa_attention", "pool_keys", "latent_rot_prep", "ssm", "add_conv_normed", "expert_rows"} <= set(eng.bounds.checked)
    with pytest.raises(IndexError, match="experts of the layer"):
        eng.ex.ops.expert_rows(torch.zeros(1, 192), i32([[7]]), torch.zeros(6, 128, 192), torch.zeros(6, 192, 64), 1.0,
                               (torch.zeros(1, 128, 192), torch.zeros(1, 192, 64), 1.0))


def test_reference_model_agrees():
    cfg = tiny_pironex()
    w = init_weights(cfg, seed=4, std=0.1)
    ids = torch.randint(0, cfg.vocab, (100,), generator=torch.Generator().manual_seed(1)).tolist()
    ref = RefModel(cfg, w)
    st = ref.new_state()
    want = ref.forward(ids[:60], st)
    want = torch.cat([want, ref.forward(ids[60:], st.clone())])
    eng = Engine(cfg, w, EngineConfig(n_slots=1, max_ctx=128), device="cpu")
    lg, _, _ = eng.forward([Segment(0, 0, ids, "all")], greedy=False)
    assert error(lg, want) < LIM
    c = pironex(64, 6, 4, 2, 50, dim=16, kv_rank=24, rot_dim=8, state=8, ssm_heads=4, ssm_vdim=16, window=9, pool=4, experts=4, top=2, expert_ff=32, shared_ff=32)
    assert [l.mixer for l in c.layers] == ["latent", "gqa", "ssm", "ssm", "latent", "gqa"] and c.layers[5].kv_from == 1
    assert Engine(c, None, EngineConfig(n_slots=1, max_ctx=64), device="cpu").generate(list(range(20)), 3)


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


def test_means_reach_further_than_the_window(tmp_path):
    """With and without blocks a model agrees until the first block has left the window, and nowhere behind it."""
    cfg = config(64, 90, [pooled(2, 1, 16, 16, 40, 8, moe(2, 1, 32), rot=0)])
    w = weights(cfg, seed=5)
    ids = tokens(cfg, 130, 1)
    got = run_cuts(engine(write(cfg, w, tmp_path / "m")), ids, [130])
    free = copy.deepcopy(cfg)
    free["layers"][0]["mixer"]["mask"]["pool"] = 1000
    window = plain.forward(free, w, ids)[0]
    assert error(got[:47], window[:47]) < LIM and error(got[47:48], window[47:48]) > 50 * LIM


def test_a_window_without_blocks(tmp_path):
    """mask.pool may be left out: a window alone."""
    cfg = config(64, 90, [pooled(2, 1, 16, 16, 12, 8, moe(2, 1, 32))])
    w, ids = weights(cfg, seed=6), tokens(cfg, 60, 2)
    free = copy.deepcopy(cfg)
    free["layers"][0]["mixer"]["mask"]["pool"] = 1000
    del cfg["layers"][0]["mixer"]["mask"]["pool"]
    assert error(run_cuts(engine(write(cfg, w, tmp_path / "m")), ids, [37, 1]), plain.forward(free, w, ids)[0]) < LIM
