"""The Zototar design on the fp32 CPU engine against a plain statement of it (`plain_latent.py`): configuration and checkpoint
reading, each mechanism, prompts, decoding, portions, batches, reused pages, speculation, the scheduler and two ranks."""
import copy
import io
import json
import sys

import pytest
import torch

import plain_latent as plain
from ferrite_b200.config import EngineConfig, ModelConfig, tiny_zototar
from ferrite_b200.engine.engine import Engine
from ferrite_b200.engine.executor import Segment
from ferrite_b200.engine.sampler import Sampling
from ferrite_b200.engine.scheduler import SchedOptions, Scheduler, generate
from ferrite_b200.formats.loader import load_model_weights
from ferrite_b200.models.weights import init_weights, latent_dims, pack_listed
from ferrite_b200.ops.torch_ops import TorchOps
from zototar_cases import CASES, engine, error, run_cuts, tokens, weights, write

LIM = 2e-5


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
    root = tmp_path_factory.mktemp("zototar")
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
    assert [l.kv_from for l in c.layers] == [None, None, 0, 1, 0] and c.layers[1].ff == 0 and c.layers[3].scale == 0.1
    assert (c.gram_buckets, c.gram_mul_prev, c.gram_mul_cur, c.embed_scale, c.logit_softcap) == (101, 13, 7, 7.5, 20.0)
    assert c.layer_kinds == ["latent"] * 5 and c.n_attn == 2
    b = read(CASES["bare"])
    assert b.gram_buckets == 0 and b.logit_softcap == 0.0 and b.eps == 1e-3
    for change, what in (((lambda c: c.update(architecture="Zotobar")), "architecture"),
                         ((lambda c: c["layers"][0].update(type="conv")), "type"),
                         ((lambda c: c["layers"][0]["mlp"].update(kind="routed")), "kind"),
                         ((lambda c: c["layers"][2]["mixer"].update(kv_from=3)), "kv_from"),
                         ((lambda c: c["layers"][4]["mixer"].update(kv_from=2)), "kv_from"),
                         ((lambda c: c["layers"][2]["mixer"].update(kv_rank=48)), "kv_from")):
        bad = copy.deepcopy(CASES["ragged"])
        change(bad)
        with pytest.raises(ValueError, match=what):
            read(bad)


def test_checkpoint_shapes_are_checked(tmp_path):
    cfg = CASES["bare"]
    w = weights(cfg)
    for change, what in (((lambda w: w.pop("l0.mix.uk")), "l0.mix.uk"),
                         ((lambda w: w.update({"l0.norm1": w["l0.norm1"][:-1]})), "l0.norm1")):
        bad = dict(w)
        change(bad)
        d = write(cfg, bad, tmp_path / what.replace(".", "_"))
        with pytest.raises((KeyError, ValueError), match=what):
            load_model_weights(d, ModelConfig.from_hf(d + "/config.json"))


def test_kernel_layout_pads_with_zeros():
    cfg = tiny_zototar()
    w = init_weights(cfg, seed=3)
    pk = pack_listed(cfg, w)
    for i, l in enumerate(cfg.layers):
        d, p = latent_dims(cfg, i), f"l{i}."
        assert d.qr % 64 == d.lat % 64 == 0 and d.hp in (64, 128, 256)
        q = pk[p + "q_b"].view(l.heads, d.hp, d.qr)
        assert torch.equal(q[:, :l.dim, :l.q_rank], w[p + "q_b"].view(l.heads, l.dim, l.q_rank))
        assert float(q[:, l.dim:].abs().sum() + q[:, :, l.q_rank:].abs().sum()) == 0.0
        assert torch.equal(pk[p + "k_abs"][:, :l.kv_rank, :l.dim].transpose(1, 2).reshape(-1, l.kv_rank), w[p + "k_b"])
        assert pk[p + "q_a_norm"].dtype == torch.float32


# ---- mechanisms -------------------------------------------------------------------------------------------------------

def rnd(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


def test_embedding_with_bigrams_across_steps_and_pages():
    ops, kvb, W = TorchOps("cpu"), 4, 8
    table, grams = rnd(30, W, seed=1), rnd(12, W, seed=2)
    w = {"embed": table, "bigram": grams}
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": 11, "mul_prev": 5, "mul_cur": 3}}}
    a, b = tokens({"vocab": 30}, 11, 3), tokens({"vocab": 30}, 6, 4)
    want_a, want_b = plain.embed(cfg, w, a), plain.embed(cfg, w, b)
    assert torch.equal(want_a[0], table[a[0]] * 2.5 + grams[11])
    bt = torch.tensor([[3, 0, 5], [2, 4, 1]], dtype=torch.int32)
    pages = torch.zeros(6, kvb, dtype=torch.int32)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    got_a, got_b = [], []
    for ra, rb in ((range(0, 3), range(0, 1)), (range(3, 4), range(1, 4)), (range(4, 9), ()), (range(9, 11), range(4, 6))):
        tok = i32([b[i] for i in rb] + [a[i] for i in ra])
        slot, pos = i32([1] * len(rb) + [0] * len(ra)), i32(list(rb) + list(ra))
        x, xb = ops.embed_grams(table, grams, tok, slot, pos, bt, pages, kvb, 2.5, 11, 5, 3)
        got_b.append(x[:len(rb)])
        got_a.append(x[len(rb):])
    assert torch.allclose(torch.cat(got_a), want_a) and torch.allclose(torch.cat(got_b), want_b)


def test_norms_activation_softcap():
    ops = TorchOps("cpu")
    x, y, w = rnd(5, 12), rnd(5, 12, seed=1) * 3, rnd(12, seed=2)
    want = x + plain.rms_norm(y, w, 1e-3)
    xx = x.clone()
    assert torch.allclose(ops.add_normed(xx, y, w, 12, 1e-3), want) and torch.allclose(xx, want)
    pad = torch.nn.functional.pad
    xp = pad(x, (0, 4))
    ops.add_normed(xp, pad(y, (0, 4)), pad(w, (0, 4)), 12, 1e-3)                 # padded columns leave the mean alone
    assert torch.allclose(xp[:, :12], want) and float(xp[:, 12:].abs().sum()) == 0
    assert torch.allclose(ops.norm_rows(x, torch.tensor([3, 0]), w, 12, 1e-3), plain.rms_norm(x[[3, 0]], w, 1e-3))
    assert float(plain.rms(torch.full((1, 4), 1e-3), 1e-5)[0, 0]) == pytest.approx(1e-3 / (1e-6 + 1e-5) ** 0.5)
    m = rnd(7, 12, seed=3)
    assert torch.allclose(ops.linear(x, m, act="relu2"), plain.relu_squared(x @ m.t()))
    z = rnd(3, 9) * 50
    assert torch.allclose(ops.softcap(z.clone(), 20.0), plain.softcap(z, 20.0)) and float(ops.softcap(z, 20.0).abs().max()) <= 20.0


@pytest.mark.parametrize("at", [0, 3, 4, 7, 8, 9, 10])
def test_one_key_stands_out(at):
    """A single latent that every query points at: seen when it is at or before the row, invisible one position later."""
    ops, kvb, L, heads = TorchOps("cpu"), 4, 16, 2
    cache = torch.zeros(3, kvb, L)
    bt = torch.tensor([[2, 0, 1]], dtype=torch.int32)
    c = rnd(12, L) * 0.1
    c[at] = torch.ones(L)
    for t in range(12):
        cache[int(bt[0, t // kvb]), t % kvb] = c[t]
    q = torch.ones(1, heads, L) * 3
    for kvlen in (at, at + 1, 11):
        if kvlen == 0:
            continue
        o = ops.latent_attention(q, cache, None, torch.zeros(1, dtype=torch.int32), torch.tensor([kvlen]), None, bt, kvb, 0.5)
        assert torch.allclose(o[0, 0], c[at], atol=1e-4) == (kvlen > at)


def test_plain_mask_and_shared_latents():
    p = plain.causal_softmax(torch.zeros(1, 3, 3))
    assert torch.allclose(p[0], torch.tensor([[1.0, 0, 0], [0.5, 0.5, 0], [1 / 3, 1 / 3, 1 / 3]]))
    cfg, w = CASES["grid"], weights(CASES["grid"])
    h, lat = rnd(4, 128), {}
    w = {k: v.float() for k, v in w.items()}
    plain.mixer(cfg, w, 0, h, lat)
    before = plain.mixer(cfg, w, 1, h, lat)
    lat[0] = lat[0] * 1.5
    assert not torch.allclose(before, plain.mixer(cfg, w, 1, h, lat)) and 1 not in lat


# ---- whole models ------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", list(CASES))
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [63, 2, 1, 64, 3, 65, 2]], ids=["whole", "single", "pairs", "mixed"])
def test_sequence_in_portions(models, name, cuts):
    cfg, w, d = models[name]
    ids = tokens(cfg, 150 if cuts[0] > 2 else 70, 11)
    want, _ = plain.forward(cfg, w, ids)
    assert error(run_cuts(engine(d), ids, cuts), want) < LIM


def test_far_tokens_show_in_the_logits(models):
    """The power of the comparisons: a token 140 places back moves the last logits by far more than the tolerance."""
    for name in ("grid", "ragged"):
        cfg, w, d = models[name]
        ids = tokens(cfg, 150, 11)
        base = plain.forward(cfg, w, ids)[0][-1:]
        moved = [error(plain.forward(cfg, w, ids[:t] + [(ids[t] + 1) % cfg["vocab"]] + ids[t + 1:])[0][-1:], base) for t in range(0, 12)]
        assert max(moved) > 1000 * LIM and min(moved) > 5 * LIM, moved


def test_residual_rows_after_every_layer(models):
    cfg, w, d = models["ragged"]
    eng = engine(d)
    eng.cfg.tap_layers[:] = range(len(cfg["layers"]))
    ids = tokens(cfg, 40, 12)
    eng.forward([Segment(0, 0, ids, "none")])
    _, after = plain.forward(cfg, w, ids)
    assert len(eng.taps) == len(cfg["layers"])
    for got, want in zip(eng.taps, after):
        assert float((got.double() - want).abs().max()) < 1e-4 * float(want.abs().max())


def test_unequal_requests_together_and_reused_pages(models):
    """Portions of some requests beside single tokens of others, in a pool that only holds what is live: requests end, their
    pages and slots go to the next ones, one request pauses for some steps."""
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


def test_wanted_rows_by_index(models):
    cfg, w, d = models["grid"]
    eng, ids = engine(d), tokens(cfg, 30, 5)
    want, _ = plain.forward(cfg, w, ids)
    lg, _, rows = eng.forward([Segment(0, 0, ids, [4, 0, 29]), Segment(1, 0, ids[:7], "last"), Segment(2, 0, ids[:3], [])], greedy=False)
    assert rows == [4, 0, 29, 36] and error(lg, want[[4, 0, 29, 6]]) < LIM
    with pytest.raises(AssertionError, match="want_logits"):
        eng.forward([Segment(3, 0, ids[:3], [3])], greedy=False)


def test_rejected_rows_leave_no_trace(models):
    """Verify rows that are not kept: the next token follows the last kept one, in the cache and in the bigram."""
    cfg, w, d = models["grid"]
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


def test_greedy_generation_and_scheduler(models):
    """Engine.generate, and the scheduler with more requests than slots, copy-drafted verify rows, a shared prefix resumed from
    the prompt cache, forks, parking and a page pool below slots x context."""
    cfg, w, d = models["grid"]
    prompts = [tokens(cfg, n, 30 + n) for n in (5, 70, 33, 1)]
    prompts.append(prompts[1] + tokens(cfg, 9, 77))
    prompts.append((tokens(cfg, 6, 78) * 6)[:34])
    want = [plain.greedy(cfg, w, p, 8) for p in prompts]
    eng = engine(d, slots=1, max_ctx=128)
    assert eng.generate(prompts[1], 8) == want[1]
    for spec, pool in ((0, 0), (0, 320), (4, 0), (3, 384)):
        eng = engine(d, slots=3, max_ctx=192, pool=pool, prefill_chunk=32)
        sched = Scheduler(eng, SchedOptions(spec=spec, arrival_ms=0, share_min=32))
        out = generate(sched, prompts, Sampling(max_tokens=8), snapshots=[[64] if len(p) > 64 else [] for p in prompts])
        assert out == want, (spec, pool)
        again = generate(sched, [prompts[4]], Sampling(max_tokens=8), snapshots=[[64]])      # from a kept or parked prefix
        assert again[0] == want[4]
        held = sum(len(b) for b in eng.ex.slot_blocks) + sum(len(e.blocks) for e in sched.park.entries.values())
        assert held + eng.ex.pool.n_free == eng.ex.pool.n_blocks


def test_small_pool_queues_requests_instead_of_failing_them(models):
    cfg, w, d = models["bare"]
    prompts = [tokens(cfg, 60 + i, i) for i in range(5)]
    eng = engine(d, slots=4, max_ctx=128, pool=256)                               # two requests of two pages at a time
    sched = Scheduler(eng, SchedOptions(arrival_ms=0))
    assert generate(sched, prompts, Sampling(max_tokens=6)) == [plain.greedy(cfg, w, p, 6) for p in prompts]


def test_long_decode_over_page_borders(models):
    cfg, w, d = models["ragged"]
    ids = tokens(cfg, 135, 9)
    want, _ = plain.forward(cfg, w, ids)
    assert error(run_cuts(engine(d), ids, [3, 1]), want) < LIM


def test_shared_latents_are_cached_once():
    cfg = tiny_zototar()
    eng = Engine(cfg, None, EngineConfig(n_slots=1, max_ctx=64), device="cpu")
    assert sorted(eng.ex.k_cache) == [i for i, l in enumerate(cfg.layers) if l.kv_from is None]
    rows = sum(t.shape[-1] for t in eng.ex.k_cache.values())
    assert eng.ex.kv_block_bytes() == 64 * (4 * rows + 4)


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


# ---- two ranks ----------------------------------------------------------------------------------------------------------

def test_two_ranks_equal_one():
    import torch.multiprocessing as mp

    from test_tp_cpu import _free_port, _worker, gather
    cfg = tiny_zototar()
    prompt = torch.randint(0, cfg.vocab, (70,), generator=torch.Generator().manual_seed(6)).tolist()
    eng = Engine(cfg, init_weights(cfg, seed=0), EngineConfig(n_slots=1, max_ctx=128), device="cpu")
    want, wp, _ = eng.forward([Segment(0, 0, prompt, "all")])
    want2, _, _ = eng.forward([Segment(0, len(prompt), [int(wp[0][-1])], "last")])
    ctx = mp.get_context("spawn")
    q, port = ctx.Queue(), _free_port()
    procs = [ctx.Process(target=_worker, args=(r, 2, port, prompt, q, "tiny-zototar")) for r in range(2)]
    for p in procs:
        p.start()
    outs = gather(q, 2)
    for p in procs:
        p.join(timeout=60)
    for rank, logits, ids, l2 in outs:
        assert error(logits, want) < LIM and error(l2, want2) < LIM and ids.tolist() == wp[0].tolist()
    assert torch.equal(outs[0][1], outs[1][1]) and torch.equal(outs[0][3], outs[1][3])
