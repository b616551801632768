"""Layered models on the GPU against the plain oracle: mechanisms alone, prompts, token-by-token decoding, portions, unequal batches,
slots that are used again, far keys and first tokens, long decoding, snapshots and beams, the slot scheduler and the command line."""
import io

import numpy as np
import pytest

from seq2seqsharp_b200.gpt import DecodingOptions, DecodingStrategyEnums as DS, KvCachePool, generate_with_pool
from seq2seqsharp_b200.layered import LayeredGPT
from seq2seqsharp_b200.pepilix import config_from_json, engine_name
from seq2seqsharp_b200.safetensors_file import to_bfloat16
from seq2seqsharp_b200.scheduler import ContinuousBatcher, Request
from tests import layered_models as M

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
GREEDY = DecodingOptions(DecodingStrategy=DS.GreedySearch)


def engine(cfg, w, dtype, max_batch=1, max_tokens=512):
    g = LayeredGPT(config_from_json(cfg, dtype), max_batch=max_batch, max_tokens=max_tokens)
    g.LoadWeights({engine_name(k): v if v.dtype == np.int32 else to_bfloat16(v) for k, v in w.items()})
    return g


def score(g, ids, slot=0, cuts=None):
    """Logits of every position, the text cut into portions of the given sizes."""
    g.SlotReset(slot)
    out, at = [], 0
    for n in (cuts or [len(ids)]):
        n = min(n, len(ids) - at)
        if n <= 0:
            break
        out.append(g.SlotLogits(slot, ids[at:at + n], range(n)))
        at += n
    if at < len(ids):
        out.append(g.SlotLogits(slot, ids[at:], range(len(ids) - at)))
    return np.concatenate(out)


# ---- each mechanism alone -------------------------------------------------------------------------------------------------------
def _only(**keep):
    """One layer in which everything but the named mechanism is switched off by its weights."""
    cfg = M.config([M.layer(3, 16, 8, 16, 24, scale=1.5, experts=5 if keep.get("experts") else None, top=2, ff=24, limit=0.5)], 48, 67, groups=4, taps=4)
    w = M.weights(cfg, 5)
    if not keep.get("conv"):
        w["l0.canon1"] = np.zeros_like(w["l0.canon1"])
    if not keep.get("gate"):
        w["l0.rg1"] = np.zeros_like(w["l0.rg1"])
        w["l0.rg1.b"] = np.full_like(w["l0.rg1.b"], 8.0)
    if keep.get("experts"):
        w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    return cfg, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("keep", ["attention", "conv", "gate", "experts"])
def test_mechanism_alone(cuda, keep, dtype):
    cfg, w = _only(**{keep: True})
    ids = M.tokens(cfg, 37)
    g = engine(cfg, w, dtype)
    assert M.rel(score(g, ids), M.oracle(cfg, w).forward(ids)) < M.TOL[dtype]
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups,taps,embed,logit,eps", [(48, 1, 2, 1.0, 1.0, 1e-6), (48, 6, 3, 7.0, 0.25, 0.5), (48, 12, 9, 1.5, 3.0, 1e-3), (256, 1, 4, 2.0, 1.0, 1e-6),
                                                               (256, 2, 1, 1.0, 1.0, 1e-5), (256, 64, 2, 1.0, 1.0, 1e-5), (2560, 4, 3, 1.0, 1.0, 1e-5), (2304, 18, 4, 1.0, 1.0, 1e-5)])
def test_norm_groups_taps_and_scales(cuda, width, groups, taps, embed, logit, eps, dtype):
    cfg = M.config([M.layer(2, 8, 8, 8, 16, experts=3, top=2, ff=16), M.layer(1, 8, 8, 8, 16)], width, 40, groups=groups, taps=taps, eps=eps, embed=embed, logit=logit)
    w = M.weights(cfg, 6)
    ids = M.tokens(cfg, 14)
    want = M.oracle(cfg, w).forward(ids)
    g = engine(cfg, w, dtype)
    assert M.rel(score(g, ids), want) < M.TOL[dtype]
    assert M.rel(score(g, ids, cuts=[1] * 14), want) < M.TOL[dtype]
    g.close()


# ---- whole prompts, decoding, portions ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_prompt_decode_and_portions_match_the_oracle(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 7)
    ids = M.tokens(cfg, 150 if name == "wide" else 45)
    want = M.oracle(cfg, w).forward(ids)
    g = engine(cfg, w, dtype, max_batch=2)
    tol = M.TOL[dtype]
    assert M.rel(score(g, ids), want) < tol
    for cuts in ([2] * 40, [3, 2, 17, 2, 9], [1, 2, 3, 4, 5], [7] * 30, [20, 100], [16, 17, 2]):
        assert M.rel(score(g, ids, cuts=cuts), want) < tol, cuts
    # token by token through the captured step, from the very first tokens on
    for start in (1, 2, 21):
        g.Reset()
        rows = [g.SlotLogits(0, ids[:start], [start - 1])[0]]
        for t in ids[start:]:
            g.StepHost([t], GREEDY)
            rows.append(g.Logits(want_probs=False)[0][0])
        assert M.rel(rows, want[start - 1:]) < tol, start
    # places out of order and more than once; an empty list
    g.Reset()
    got = g.SlotLogits(0, ids[:8], [7, 0, 7])
    assert M.rel(got, want[[7, 0, 7]]) < tol
    assert g.SlotLogits(0, ids[8:10], []).shape == (0, cfg["vocab"])
    assert M.rel(g.SlotLogits(0, ids[10:12], [1]), want[11:12]) < tol
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_in_large_and_small_portions(cuda, dtype):
    """Several tiles of keys, queries and rows in every kernel; portion borders inside and at the edges of the tiles."""
    cfg = M.CONFIGS["wide"]
    w = M.weights(cfg, 8)
    ids = M.tokens(cfg, 420)
    want = M.oracle(cfg, w).forward(ids)
    g = engine(cfg, w, dtype)
    for cuts in (None, [256, 100], [63, 65, 1, 127, 2], [128, 128, 128], [129, 2, 2, 200]):
        assert M.rel(score(g, ids, cuts=cuts), want) < M.TOL[dtype], cuts
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,rot", [(24, 8), (256, 16), (256, 96), (264, 8), (512, 64), (512, 96), (648, 32), (1024, 16), (1000, 88)])
def test_latent_sizes(cuda, rank, rot, dtype):
    """Every register and staging variant of the absorbed form."""
    cfg = M.config([M.layer(5, 16, rot, 24, rank, scale=0.2), M.layer(3, 24, rot, 40, rank, kv_from=0, scale=0.2)], 64, 50, groups=2, taps=3)
    w = M.weights(cfg, 18)
    ids = M.tokens(cfg, 150)
    want = M.oracle(cfg, w).forward(ids)
    g = engine(cfg, w, dtype)
    tol = M.TOL[dtype]
    assert M.rel(score(g, ids, cuts=[13, 5, 2, 40, 64, 3]), want) < tol
    g.Reset()
    rows = [g.SlotLogits(0, ids[:120], [119])[0]]
    for t in ids[120:]:
        g.StepHost([t], GREEDY)
        rows.append(g.Logits(want_probs=False)[0][0])
    assert M.rel(rows, want[119:]) < tol
    g.CheckGuards()
    g.close()


# ---- keys far away, at tile borders, the first tokens ----------------------------------------------------------------------------
def _needle(scale=6.0, n=200, at=0):
    """A model whose attention is nearly one-hot: the marker token's key stands out for every query."""
    cfg = M.config([M.layer(2, 16, 8, 16, 32, scale=scale, base=1e6)], 64, 50, groups=1, taps=1)
    w = M.weights(cfg, 9)
    ids = [t if t != 49 else 48 for t in M.tokens(cfg, n, at)]
    ids[at] = 49
    w["embed"] = w["embed"].copy()
    w["embed"][49] *= 1.0
    # one latent direction says "marker", and every head's unrotated query has a constant part along its key
    u = np.sign(np.random.default_rng(3).normal(size=64)).astype(np.float32)
    w["embed"][:, 0] = 2.0
    w["embed"][49] = 2.0 * u
    w["embed"][49, 0] = 2.0
    w["l0.mix.dkv"][0] = u / 8
    w["l0.mix.q"] *= 0.25
    for h in range(2):
        w["l0.mix.uk"][16 * h] = 0
        w["l0.mix.uk"][16 * h, 0] = 2.0
        w["l0.mix.q"][24 * h] = 0
        w["l0.mix.q"][24 * h, 0] = 1.0
    for k in ("l0.mix.dkv", "l0.mix.q", "l0.mix.uk", "embed"):
        from seq2seqsharp_b200.safetensors_file import to_float32
        w[k] = to_float32(to_bfloat16(w[k]))
    return cfg, w, ids


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 65, 127, 128, 198])
def test_one_key_among_many(cuda, at, dtype):
    cfg, w, ids = _needle(at=at)
    orc = M.oracle(cfg, w)
    want = orc.forward(ids)
    other = list(ids)
    other[at] = 48
    assert M.rel(orc.forward(other)[-1:], want[-1:]) > 0.2     # the answer hangs on that one key
    g = engine(cfg, w, dtype)
    tol = M.TOL[dtype]
    assert M.rel(score(g, ids), want) < tol
    assert M.rel(score(g, ids, cuts=[at + 1, 2, 2, 37, 64]), want) < tol
    assert M.rel(score(g, ids, cuts=[max(at, 1), 1, 1, 3]), want) < tol
    g.Reset()
    g.SlotLogits(0, ids[:at + 1], [])
    rows = []
    for t in ids[at + 1:]:
        g.StepHost([t], GREEDY)
        rows.append(g.Logits(want_probs=False)[0][0])
    assert M.rel(rows, want[at + 1:]) < tol
    g.close()


# ---- batches, slots ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batch_matches_each_alone(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 10)
    lens = [1, 2, 3, 29, 17, 70]
    prompts = [M.tokens(cfg, n, i) for i, n in enumerate(lens)]
    orc = M.oracle(cfg, w)
    g = engine(cfg, w, dtype, max_batch=6, max_tokens=128)
    tol = M.TOL[dtype]
    g.PrefillRagged(prompts, GREEDY)
    full = [orc.forward(p) for p in prompts]
    assert M.rel(g.Logits(want_probs=False)[0], [f[-1] for f in full]) < tol
    # every sequence goes on with tokens of its own choosing
    texts = [list(p) for p in prompts]
    for step in range(6):
        nxt = [M.tokens(cfg, 1, 50 + 7 * step + i)[0] for i in range(6)]
        g.StepHost(nxt, GREEDY)
        for t, n in zip(texts, nxt):
            t.append(n)
        got = g.Logits(want_probs=False)[0]
        assert M.rel(got, [orc.forward(t)[-1] for t in texts]) < tol, step
    # equal lengths in one prefill
    g.Reset()
    same = [M.tokens(cfg, 24, 90 + i) for i in range(6)]
    g.Prefill(same, GREEDY)
    assert M.rel(g.Logits(want_probs=False)[0], [orc.forward(p)[-1] for p in same]) < tol
    ext = [M.tokens(cfg, 5, 190 + i) for i in range(6)]
    g.Extend(ext, GREEDY)
    assert M.rel(g.Logits(want_probs=False)[0], [orc.forward(p + e)[-1] for p, e in zip(same, ext)]) < tol
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_slots_used_again_and_neighbours_undisturbed(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 11)
    orc = M.oracle(cfg, w)
    g = engine(cfg, w, dtype, max_batch=3, max_tokens=160)
    tol = M.TOL[dtype]
    a, b = M.tokens(cfg, 90, 1), M.tokens(cfg, 33, 2)
    g.SlotReset(0)
    g.SlotLogits(0, a[:60], [])
    g.SlotReset(1)
    g.SlotLogits(1, M.tokens(cfg, 120, 3), [])
    g.SlotReset(1)                                     # a long request leaves, a short one takes its place
    assert M.rel(g.SlotLogits(1, b[:1], [0]), orc.forward(b[:1])) < tol
    assert M.rel(g.SlotLogits(1, b[1:20], range(19)), orc.forward(b)[1:20]) < tol
    assert M.rel(g.SlotLogits(0, a[60:], range(30)), orc.forward(a)[60:]) < tol
    # park, run something else in the slot, come back: the convolution state travels with the cache
    snap = g.SlotSnapshot(1)
    g.SlotReset(1)
    g.SlotLogits(1, M.tokens(cfg, 50, 4), [])
    g.SlotRestore(snap, 1)
    assert M.rel(g.SlotLogits(1, b[20:22], [0, 1]), orc.forward(b)[20:22]) < tol
    g.SlotRestore(snap, 2)
    assert M.rel(g.SlotLogits(2, b[20:], range(13)), orc.forward(b)[20:]) < tol
    snap.close()
    g.CheckGuards()
    g.close()


def test_sequences_that_stand_still_keep_their_state(cuda):
    """A finished sequence is stepped with the others at its own position; what it holds must not change."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 12)
    orc = M.oracle(cfg, w)
    g = engine(cfg, w, "float32", max_batch=2, max_tokens=128)
    g.SetPerSequenceState(True)
    a, b = M.tokens(cfg, 11, 1), M.tokens(cfg, 20, 2)
    for s, t in ((0, a), (1, b)):
        g.SlotReset(s)
        g.SlotExtend(s, t, GREEDY)
    # the pending id of slot 0 becomes </s>: it stands still from now on
    snap = g.SlotSnapshot(0)
    g.SlotReset(0)
    g.SlotLogits(0, a, [])
    ids = g.Decode(9, GREEDY, stop_on_eos=True)
    assert list(g.CacheLengths())[0] == len(a) and ids.shape[1] >= 1
    tail = M.tokens(cfg, 4, 3)
    assert M.rel(g.SlotLogits(0, tail, range(4)), orc.forward(a + tail)[-4:]) < M.TOL["float32"]
    snap.close()
    g.SetPerSequenceState(False)
    g.close()


# ---- generation --------------------------------------------------------------------------------------------------------------------
def greedy(orc, prompt, n):
    """Oracle continuation and the smallest margin between the best two logits on the way."""
    ids, margin = list(prompt), np.inf
    for _ in range(n):
        z = orc.forward(ids)[-1]
        top = np.sort(z)[-2:]
        margin = min(margin, float((top[1] - top[0]) / z.std()))
        ids.append(int(z.argmax()))
        if ids[-1] == 0:
            break
    return ids[len(prompt):], margin


@pytest.mark.parametrize("name", ["mixed", "odd", "plain"])
def test_scheduler_generates_what_the_oracle_does(cuda, name):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 13)
    orc = M.oracle(cfg, w)
    reqs = [Request(i, M.tokens(cfg, n, i), k) for i, (n, k) in enumerate([(3, 9), (1, 12), (25, 4), (8, 8), (2, 2), (40, 6), (5, 10)])]
    g = engine(cfg, w, "float32", max_batch=3, max_tokens=64)
    pool = KvCachePool()
    got = ContinuousBatcher(g, GREEDY, slots=3, max_tokens=64, chunk=3, pool=pool).run(reqs)
    for r in reqs:
        want, margin = greedy(orc, r.tokens, r.max_new)
        assert list(got[r.rid]) == want or margin < 1e-4, (r.rid, list(got[r.rid]), want, margin)
    # a request that starts with a parked text goes on from its cache and convolution state
    first = next(r for r in reqs if len(got[r.rid]) and got[r.rid][-1] != 0 and len(r.tokens) + len(got[r.rid]) < 50)
    follow = first.tokens + [int(t) for t in got[first.rid]] + [7, 9]
    b = ContinuousBatcher(g, GREEDY, slots=3, max_tokens=64, pool=pool)
    out = b.run([Request("f", follow, 6)])["f"]
    want, margin = greedy(orc, follow, 6)
    assert b.stats["pool_hits"] == 1 and (list(out) == want or margin < 1e-4)
    pool.clear()
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda, dtype):
    """Hundreds of steps of the captured token loop; the text it wrote, read again as a prompt and by the oracle, gives its logits."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 14)
    g = engine(cfg, w, dtype, max_batch=2, max_tokens=400)
    opts = DecodingOptions(DecodingStrategy=DS.GreedySearch, BlockedTokens=[0])
    prompts = [M.tokens(cfg, 5, 1), M.tokens(cfg, 5, 2)]
    first = g.Prefill(prompts, opts)
    ids = g.Decode(330, opts)
    text = [p + [int(f)] + [int(t) for t in i] for p, f, i in zip(prompts, first, ids)]
    last = g.Logits(want_probs=False)[0]
    want = [M.oracle(cfg, w).forward(t[:-1])[-1] for t in text]
    assert M.rel(last, want) < M.TOL[dtype]
    for b in range(2):
        assert M.rel(score(g, text[b][:-1], slot=b)[-1:], want[b:b + 1]) < M.TOL[dtype]
    g.close()


def test_generation_entry_points(cuda):
    """RunForwardOnSingleDevice, the KV pool, Top-P sampling and beam search run on a layered engine as on any other."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 15)
    g = engine(cfg, w, "float32", max_batch=6, max_tokens=96)
    orc = M.oracle(cfg, w)
    p = M.tokens(cfg, 12, 5)
    opts = DecodingOptions(MaxTgtSentLength=30, BlockedTokens=[0])
    ids = g.RunForwardOnSingleDevice([p, p], opts)
    assert (ids[0] == ids[1]).all() and ids.shape == (2, 18)
    z = orc.forward(p + [int(t) for t in ids[0][:-1]])
    for k, t in enumerate(ids[0]):
        row = z[len(p) - 1 + k].copy()
        row[0] = -np.inf
        assert row[int(t)] >= row.max() - 1e-4 * z.std()
    pool = KvCachePool()
    a = generate_with_pool(g, pool, p, opts)
    assert list(a) == list(ids[0])
    b = generate_with_pool(g, pool, p + [int(t) for t in a] + [3], DecodingOptions(MaxTgtSentLength=36, BlockedTokens=[0]))
    z = orc.forward(p + [int(t) for t in a] + [3])[-1]
    assert pool.hits == 1 and len(b) == 5 and z[int(b[0])] >= z[1:].max() - 1e-4 * z.std()
    pool.clear()
    s = DecodingOptions(MaxTgtSentLength=30, TopP=0.98, Temperature=20.0, DecodingStrategy=DS.Sampling, Seed=3, BlockedTokens=[0])
    x, y = g.RunForwardOnSingleDevice([p, p], s), g.RunForwardOnSingleDevice([p, p], s)
    assert (x == y).all() and not (x[0] == x[1]).all()
    # every hypothesis' score is what the oracle gives its text: the caches of the copied sequences are whole
    beam = g.BeamSearch([p], DecodingOptions(MaxTgtSentLength=20, BeamSearchSize=3))
    assert len(beam.ids) == 3 and beam.copies > 0
    for hyp, score_ in zip(beam.ids, beam.scores):
        z = orc.forward(p + [int(t) for t in hyp[0][:-1]])[len(p) - 1:]
        lp = z - z.max(1, keepdims=True)
        lp = lp - np.log(np.exp(lp).sum(1, keepdims=True))
        assert abs(1.0 - sum(lp[k][t] for k, t in enumerate(hyp[0])) - score_[0]) < 1e-3
    g.CheckGuards()
    g.close()


def test_command_line_and_model_folder(cuda, tmp_path, monkeypatch, capsys):
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 16)
    path = M.save(tmp_path / "model", cfg, w)
    from seq2seqsharp_b200 import cli
    prompts = [M.tokens(cfg, n, n) for n in (4, 19, 7)]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(" ".join(map(str, p)) for p in prompts) + "\n"))
    assert cli.main(["generate", "--model", path, "--dtype", "float32", "--max-new", "7", "--slots", "2"]) == 0
    lines = [[int(t) for t in line.split()] for line in capsys.readouterr().out.strip().splitlines()]
    orc = M.oracle(cfg, w)
    for p, got in zip(prompts, lines):
        want, margin = greedy(orc, p, 7)
        assert got == want or margin < 1e-4
    # the trace runner on the same folder
    from seq2seqsharp_b200 import trace
    steps = ['{"step": 0, "entries": [{"id": "q", "tokens": %s, "want": [0, 3]}], "end": []}' % prompts[1][:4],
             '{"step": 1, "entries": [{"id": "q", "tokens": %s, "want": [0]}], "end": []}' % prompts[1][4:5],
             '{"step": 2, "entries": [{"id": "q", "tokens": %s, "want": []}], "end": ["q"]}' % prompts[1][5:9],
             '{"step": 3, "entries": [{"id": "z", "tokens": %s, "want": [6]}], "end": ["z"]}' % prompts[2]]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(steps) + "\n"))
    assert trace.main(["--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
    full = orc.forward(prompts[1])
    for k, rows in ((0, full[[0, 3]]), (1, full[[4]]), (3, orc.forward(prompts[2])[[6]])):
        got = np.fromfile(str(tmp_path / ("%d.f32" % k)), "<f4").reshape(-1, cfg["vocab"])
        assert M.rel(got, rows) < M.TOL["float32"]
    assert not (tmp_path / "2.f32").exists()


def test_scoring_works_for_uniform_models_too(cuda):
    """SlotLogits on a GPTDecoder engine: the last place equals what SlotExtend leaves in the logits buffer."""
    from seq2seqsharp_b200.gpt import GPT, GPTConfig, synthetic_weights
    for dtype in ("float32", "float16"):
        cfg = GPTConfig(L=2, d=128, H=4, hd=32, F=256, V=211, dtype=dtype)
        g = GPT(cfg, max_batch=2, max_tokens=64)
        g.LoadWeights(synthetic_weights(cfg, 4, std=0.08, bias_std=0.02))
        ids = [int(t) for t in np.random.default_rng(0).integers(1, 211, size=20)]
        g.SlotReset(0)
        g.SlotExtend(0, ids, GREEDY)
        want = g.Logits(want_probs=False)[0][0]
        g.SlotReset(0)
        got = g.SlotLogits(0, ids[:12], [3, 11])
        got2 = g.SlotLogits(0, ids[12:], [7])
        assert M.rel(got2, want[None]) < (1e-5 if dtype == "float32" else 2e-2) and got.shape == (2, 211)
        g.CheckGuards()
        g.close()


def test_errors_leave_the_engine_usable(cuda):
    cfg = M.CONFIGS["plain"]
    w = M.weights(cfg, 17)
    c = config_from_json(cfg, "float32")
    g = LayeredGPT(c, max_batch=1, max_tokens=24)
    from seq2seqsharp_b200._native import TSB200Error
    names = {engine_name(k): v for k, v in w.items()}
    held = names.pop("layer.0.attn.uv")
    g.LoadWeights(names)
    g.SlotReset(0)
    with pytest.raises(TSB200Error, match="attn.uv"):
        g.SlotLogits(0, [1, 2], [0])
    with pytest.raises(TSB200Error, match="expects"):
        g.SetWeight("layer.0.attn.uv", held.T)
    bad = names["layer.0.experts.table"].copy()
    bad[3, 0] = 2
    with pytest.raises(TSB200Error, match="expert"):
        g.SetWeight("layer.0.experts.table", bad)
    g.SetWeight("layer.0.attn.uv", held)
    ids = M.tokens(cfg, 24)
    with pytest.raises(TSB200Error, match="OOM"):
        g.SlotLogits(0, ids + [1], [0])
    with pytest.raises(TSB200Error, match="outside the portion"):
        g.SlotLogits(0, ids, [24])
    with pytest.raises(TSB200Error, match="out of range"):
        g.SlotLogits(0, [cfg["vocab"]], [0])
    g.Reset()
    assert M.rel(score(g, ids), M.oracle(cfg, w).forward(ids)) < M.TOL["float32"]     # the cache to its last row
    g.close()


def test_synthetic_fill_runs(cuda):
    g = LayeredGPT(config_from_json(M.CONFIGS["wide"], "bfloat16"), max_batch=2, max_tokens=64)
    g.FillSynthetic(5, 0.05, 0.1)
    g.Prefill([M.tokens(M.CONFIGS["wide"], 20, 1)] * 2, GREEDY)
    ids = g.Decode(4, GREEDY)
    assert (ids[0] == ids[1]).all() and np.isfinite(g.Logits(want_probs=False)[0]).all() and g.StepBytes(2, 24) > 0
    assert sum(n for _, n in g.ProfileDecode(2, GREEDY).values()) > 0
    g.close()
