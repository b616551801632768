"""The design Gunuvik on the GPU against the plain oracle: mechanisms alone, prompts, token-by-token decoding, portions, unequal batches,
slots that are used again, keys at the edges of windows and among the first tokens, chunk edges of the memories, long decoding, snapshots and
beams, the slot scheduler and the command line."""
import io

import numpy as np
import pytest

from seq2seqsharp_b200.gpt import DecodingOptions, DecodingStrategyEnums as DS, KvCachePool, generate_with_pool
from seq2seqsharp_b200.layered import LayeredGPT
from seq2seqsharp_b200.scheduler import ContinuousBatcher, Request
from tests import gunuvik_models as M

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
GREEDY = DecodingOptions(DecodingStrategy=DS.GreedySearch)


def engine(cfg, w, dtype, max_batch=1, max_tokens=512, rows=None):
    g = LayeredGPT(M.layered(cfg, dtype, rows), max_batch=max_batch, max_tokens=max_tokens)
    g.LoadWeights(M.engine_weights(cfg, w, rows))
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


def decoded(g, ids, start):
    """Logits from position start - 1 on: a prompt of `start` tokens, then token by token through the captured step."""
    g.Reset()
    rows = [g.SlotLogits(0, ids[:start], [start - 1])[0]]
    for t in ids[start:]:
        g.StepHost([t], GREEDY)
        rows.append(g.Logits(want_probs=False)[0][0])
    return np.array(rows)


# ---- each mechanism alone -------------------------------------------------------------------------------------------------------
NEUTRAL = {"mix.rel": 0.0, "mix.sink": -60.0, "mix.g": 0.0, "mix.q.b": 0.0, "mix.k.b": 0.0, "mix.v.b": 0.0, "mix.q.norm": 1.0, "mix.k.norm": 1.0, "ls1": 1.0,
           "norm1b": 1.0, "ls2": 1.0, "norm2b": 1.0}
KEEP = {"plain": (), "bias": ("mix.rel",), "sink": ("mix.sink",), "gate": ("mix.g",), "qkv_bias": ("mix.q.b", "mix.k.b", "mix.v.b"), "qk_norm": ("mix.q.norm", "mix.k.norm"),
        "post_norm": ("norm1b", "norm2b"), "layer_scale": ("ls1", "ls2")}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("keep", list(KEEP))
def test_attention_mechanism_alone(cuda, keep, dtype):
    """One layer in which everything but the named mechanism is made neutral by its weights."""
    cfg = M.config([M.attention(4, 2, 16, 24, 11, 3, far=30, ff=40 if keep in ("post_norm", "layer_scale") else None)], 48, 67)
    w = M.weights(cfg, 5)
    for n, v in NEUTRAL.items():
        if n not in KEEP[keep] and "l0." + n in w:
            w["l0." + n] = np.full_like(w["l0." + n], v)
    ids = M.tokens(cfg, 50)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype)
    assert want.worst(score(g, ids)) < 1
    assert want.worst(decoded(g, ids, 2), slice(1, None)) < 1
    g.CheckGuards()
    g.close()


# gates: (input bias, forget bias); the state keeps, forgets at once, saturates the cap, or hardly takes anything in
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ib,fb,cap", [(0.0, 3.0, 12.0), (0.0, 8.0, 12.0), (0.0, -8.0, 12.0), (40.0, 40.0, 5.0), (-30.0, 5.0, 15.0), (9.0, -30.0, 20.0), (0.0, 1.0, 0.5)])
def test_memory_alone(cuda, ib, fb, cap, dtype):
    cfg = M.config([M.memory(3, 16, 24, cap=cap)], 48, 67)
    w = M.weights(cfg, 6)
    w["l0.mix.i.b"][:] = ib
    w["l0.mix.f.b"][:] = fb
    ids = M.tokens(cfg, 300)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype)
    assert want.worst(score(g, ids)) < 1
    for cuts in ([127, 2, 33, 2], [128, 128], [129, 40], [2] * 20 + [64], [31, 32, 33, 34], [1, 1, 1]):
        assert want.worst(score(g, ids, cuts=cuts)) < 1, cuts
    assert want.worst(decoded(g, ids[:160], 1), slice(0, 160)) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(1, 8, 8), (2, 24, 40), (4, 64, 64), (2, 128, 256), (1, 256, 512), (2, 72, 136), (3, 9, 14), (2, 264, 16), (5, 16, 4), (1, 300, 7)])
def test_memory_sizes(cuda, heads, dim, vdim, dtype):
    cfg = M.config([M.memory(heads, dim, vdim)], 64, 50)
    w = M.weights(cfg, 7)
    ids = M.tokens(cfg, 200)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype, max_batch=2)
    assert want.worst(score(g, ids)) < 1
    assert want.worst(score(g, ids, slot=1, cuts=[70, 3, 64, 1])) < 1
    assert want.worst(decoded(g, ids, 150), slice(149, None)) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 4, 32, 32), (8, 1, 32, 48), (3, 1, 64, 40), (10, 2, 80, 64), (20, 1, 32, 32), (40, 2, 16, 8), (70, 1, 8, 8), (4, 2, 96, 128),
                                                      (2, 1, 192, 64), (2, 2, 64, 192), (2, 1, 256, 256), (16, 1, 256, 32), (2, 1, 264, 16), (6, 3, 10, 7), (5, 5, 12, 6)])
def test_attention_sizes(cuda, heads, kv_heads, dim, vdim, dtype):
    """Every tile size, heads that do not fill a tile, groups larger than a tile, sizes that only the CUDA-core kernel takes."""
    cfg = M.config([M.attention(heads, kv_heads, dim, vdim, 50, 5, far=70), M.attention(heads, kv_heads, dim, vdim, 90, 9, far=130, kv_from=0)], 64, 50)
    w = M.weights(cfg, 8)
    ids = M.tokens(cfg, 160)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype)
    assert want.worst(score(g, ids)) < 1
    assert want.worst(score(g, ids, cuts=[40, 3, 2, 64, 1])) < 1
    assert want.worst(decoded(g, ids, 30), slice(29, None)) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,eps,embed", [(48, 1e-6, 1.0), (50, 0.5, 7.0), (129, 1e-3, 1.5), (1000, 1e-6, 3.0), (2048, 1e-6, 1.0), (4096, 1e-5, 2.0), (2560, 1e-5, 1.0)])
def test_widths_and_scales(cuda, width, eps, embed, dtype):
    cfg = M.config([M.attention(2, 1, 8, 8, 6, 1, ff=24), M.memory(2, 8, 8, ff=16)], width, 40, eps=eps, embed=embed)
    w = M.weights(cfg, 9)
    ids = M.tokens(cfg, 14)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype)
    assert want.worst(score(g, ids)) < 1
    assert want.worst(score(g, ids, cuts=[1] * 14)) < 1
    g.close()


# ---- whole prompts, decoding, portions ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_prompt_decode_and_portions_match_the_oracle(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 7)
    ids = M.tokens(cfg, 260 if name == "wide" else 70)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype, max_batch=2)
    assert want.worst(score(g, ids)) < 1
    for cuts in ([2] * 60, [3, 2, 17, 2, 9], [1, 2, 3, 4, 5], [7] * 30, [20, 100], [16, 17, 2], [64, 2, 63, 65]):
        assert want.worst(score(g, ids, cuts=cuts)) < 1, cuts
    for start in (1, 2, 41):
        assert want.worst(decoded(g, ids, start), slice(start - 1, None)) < 1, start
    # places out of order and more than once; an empty list
    g.Reset()
    got = g.SlotLogits(0, ids[:8], [7, 0, 7])
    assert want.worst(got, [7, 0, 7]) < 1
    assert g.SlotLogits(0, ids[8:10], []).shape == (0, cfg["vocab"])
    assert want.worst(g.SlotLogits(0, ids[10:12], [1]), 11) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_in_large_and_small_portions(cuda, dtype):
    """Several tiles of keys, queries and rows and several memory chunks; portion borders inside and at the edges of both."""
    cfg = M.CONFIGS["wide"]
    w = M.weights(cfg, 8)
    ids = M.tokens(cfg, 700)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype, max_tokens=800)
    for cuts in (None, [256, 100], [63, 65, 1, 127, 2], [128, 128, 128], [129, 2, 2, 200]):
        assert want.worst(score(g, ids, cuts=cuts)) < 1, cuts
    assert want.worst(decoded(g, ids, 640), slice(639, None)) < 1
    g.CheckGuards()
    g.close()


# ---- keys at the edges of a window, among the first tokens, far away --------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(16, 4), (1, 3), (64, 0), (65, 17), (5, 70), (130, 1)])
def test_one_key_among_many(cuda, window, keep, dtype):
    n = max(2 * window, keep) + 40
    for at in sorted(x for x in {0, max(0, keep - 1), keep, keep + 1, 15, 16, 63, 64, n // 3} if x < n - 14):
        cfg, w, ids = M.needle(at, n, window, keep, layers=2)
        want = M.Expected(cfg, w, ids, dtype)
        g = engine(cfg, w, dtype)
        edge = at + window
        assert want.worst(score(g, ids)) < 1, at
        for cuts in ([at + 1, 2, 2, 37, 64], [max(at, 1), 1, 1, 3], [max(1, min(edge, n - 3)), 2], [max(1, min(edge - 1, n - 3)), 2, 2], [max(1, min(edge - 2, n - 3)), 2, 3]):
            assert want.worst(score(g, ids, cuts=cuts)) < 1, (at, cuts)
        start = max(1, min(edge - 3, n - 12))
        assert want.worst(decoded(g, ids[:min(n, start + 12)], start), slice(start - 1, start + 12)) < 1, at
        assert want.worst(decoded(g, ids[:at + 14], at + 1), slice(at, at + 14)) < 1, at
        g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_kept_keys_over_many_splits(cuda, dtype):
    """A first token that is kept while a long window, cut into several splits, passes over the decoded tokens."""
    cfg, w, ids = M.needle(2, 900, 600, 3, heads=8, kv_heads=1, dim=64, vdim=64)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype, max_tokens=1000)
    assert want.worst(score(g, ids)) < 1
    assert want.worst(decoded(g, ids, 860), slice(859, None)) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_cache_of_another_layer_seen_through_a_wider_window(cuda, dtype):
    """The reading layer looks further back than the layer that owns the cache."""
    cfg = M.config([M.attention(4, 2, 16, 16, 3, 0, ff=48), M.attention(4, 2, 16, 16, 80, 2, kv_from=0, ff=32), M.attention(4, 2, 16, 16, 2, 30, kv_from=0)], 64, 50)
    w = M.weights(cfg, 10)
    ids = M.tokens(cfg, 130)
    want = M.Expected(cfg, w, ids, dtype)
    g = engine(cfg, w, dtype)
    assert want.worst(score(g, ids, cuts=[50, 2, 30])) < 1
    assert want.worst(decoded(g, ids, 60), slice(59, None)) < 1
    g.close()


# ---- batches, slots ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batch_matches_each_alone(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 10)
    lens = [1, 2, 3, 29, 17, 140]
    texts = [M.Expected(cfg, w, M.tokens(cfg, n + 6, i), dtype) for i, n in enumerate(lens)]
    g = engine(cfg, w, dtype, max_batch=6, max_tokens=200)
    g.PrefillRagged([t.ids[:n] for t, n in zip(texts, lens)], GREEDY)
    # every sequence goes on with tokens of its own choosing
    for step in range(7):
        if step:
            g.StepHost([t.ids[n + step - 1] for t, n in zip(texts, lens)], GREEDY)
        got = g.Logits(want_probs=False)[0]
        for z, t, n in zip(got, texts, lens):
            assert t.worst(z, n + step - 1) < 1, (n, step)
    # equal lengths in one prefill, and more text on top
    g.Reset()
    same = [M.Expected(cfg, w, M.tokens(cfg, 87, 90 + i), dtype) for i in range(6)]
    g.Prefill([t.ids[:50] for t in same], GREEDY)
    for z, t in zip(g.Logits(want_probs=False)[0], same):
        assert t.worst(z, 49) < 1
    g.Extend([t.ids[50:] for t in same], GREEDY)
    for z, t in zip(g.Logits(want_probs=False)[0], same):
        assert t.worst(z, 86) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("rows", [20, 70])
def test_more_sequences_than_a_row_tile(cuda, rows):
    """Row counts that every form of the linears serves."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 10)
    texts = [M.Expected(cfg, w, M.tokens(cfg, 2 + (7 * i) % 23, i), "bfloat16") for i in range(rows)]
    g = engine(cfg, w, "bfloat16", max_batch=rows, max_tokens=64)
    g.PrefillRagged([t.ids[:-1] for t in texts], GREEDY)
    g.StepHost([t.ids[-1] for t in texts], GREEDY)
    for z, t in zip(g.Logits(want_probs=False)[0], texts):
        assert t.worst(z, -1) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_slots_used_again_and_neighbours_undisturbed(cuda, name, dtype):
    cfg = M.CONFIGS[name]
    w = M.weights(cfg, 11)
    g = engine(cfg, w, dtype, max_batch=3, max_tokens=160)
    ea, eb = M.Expected(cfg, w, M.tokens(cfg, 90, 1), dtype), M.Expected(cfg, w, M.tokens(cfg, 73, 2), dtype)
    a, b = ea.ids, eb.ids
    g.SlotReset(0)
    g.SlotLogits(0, a[:60], [])
    g.SlotReset(1)
    g.SlotLogits(1, M.tokens(cfg, 120, 3), [])
    g.SlotReset(1)                                     # a long request leaves, a short one takes its place
    assert eb.worst(g.SlotLogits(1, b[:1], [0]), 0) < 1
    assert eb.worst(g.SlotLogits(1, b[1:20], range(19)), slice(1, 20)) < 1
    assert ea.worst(g.SlotLogits(0, a[60:], range(30)), slice(60, None)) < 1
    # park, run something else in the slot, come back: the memories travel with the cache
    snap = g.SlotSnapshot(1)
    g.SlotReset(1)
    g.SlotLogits(1, M.tokens(cfg, 50, 4), [])
    g.SlotRestore(snap, 1)
    assert eb.worst(g.SlotLogits(1, b[20:22], [0, 1]), slice(20, 22)) < 1
    g.SlotRestore(snap, 2)
    assert eb.worst(g.SlotLogits(2, b[20:], range(53)), slice(20, None)) < 1
    snap.close()
    # a slot whose first portion is long enough for the chunk kernels, after another text
    g.SlotReset(1)
    assert eb.worst(g.SlotLogits(1, b, range(73))) < 1
    g.CheckGuards()
    g.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_that_stand_still_keep_their_state(cuda, dtype):
    """A finished sequence is stepped with the others at its own position; what it holds must not change."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 12)
    g = engine(cfg, w, dtype, max_batch=2, max_tokens=128)
    g.SetPerSequenceState(True)
    a, b = M.tokens(cfg, 11, 1), M.tokens(cfg, 20, 2)
    for s, t in ((0, a), (1, b)):
        g.SlotReset(s)
        g.SlotExtend(s, t, GREEDY)
    # the pending id of slot 0 becomes </s>: it stands still from now on
    g.SlotReset(0)
    g.SlotLogits(0, a, [])
    ids = g.Decode(9, GREEDY, stop_on_eos=True)
    assert list(g.CacheLengths())[0] == len(a) and ids.shape[1] >= 1
    tail = M.tokens(cfg, 4, 3)
    assert M.Expected(cfg, w, a + tail, dtype).worst(g.SlotLogits(0, tail, range(4)), slice(-4, None)) < 1
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
    # a request that starts with a parked text goes on from its cache and memories
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
    for b in range(2):
        want = M.Expected(cfg, w, text[b][:-1], dtype)
        assert want.worst(last[b], -1) < 1
        assert want.worst(score(g, text[b][:-1], slot=b)) < 1
    g.close()


def test_generation_entry_points(cuda):
    """RunForwardOnSingleDevice, the KV pool, Top-P sampling and beam search run as on any other model."""
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
    # every hypothesis' score is what the oracle gives its text: the caches and memories of the copied sequences are whole
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
    from seq2seqsharp_b200 import cli, trace
    prompts = [M.tokens(cfg, n, n) for n in (4, 19, 7)]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(" ".join(map(str, p)) for p in prompts) + "\n"))
    assert cli.main(["generate", "--model", path, "--dtype", "float32", "--max-new", "7", "--slots", "2"]) == 0
    lines = [[int(t) for t in line.split()] for line in capsys.readouterr().out.strip().splitlines()]
    orc = M.oracle(cfg, w)
    for p, got in zip(prompts, lines):
        want, margin = greedy(orc, p, 7)
        assert got == want or margin < 1e-4
    # the trace runner on the same folder: two live requests, then one alone
    steps = ['{"step": 0, "entries": [{"id": "q", "tokens": %s, "want": [0, 3]}, {"id": "r", "tokens": %s, "want": [3]}], "end": []}' % (prompts[1][:4], prompts[0]),
             '{"step": 1, "entries": [{"id": "q", "tokens": %s, "want": [0]}], "end": ["r"]}' % prompts[1][4:5],
             '{"step": 2, "entries": [{"id": "q", "tokens": %s, "want": []}], "end": ["q"]}' % prompts[1][5:9],
             '{"step": 3, "entries": [{"id": "z", "tokens": %s, "want": [5]}], "end": []}' % prompts[2][:6],
             '{"step": 4, "entries": [{"id": "z", "tokens": %s, "want": [0]}], "end": ["z"]}' % prompts[2][6:]]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(steps) + "\n"))
    assert trace.main(["--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2", "done", "3", "done", "4"]
    full, last = orc.forward(prompts[1]), orc.forward(prompts[2])
    for k, rows in ((0, np.stack([full[0], full[3], orc.forward(prompts[0])[3]])), (1, full[[4]]), (3, last[[5]]), (4, last[[6]])):
        got = np.fromfile(str(tmp_path / ("%d.f32" % k)), "<f4").reshape(-1, cfg["vocab"])
        assert M.rel(got, rows) < M.TOL["float32"]
    assert not (tmp_path / "2.f32").exists()


def test_errors_leave_the_engine_usable(cuda):
    cfg = M.CONFIGS["plain"]
    w = M.weights(cfg, 17)
    from seq2seqsharp_b200._native import TSB200Error
    g = LayeredGPT(M.layered(cfg), max_batch=1, max_tokens=24)
    names = M.engine_weights(cfg, w)
    held = names.pop("layer.1.mem.v")
    g.LoadWeights(names)
    g.SlotReset(0)
    with pytest.raises(TSB200Error, match="mem.v"):
        g.SlotLogits(0, [1, 2], [0])
    with pytest.raises(TSB200Error, match="expects"):
        g.SetWeight("layer.1.mem.v", held.T)
    with pytest.raises(TSB200Error, match="unknown weight"):
        g.SetWeight("layer.0.mem.v", held)
    g.SetWeight("layer.1.mem.v", held)
    ids = M.tokens(cfg, 24)
    with pytest.raises(TSB200Error, match="OOM"):
        g.SlotLogits(0, ids + [1], [0])
    g.Reset()
    assert M.Expected(cfg, w, ids, "float32").worst(score(g, ids)) < 1     # the cache to its last row
    g.close()


def test_synthetic_fill_runs(cuda):
    g = LayeredGPT(M.layered(M.CONFIGS["wide"], "bfloat16"), max_batch=2, max_tokens=64)
    g.FillSynthetic(5, 0.05, 0.1)
    g.Prefill([M.tokens(M.CONFIGS["wide"], 20, 1)] * 2, GREEDY)
    ids = g.Decode(4, GREEDY)
    assert (ids[0] == ids[1]).all() and np.isfinite(g.Logits(want_probs=False)[0]).all() and g.StepBytes(2, 24) > 0
    prof = g.ProfileDecode(2, GREEDY)
    assert prof["memory"][1] == 4 and prof["attention"][1] == 6
    g.close()
