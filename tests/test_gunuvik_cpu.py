"""CPU tests of the design Gunuvik: the oracle's mechanisms one by one, what the GPU tests' comparisons are sensitive to, configuration and
tensor names, the registry, and what the engine refuses before it touches a device."""
import copy
import ctypes as C
import math

import numpy as np
import pytest

from oracle import gunuvik_oracle as GO
from seq2seqsharp_b200 import _native as N
from seq2seqsharp_b200 import gunuvik, registry
from seq2seqsharp_b200.layered import GroupedAttention, MatrixMemory, synthetic_layered_weights
from tests import gunuvik_models as M


# ---- the oracle's mechanisms -------------------------------------------------------------------------------------------------
def test_distance_buckets_are_single_then_logarithmic():
    b = [GO.distance_bucket(n, 8, 64) for n in range(80)]
    assert b[:4] == [0, 1, 2, 3] and b[4] == 4 and b[63] == 7 and b[79] == 7
    assert b[4:9] == [4, 4, 4, 4, 5] and b[15:17] == [5, 6] and b[31:33] == [6, 7]     # powers of two open a new row: 4 * 2^k
    assert all(x <= y for x, y in zip(b, b[1:]))
    t = np.arange(16.0).reshape(8, 2)
    bias = GO.distance_bias(10, t, 64)
    assert bias[0, 9, 9] == 0 and bias[1, 9, 0] == t[5, 1] and bias[0, 7, 4] == t[3, 0]


def test_window_keeps_the_first_tokens():
    m = GO.window_mask(9, 3, 2)
    assert m[8].tolist() == [True, True, False, False, False, False, True, True, True]
    assert m[2].tolist() == [True, True, True] + [False] * 6 and m[0].sum() == 1
    assert GO.window_mask(4, 1, 0).sum() == 4 and GO.window_mask(6, 2, 5)[5].sum() == 6


def test_sink_joins_the_denominator_only():
    z = np.array([[0.0, 1.0, -np.inf]])
    p = GO.softmax_with_sink(z, 2.0)
    e = np.exp([0.0, 1.0, 2.0])
    assert np.allclose(p[0, :2], e[:2] / e.sum()) and p[0, 2] == 0
    assert np.allclose(GO.softmax_with_sink(z, -1e9)[0, :2], e[:2] / e[:2].sum())
    assert np.allclose(GO.softmax_with_sink(z + 900.0, 902.0), p)


def test_matrix_memory_equals_its_sum_over_the_past():
    rng = np.random.default_rng(1)
    S, dim, vdim = 9, 3, 4
    q, k, v = rng.normal(size=(S, dim)), rng.normal(size=(S, dim)), rng.normal(size=(S, vdim))
    i, f = rng.normal(size=S) * 3, -np.abs(rng.normal(size=S))
    got = GO.matrix_memory(q, k, v, i, f)
    for t in range(S):
        m = 0.0
        for s in range(t + 1):
            m = max(f[s] + m, i[s])
        wts = np.array([math.exp(i[s] + f[s + 1:t + 1].sum() - m) for s in range(t + 1)])
        num, n = (wts * (k[:t + 1] @ q[t])) @ v[:t + 1], wts @ k[:t + 1]
        assert np.allclose(got[t], num / (max(abs(n @ q[t]), math.exp(-m)) + 1e-6))


def test_grouped_heads_gate_and_shared_keys():
    cfg = M.config([M.attention(4, 2, 6, 4, 5, 1)], 12, 20)
    w = M.weights(cfg, 3)
    mw = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
    h = np.random.default_rng(0).normal(size=(7, 12))
    m = cfg["layers"][0]["mixer"]
    k, v = GO.attention_keys(h, m, mw, 1e-5)
    base = GO.attention(h, m, mw, k, v, 1e-5)
    v2 = v.copy()
    v2[:, 1] = 0.0                                    # the second key/value head serves heads 2 and 3
    shut = dict(mw, g=mw["g"].copy())
    mo = mw["o"].copy()
    mo[:, 8:] = 0.0
    assert np.allclose(GO.attention(h, m, dict(mw, o=mo), k, v2, 1e-5), GO.attention(h, m, dict(mw, o=mo), k, v, 1e-5))
    assert not np.allclose(GO.attention(h, m, mw, k, v2, 1e-5), base)
    shut["g"][:] = 0.0
    half = GO.attention(h, m, shut, k, v, 1e-5)
    gate = GO.sigmoid(h @ mw["g"].T)
    assert not np.allclose(half, base) and gate.shape == (7, 4)
    assert np.allclose(np.sqrt(np.mean((k / mw["k.norm"]) ** 2, axis=-1)), 1.0, atol=1e-3)


def test_a_mistake_in_a_mechanism_shows_in_the_logits(monkeypatch):
    """What the GPU tests compare with is sensitive: each planted mistake moves the logits far beyond their tolerance."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 3)
    ids = M.tokens(cfg, 60)
    want = M.oracle(cfg, w).forward(ids)

    def moved(c=cfg, ww=w):
        return M.rel(M.oracle(c, ww).forward(ids), want)

    bound = 500 * M.TOL["float32"]
    for layer, key in ((0, "size"), (1, "size"), (3, "size"), (0, "keep_first"), (1, "keep_first")):
        c = copy.deepcopy(cfg)
        c["layers"][layer]["mixer"]["mask"][key] += 1
        assert moved(c) > 50 * M.TOL["float32"], (layer, key)
    for i, name in ((0, "bias_max"), (2, "gate_cap"), (0, "scale")):
        c = copy.deepcopy(cfg)
        c["layers"][i]["mixer"][name] *= 0.7
        assert moved(c) > 50 * M.TOL["float32"], name
    for name in ("l0.mix.sink", "l0.mix.g", "l0.mix.rel", "l0.ls1", "l0.ls2", "l0.norm1b", "l1.mix.q.norm", "l2.mix.norm", "l2.mix.f.b", "l2.mix.i.b", "l0.mix.v.b"):
        assert moved(ww=dict(w, **{name: np.zeros_like(w[name]) + 0.1})) > bound, name
    real = GO.matrix_memory
    monkeypatch.setattr(GO, "matrix_memory", lambda q, k, v, i, f: np.concatenate([real(q[:30], k[:30], v[:30], i[:30], f[:30]),
                                                                                   real(q[30:], k[30:], v[30:], i[30:], f[30:])]))
    assert moved() > bound                                 # the state is lost half way


@pytest.mark.parametrize("window,keep", [(16, 4), (9, 0), (5, 12)])
def test_the_marker_decides_at_the_edges(window, keep):
    """The inputs of the edge tests: whether the marker is inside or outside changes the logits a lot."""
    for at in (keep, max(0, keep - 1), 20):
        cfg, w, ids = M.needle(at, 48, window, keep)
        orc = M.oracle(cfg, w)
        want = orc.forward(ids)
        wide, narrow = copy.deepcopy(cfg), copy.deepcopy(cfg)
        wide["layers"][0]["mixer"]["mask"]["size"] += 1
        last_in, first_out = at + window - 1, at + window
        if at >= keep and first_out < len(ids):
            assert M.rel(M.oracle(wide, w).forward(ids)[first_out:first_out + 1], want[first_out:first_out + 1]) > 0.15
            if window > 1:
                narrow["layers"][0]["mixer"]["mask"]["size"] -= 1
                assert M.rel(M.oracle(narrow, w).forward(ids)[last_in:last_in + 1], want[last_in:last_in + 1]) > 0.15
        kept = copy.deepcopy(cfg)
        kept["layers"][0]["mixer"]["mask"]["keep_first"] += 1 if at == keep else (-1 if at == keep - 1 else 0)
        if kept != cfg:
            assert M.rel(M.oracle(kept, w).forward(ids)[-1:], want[-1:]) > 0.15


# ---- configuration, names, registry -----------------------------------------------------------------------------------------
def test_config_reader_takes_every_value_from_the_file():
    c = M.layered(M.CONFIGS["mixed"])
    assert (c.d, c.V, c.L, c.embed_scale, c.eps, c.block, c.tied_head) == (96, 101, 6, 2.5, 1e-5, "sandwich", False)
    assert c.layers[1].mixer == GroupedAttention(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.4, window=33, keep_first=5, bias_rows=12, bias_max=25, qk_norm=True,
                                                 qkv_bias=True, sink=True, head_gate=True, kv_from=0)
    assert c.layers[2].mixer == MatrixMemory(heads=3, dim=16, vdim=24, gate_cap=9.0)
    assert [x.dense.ff if x.dense else 0 for x in c.layers] == [40, 0, 56, 24, 0, 72]
    s = c.weight_shapes()
    assert "layer.1.attn.k" not in s and "layer.1.norm2" not in s and s["layer.0.attn.k"] == (32, 96) and s["layer.3.attn.bias"] == (6, 4)
    assert s["layer.2.mem.gate"] == (72, 96) and s["head"] == (101, 96) and c.active_matmul_params() > 0


def test_config_reader_refuses_what_it_does_not_know():
    for edit in (lambda c: c.update(logit_scale=5), lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0]["mixer"].update(rot={}),
                 lambda c: c["layers"][0]["mlp"].update(kind="moe"), lambda c: c.update(architecture="Other"), lambda c: c["layers"][2]["mixer"].update(conv=4),
                 lambda c: c["layers"][0]["mixer"]["mask"].update(chunk=4), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)):
        c = copy.deepcopy(M.CONFIGS["mixed"])
        edit(c)
        with pytest.raises(ValueError):
            M.layered(c, rows=M.REL_ROWS["mixed"])
    with pytest.raises(ValueError, match="mix.rel"):
        gunuvik.config_from_json(M.CONFIGS["mixed"])


def test_tensor_names_map_one_to_one():
    for cfg in M.CONFIGS.values():
        c = M.layered(cfg)
        names = gunuvik.file_names(c)
        assert set(names) == set(c.weight_shapes())
        assert {gunuvik.engine_name(n, c): n for n in names.values()} == names
        assert set(synthetic_layered_weights(c, 1)) == set(names)
    c = M.layered(M.CONFIGS["mixed"])
    for bad in ("l0.mix.foo", "lm_head", "l0.mix.i", "l2.mix.rel", "l9.norm1", "x0.norm1"):
        with pytest.raises(KeyError):
            gunuvik.engine_name(bad, c)


def test_registry_reads_table_sizes_from_the_file(tmp_path, capsys):
    cfg = M.CONFIGS["odd"]
    w = M.weights(cfg)
    path = M.save(tmp_path / "m", cfg, w)
    arch, c = registry.read_config(path, "float32")
    assert arch is registry.ARCHITECTURES["Gunuvik"] and [x.mixer.bias_rows for x in (c.layers[0], c.layers[2])] == [5, 7]
    from seq2seqsharp_b200 import cli
    assert cli.main(["info", "--model", path]) == 0
    assert "Gunuvik: 3 layers, width 50" in capsys.readouterr().out
    del w["l1.mix.f"]
    M.save(path, cfg, w)
    with pytest.raises(ValueError, match="mem.f"):
        registry.load_model(path)


# ---- what the engine refuses before it needs a device -----------------------------------------------------------------------
def _create(cfg_edit=None, layer_edit=None, n=3):
    c = N.LayeredConfigC()
    c.L, c.d, c.V, c.dtype, c.norm_groups, c.conv_taps, c.max_batch, c.max_tokens = n, 32, 50, N.F32, 1, 1, 1, 16
    c.eps = c.embed_scale = c.logit_scale = 1.0
    c.block = N.BLOCK_SANDWICH
    ls = (N.LayerDescC * n)()
    for i, t in enumerate(ls):
        t.mixer, t.heads, t.kv_heads, t.dim, t.vdim, t.kv_from, t.scale, t.window, t.bias_rows, t.bias_max = N.MIXER_GROUPED, 4, 2, 8, 8, -1, 1.0, 4, 4, 9
    ls[1].mixer, ls[1].gate_cap = N.MIXER_MEMORY, 2.0
    if cfg_edit:
        cfg_edit(c)
    if layer_edit:
        layer_edit(ls)
    h = C.c_void_p()
    ok = N.lib().TSB200_GptCreateLayered(C.byref(c), ls, C.byref(h))
    if ok:
        N.lib().TSB200_GptDestroy(h)
    return ok, N.last_error()


def test_engine_refuses_inconsistent_layers(native):
    def put(i, **kw):
        def edit(ls):
            for k, v in kw.items():
                setattr(ls[i], k, v)
        return edit

    for edit, word in ((put(0, mixer=N.MIXER_LATENT), "unknown mixer"), (put(0, kv_heads=3), "do not share"), (put(2, kv_from=1), "earlier layer"), (put(0, kv_from=2), "earlier layer"),
                       (put(2, kv_from=0, dim=16), "differ in the key/value heads"), (put(1, gate_cap=0.0), "gate cap"), (put(0, bias_max=2), "distance bias"),
                       (put(0, window=-1), "window"), (put(0, experts=2), "bad sizes")):
        ok, msg = _create(layer_edit=edit)
        assert not ok and word in msg, msg

    def groups(c):
        c.norm_groups = 2

    def block(c):
        c.block = 7

    for edit, word in ((groups, "norm group"), (block, "kind of block")):
        ok, msg = _create(cfg_edit=edit)
        assert not ok and word in msg, msg
