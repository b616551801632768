"""CPU tests of the layered models: the oracle's mechanisms one by one, configuration and tensor names, the file reader, the registry,
the command line's `info`, the trace replay's slot bookkeeping, and what the engine refuses before it touches a device."""
import copy
import ctypes as C
import json

import numpy as np
import pytest

from oracle import latent_oracle as LO
from seq2seqsharp_b200 import _native as N
from seq2seqsharp_b200 import pepilix, registry
from seq2seqsharp_b200.safetensors_file import SafetensorsFile, to_bfloat16, to_float32, write_safetensors
from seq2seqsharp_b200.trace import TraceReplay
from tests import layered_models as M


# ---- the oracle's mechanisms -------------------------------------------------------------------------------------------------
def test_group_norm_parts_are_independent():
    rng = np.random.default_rng(0)
    x, w = rng.normal(size=(3, 12)), rng.normal(size=12)
    y = LO.group_rms(x, w, 3, 1e-5)
    for g in range(3):
        s = slice(4 * g, 4 * g + 4)
        assert np.allclose(y[:, s], LO.rms(x[:, s], w[s], 1e-5))
    x2 = x.copy()
    x2[:, :4] *= 10
    assert np.allclose(LO.group_rms(x2, w, 3, 1e-5)[:, 4:], y[:, 4:])
    assert np.allclose(LO.group_rms(x, w, 1, 1e-5), LO.rms(x, w, 1e-5))
    assert abs(float(LO.rms(np.full((1, 4), 2.0), np.ones(4), 12.0)[0, 0]) - 2.0 / 4.0) < 1e-12     # eps is inside the root


def test_short_conv_is_causal_and_newest_tap_is_last():
    h = np.arange(1.0, 6.0)[:, None]
    assert np.allclose(LO.short_conv(h, np.array([[0.0, 0.0, 1.0]]))[:, 0], h[:, 0])
    assert np.allclose(LO.short_conv(h, np.array([[1.0, 0.0, 0.0]]))[:, 0], [0, 0, 1, 2, 3])
    assert np.allclose(LO.short_conv(h, np.array([[0.0, 10.0, 1.0]]))[:, 0], [1, 12, 23, 34, 45])


def test_rotation_pairs_halves_and_scores_depend_on_distance():
    rng = np.random.default_rng(1)
    x = np.zeros((1, 6))
    x[0, 0] = 1.0
    y = LO.rotate_half(x, [1], 6, 100.0)
    assert np.isclose(y[0, 0], np.cos(1.0)) and np.isclose(y[0, 3], np.sin(1.0)) and np.allclose(y[0, [1, 2, 4, 5]], 0)
    z = np.zeros((1, 6))
    z[0, 1] = 1.0
    assert np.isclose(LO.rotate_half(z, [2], 6, 100.0)[0, 4], np.sin(2.0 * 100.0 ** (-2 / 6)))
    q, k = rng.normal(size=8), rng.normal(size=8)
    dot = [LO.rotate_half(q[None], [p + 5], 8, 1e4)[0] @ LO.rotate_half(k[None], [p], 8, 1e4)[0] for p in (0, 3, 77)]
    assert np.allclose(dot, dot[0])
    assert np.allclose(LO.rotate_half(q[None], [9], 4, 1e4)[0, 4:], q[4:])      # dimensions beyond `dims` pass


def test_latent_attention_equals_attention_over_its_keys_and_values():
    """Absorbing W_uk into the query and W_uv into the output gives the same result."""
    rng = np.random.default_rng(2)
    m = {"heads": 2, "dim": 4, "rot_dim": 2, "vdim": 3, "kv_rank": 5, "scale": 0.7, "rot": {"base": 50.0, "dims": 2}}
    S, d = 6, 8
    h = rng.normal(size=(S, d))
    w = {"q": rng.normal(size=(12, d)), "uk": rng.normal(size=(8, 5)), "uv": rng.normal(size=(6, 5)), "o": rng.normal(size=(d, 6))}
    c, kr = LO.latent_keys(h, rng.normal(size=(7, d)), np.ones(5), 5, 2, 50.0, 1e-6)
    got = LO.latent_attention(h, m, w, c, kr)
    q = (h @ w["q"].T).reshape(S, 2, 6)
    out = np.zeros((S, 6))
    for a in range(2):
        ql = q[:, a, :4] @ w["uk"][4 * a:4 * a + 4]
        qr = LO.rotate_half(q[:, a, 4:], range(S), 2, 50.0)
        for s in range(S):
            p = LO.softmax((c[:s + 1] @ ql[s] + kr[:s + 1] @ qr[s]) * 0.7)
            out[s, 3 * a:3 * a + 3] = w["uv"][3 * a:3 * a + 3] @ (p @ c[:s + 1])
    assert np.allclose(got, out @ w["o"].T)


def test_experts_follow_the_table_and_clamp():
    one = {"gate": np.array([[1.0]]), "up": np.array([[1.0]]), "down": np.array([[1.0]])}
    two = {k: v * (3.0 if k == "down" else 1.0) for k, v in one.items()}
    table = np.array([[0], [1]])
    h = np.array([[5.0], [5.0]])
    y = LO.table_experts(h, [0, 1], table, [one, two], 2.0)
    a = 2.0 / (1 + np.exp(-1.702 * 2.0)) * 3.0            # gate and up are cut to 2
    assert np.allclose(y[:, 0], [a, 3 * a])
    low = LO.clamped_expert(np.array([[-5.0]]), one["gate"], one["up"], one["down"], 2.0)
    assert np.allclose(low, -5.0 / (1 + np.exp(1.702 * 5.0)) * (-2.0 + 1.0))     # the gate has no lower bound
    both = LO.table_experts(h[:1], [0], np.array([[0, 1]]), [one, two], 2.0)
    assert np.allclose(both[0, 0], 2 * a)                 # mean of a and 3 a


def test_a_mistake_in_a_mechanism_shows_in_the_logits(monkeypatch):
    """What the GPU tests compare with is sensitive: each planted mistake moves the logits far beyond their tolerance."""
    cfg = M.CONFIGS["mixed"]
    w = M.weights(cfg, 3)
    ids = M.tokens(cfg, 40)
    want = M.oracle(cfg, w).forward(ids)

    def moved(c=cfg, ww=w):
        return M.rel(M.oracle(c, ww).forward(ids), want)

    for edit in (lambda c: c["norm"].update(groups=1), lambda c: c["layers"][3]["mixer"].update(kv_from=None),
                 lambda c: c["layers"][0]["mixer"]["rot"].update(base=9000.0), lambda c: c["layers"][2]["mlp"]["expert"].update(limit=0.7)):
        c = copy.deepcopy(cfg)
        edit(c)
        ww = w
        if c["layers"][3]["mixer"].get("kv_from", 0) is None:
            ww = dict(w, **{"l3.mix.dkv": w["l2.mix.dkv"], "l3.mix.dkv.norm": w["l2.mix.dkv.norm"]})
        assert moved(c, ww) > 20 * M.TOL["float32"]
    shifted = dict(w, **{"l1.canon1": np.roll(w["l1.canon1"], 1, axis=1)})
    assert moved(ww=shifted) > 0.1
    real = LO.softmax
    monkeypatch.setattr(LO, "softmax", lambda z: real(np.concatenate([z[:1], np.where(np.arange(z.shape[1])[None] == 0, -np.inf, z[1:])])))
    assert moved() > 1e-3                                  # the first token is left out
    monkeypatch.setattr(LO, "softmax", real)


# ---- configuration, names, files, registry --------------------------------------------------------------------------------
def test_config_reader_takes_every_value_from_the_file():
    c = pepilix.config_from_json(M.CONFIGS["mixed"], "float32")
    assert (c.d, c.V, c.L, c.norm_groups, c.conv_taps) == (96, 101, 4, 3, 3)
    assert (c.embed_scale, c.logit_scale, c.eps, c.dtype) == (2.5, 0.7, 1e-5, "float32")
    assert [x.mixer.kv_from for x in c.layers] == [-1, 0, -1, 2] and c.layers[1].experts is None
    assert c.layers[3].experts.top == 3 and c.layers[2].experts.limit == 0.6 and c.layers[2].mixer.rot_base == 500.0
    s = c.weight_shapes()
    assert "layer.1.attn.dkv" not in s and "layer.1.norm2" not in s and s["layer.3.experts.6.down"] == (96, 16)
    assert s["layer.2.attn.q"] == (5 * 24, 96) and s["layer.0.experts.table"] == (101, 2)


def test_config_reader_refuses_what_it_does_not_know():
    for edit in (lambda c: c.update(window=5), lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0]["mixer"].update(window=3),
                 lambda c: c["layers"][0]["mlp"].update(kind="dense"), lambda c: c.update(architecture="Other")):
        c = copy.deepcopy(M.CONFIGS["mixed"])
        edit(c)
        with pytest.raises(ValueError):
            pepilix.config_from_json(c)


def test_tensor_names_map_one_to_one():
    for cfg in M.CONFIGS.values():
        c = pepilix.config_from_json(cfg)
        names = pepilix.file_names(c)
        assert set(names) == set(c.weight_shapes())
        assert {pepilix.engine_name(n): n for n in names.values()} == names
    for bad in ("l0.mix.foo", "lm_head", "l0.mlp.e0.bias", "x0.norm1"):
        with pytest.raises(KeyError):
            pepilix.engine_name(bad)


def test_bfloat16_conversion_rounds_to_nearest_even():
    v = np.array([1.0, 1.00390625, 1.01171875, -2.5, 3.0e-3, 0.0], dtype=np.float32)
    back = to_float32(to_bfloat16(v))
    assert np.array_equal(back[[0, 3, 5]], v[[0, 3, 5]])
    assert back[1] == 1.0 and back[2] == np.float32(1.015625)      # ties go to the even pattern
    import torch
    r = np.random.default_rng(0).normal(size=1000).astype(np.float32)
    assert np.array_equal(to_float32(to_bfloat16(r)), torch.from_numpy(r).to(torch.bfloat16).float().numpy())


def test_safetensors_roundtrip_and_damage(tmp_path):
    p = str(tmp_path / "a.safetensors")
    t = {"a": np.arange(6, dtype=np.float32).reshape(2, 3), "b": np.array([[1], [2]], dtype=np.int32), "c": to_bfloat16(np.ones((3, 1)))}
    write_safetensors(p, t)
    f = SafetensorsFile(p)
    assert f.names() == ["a", "b", "c"] and f.shape("a") == (2, 3) and "c" in f
    for k, v in f.items():
        assert np.array_equal(v, t[k]) and v.dtype == t[k].dtype
    raw = open(p, "rb").read()
    for damaged in (raw[:4], raw[:-1], b"\xff" * 8 + raw[8:]):
        open(p, "wb").write(damaged)
        with pytest.raises(ValueError):
            SafetensorsFile(p)


def test_registry_finds_the_architecture_and_missing_tensors(tmp_path, capsys):
    cfg = M.CONFIGS["plain"]
    w = M.weights(cfg)
    path = M.save(tmp_path / "m", cfg, w)
    arch, c = registry.read_config(path)
    assert c.d == 64 and arch is registry.ARCHITECTURES["Pepilix"]
    from seq2seqsharp_b200 import cli
    assert cli.main(["info", "--model", path]) == 0
    assert "1 layers, width 64" in capsys.readouterr().out
    del w["l0.mix.uk"]
    M.save(path, cfg, w)
    with pytest.raises(ValueError, match="attn.uk"):
        registry.load_model(path)
    json.dump({"architecture": "nobody"}, open(path + "/config.json", "w"))
    with pytest.raises(ValueError, match="nobody"):
        registry.read_config(path)


# ---- trace replay on a fake engine ---------------------------------------------------------------------------------------------
class FakeEngine:
    """Logits = what the sequence has seen so far, so that a lost or mixed-up slot shows."""
    max_batch = 3

    class cfg:
        V = 2

    def __init__(self):
        self.slots, self.calls = {}, []

    def Reset(self):
        self.slots = {}

    def Batch(self):
        return len(self.slots)

    def SlotReset(self, s):
        assert s <= len(self.slots)
        self.slots[s] = []

    def SlotLogits(self, s, toks, want):
        self.calls.append(("portion", len(toks)))
        base = list(self.slots[s])
        self.slots[s] = base + list(toks)
        return np.array([[len(base) + w + 1, sum((base + list(toks))[:len(base) + w + 1])] for w in want], dtype=np.float32).reshape(-1, 2)

    def StepHost(self, ids, opts):
        self.calls.append(("step", 1))
        self.slots[0].append(int(ids[0]))

    def Logits(self, want_probs=False):
        return np.array([[len(self.slots[0]), sum(self.slots[0])]], dtype=np.float32), None


def test_replay_keeps_requests_apart_and_gives_slots_back():
    e = FakeEngine()
    r = TraceReplay(e)
    out = r.step([{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}], [])
    assert out.tolist() == [[1, 1], [3, 6]]
    assert r.step([{"id": "a", "tokens": [4], "want": [0]}], []).tolist() == [[4, 10]] and e.calls[-1][0] == "step"
    assert r.step([{"id": "b", "tokens": [7], "want": [0]}, {"id": "a", "tokens": [1], "want": [0]}], ["a"]).tolist() == [[1, 7], [5, 11]]
    assert e.calls[-1][0] == "portion"                   # two live requests: not the step of the whole batch
    assert r.step([{"id": "c", "tokens": [5, 5], "want": [1]}], ["b", "c"]).tolist() == [[2, 10]] and not e.slots
    assert r.step([{"id": "a", "tokens": [9], "want": []}], []).shape == (0, 2)
    for i in range(2):
        r.step([{"id": "x%d" % i, "tokens": [1, 1], "want": []}], [])
    with pytest.raises(ValueError):
        r.step([{"id": "y", "tokens": [1], "want": []}], [])


# ---- what the engine refuses before it needs a device -----------------------------------------------------------------------
def _create(cfg_edit=None, layer_edit=None, n=2):
    c = N.LayeredConfigC()
    c.L, c.d, c.V, c.dtype, c.norm_groups, c.conv_taps, c.max_batch, c.max_tokens = n, 32, 50, N.F32, 2, 2, 1, 16
    c.eps = c.embed_scale = c.logit_scale = 1.0
    c.tied_head = 1
    ls = (N.LayerDescC * n)()
    for t in ls:
        t.heads, t.dim, t.rot_dim, t.rot_dims, t.vdim, t.kv_rank, t.kv_from, t.scale, t.rot_base = 2, 8, 4, 4, 8, 16, -1, 1.0, 100.0
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
    def own(ls):
        ls[1].kv_from = 1

    def differs(ls):
        ls[1].kv_from, ls[1].kv_rank = 0, 8

    def odd(ls):
        ls[0].rot_dims = 3

    def many(ls):
        ls[0].experts, ls[0].top, ls[0].ff = 2, 3, 8

    for edit, word in ((own, "earlier layer"), (differs, "differ in the latent"), (odd, "rotation"), (many, "per token")):
        ok, msg = _create(layer_edit=edit)
        assert not ok and word in msg, msg

    def groups(c):
        c.norm_groups = 5

    def half(c):
        c.dtype = N.F16

    for edit, word in ((groups, "norm groups"), (half, "dtype")):
        ok, msg = _create(cfg_edit=edit)
        assert not ok and word in msg, msg
