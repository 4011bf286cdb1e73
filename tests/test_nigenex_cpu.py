"""Host-side parts of the Nigenex design: configuration, files, the trace runner's bookkeeping, the oracle's mechanisms."""
import copy
import json

import numpy as np
import pytest

from oracle import nigenex_oracle as no
from tests import nigenex_models as nm
from turbospark_b200 import build, nigenex, plain, registry, safetensors, trace


# ---- configuration
def test_every_size_and_constant_comes_from_the_configuration():
    cfg = nm.config(72, 31, [nm.layer(6, 2, 20, 11, 40, scale=0.3, softcap=5.0), nm.layer(4, 4, 12, 3, None, scale=0.7, softcap=9.0)], eps=3e-4,
                    logit_softcap=17.0)
    pc, layers = nigenex.parse_config(cfg, max_context=99, compute=plain.F32)
    assert (pc.n_layers, pc.d_model, pc.vocab, pc.max_context, pc.compute) == (2, 72, 31, 99, plain.F32)
    assert abs(pc.norm_eps - 3e-4) < 1e-9 and pc.logit_cap == 17.0
    a, b = layers
    assert (a.n_q_heads, a.n_kv_heads, a.head_dim, a.window, a.ffn) == (6, 2, 20, 11, 40)
    assert (b.n_q_heads, b.n_kv_heads, b.head_dim, b.window, b.ffn) == (4, 4, 12, 3, 0)
    assert abs(a.score_scale - 0.3) < 1e-7 and a.score_cap == 5.0 and abs(b.score_scale - 0.7) < 1e-7 and b.score_cap == 9.0
    assert all(l.log_bias and l.head_gate and l.token_shift and l.act == plain.GELU_TANH for l in layers)


@pytest.mark.parametrize("break_it", [
    lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c.pop("logit_softcap"), lambda c: c["layers"][0].pop("mlp"),
    lambda c: c["layers"][0]["mixer"].pop("mask"), lambda c: c["layers"][0]["mixer"].update(vdim=7), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mlp"].update(kind="routed"), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)])
def test_a_configuration_that_says_something_else_is_refused(break_it):
    cfg = copy.deepcopy(nm.CONFIGS["odd"])
    break_it(cfg)
    with pytest.raises(ValueError):
        nigenex.parse_config(cfg, 64)


def test_the_registry_goes_by_the_architecture_name(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="Unknown"):
        registry.load(None, str(tmp_path), 64)
    assert nigenex.ARCHITECTURE in registry.ARCHITECTURES


def test_loading_asks_for_exactly_the_tensors_of_the_design():
    class Fake:
        def __init__(self, layers):
            self.layers, self.got = layers, {}

        def set(self, which, array, layer=-1):
            self.got[(layer, which)] = array

    cfg = nm.CONFIGS["mixed_layers"]
    w = nm.random_weights(cfg, 0)
    asked = []
    fake = Fake(nigenex.parse_config(cfg, 64)[1])
    nigenex.load_tensors(fake, lambda name: (asked.append(name), w[name])[1])
    assert sorted(asked) == sorted(w)
    assert fake.got[(1, plain.P_FF_DOWN)].shape == (128, 100) and (0, plain.P_FF_DOWN) not in fake.got


# ---- files
def test_safetensors_round_trip_and_malformed_files(tmp_path):
    p = str(tmp_path / "m.safetensors")
    rng = np.random.default_rng(0)
    # a scalar first, so that the following data start on an odd boundary
    t = {"s": np.array(plain.bf16_bits(np.float32(1.5))).reshape(()), "a": plain.bf16_bits(rng.standard_normal((3, 5))).reshape(3, 5),
         "f": rng.standard_normal((2, 4)).astype(np.float32), "i": np.arange(6, dtype=np.int32)}
    safetensors.write(p, t)
    f = safetensors.SafeTensors(p)
    assert f.names() == list(t) and f.dtype("a") == "BF16" and f.shape("s") == ()
    for k, v in t.items():
        assert np.array_equal(f.get(k), v)
    with pytest.raises(KeyError):
        f.get("absent")
    raw = open(p, "rb").read()
    (tmp_path / "short").write_bytes(raw[:-9])
    with pytest.raises(ValueError):
        safetensors.SafeTensors(str(tmp_path / "short")).get("i")
    (tmp_path / "none").write_bytes(b"\xff" * 16)
    with pytest.raises(ValueError):
        safetensors.SafeTensors(str(tmp_path / "none"))


def test_bf16_rounding_is_to_nearest_even():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.14159, 1e-20, 65504.0], dtype=np.float32)
    assert plain.bf16_to_f32(plain.bf16_bits(x))[1] == 1.0 and plain.bf16_to_f32(plain.bf16_bits(x))[2] == np.float32(1.015625)
    assert np.all(np.abs(plain.bf16_to_f32(plain.bf16_bits(x)) - x) <= np.abs(x) * 2.0 ** -8)


# ---- units of the library
def test_every_unit_belongs_to_one_family_or_to_all():
    everything = set(build._sources())
    blocks, plain_units = set(build._sources("blocks")), set(build._sources("plain"))
    assert blocks | plain_units == everything and build.FAMILY_UNITS["blocks"] <= everything and build.FAMILY_UNITS["plain"] <= everything
    assert not build.FAMILY_UNITS["blocks"] & plain_units and not build.FAMILY_UNITS["plain"] & blocks


# ---- trace replay
class FakeSession:
    """Logits that name the stream and the position they belong to."""
    n_streams = 2

    def __init__(self):
        self.at, self.resets = {}, []

    def step(self, entries):
        assert len({s for s, _, _ in entries}) == len(entries)
        rows = []
        for s, tokens, places in entries:
            assert list(places) == sorted(set(places))
            base = self.at.get(s, 0)
            rows += [[s, base + p, tokens[p]] for p in places]
            self.at[s] = base + len(tokens)
        return np.array(rows, dtype=np.float32).reshape(-1, 3)

    def reset(self, s):
        self.resets.append(s)
        self.at[s] = 0


def test_trace_replay_orders_rows_and_hands_streams_on(tmp_path):
    s, said = FakeSession(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [7, 8, 9], "want": [2, 0]}, {"id": "b", "tokens": [5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [6], "want": [0]}, {"id": "a", "tokens": [1], "want": [0, 0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [3, 4], "want": [1]}], "end": ["c", "b"]}]
    trace.replay(s, [json.dumps(x) for x in steps], str(tmp_path), said.append)
    assert said == [0, 1, 2]
    read = lambda n: np.fromfile(tmp_path / ("%d.f32" % n), dtype="<f4").reshape(-1, 3).tolist()
    assert read(0) == [[0, 2, 9], [0, 0, 7]]
    assert read(1) == [[1, 1, 6], [0, 3, 1], [0, 3, 1]]
    assert read(2) == [[0, 1, 4]] and s.resets == [0, 0, 1]  # the freed stream, from position 0 again
    s2 = FakeSession()
    over = {"step": 0, "entries": [{"id": str(i), "tokens": [1], "want": []} for i in range(3)]}
    with pytest.raises(RuntimeError, match="taken"):
        trace.replay(s2, [json.dumps(over)], str(tmp_path), said.append)


# ---- the oracle's mechanisms, each on numbers worked out by hand or by another route
def test_oracle_token_shift_and_norm():
    h = np.array([[1.0, 2.0], [3.0, 6.0]])
    assert np.allclose(no.token_shift(h, np.array([0.5, 0.25])), [[0.5, 1.5], [2.0, 5.0]])
    assert np.allclose(no.token_shift(h, np.array([0.5, 0.25]), previous=np.array([3.0, 2.0])), [[2.0, 2.0], [2.0, 5.0]])
    assert np.allclose(no.rms_norm_scalar(np.array([[3.0, 4.0]]), 2.0, 12.5), [[6.0 / 5.0, 8.0 / 5.0]])


def test_oracle_window_gate_cap_and_bias():
    m = no.window_mask(4, 4, 0, 2)
    assert m.tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert no.window_mask(1, 6, 5, 3).tolist() == [[0, 0, 0, 1, 1, 1]]
    assert np.allclose(no.soft_cap(np.array([0.0, 1e9, -1e9]), 5.0), [0.0, 5.0, -5.0])
    assert abs(no.log_distance_bias(2.0, 0.5, 4.0) - 2.0 * np.log(3.0)) < 1e-12
    # one visible key: the output is that key whatever the score; the gate halves it at 0
    q, k = np.full((1, 2, 3), 9.0), np.arange(3.0).reshape(1, 1, 3)
    o = no.attention(q, k, k, 1.0, 2.0, np.ones(2), np.ones(2), 5)
    assert np.allclose(o, np.arange(3.0)) and np.allclose(no.head_gate(o, np.zeros((1, 2))), np.arange(3.0) / 2)


def test_oracle_attention_weights_follow_the_equations():
    rng = np.random.default_rng(3)
    q, k = rng.standard_normal((5, 4, 6)), rng.standard_normal((5, 2, 6))
    r1, r2 = rng.uniform(0.1, 1, 4), rng.uniform(0.1, 1, 4)
    got = no.attention(q, k, k, 0.4, 3.0, r1, r2, 3)
    for i in range(5):
        for h in range(4):
            js = range(max(0, i - 2), i + 1)
            e = np.array([np.exp(3.0 * np.tanh(0.4 * q[i, h] @ k[j, h // 2] / 3.0)) / (1 + r2[h] * (i - j)) ** r1[h] for j in js])
            want = sum(p * k[j, h // 2] for p, j in zip(e / e.sum(), js))
            assert np.allclose(got[i, h], want)


def test_oracle_logits_do_not_see_the_future():
    cfg = nm.CONFIGS["one_kv"]
    w = nm.random_weights(cfg, 5)
    toks = np.arange(40) * 7 % cfg["vocab"]
    a = no.forward(w, cfg, toks)
    toks2 = toks.copy()
    toks2[30:] = 3
    assert np.allclose(a[:30], no.forward(w, cfg, toks2)[:30]) and not np.allclose(a[30:], no.forward(w, cfg, toks2)[30:])


def test_every_mechanism_shows_in_the_test_models_logits():
    """Each mechanism changed moves the logits by a hundred times what the f32 comparisons on the GPU allow (2e-5)."""
    cfg = nm.CONFIGS["odd"]
    w = nm.random_weights(cfg, 0)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=140)
    want = no.forward(w, cfg, toks)

    def moved(edit_layer=None, zero=None, **top):
        c, v = dict(copy.deepcopy(cfg), **top), dict(w)
        for l in c["layers"]:
            if edit_layer:
                edit_layer(l)
        if zero:
            v.update({k: np.zeros_like(x) for k, x in v.items() if k.endswith(zero)})
        return nm.logit_error(no.forward(v, c, toks), want).max()

    least = 100 * 2e-5
    assert moved(lambda l: l["mixer"]["mask"].update(size=36)) > least and moved(lambda l: l["mixer"]["mask"].update(size=38)) > least
    assert moved(lambda l: l["mixer"].update(softcap=1e6)) > least and moved(lambda l: l["mixer"].update(scale=l["mixer"]["scale"] * 1.05)) > least
    assert moved(norm={"eps": 2e-2}) > least and moved(logit_softcap=5.0) > least
    for zero in (".shift", ".r1", ".r2", "mix.g", "mlp.up"):
        assert moved(zero=zero) > least, zero
