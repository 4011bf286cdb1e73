"""Host-side parts of the Gimozen design: configuration, tensor names, the oracle's mechanisms."""
import copy

import numpy as np
import pytest

from oracle import gimozen_oracle as go
from tests import gimozen_models as gm
from turbospark_b200 import gimozen, plain, registry


# ---- configuration
def test_every_size_and_constant_comes_from_the_configuration():
    cfg = gm.config(72, 31, [gm.latent(6, 20, 8, 12, 44, 40, scale=0.3, base=700.0, scaling={"factor": 8.0, "original": 64, "fast": 5.0, "slow": 2.0}),
                             gm.attention(4, 2, 12, 28, None, scale=0.7, temp=(0.25, 9)), gm.latent(3, 16, 8, 20, 44, 16, base=700.0,
                             scaling={"factor": 8.0, "original": 64, "fast": 5.0, "slow": 2.0}, kv_from=0)], eps=3e-4, alpha=1.25, embed=6.0)
    pc, (a, b, c) = gimozen.parse_config(cfg, max_context=99, compute=plain.F32)
    assert (pc.n_layers, pc.d_model, pc.vocab, pc.max_context, pc.compute, pc.post_norm) == (3, 72, 31, 99, plain.F32, 1)
    assert abs(pc.norm_eps - 3e-4) < 1e-9 and pc.residual_scale == 1.25 and pc.embed_scale == 6.0 and pc.logit_cap == 0.0
    assert (a.n_q_heads, a.head_dim, a.rot_dim, a.value_dim, a.kv_rank, a.ffn, a.kv_source) == (6, 20, 8, 12, 44, 40, 0)
    assert (a.rot_base, a.rot_factor, a.rot_original, a.rot_fast, a.rot_slow) == (700.0, 8.0, 64.0, 5.0, 2.0)
    assert abs(a.score_scale - 0.3) < 1e-7 and a.sink and a.value_gate and not a.qk_norm and a.act == plain.SILU
    assert (b.n_q_heads, b.n_kv_heads, b.head_dim, b.value_dim, b.ffn, b.kv_rank, b.q_temp_every) == (4, 2, 12, 28, 0, 0, 9)
    assert abs(b.score_scale - 0.7) < 1e-7 and b.q_temp_coef == 0.25 and b.qk_norm and not b.sink and not b.value_gate
    assert (c.n_q_heads, c.head_dim, c.value_dim, c.kv_source) == (3, 16, 20, 1)
    for l in gimozen.parse_config(gm.CONFIGS["borrow"], 64)[1][1:2]:
        assert l.rot_factor == 0.0  # unscaled


def _latent_layer(c):
    return c["layers"][0]["mixer"]


@pytest.mark.parametrize("break_it", [
    lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c.pop("postln_alpha"), lambda c: c["embedding"].pop("scale"),
    lambda c: c["layers"][0].pop("mlp"), lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="routed"),
    lambda c: _latent_layer(c).pop("kv_rank"), lambda c: _latent_layer(c)["rot"].update(dims=4), lambda c: _latent_layer(c)["rot"]["scaling"].pop("fast"),
    lambda c: _latent_layer(c)["rot"]["scaling"].update(factor=0.0), lambda c: c["layers"][1]["mixer"].pop("kv_heads"),
    lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=2.5),
    lambda c: c["layers"][2]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=-1), lambda c: c["layers"][2]["mixer"].update(kv_from=1),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=80), lambda c: c["layers"][2]["mixer"]["rot"].update(base=10.0)])
def test_a_configuration_that_says_something_else_is_refused(break_it):
    cfg = copy.deepcopy(gm.CONFIGS["odd"])
    break_it(cfg)
    with pytest.raises(ValueError):
        gimozen.parse_config(cfg, 64)


def test_a_latent_is_borrowed_from_a_layer_that_has_one():
    cfg = copy.deepcopy(gm.CONFIGS["borrow"])
    gimozen.parse_config(cfg, 64)
    cfg["layers"][4]["mixer"]["kv_from"] = 3  # itself a borrower
    with pytest.raises(ValueError, match="kv_from"):
        gimozen.parse_config(cfg, 64)


def test_the_registry_knows_the_design():
    assert registry.ARCHITECTURES[gimozen.ARCHITECTURE] is gimozen.build


@pytest.mark.parametrize("name", list(gm.CONFIGS))
def test_loading_asks_for_exactly_the_tensors_of_the_design(name):
    class Fake:
        def __init__(self, layers):
            self.layers, self.got = layers, {}

        def set(self, which, array, layer=-1):
            assert (layer, which) not in self.got
            self.got[(layer, which)] = array

    cfg = gm.CONFIGS[name]
    w = gm.random_weights(cfg, 0)
    asked = []
    gimozen.load_tensors(Fake(gimozen.parse_config(cfg, 64)[1]), lambda n: (asked.append(n), w[n])[1])
    assert sorted(asked) == sorted(w)


# ---- the oracle's mechanisms, each on numbers worked out by hand or by another route
def test_oracle_norms():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(go.rms_norm(x, np.array([2.0, 10.0]), 12.5), [[6.0 / 5.0, 8.0]])
    assert np.allclose(go.rms_norm_zero_centred(x, np.array([0.0, -1.0]), 12.5), [[3.0 / 5.0, 0.0]])


def test_oracle_rotation_keeps_lengths_and_relative_angles():
    rot = {"dims": 6, "base": 50.0}
    rng = np.random.default_rng(0)
    x = rng.standard_normal((1, 2, 9))
    a, b = go.rotate(x, [4], rot), go.rotate(x, [0], rot)
    assert np.allclose(b, x) and np.allclose(a[..., 6:], x[..., 6:]) and np.allclose((a ** 2).sum(-1), (x ** 2).sum(-1))
    # pair (i, i + 3) as a complex number is multiplied by e^(i p f)
    z = (x[..., :3] + 1j * x[..., 3:6]) * np.exp(1j * 4 * 50.0 ** (-np.arange(3) / 3))
    assert np.allclose(a[..., :3], z.real) and np.allclose(a[..., 3:6], z.imag)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    dot = lambda p, r: float((go.rotate(q, [p], rot) * go.rotate(k, [r], rot)).sum())
    assert abs(dot(9, 5) - dot(104, 100)) < 1e-9 and abs(dot(9, 5) - dot(9, 6)) > 1e-3


def test_oracle_scaled_frequencies_go_from_the_unscaled_to_the_divided_ones():
    s = {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}
    f, g = go.rotary_frequencies(64, 10000.0), go.rotary_frequencies(64, 10000.0, s)
    turns = f * 2048 / (2 * np.pi)
    assert np.allclose(g[turns > 45], f[turns > 45]) and np.allclose(g[turns < 0.7], f[turns < 0.7] / 4)
    between = (turns < 30) & (turns > 1.3)
    assert between.sum() > 4 and np.all(g[between] < f[between]) and np.all(g[between] > f[between] / 4) and np.all(np.diff(g) < 0)
    assert abs(go.rotary_magnitude(s) - (1 + 0.1 * np.log(4.0))) < 1e-12 and go.rotary_magnitude() == 1.0
    # both ends of the ramp on the same pair: a step
    h = go.rotary_frequencies(4, 10.0, {"factor": 2.0, "original": 1.0, "fast": 30.0, "slow": 30.0})
    assert np.allclose(h[1:], go.rotary_frequencies(4, 10.0)[1:] / 2)


def test_oracle_temperature_grows_at_multiples():
    t = go.query_temperature(np.array([0, 8, 9, 18, 19]), 0.5, 10)
    assert np.allclose(t, [1, 1, 1 + 0.5 * np.log(2), 1 + 0.5 * np.log(2), 1 + 0.5 * np.log(3)])


def test_oracle_attention_weights_follow_the_equations():
    rng = np.random.default_rng(3)
    q, k, v, sink = rng.standard_normal((5, 4, 6)), rng.standard_normal((7, 2, 6)), rng.standard_normal((7, 2, 3)), rng.uniform(-1, 3, 4)
    got, plain_ = go.causal_attention(q, k, v, 0.4, sink, first_query=2), go.causal_attention(q, k, v, 0.4, first_query=2)
    for i in range(5):
        for h in range(4):
            e = np.array([np.exp(0.4 * q[i, h] @ k[j, h // 2]) for j in range(i + 3)])
            num = sum(p * v[j, h // 2] for j, p in enumerate(e))
            assert np.allclose(got[i, h], num / (e.sum() + np.exp(sink[h]))) and np.allclose(plain_[i, h], num / e.sum())


def test_a_latent_row_serves_as_key_and_value_in_the_latents_space():
    """Scores and outputs through a head's own keys and values equal those of queries and sums taken to the latent and back."""
    rng = np.random.default_rng(4)
    H, D, R, E, K, n = 3, 5, 4, 6, 7, 9
    c, kr, q = rng.standard_normal((n, K)), rng.standard_normal((n, R)), rng.standard_normal((n, H, D + R))
    uk, uv, sink = rng.standard_normal((H, D, K)), rng.standard_normal((H, E, K)), rng.uniform(-1, 2, H)
    k = np.concatenate([np.einsum("hdk,nk->nhd", uk, c), np.broadcast_to(kr[:, None], (n, H, R))], axis=-1)
    want = go.causal_attention(q, k, np.einsum("hek,nk->nhe", uv, c), 0.3, sink)
    row = np.concatenate([c, kr], axis=-1)[:, None]
    absorbed = np.concatenate([np.einsum("hdk,nhd->nhk", uk, q[..., :D]), q[..., D:]], axis=-1)
    sums = go.causal_attention(absorbed, row, row[..., :K], 0.3, sink)
    assert np.allclose(np.einsum("hek,nhk->nhe", uv, sums), want)


def test_oracle_logits_do_not_see_the_future():
    cfg = gm.CONFIGS["odd"]
    w = gm.random_weights(cfg, 5)
    toks = np.arange(40) * 7 % cfg["vocab"]
    a = go.forward(w, cfg, toks)
    toks2 = toks.copy()
    toks2[30:] = 3
    assert np.allclose(a[:30], go.forward(w, cfg, toks2)[:30]) and not np.allclose(a[30:], go.forward(w, cfg, toks2)[30:])


def test_every_mechanism_shows_in_the_test_models_logits():
    """Each mechanism changed moves the logits by a hundred times what the f32 comparisons on the GPU allow (2e-5)."""
    cfg = gm.CONFIGS["odd"]
    w = gm.random_weights(cfg, 0)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=140)
    want = go.forward(w, cfg, toks)

    def moved(edit=None, zero=None, change=None):
        c, v = copy.deepcopy(cfg), dict(w)
        if edit:
            edit(c)
        if zero:
            v.update({k: np.zeros_like(x) for k, x in v.items() if k.endswith(zero)})
        if change:
            v.update(change(v))
        return gm.logit_error(go.forward(v, c, toks), want).max()

    def each(kind, f):
        return lambda c: [f(l["mixer"]) for l in c["layers"] if l["type"] == kind]

    least = 100 * 2e-5
    lat, att = "latent_attention", "attention"
    assert moved(lambda c: c.update(postln_alpha=1.72)) > least and moved(lambda c: c["embedding"].update(scale=2.6)) > least
    assert moved(lambda c: c["norm"].update(eps=3e-2)) > least
    for kind in (lat, att):
        assert moved(each(kind, lambda m: m.update(scale=m["scale"] * 1.05))) > least
    assert moved(each(lat, lambda m: m["rot"].update(base=5500.0))) > least and moved(each(lat, lambda m: m["rot"].pop("scaling"))) > least
    for key, value in (("factor", 3.2), ("original", 100), ("fast", 20.0), ("slow", 6.0)):
        assert moved(each(lat, lambda m: m["rot"].update(scaling=dict(m["rot"]["scaling"], **{key: value})))) > least, key
    assert moved(each(att, lambda m: m.pop("q_temp", None))) > least
    assert moved(each(att, lambda m: m.update(q_temp={"coef": 0.4, "every": 38}) if "q_temp" in m else None)) > least
    for zero in ("mix.sink", "mix.g", "norm1", "norm2", "final.norm", "mlp.up", "mix.uv", "mix.uk"):
        assert moved(zero=zero) > least, zero
    for one in ("q.norm", "k.norm", "dkv.norm"):
        assert moved(change=lambda v: {k: np.ones_like(x) for k, x in v.items() if k.endswith(one)}) > least, one
    # a layer that borrows reads the named layer's latent, not one of its own
    own = lambda v: {"l2.mix.dkv": np.roll(v["l0.mix.dkv"], 1, axis=0), "l2.mix.dkv.norm": v["l0.mix.dkv.norm"]}
    assert moved(edit=lambda c: c["layers"][2]["mixer"].pop("kv_from"), change=own) > least
