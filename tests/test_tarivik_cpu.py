"""Host-side parts of the Tarivik design: configuration, tensor names, the oracle's mechanisms."""
import copy

import numpy as np
import pytest

from oracle import tarivik_oracle as to
from tests import tarivik_models as tm
from turbospark_b200 import plain, registry, tarivik


# ---- configuration
def test_every_size_and_constant_comes_from_the_configuration():
    cfg = tm.config(72, 31, [tm.parallel((6, 2, 12, 28, 19), (4, 2, 10, 14, 5, 3), tm.moe(24, 12, 3, 4, 2), scales=(0.3, 0.6), scale=0.7), tm.hgrn2(3, 16, 20, None),
                             tm.mlstm(5, 8, 12, tm.moe(9, 4, 2, 1, 1), cap=3.5)], groups=6, taps=5, eps=3e-4, positions=77)
    pc, (a, b, c) = tarivik.parse_config(cfg, max_context=99, compute=plain.F32)
    assert (pc.n_layers, pc.d_model, pc.vocab, pc.max_context, pc.compute, pc.output_norm, pc.post_norm) == (3, 72, 31, 77, plain.F32, 1, 0)
    assert abs(pc.norm_eps - 3e-4) < 1e-9 and (pc.norm_groups, pc.conv_taps, pc.positions) == (6, 5, 77)
    assert tarivik.parse_config(cfg, max_context=50)[0].max_context == 50
    assert (a.n_q_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.chunk, a.window) == (6, 2, 12, 28, 19, 0)
    assert abs(a.score_scale - 0.7) < 1e-7 and abs(a.attn_scale - 0.3) < 1e-7 and abs(a.rec_scale - 0.6) < 1e-7
    assert a.sink and a.value_gate and a.qkv_bias and a.linear_bias and a.qk_norm == plain.NORM_PROJECTION
    assert (a.recurrence, a.rec_heads, a.rec_groups, a.rec_vdim, a.rec_dim, a.rec_taps, a.rec_norm_groups) == (plain.REC_SSD, 4, 2, 10, 14, 5, 3)
    assert (a.ffn, a.experts, a.expert_top, a.expert_groups, a.expert_keep, a.act) == (24, 12, 3, 4, 2, plain.SILU)
    assert (b.n_q_heads, b.recurrence, b.rec_heads, b.rec_dim, b.rec_vdim, b.ffn, b.experts) == (0, plain.REC_FORGET, 3, 16, 20, 0, 0)
    assert (c.recurrence, c.rec_heads, c.rec_dim, c.rec_vdim, c.rec_cap, c.experts) == (plain.REC_MLSTM, 5, 8, 12, 3.5, 4)


@pytest.mark.parametrize("break_it", [
    lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c["norm"].pop("groups"), lambda c: c["canon"].pop("taps"), lambda c: c.pop("max_positions"),
    lambda c: c["layers"][0].pop("mlp"), lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mlp"]["router"].pop("top"), lambda c: c["layers"][0]["mlp"]["router"]["groups"].pop("keep"), lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"),
    lambda c: c["layers"][0]["mixer"].pop("left_scale"), lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"]["right"].pop("norm_groups"), lambda c: c["layers"][1]["mixer"].pop("dim"), lambda c: c["layers"][2]["mixer"].pop("gate_cap")])
def test_a_configuration_that_says_something_else_is_refused(break_it):
    cfg = copy.deepcopy(tm.CONFIGS["odd"])
    break_it(cfg)
    with pytest.raises(ValueError):
        tarivik.parse_config(cfg, 64)


def test_the_registry_knows_the_design():
    assert registry.ARCHITECTURES[tarivik.ARCHITECTURE] is tarivik.build


@pytest.mark.parametrize("name", list(tm.CONFIGS))
def test_loading_asks_for_exactly_the_tensors_of_the_design(name):
    class Fake:
        def __init__(self, cfg, layers):
            self.cfg, self.layers, self.got = cfg, layers, {}

        def set(self, which, array, layer=-1):
            assert (layer, which) not in self.got
            self.got[(layer, which)] = array

    cfg = tm.CONFIGS[name]
    w = tm.random_weights(cfg, 0)
    asked, model = [], Fake(*tarivik.parse_config(cfg, 64))
    tarivik.load_tensors(model, lambda n: (asked.append(n), w[n])[1])
    assert sorted(asked) == sorted(w)
    for i, l in enumerate(model.layers):  # the experts' matrices one after another
        if l.experts:
            assert np.array_equal(model.got[i, plain.P_FF_UP][l.ffn * (l.experts - 1):], w["l%d.mlp.e%d.up" % (i, l.experts - 1)])
            assert model.got[i, plain.P_FF_DOWN].shape == (l.experts * cfg["width"], l.ffn)


# ---- the oracle's mechanisms, each on numbers worked out by hand or by another route
def test_oracle_grouped_norm():
    x = np.array([[3.0, 4.0, 0.0, 2.0]])
    assert np.allclose(to.grouped_rms_norm(x, np.array([1.0, 2.0, 5.0, 3.0]), 2, 0.0), [[3 / 12.5 ** 0.5, 8 / 12.5 ** 0.5, 0.0, 6 / 2 ** 0.5]])
    assert np.allclose(to.grouped_rms_norm(x, np.ones(4), 1, 0.0), x / 7.25 ** 0.5) and np.allclose(to.grouped_rms_norm(x, np.ones(4), 4, 16.0)[0, :2], [0.6, 4 / 32 ** 0.5])


def test_oracle_convolution_ends_at_the_token_itself():
    h = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(to.short_conv(h, np.array([[3.0, 2.0, 1.0]])), [[1.0], [12.0], [123.0]])
    assert np.allclose(to.short_conv(h, np.array([[5.0]]), np.array([1.0])), [[6.0], [51.0], [501.0]])


def test_oracle_attention_weights_follow_the_equations():
    rng = np.random.default_rng(3)
    n, chunk = 11, 4
    q, k, v, sink = rng.standard_normal((n, 4, 6)), rng.standard_normal((n, 2, 6)), rng.standard_normal((n, 2, 3)), rng.uniform(-1, 3, 4)
    slopes = to.alibi_slopes(4)
    assert np.allclose(slopes, [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8]) and np.allclose(to.alibi_slopes(3)[0], 2.0 ** (-8 / 3))
    got = to.chunked_attention(q, k, v, 0.4, chunk, slopes, sink)
    for i in range(n):
        for h in range(4):
            seen = range(i - i % chunk, i + 1)
            e = np.array([np.exp(0.4 * q[i, h] @ k[j, h // 2] - slopes[h] * (i - j)) for j in seen])
            assert np.allclose(got[i, h], sum(p * v[j, h // 2] for p, j in zip(e, seen)) / (e.sum() + np.exp(sink[h])))


def test_oracle_recurrence_is_a_weighted_sum_of_the_past():
    rng = np.random.default_rng(4)
    n, H, D, E = 7, 2, 3, 4
    q, k, v, f = rng.standard_normal((n, H, D)), rng.standard_normal((n, H, D)), rng.standard_normal((n, H, E)), rng.uniform(0.2, 1, (n, H, D))
    got = to.decayed_outer_products(q, k, v, f)
    for t in range(n):
        for h in range(H):
            want = sum((q[t, h] * k[s, h] * np.prod(f[s + 1:t + 1, h], axis=0)).sum() * v[s, h] for s in range(t + 1))
            assert np.allclose(got[t, h], want)
    # carried over: the state of the first rows goes on
    S = np.zeros((H, D, E))
    for t in range(3):
        S = f[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
    assert np.allclose(to.decayed_outer_products(q[3:], k[3:], v[3:], f[3:], S), got[3:])


def test_oracle_mlstm_needs_no_maximum_where_nothing_overflows():
    """The same numbers without the running maximum: S, n decay with the plain forget gates, the floor is one."""
    rng = np.random.default_rng(5)
    m = {"heads": 2, "dim": 3, "vdim": 4, "gate_cap": 2.0}
    d, n = 6, 9
    w = {"q": rng.standard_normal((6, d)), "k": rng.standard_normal((6, d)), "v": rng.standard_normal((8, d)), "g": rng.standard_normal((8, d)), "o": rng.standard_normal((d, 8)),
         "norm": rng.uniform(0.5, 1.5, 8), "i": rng.standard_normal((2, d)), "i.b": rng.standard_normal(2), "f": rng.standard_normal((2, d)), "f.b": rng.standard_normal(2)}
    h = rng.standard_normal((n, d))
    i = 2 * np.tanh((h @ w["i"].T + w["i.b"]) / 2)
    f = 1 / (1 + np.exp(-2 * np.tanh((h @ w["f"].T + w["f.b"]) / 2)))
    q, k, v = (h @ w["q"].T).reshape(n, 2, 3) / 3 ** 0.5, (h @ w["k"].T).reshape(n, 2, 3), (h @ w["v"].T).reshape(n, 2, 4)
    ke = k * np.exp(i)[..., None]
    decay = np.broadcast_to(f[..., None], k.shape)
    o = to.decayed_outer_products(q, ke, v, decay)
    nq = to.decayed_outer_products(q, ke, np.ones((n, 2, 1)), decay)[..., 0]
    o = o / np.maximum(np.abs(nq), 1.0)[..., None]
    want = (to.rms(o, 1e-4).reshape(n, 8) * w["norm"] * to.sigmoid(h @ w["g"].T)) @ w["o"].T
    assert np.allclose(to.mlstm(w, "", m, h, 1e-4), want, rtol=1e-4)


def test_oracle_choice_of_experts():
    s = np.array([[0.9, 0.1, 0.5, 0.5, 0.8, 0.0]])
    # groups of two: worth 1.0, 1.0, 0.8; ties go to the lower index
    assert to.choose_experts(s, np.zeros(6), 3, 2, 2).tolist() == [[0, 2]]
    assert to.choose_experts(s, np.zeros(6), 1, 1, 3).tolist() == [[0, 4, 2]]
    # corrections move the choice, also below zero: an expert outside the groups that stay is worse than any
    assert to.choose_experts(s, np.array([-5.0, -5.0, 0, 0, -6.0, -6.0]), 3, 2, 4).tolist() == [[2, 3, 0, 1]]
    w = {"router": np.zeros((2, 3)), "correction": np.array([0.0, -1.0])}
    for e in range(2):
        w.update({"e%d.gate" % e: np.eye(1, 3), "e%d.up" % e: np.eye(1, 3), "e%d.down" % e: np.full((3, 1), e + 1.0)})
    m = {"router": {"experts": 2, "top": 1, "groups": {"count": 1, "keep": 1}}}
    h = np.array([[2.0, 0.0, 0.0]])
    assert np.allclose(to.mixture(w, "", m, h), 0.5 * to.silu(2.0) * 2.0)  # the score, not the choice, weighs; no renormalising


def test_oracle_logits_do_not_see_the_future():
    cfg = tm.CONFIGS["odd"]
    w = tm.random_weights(cfg, 5)
    toks = np.arange(40) * 7 % cfg["vocab"]
    a = to.forward(w, cfg, toks)
    toks2 = toks.copy()
    toks2[30:] = 3
    assert np.allclose(a[:30], to.forward(w, cfg, toks2)[:30]) and not np.allclose(a[30:], to.forward(w, cfg, toks2)[30:])


def test_steady_weights_leave_no_close_choice():
    cfg = tm.CONFIGS["odd"]
    w = tm.steady_weights(cfg, 0)
    rows = []
    mixture = to.mixture

    def spy(w_, p, m, h):
        rows.append(tm.margin(to.sigmoid(h @ w_[p + "router"].T), w_[p + "correction"], m["router"]).min())
        return mixture(w_, p, m, h)
    to.mixture = spy
    try:
        to.forward(w, cfg, np.random.default_rng(1).integers(0, cfg["vocab"], size=60))
    finally:
        to.mixture = mixture
    assert len(rows) == 3 and min(rows) > 0.02


def test_every_mechanism_shows_in_the_test_models_logits():
    """Each mechanism changed moves the logits by forty times what the f32 comparisons on the GPU allow (5e-5)."""
    cfg = tm.CONFIGS["odd"]
    w = tm.random_weights(cfg, 0)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=140)
    want = to.forward(w, cfg, toks)

    def moved(edit=None, change=None):
        c, v = copy.deepcopy(cfg), dict(w)
        if edit:
            edit(c)
        if change:
            v.update(change(v))
        return tm.logit_error(to.forward(v, c, toks), want).max()

    def each(kind, f):
        return lambda c: [f(l["mixer"]) for l in c["layers"] if l["type"] == kind]

    def tensors(end, f):
        return lambda v: {k: f(x) for k, x in v.items() if k.endswith(end)}

    least = 40 * 5e-5
    assert moved(lambda c: c["norm"].update(eps=3e-2)) > least and moved(lambda c: c["norm"].update(groups=4)) > least
    for f in (lambda m: m.update(left_scale=0.85), lambda m: m.update(right_scale=1.15), lambda m: m["left"].update(scale=m["left"]["scale"] * 1.05),
              lambda m: m["left"]["mask"].update(size=m["left"]["mask"]["size"] + 1), lambda m: m["left"]["mask"].update(size=m["left"]["mask"]["size"] - 1),
              lambda m: m["right"].update(norm_groups=1 if m["right"]["norm_groups"] == 2 else 3)):
        assert moved(each("parallel", f)) > least
    assert moved(each("mlstm", lambda m: m.update(gate_cap=8.0))) > least
    assert moved(lambda c: [l["mlp"]["router"].update(top=l["mlp"]["router"]["top"] - 1) for l in c["layers"] if l["mlp"]]) > least
    assert moved(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3)) > least
    for end in ("q.b", "k.b", "v.b", "sink", "f.b", "i.b", "lower", "conv.b", "dt_bias", "A_log", "right.D", "correction", "pos", "canon1", "canon2", "left.g", "mix.g"):
        assert moved(change=tensors(end, np.zeros_like)) > least, end
    for end in ("q.norm", "k.norm", "mix.norm", "right.norm", "norm1", "norm2", "final.norm"):
        assert moved(change=tensors(end, np.ones_like)) > least, end
    assert moved(change=tensors("right.conv", lambda x: np.roll(x, 1, axis=1))) > least
