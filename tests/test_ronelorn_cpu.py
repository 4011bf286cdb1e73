"""Host-side parts of the Ronelorn design: configuration, tensor names, the oracle's mechanisms."""
import copy

import numpy as np
import pytest

from oracle import ronelorn_oracle as ro
from tests import ronelorn_models as rm
from turbospark_b200 import plain, registry, ronelorn


# ---- configuration
def test_every_size_and_constant_comes_from_the_configuration():
    a0 = rm.pooled(6, 2, 12, 28, 19, 7, 24, rot=10, factor=3.5, base=321.0, cap=4.5, scale=0.7)
    cfg = rm.config(72, 31, [a0, rm.kept(4, 1, 16, 20, 33, 9, None, rot=6, base=55.0, scale=0.2), rm.mingru(44, mlp=12), rm.again(0, a0)], mult=0.45, eps=3e-4, embed=2.5)
    pc, (a, b, c, e) = ronelorn.parse_config(cfg, max_context=99, compute=plain.F32)
    assert (pc.n_layers, pc.d_model, pc.vocab, pc.max_context, pc.compute, pc.pre_norm, pc.output_norm, pc.post_norm) == (4, 72, 31, 99, plain.F32, 1, 0, 0)
    assert abs(pc.norm_eps - 3e-4) < 1e-9 and abs(pc.sublayer_scale - 0.45) < 1e-7 and pc.embed_scale == 2.5 and pc.logit_cap == 0
    assert (a.n_q_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.window, a.pool, a.keep_first) == (6, 2, 12, 28, 19, 7, 0)
    assert abs(a.score_scale - 0.7) < 1e-7 and a.score_cap == 4.5 and (a.rot_dim, a.rot_base, a.rot_factor, a.rot_original) == (10, 321.0, 3.5, 0.0)
    assert a.qk_norm == plain.NORM_HEAD and a.value_rot and not a.sink and (a.ffn, a.ff_plain, a.act) == (24, 1, plain.RELU2)
    assert (b.n_q_heads, b.n_kv_heads, b.head_dim, b.value_dim, b.window, b.pool, b.keep_first, b.ffn) == (4, 1, 16, 20, 33, 0, 9, 0)
    assert b.qk_norm == plain.NORM_PROJECTION and b.sink == plain.SINK_ZERO and not b.value_rot and b.score_cap == 0 and (b.rot_dim, b.rot_base, b.rot_factor) == (6, 55.0, 0.0)
    assert (c.n_q_heads, c.recurrence, c.rec_heads, c.rec_dim, c.rec_vdim, c.ffn) == (0, plain.REC_MINGRU, 1, 1, 44, 12)
    assert e.weights_of == 1 and not (a.weights_of or b.weights_of or c.weights_of)


@pytest.mark.parametrize("break_it", [
    lambda c: c.pop("width"), lambda c: c["norm"].pop("eps"), lambda c: c.pop("residual_mult"), lambda c: c["embedding"].pop("scale"), lambda c: c["layers"][1].pop("mlp"),
    lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="moe"), lambda c: c["layers"][0]["mlp"].pop("ff"),
    lambda c: c["layers"][0]["mixer"].pop("softcap"), lambda c: c["layers"][0]["mixer"].pop("scale"), lambda c: c["layers"][0]["mixer"]["mask"].pop("pool"),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), lambda c: c["layers"][0]["mixer"]["mask"].update(pool=0), lambda c: c["layers"][0]["mixer"].update(vdim=7),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=400), lambda c: c["layers"][0]["mixer"]["rot"].pop("base"),
    lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("factor"), lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), lambda c: c["layers"][1]["mixer"].pop("width"),
    lambda c: c["layers"][2]["mixer"]["mask"].pop("keep_first"), lambda c: c["layers"][2]["mixer"]["mask"].update(keep_first=-1), lambda c: c["layers"][0]["mixer"].pop("mask"),
    lambda c: c["layers"][3].update(weights_of=1), lambda c: c["layers"][3].update(weights_of=9), lambda c: c["layers"][3].update(weights_of=3),
    lambda c: c["layers"][0].update(weights_of=3), lambda c: c["layers"][3]["mixer"].update(scale=0.9), lambda c: c.update(residual_mult=0)])
def test_a_configuration_that_says_something_else_is_refused(break_it):
    cfg = copy.deepcopy(rm.CONFIGS["odd"])
    break_it(cfg)
    with pytest.raises(ValueError):
        ronelorn.parse_config(cfg, 64)


def test_tensors_of_a_layer_that_has_none_itself():
    a = rm.mingru(16)
    _, layers = ronelorn.parse_config(rm.config(32, 9, [rm.again(1, a), rm.again(2, a), a, rm.again(0, a)]), 64)
    assert [l.weights_of for l in layers] == [3, 3, 0, 3]


def test_the_registry_knows_the_design():
    assert registry.ARCHITECTURES[ronelorn.ARCHITECTURE] is ronelorn.build


@pytest.mark.parametrize("name", list(rm.CONFIGS))
def test_loading_asks_for_exactly_the_tensors_of_the_design(name):
    class Fake:
        def __init__(self, cfg, layers):
            self.cfg, self.layers, self.got = cfg, layers, set()

        def set(self, which, array, layer=-1):
            assert (layer, which) not in self.got
            self.got.add((layer, which))

    w = rm.random_weights(rm.CONFIGS[name], 0)
    asked = []
    ronelorn.load_tensors(Fake(*ronelorn.parse_config(rm.CONFIGS[name], 64)), lambda n: (asked.append(n), w[n])[1])
    assert sorted(asked) == sorted(w)


# ---- the oracle's mechanisms, each on numbers worked out by hand or by another route
def test_oracle_norm_and_activations():
    x = np.array([[3.0, 4.0, 0.0, 1.0]])
    assert np.allclose(ro.shifted_rms_norm(x, np.array([0.0, 1.0, 4.0, -0.5]), 0.0), [[3 / 6.5 ** 0.5, 8 / 6.5 ** 0.5, 0.0, 0.5 / 6.5 ** 0.5]])
    assert np.allclose(ro.shifted_rms_norm(x, np.zeros(4), 2.5), x / 3.0)
    assert np.allclose(ro.squared_relu(np.array([-2.0, 0.0, 3.0])), [0.0, 0.0, 9.0])
    assert np.allclose(ro.positive(np.array([0.0, 2.0, -1e-9, -1.0])), [0.5, 2.5, 0.5, 1 / (1 + np.e)])
    assert np.allclose(ro.softcap(np.array([0.1, 100.0]), 2.0), [2 * np.tanh(0.05), 2.0])


def test_oracle_rotation_pairs_halves_and_leaves_the_rest():
    f = ro.frequencies(10000.0, 4)
    assert np.allclose(f, [1.0, 0.01]) and np.allclose(ro.frequencies(10000.0, 4, 5.0), [0.2, 0.002])
    x = np.arange(1.0, 7.0).reshape(1, 1, 6)
    got = ro.rotate_half(x, [2], f)[0, 0]
    z = (x[0, 0, 0] + 1j * x[0, 0, 2]) * np.exp(2j), (x[0, 0, 1] + 1j * x[0, 0, 3]) * np.exp(0.02j)
    assert np.allclose(got, [z[0].real, z[1].real, z[0].imag, z[1].imag, 5.0, 6.0])
    assert np.allclose(ro.rotate_half(ro.rotate_half(x, [7], f), [-7], f), x)


def test_oracle_masks_are_their_definitions():
    n, size, keep, pool = 23, 6, 4, 3
    kept, window, blocks = ro.kept_mask(n, size, keep), ro.window_mask(n, size), ro.block_mask(n, size, pool)
    for i in range(n):
        for j in range(n):
            assert window[i, j] == (0 <= i - j < size) and kept[i, j] == (j <= i and (i - j < size or j < keep))
        for b in range(n // pool):
            assert blocks[i, b] == all(i - j >= size for j in range(b * pool, (b + 1) * pool))
    assert not blocks[size + pool - 2].any() and blocks[size + pool - 1].tolist() == [True] + [False] * (n // pool - 1)
    x = np.arange(10.0).reshape(10, 1, 1)
    assert ro.block_means(x, 4).ravel().tolist() == [1.5, 5.5]


def test_oracle_attention_weights_follow_the_equations():
    rng = np.random.default_rng(3)
    q, k, v = rng.standard_normal((5, 4, 6)), rng.standard_normal((7, 2, 6)), rng.standard_normal((7, 2, 3))
    seen = rng.random((5, 7)) < 0.6
    seen[:, 0] = True
    for cap, one in ((None, False), (1.5, False), (None, True)):
        got = ro.grouped_attention(q, k, v, seen, 0.8, cap, one)
        for i in range(5):
            for h in range(4):
                s = np.array([0.8 * q[i, h] @ k[j, h // 2] for j in range(7)])
                e = np.exp(s if cap is None else cap * np.tanh(s / cap)) * seen[i]
                assert np.allclose(got[i, h], e @ v[:, h // 2] / (e.sum() + one))


def test_oracle_scan_is_a_weighted_sum_of_the_past():
    rng = np.random.default_rng(4)
    z, c = rng.uniform(0, 1, (9, 3)), rng.standard_normal((9, 3))
    got = ro.gated_scan(z, c)
    for t in range(9):
        want = sum(np.prod(1 - z[s + 1:t + 1], axis=0) * z[s] * c[s] for s in range(t + 1))
        assert np.allclose(got[t], want)
    assert np.allclose(ro.gated_scan(z[4:], c[4:], got[3]), got[4:])


def test_oracle_turning_values_make_a_sum_that_depends_on_distances():
    """Shifting all positions of a single-block window by a constant leaves the output."""
    rng = np.random.default_rng(6)
    m = rm.pooled(2, 1, 8, 6, 50, 4, None, rot=4)["mixer"]
    w = {"q": rng.standard_normal((16, 10)), "k": rng.standard_normal((8, 10)), "v": rng.standard_normal((6, 10)), "o": rng.standard_normal((10, 12)),
         "q.norm": rng.uniform(0.5, 1.5, 8), "k.norm": rng.uniform(0.5, 1.5, 8)}
    h = rng.standard_normal((5, 10))
    f, turn = ro.frequencies(m["rot"]["base"], 4), ro.frequencies(m["rot"]["base"], 6)
    outs = []
    for shift in (0, 11):
        pos = np.arange(5) + shift
        q = ro.rotate_half(ro.rms((h @ w["q"].T).reshape(5, 2, 8), 1e-5) * w["q.norm"], pos, f)
        k = ro.rotate_half(ro.rms((h @ w["k"].T).reshape(5, 1, 8), 1e-5) * w["k.norm"], pos, f)
        v = ro.rotate_half((h @ w["v"].T).reshape(5, 1, 6), pos, turn)
        o = ro.grouped_attention(q, k, v, ro.window_mask(5, 50), m["scale"], cap=m["softcap"])
        outs.append(ro.rotate_half(o, -pos, turn).reshape(5, 12) @ w["o"].T)
    assert np.allclose(outs[0], outs[1]) and np.allclose(outs[0], ro.pooled_window_attention(w, "", m, h, 1e-5))


def test_oracle_logits_do_not_see_the_future():
    cfg = rm.CONFIGS["odd"]
    w = rm.random_weights(cfg, 5)
    toks = np.arange(80) * 7 % cfg["vocab"]
    a = ro.forward(w, cfg, toks)
    toks2 = toks.copy()
    toks2[60:] = 3
    assert np.allclose(a[:60], ro.forward(w, cfg, toks2)[:60]) and not np.allclose(a[60:], ro.forward(w, cfg, toks2)[60:])


def test_every_mechanism_shows_in_the_test_models_logits():
    """Each mechanism changed moves the logits by forty times what the f32 comparisons on the GPU allow (5e-5)."""
    cfg = rm.CONFIGS["odd"]
    w = rm.random_weights(cfg, 0)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], size=140)
    want = ro.forward(w, cfg, toks)

    def moved(edit=None, change=None):
        c, v = copy.deepcopy(cfg), dict(w)
        if edit:
            edit(c)
        if change:
            v.update(change(v))
        return rm.logit_error(ro.forward(v, c, toks), want).max()

    def each(kind, f):
        return lambda c: [f(l["mixer"]) for l in c["layers"] if l["type"] == kind]

    def tensors(end, f):
        return lambda v: {k: f(x) for k, x in v.items() if k.endswith(end)}

    least = 40 * 5e-5
    assert moved(lambda c: c["norm"].update(eps=3e-2)) > least and moved(lambda c: c.update(residual_mult=0.62)) > least and moved(lambda c: c["embedding"].update(scale=1.4)) > least
    for f in (lambda m: m["mask"].update(size=38), lambda m: m["mask"].update(size=36), lambda m: m["mask"].update(pool=6), lambda m: m["mask"].update(pool=400),
              lambda m: m.update(softcap=8.0), lambda m: m.update(scale=m["scale"] * 1.05), lambda m: m["rot"].update(base=1100.0), lambda m: m["rot"].update(dims=18),
              lambda m: m["rot"].pop("scaling"), lambda m: m["rot"]["scaling"].update(factor=2.6)):
        assert moved(each("attention", f)) > least
    for f in (lambda m: m["mask"].update(size=51), lambda m: m["mask"].update(size=49), lambda m: m["mask"].update(keep_first=6), lambda m: m["mask"].update(keep_first=8),
              lambda m: m.update(scale=m["scale"] * 1.05), lambda m: m["rot"].update(base=800.0), lambda m: m["rot"].update(dims=22)):
        assert moved(each("attention_2", f)) > least
    for end in ("z.b", "x.b", "mix.g", "mlp.up"):
        assert moved(change=tensors(end, np.zeros_like)) > least, end
    for end in ("q.norm", "k.norm"):
        assert moved(change=tensors(end, np.ones_like)) > least, end
    for end in ("norm1", "norm2", "final.norm"):
        assert moved(change=tensors(end, np.zeros_like)) > least, end
    for name in ("rotate_half", "sigmoid", "positive", "squared_relu"):  # mechanisms that have no constant
        old = getattr(ro, name)
        setattr(ro, name, (lambda x, pos, f: x if len(f) == 12 else old(x, pos, f)) if name == "rotate_half" else (lambda x: 0.9 * old(x)))
        try:
            assert moved() > least, name  # rotate_half: the values of the pooled layers stay where they are
        finally:
            setattr(ro, name, old)
    old = ro.softmax_sum
    ro.softmax_sum = lambda s, seen, v, one: old(s, seen, v, False)
    try:
        assert moved() > least
    finally:
        ro.softmax_sum = old
