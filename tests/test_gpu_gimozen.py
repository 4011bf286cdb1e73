"""Gimozen models through the framework's own sessions, steps, loops and entry points, against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import gimozen_oracle as go
from tests import gimozen_models as gm
from turbospark_b200 import gimozen
from turbospark_b200.plain import BF16, F32

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {F32: 2e-5, BF16: 4e-2}
CONTEXT = 512


@pytest.fixture(scope="module")
def rig():
    """Models by (configuration, type), oracle logits by (configuration, tokens), made once."""
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    weights = {n: gm.random_weights(c, i) for i, (n, c) in enumerate(gm.CONFIGS.items())}
    models, logits = {}, {}

    class Rig:
        def model(self, name, type_):
            if (name, type_) not in models:
                models[name, type_] = gimozen.build(ctx, gm.CONFIGS[name], weights[name].__getitem__, CONTEXT, type_)
            return models[name, type_]

        def logits(self, name, tokens):
            key = (name, tuple(tokens))
            if key not in logits:
                logits[key] = go.forward(weights[name], gm.CONFIGS[name], list(tokens))
            return logits[key]

        def tokens(self, name, n, seed):
            return np.random.default_rng(seed).integers(0, gm.CONFIGS[name]["vocab"], size=n).tolist()

        def session(self, name, type_, streams=3, max_rows=1, pool=0, rows=700, draft=None):
            return tsb.Session(ctx, self.model(name, type_), draft, streams, max_rows, pool_tokens=pool, step_rows=rows)

    r = Rig()
    r.ctx, r.tsb, r.weights = ctx, tsb, weights
    yield r
    for m in models.values():
        m.close()
    ctx.close()


def check(got, want, type_, at=""):
    e = gm.logit_error(got, want)
    assert e.max() < LIMIT[type_], (at, int(e.argmax()), float(e.max()))


NAMES = list(gm.CONFIGS)


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(rig, name, type_):
    """Lengths on both sides of where latents are expanded, of key tiles and of pages."""
    s = rig.session(name, type_)
    for i, n in enumerate([1, 2, 31, 63, 64, 65, 127, 129, 300]):
        t = rig.tokens(name, n, i)
        check(s.step([(i % 3, t, list(range(n)))]), rig.logits(name, t), type_, n)
        s.reset(i % 3)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_equals_the_whole_prompt(rig, name, type_):
    s = rig.session(name, type_, streams=1)
    t = rig.tokens(name, 150, 1)
    got = np.stack([s.produce(tok, i) for i, tok in enumerate(t)])
    check(got, rig.logits(name, t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "borrow", "wide_heads", "large"])
@pytest.mark.parametrize("size", [2, 3, 17, 63, 64, 65, 129])
def test_portions(rig, name, type_, size):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 300, 2)
    got = [s.step([(1, t[i:i + size], list(range(len(t[i:i + size]))))]) for i in range(0, len(t), size)]
    check(np.concatenate(got), rig.logits(name, t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_a_step_larger_than_a_pass_and_than_the_logit_rows(rig, type_):
    """Steps are cut where they exceed what a pass holds; the answer stays the same."""
    t, u = rig.tokens("odd", 300, 2), rig.tokens("odd", 40, 3)
    for rows in (50, 100):
        s = rig.session("odd", type_, streams=2, rows=rows)
        got = s.step([(0, u, [0, 39]), (1, t, list(range(300)))])
        check(got[:2], rig.logits("odd", u)[[0, 39]], type_)
        check(got[2:], rig.logits("odd", t), type_)
        s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_with_pages_and_streams_used_again(rig, name, type_):
    """Requests of unequal lengths in random portions, three at a time in a pool that holds little more: every logit row
    equals the request alone, whatever pages and streams it got."""
    rng = np.random.default_rng(11)
    s = rig.session(name, type_, streams=3, pool=576)
    reqs = [rig.tokens(name, n, 20 + i) for i, n in enumerate([200, 3, 130, 65, 1, 190, 64, 7, 150])]
    waiting, live, free, rows = list(range(len(reqs))), {}, [2, 0, 1], {i: [] for i in range(len(reqs))}
    while waiting or live:
        while waiting and free and sum((len(reqs[i]) + 63) // 64 for i in [*live, waiting[0]]) <= 9:
            live[waiting.pop(0)] = [free.pop(0), 0]
        entries, order = [], []
        for i in rng.permutation(list(live)):
            stream, at = live[i]
            if len(live) > 1 and rng.random() < 0.2:
                continue  # left out of this step
            n = min(int(rng.choice([1, 1, 2, 5, 33, 64, 90, 128])), len(reqs[i]) - at)
            entries.append((stream, reqs[i][at:at + n], list(range(n))))
            order.append((i, n))
        if not entries:
            continue
        got, r = s.step(entries), 0
        for i, n in order:
            rows[i].append(got[r:r + n])
            r += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                s.reset(live[i][0])
                free.append(live.pop(i)[0])
    for i, t in enumerate(reqs):
        check(np.concatenate(rows[i]), rig.logits(name, t), type_, i)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "borrow"])
def test_long_decoding(rig, name, type_):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 420, 4)
    got = [s.step([(0, t[:20], [19])])]
    for i in range(20, 420):
        got.append(s.step([(0, t[i:i + 1], [0])]))
    check(np.concatenate(got), rig.logits(name, t)[19:], type_)
    s.close()


def test_f32_and_bf16_stay_close_over_every_way_to_cut_a_long_prompt(rig):
    """The same positions through short portions (absorbed), long ones (expanded) and single tokens differ by rounding only."""
    t = rig.tokens("wide_heads", 400, 9)
    want = rig.logits("wide_heads", t)
    outs = []
    for cuts in ([400], [40] * 10, [64] * 6 + [16], [300, 100], [63, 337]):
        s = rig.session("wide_heads", BF16, streams=1)
        at, got = 0, []
        for n in cuts:
            got.append(s.step([(0, t[at:at + n], list(range(n)))]))
            at += n
        outs.append(np.concatenate(got))
        check(outs[-1], want, BF16, cuts)
        s.close()
    assert max(gm.logit_error(a, b).max() for a in outs for b in outs) < LIMIT[BF16]


# ------------------------------------------------------------------ a far token that decides
def sharp_model(cfg_layer, seed):
    """A one-layer model in which the marked token's key answers the query of the asking token far above all others."""
    cfg = gm.config(64, 48, [cfg_layer], alpha=1.0, embed=1.0)
    w = gm.random_weights(cfg, seed)
    m = cfg_layer["mixer"]
    H, D, d = m["heads"], m["dim"], 64
    mark, ask = 5, 7
    e = w["embed"]
    e[:, :2] = 0.0
    e[mark, 0], e[ask, 1] = 12.0, 12.0  # coordinate 0: "I am marked", coordinate 1: "I am asking"
    w["l0.mix.q"] = w["l0.mix.q"] * 0.3
    if cfg_layer["type"] == "latent_attention":
        R, K = m["rot_dim"], m["kv_rank"]
        q = w["l0.mix.q"].reshape(H, D + R, d)
        q[:, 0, 1] = 1.0
        w["l0.mix.dkv"] = w["l0.mix.dkv"] * 0.3
        w["l0.mix.dkv"][0, 0] = 1.0
        w["l0.mix.uk"] = w["l0.mix.uk"] * 0.3
        w["l0.mix.uk"].reshape(H, D, K)[:, 0, 0] = 1.0
    else:
        G = m["kv_heads"]
        w["l0.mix.q"].reshape(H, D, d)[:, 0, 1] = 1.0
        w["l0.mix.k"] = w["l0.mix.k"] * 0.3
        w["l0.mix.k"].reshape(G, D, d)[:, 0, 0] = 1.0
        w["l0.mix.q.norm"][0] = w["l0.mix.k.norm"][0] = 1.5
    w = {k: gm.bf16_to_f32(gm.bf16_bits(v)).reshape(np.shape(v)) for k, v in w.items()}
    return cfg, w, mark, ask


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("kind", ["latent", "attention"])
def test_one_far_key_decides_wherever_it_stands_and_however_it_is_asked(rig, kind, type_):
    layer = gm.latent(4, 24, 8, 24, 40, None, scale=0.6) if kind == "latent" else gm.attention(4, 2, 24, 24, None, scale=0.6, temp=(0.5, 64))
    cfg, w, mark, ask = sharp_model(layer, 3)
    model = gimozen.build(rig.ctx, cfg, w.__getitem__, CONTEXT, type_)
    s = rig.tsb.Session(rig.ctx, model, None, 2, 1, step_rows=512)
    rng = np.random.default_rng(1)
    base = rng.integers(10, 48, size=400).tolist()
    for place in [0, 1, 2, 63, 64, 65, 127, 128, 191, 192, 255, 256, 300]:
        t = list(base)
        t[place], t[399] = mark, ask
        want = go.forward(w, cfg, t)
        plain = list(base)
        plain[399] = ask
        assert gm.logit_error(go.forward(w, cfg, plain)[399:], want[399:]).max() > 10 * LIMIT[BF16]  # the key shows
        for cut in ([400], [399, 1], [330, 69, 1], [337, 63]):
            at, got = 0, None
            for n in cut:
                got = s.step([(place % 2, t[at:at + n], [n - 1])])
                at += n
            s.reset(place % 2)
            check(got, want[399:], type_, (place, cut))
    s.close(), model.close()


# ------------------------------------------------------------------ pool, refusals, rewinding
def test_a_step_that_does_not_fit_is_refused_and_changes_nothing(rig):
    s = rig.session("odd", F32, streams=3, pool=192)
    t = rig.tokens("odd", 130, 5)
    s.step([(0, t[:100], [])])
    with pytest.raises(rig.tsb.TsbError, match="pages"):
        s.step([(1, t[:70], [0]), (0, t[100:], [0])])
    check(s.step([(0, t[100:], list(range(30)))]), rig.logits("odd", t)[100:], F32)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_cursors_go_back_anywhere(rig, type_):
    """No state but the cache: rejected rows are overwritten, prefixes are taken up again."""
    s = rig.session("odd", type_, streams=1, max_rows=6)
    t, u = rig.tokens("odd", 90, 6), rig.tokens("odd", 90, 7)
    for i in range(60):
        s.produce(t[i], i)
    s.verify(t[60:66], 60)
    s.rollback_retaining(60, 2)
    mixed = t[:62] + u[:20]
    got = [s.produce(tok, 62 + i) for i, tok in enumerate(u[:20])]
    check(np.stack(got), rig.logits("odd", mixed)[62:], type_)
    assert s.try_reuse_prefix(mixed[:30] + [5, 6]) == 30
    check(np.stack([s.produce(5, 30), s.produce(6, 31)]), rig.logits("odd", mixed[:30] + [5, 6])[30:], type_)
    with pytest.raises(rig.tsb.TsbError, match="chains"):
        s.verify_tree([1, 2, 3], [-1, 0, 0], 32)
    s.close()


# ------------------------------------------------------------------ generation
def greedy(rig, name, prompt, n):
    """Oracle greedy continuation; it ends at a step whose two best logits are closer than rounding could tell."""
    toks, out = list(prompt), []
    for _ in range(n):
        l = rig.logits(name, toks)[-1]
        top = np.sort(l)[-2:]
        if top[1] - top[0] < 1e-3:
            break
        out.append(int(l.argmax()))
        toks.append(out[-1])
    return out


@pytest.mark.parametrize("name", ["odd", "borrow"])
def test_greedy_generation_one_request_many_requests_and_speculation(rig, name):
    tsb = rig.tsb
    s = rig.session(name, F32, streams=3, pool=640, rows=100)
    prompts = [rig.tokens(name, n, 40 + i) for i, n in enumerate([5, 90, 1, 33, 64, 150, 12])]
    budgets = [24, 10, 30, 1, 16, 20, 8]
    want = [greedy(rig, name, p, b) for p, b in zip(prompts, budgets)]
    assert sum(map(len, want)) > 0.7 * sum(budgets)
    rc = tsb.run_config(tsb.shaping(temperature=0.0), max(budgets), 3)
    out, reasons, stats = s.serve(prompts, budgets, rc, prefill_chunk=80)
    assert [len(o) for o in out] == budgets and not reasons.any() and stats.most_live == 3
    for o, w in zip(out, want):
        assert o[:len(w)].tolist() == w
    # the single-request loop gives the same tokens
    for i in (0, 3, 4):
        _, seq, _ = s.sequential_run(prompts[i], tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 3), stream=1)
        assert np.array_equal(seq, out[i])
    s.close()
    # speculation with the model's first layers as the drafter commits the same greedy tokens
    small = dict(gm.CONFIGS[name], layers=gm.CONFIGS[name]["layers"][:2])
    draft = gimozen.build(rig.ctx, small, rig.weights[name].__getitem__, CONTEXT, F32)
    s = rig.session(name, F32, streams=2, max_rows=6, draft=draft)
    for i in (0, 4, 5):
        _, spec, res = s.spec_run(prompts[i], tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 4), stream=i % 2)
        assert np.array_equal(spec, out[i]) and res.rounds > 0
    s.close(), draft.close()


def test_speculative_rounds_of_several_streams_replay_as_a_graph(rig):
    """Lockstep rounds (a CUDA graph after the first) leave the tokens that the streams decode alone."""
    tsb, name = rig.tsb, "borrow"
    small = dict(gm.CONFIGS[name], layers=gm.CONFIGS[name]["layers"][:2])
    draft = gimozen.build(rig.ctx, small, rig.weights[name].__getitem__, CONTEXT, F32)
    s = rig.session(name, F32, streams=2, max_rows=5, draft=draft)
    prompts = [rig.tokens(name, 17, 60), rig.tokens(name, 17, 61)]
    rc = tsb.run_config(tsb.shaping(temperature=0.0), 1 << 20, 4)
    nxt = np.zeros(2, dtype=np.int32)
    for q, p in enumerate(prompts):
        s.step([(q, p[:-1], [])])
        nxt[q] = int(s.produce(p[-1], 16, stream=q).argmax())
        s.prime_drafter(p[-1], 15, stream=q)
    out = [[int(nxt[0])], [int(nxt[1])]]
    ctr = np.zeros(2, dtype=np.uint64)
    for _ in range(6):
        acc, toks = s.round_tokens(rc, nxt, ctr)
        for q in range(2):
            out[q] += toks[q, :acc[q] + 1].tolist()
    s.close()
    s = rig.session(name, F32, streams=1)
    for q, p in enumerate(prompts):
        _, seq, _ = s.sequential_run(p, tsb.run_config(tsb.shaping(temperature=0.0), len(out[q]), 1))
        assert seq.tolist() == out[q]
    s.close(), draft.close()


# ------------------------------------------------------------------ entry points
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_and_command_line(rig, tmp_path, dtype):
    name = "odd"
    type_ = F32 if dtype == "float32" else BF16
    folder = str(tmp_path / "model")
    gm.write_folder(folder, gm.CONFIGS[name], rig.weights[name])
    t, u = rig.tokens(name, 100, 80), rig.tokens(name, 9, 81)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:70], "want": [0, 69]}, {"id": "y", "tokens": u[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[8:], "want": [0]}, {"id": "x", "tokens": t[70:], "want": [29]}], "end": ["x", "y"]},
             {"step": 2, "entries": [{"id": "z", "tokens": t[:3], "want": []}], "end": ["z"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                       input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    V = gm.CONFIGS[name]["vocab"]
    read = lambda n: np.fromfile(out / ("%d.f32" % n), dtype="<f4").reshape(-1, V)
    check(read(0), rig.logits(name, t)[[0, 69]], type_)
    check(read(1), np.stack([rig.logits(name, u)[8], rig.logits(name, t)[99]]), type_)
    assert not (out / "2.f32").exists()
    if type_ == F32:
        r = subprocess.run([sys.executable, "-m", "turbospark_b200.generate", "--model", folder, "--dtype", dtype, "--max-new-tokens", "6", "--prompt",
                            " ".join(map(str, u)), "--prompt", "1,2"], capture_output=True, text=True, timeout=240, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        lines = [json.loads(l) for l in r.stdout.splitlines()]
        want = greedy(rig, name, u, 6)
        assert lines[0]["tokens"][:len(want)] == want and lines[0]["reason"] == "length" and len(lines[1]["tokens"]) == 6


def test_a_model_with_a_missing_tensor_or_an_unsupported_size_is_refused(rig):
    tsb = rig.tsb
    cfg, layers = gimozen.parse_config(gm.CONFIGS["single"], 64)
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    gimozen.load_tensors(m, rig.weights["single"].__getitem__)
    with pytest.raises(tsb.TsbError, match="must be"):
        m.set(5, np.zeros((3, 3), dtype=np.float32), layer=0)
    with pytest.raises(tsb.TsbError, match="no tensor"):
        m.set(tsb.plain.P_V, np.zeros((16, 64), dtype=np.float32), layer=0)
    m.close()
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    with pytest.raises(tsb.TsbError, match="missing"):
        tsb.Session(rig.ctx, m, None, 1, 1)
    m.close()
    for bad in (gm.latent(1, 16, 4, 16, 600, None), gm.attention(1, 1, 300, 16, None), gm.latent(1, 16, 5, 16, 32, None)):
        with pytest.raises(tsb.TsbError):
            tsb.PlainModel(rig.ctx, *gimozen.parse_config(gm.config(64, 40, [bad]), 64))
