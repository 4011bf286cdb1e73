"""Tarivik models through the framework's own sessions, steps, loops and entry points, against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import tarivik_oracle as to
from tests import tarivik_models as tm
from turbospark_b200 import tarivik
from turbospark_b200.plain import BF16, F32

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {F32: 5e-5, BF16: 4e-2}
CONTEXT = 512


class Expected:
    """Oracle logits of a sequence, and for bfloat16 how far they move when every matrix is off by as much as rounding: a norm of a small output or a
    normaliser next to nothing now and then lifts that to many times its usual size."""

    def __init__(self, w=None, cfg=None, tokens=None, type_=None, logits=None, moved=None):
        self.logits, self.moved = logits, moved
        if w is None:
            return
        self.logits = to.forward(w, cfg, tokens)
        if type_ == BF16:
            self.moved = np.zeros(len(tokens))
            for seed in range(2):
                rng = np.random.default_rng(seed)
                off = {k: v * (1 + 2.0 ** -8 * rng.uniform(-1, 1, v.shape)) if v.ndim == 2 and "canon" not in k else v for k, v in w.items()}
                self.moved = np.maximum(self.moved, 8 * tm.logit_error(to.forward(off, cfg, tokens), self.logits))

    def __getitem__(self, rows):
        return Expected(logits=self.logits[rows], moved=None if self.moved is None else self.moved[rows])


@pytest.fixture(scope="module")
def rig():
    """Models by (configuration, type), oracle logits by (configuration, type, tokens), made once.  bfloat16 models have routers without close
    choices."""
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    weights = {(n, t): make(c, i) for i, (n, c) in enumerate(tm.CONFIGS.items()) for t, make in ((F32, tm.random_weights), (BF16, tm.steady_weights))}
    models, logits = {}, {}

    class Rig:
        def model(self, name, type_):
            if (name, type_) not in models:
                models[name, type_] = tarivik.build(ctx, tm.CONFIGS[name], weights[name, type_].__getitem__, CONTEXT, type_)
            return models[name, type_]

        def logits(self, name, type_, tokens):
            key = (name, type_, tuple(tokens))
            if key not in logits:
                logits[key] = Expected(weights[name, type_], tm.CONFIGS[name], list(tokens), type_)
            return logits[key]

        def tokens(self, name, n, seed):
            return np.random.default_rng(seed).integers(0, tm.CONFIGS[name]["vocab"], size=n).tolist()

        def session(self, name, type_, streams=3, max_rows=1, pool=0, rows=700, draft=None):
            return tsb.Session(ctx, self.model(name, type_), draft, streams, max_rows, pool_tokens=pool, step_rows=rows)

    r = Rig()
    r.ctx, r.tsb, r.weights = ctx, tsb, weights
    yield r
    for m in models.values():
        m.close()
    ctx.close()


def check(got, want, type_, at=""):
    """want: logits, and (bfloat16) how far rounding may move each row."""
    e = tm.logit_error(got, want.logits)
    limit = LIMIT[type_] if type_ == F32 else np.maximum(LIMIT[type_], want.moved)
    worst = int((e / limit).argmax())
    assert (e <= limit).all(), (at, worst, float(e[worst]), limit if type_ == F32 else float(limit[worst]))


NAMES = list(tm.CONFIGS)


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(rig, name, type_):
    """Lengths on both sides of where recurrences go chunk by chunk, of chunks, of key tiles and of pages."""
    s = rig.session(name, type_)
    t = rig.tokens(name, 300, 7)
    for i, n in enumerate([1, 2, 3, 31, 32, 63, 64, 65, 128, 129, 300]):
        check(s.step([(i % 3, t[:n], list(range(n)))]), rig.logits(name, type_, t)[:n], type_, n)
        s.reset(i % 3)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_equals_the_whole_prompt(rig, name, type_):
    s = rig.session(name, type_, streams=1)
    t = rig.tokens(name, 300, 7)[:130]
    got = np.stack([s.produce(tok, i) for i, tok in enumerate(t)])
    check(got, rig.logits(name, type_, rig.tokens(name, 300, 7))[:130], type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("size", [2, 3, 7, 33, 64, 65, 100])
def test_portions(rig, name, type_, size):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 300, 7)
    got = [s.step([(1, t[i:i + size], list(range(len(t[i:i + size]))))]) for i in range(0, len(t), size)]
    check(np.concatenate(got), rig.logits(name, type_, t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_a_step_larger_than_a_pass_and_than_the_logit_rows(rig, type_):
    """Steps are cut where they exceed what a pass holds; the answer stays the same."""
    t, u = rig.tokens("odd", 300, 7), rig.tokens("odd", 40, 3)
    for rows in (50, 100):
        s = rig.session("odd", type_, streams=2, rows=rows)
        got = s.step([(0, u, [0, 39]), (1, t, list(range(300)))])
        check(got[:2], rig.logits("odd", type_, u)[[0, 39]], type_)
        check(got[2:], rig.logits("odd", type_, t), type_)
        s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_with_pages_and_streams_used_again(rig, name, type_):
    """Requests of unequal lengths in random portions, three at a time in a pool that holds little more: every logit row
    equals the request alone, whatever pages, states and streams it got."""
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
        check(np.concatenate(rows[i]), rig.logits(name, type_, t), type_, i)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "even"])
def test_long_decoding(rig, name, type_):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 420, 4)
    got = [s.step([(0, t[:20], [19])])]
    for i in range(20, 420):
        got.append(s.step([(0, t[i:i + 1], [0])]))
    check(np.concatenate(got), rig.logits(name, type_, t)[19:], type_)
    s.close()


def test_many_rows_and_many_slots_per_expert(rig):
    """A batch whose routed products run on the tensor-memory kernel and whose row operators walk runs of rows."""
    name = "even"
    s = rig.session(name, BF16, streams=4, rows=2048)
    reqs = [rig.tokens(name, n, 50 + i) for i, n in enumerate([500, 411, 77, 330])]
    got, r = s.step([(i, t, list(range(0, len(t), 7))) for i, t in enumerate(reqs)]), 0
    for t in reqs:
        n = len(range(0, len(t), 7))
        check(got[r:r + n], rig.logits(name, BF16, t)[::7], BF16)
        r += n
    s.close()


# ------------------------------------------------------------------ a far token that decides, a chunk's edge
def sharp_model(chunk, seed):
    """One attention layer in which the marked token's key answers the query of the asking token far above all others."""
    cfg = tm.config(64, 48, [tm.parallel((4, 2, 16, 16, chunk), (2, 1, 8, 8, 3, 1), None, scales=(1.5, 0.001), scale=2.0)], groups=1, taps=2)
    w = tm.random_weights(cfg, seed)
    mark, ask = 5, 7
    e = w["embed"]
    e[:, :2] = 0.0
    e[mark, 0], e[ask, 1] = 12.0, 12.0  # coordinate 0: "I am marked", coordinate 1: "I am asking"
    w["pos"][:, :2] = 0.0
    w["l0.canon1"][:] = 0.0
    for name, heads, coordinate in (("q", 4, 1), ("k", 2, 0)):
        m = w["l0.mix.left." + name] = w["l0.mix.left." + name] * 0.3
        m[:, :2] = 0.0
        m.reshape(heads, 16, 64)[:, 0, coordinate] = 1.0
    w["l0.mix.left.sink"][:] = 0.5
    return cfg, tm.rounded(w), mark, ask


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("chunk", [64, 150, 1000])
def test_a_far_key_and_both_sides_of_a_chunks_edge(rig, chunk, type_):
    cfg, w, mark, ask = sharp_model(chunk, 3)
    model = tarivik.build(rig.ctx, cfg, w.__getitem__, CONTEXT, type_)
    s = rig.tsb.Session(rig.ctx, model, None, 2, 1, step_rows=512)
    base = np.random.default_rng(1).integers(10, 48, size=400).tolist()
    edge = 400 // chunk * chunk  # the first position that the last one sees
    places = sorted({p for p in (edge, edge + 1, edge + 7, 399 - 63, 399 - 20, 397, edge - 1, edge - 2, edge - chunk, 0) if 0 <= p < 399 - 1})
    for place in places:
        t = list(base)
        t[place], t[399] = mark, ask
        plain = list(base)
        plain[399] = ask
        want = Expected(w, cfg, t, type_)[399:]
        shows = tm.logit_error(to.forward(w, cfg, plain)[399:], want.logits).max()
        assert (shows > 3 * LIMIT[BF16]) == (place >= edge), (place, shows)
        for cut in ([400], [399, 1], [330, 69, 1], [edge or 200, 400 - (edge or 200)], [edge + 1, 399 - edge]):
            at, got = 0, None
            for n in cut:
                got = s.step([(place % 2, t[at:at + n], [n - 1])])
                at += n
            s.reset(place % 2)
            check(got, want, type_, (place, cut))
    s.close(), model.close()


# ------------------------------------------------------------------ pool, refusals, rewinding
def test_a_step_that_does_not_fit_is_refused_and_changes_nothing(rig):
    s = rig.session("odd", F32, streams=3, pool=192)
    t = rig.tokens("odd", 300, 7)[:130]
    s.step([(0, t[:100], [])])
    with pytest.raises(rig.tsb.TsbError, match="pages"):
        s.step([(1, t[:70], [0]), (0, t[100:], [0])])
    check(s.step([(0, t[100:], list(range(30)))]), rig.logits("odd", F32, rig.tokens("odd", 300, 7))[100:130], F32)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "ones"])
def test_cursors_go_back_as_far_as_the_states(rig, name, type_):
    """Rejected rows of a verify pass leave no trace; a state that is gone is not used."""
    s = rig.session(name, type_, streams=1, max_rows=6)
    t, u = rig.tokens(name, 90, 6), rig.tokens(name, 90, 7)
    s.step([(0, t[:57], [])])
    for i in range(57, 60):
        s.produce(t[i], i)
    for keep in (2, 0, 5):  # rounds of six rows of which some are kept
        base = s.checkpoint()
        s.verify(t[60:66], base)
        s.rollback_retaining(base, keep)
    mixed = t[:60] + t[60:62] + t[60:65]
    assert s.checkpoint() == len(mixed)
    got = [s.produce(tok, len(mixed) + i) for i, tok in enumerate(u[:20])]
    check(np.stack(got), rig.logits(name, type_, mixed + u[:20])[len(mixed):], type_)
    # a prefix that ends where no state is kept: the stream starts over
    assert s.try_reuse_prefix(mixed[:30] + [5, 6]) == 0
    fresh = mixed[:30] + [5, 6]
    check(s.step([(0, fresh, list(range(32)))]), rig.logits(name, type_, fresh), type_)
    with pytest.raises(rig.tsb.TsbError, match="chains"):
        s.verify_tree([1, 2, 3], [-1, 0, 0], 32)
    s.close()


# ------------------------------------------------------------------ generation
def greedy(rig, name, prompt, n):
    """Oracle greedy continuation; it ends at a step whose two best logits are closer than rounding could tell."""
    toks, out = list(prompt), []
    for _ in range(n):
        l = rig.logits(name, F32, toks).logits[-1]
        top = np.sort(l)[-2:]
        if top[1] - top[0] < 1e-3:
            break
        out.append(int(l.argmax()))
        toks.append(out[-1])
    return out


@pytest.mark.parametrize("name", ["odd", "many_experts"])
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
    # speculation with the model's first layer as the drafter commits the same greedy tokens
    small = dict(tm.CONFIGS[name], layers=tm.CONFIGS[name]["layers"][:1])
    draft = tarivik.build(rig.ctx, small, rig.weights[name, F32].__getitem__, CONTEXT, F32)
    s = rig.session(name, F32, streams=2, max_rows=6, draft=draft)
    for i in (0, 4, 5):
        _, spec, res = s.spec_run(prompts[i], tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 4), stream=i % 2)
        assert np.array_equal(spec, out[i]) and res.rounds > 0
    s.close(), draft.close()


def test_speculative_rounds_of_several_streams_replay_as_a_graph(rig):
    """Lockstep rounds (a CUDA graph after the first) leave the tokens that the streams decode alone."""
    tsb, name = rig.tsb, "odd"
    small = dict(tm.CONFIGS[name], layers=tm.CONFIGS[name]["layers"][:2])
    draft = tarivik.build(rig.ctx, small, rig.weights[name, F32].__getitem__, CONTEXT, F32)
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
    tm.write_folder(folder, tm.CONFIGS[name], rig.weights[name, type_])
    t, u = rig.tokens(name, 300, 7)[:100], rig.tokens(name, 9, 81)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:70], "want": [0, 69]}, {"id": "y", "tokens": u[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[8:], "want": [0]}, {"id": "x", "tokens": t[70:], "want": [29]}], "end": ["x", "y"]},
             {"step": 2, "entries": [{"id": "z", "tokens": t[:3], "want": []}], "end": ["z"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "1024"],
                       input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    V = tm.CONFIGS[name]["vocab"]
    read = lambda n: np.fromfile(out / ("%d.f32" % n), dtype="<f4").reshape(-1, V)
    check(read(0), rig.logits(name, type_, t)[[0, 69]], type_)
    check(read(1)[:1], rig.logits(name, type_, u)[8:9], type_)
    check(read(1)[1:], rig.logits(name, type_, t)[99:100], type_)
    assert not (out / "2.f32").exists()
    if type_ == F32:
        r = subprocess.run([sys.executable, "-m", "turbospark_b200.generate", "--model", folder, "--dtype", dtype, "--max-new-tokens", "6", "--prompt",
                            " ".join(map(str, u)), "--prompt", "1,2"], capture_output=True, text=True, timeout=240, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        lines = [json.loads(l) for l in r.stdout.splitlines()]
        want = greedy(rig, name, u, 6)
        assert lines[0]["tokens"][:len(want)] == want and lines[0]["reason"] == "length" and len(lines[1]["tokens"]) == 6


def test_a_model_with_a_missing_tensor_or_an_unsupported_size_is_refused(rig):
    tsb, name = rig.tsb, "ones"
    cfg, layers = tarivik.parse_config(tm.CONFIGS[name], 64)
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    tarivik.load_tensors(m, rig.weights[name, F32].__getitem__)
    with pytest.raises(tsb.TsbError, match="must be"):
        m.set(tsb.plain.P_Q, np.zeros((3, 3), dtype=np.float32), layer=0)
    with pytest.raises(tsb.TsbError, match="no tensor"):
        m.set(tsb.plain.P_REC_K, np.zeros((8, 64), dtype=np.float32), layer=1)
    m.close()
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    with pytest.raises(tsb.TsbError, match="missing"):
        tsb.Session(rig.ctx, m, None, 1, 1)
    m.close()
    moe = tm.moe
    for bad in (tm.hgrn2(1, 2000, 8, None), tm.parallel((3, 2, 8, 8, 4), (1, 1, 8, 8, 2, 1), None), tm.parallel((1, 1, 8, 8, 4), (3, 2, 8, 8, 2, 1), None),
                tm.parallel((1, 1, 8, 8, 4), (3, 1, 8, 8, 2, 5), None), tm.parallel((1, 1, 8, 8, 4), (1, 1, 8, 8, 9, 1), None), tm.mlstm(1, 8, 8, None, cap=0.0),
                tm.hgrn2(1, 8, 8, moe(8, 9, 2, 2, 1)), tm.hgrn2(1, 8, 8, moe(8, 8, 5, 2, 1)), tm.hgrn2(1, 8, 8, moe(8, 8, 1, 2, 3))):
        with pytest.raises(tsb.TsbError):
            tsb.PlainModel(rig.ctx, *tarivik.parse_config(tm.config(64, 40, [bad]), 64))
    for groups, taps in ((5, 2), (1, 9)):
        with pytest.raises(tsb.TsbError):
            tsb.PlainModel(rig.ctx, *tarivik.parse_config(tm.config(64, 40, [tm.hgrn2(1, 8, 8, None)], groups=groups, taps=taps), 64))
