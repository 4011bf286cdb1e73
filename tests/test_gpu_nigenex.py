"""Nigenex models through the framework's own sessions, steps, loops and entry points, against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import nigenex_oracle as no
from tests import nigenex_models as nm
from turbospark_b200 import nigenex
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
    weights = {n: nm.random_weights(c, i) for i, (n, c) in enumerate(nm.CONFIGS.items())}
    models, logits = {}, {}

    class Rig:
        def model(self, name, type_):
            if (name, type_) not in models:
                models[name, type_] = nigenex.build(ctx, nm.CONFIGS[name], weights[name].__getitem__, CONTEXT, type_)
            return models[name, type_]

        def logits(self, name, tokens):
            key = (name, tuple(tokens))
            if key not in logits:
                logits[key] = no.forward(weights[name], nm.CONFIGS[name], list(tokens))
            return logits[key]

        def tokens(self, name, n, seed):
            return np.random.default_rng(seed).integers(0, nm.CONFIGS[name]["vocab"], size=n).tolist()

        def session(self, name, type_, streams=3, max_rows=1, pool=0, rows=700, draft=None):
            return tsb.Session(ctx, self.model(name, type_), draft, streams, max_rows, pool_tokens=pool, step_rows=rows)

    r = Rig()
    r.ctx, r.tsb, r.weights = ctx, tsb, weights
    yield r
    for m in models.values():
        m.close()
    ctx.close()


def check(got, want, type_, at=""):
    e = nm.logit_error(got, want)
    assert e.max() < LIMIT[type_], (at, int(e.argmax()), float(e.max()))


NAMES = list(nm.CONFIGS)


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(rig, name, type_):
    s = rig.session(name, type_)
    for i, n in enumerate([1, 2, 31, 64, 65, 140, 200]):
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
@pytest.mark.parametrize("name", ["odd", "mixed_layers"])
@pytest.mark.parametrize("size", [2, 3, 17, 63, 64, 65, 129])
def test_portions(rig, name, type_, size):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 262, 2)
    got = [s.step([(1, t[i:i + size], list(range(len(t[i:i + size]))))]) for i in range(0, len(t), size)]
    check(np.concatenate(got), rig.logits(name, t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_a_step_larger_than_a_pass_and_than_the_logit_rows(rig, type_):
    """Steps are cut where they exceed what a pass holds; the answer stays the same."""
    s = rig.session("odd", type_, streams=2, rows=50)
    t, u = rig.tokens("odd", 262, 2), rig.tokens("odd", 40, 3)
    got = s.step([(0, u, [0, 39]), (1, t, list(range(262)))])
    check(got[:2], rig.logits("odd", u)[[0, 39]], type_)
    check(got[2:], rig.logits("odd", t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "mixed_layers", "large_heads"])
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
            n = min(int(rng.choice([1, 1, 2, 5, 33, 64, 90])), len(reqs[i]) - at)
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
def test_long_decoding_past_every_window(rig, type_):
    s = rig.session("mixed_layers", type_, streams=2)
    t = rig.tokens("mixed_layers", 420, 4)
    got = [s.step([(0, t[:20], [19])])]
    for i in range(20, 420):
        got.append(s.step([(0, t[i:i + 1], [0])]))
    check(np.concatenate(got), rig.logits("mixed_layers", t)[19:], type_)
    s.close()


# ------------------------------------------------------------------ pool, refusals, rewinding
def test_a_step_that_does_not_fit_is_refused_and_changes_nothing(rig):
    s = rig.session("odd", F32, streams=3, pool=192)
    t = rig.tokens("odd", 130, 5)
    s.step([(0, t[:100], [])])
    with pytest.raises(rig.tsb.TsbError, match="pages"):
        s.step([(1, t[:70], [0]), (0, t[100:], [0])])
    check(s.step([(0, t[100:], list(range(30)))]), rig.logits("odd", t)[100:], F32)
    s.reset(0)
    check(s.step([(2, t, list(range(130)))]), rig.logits("odd", t), F32)
    for bad in ([(3, [1], [])], [(0, [1], [1])], [(0, [1, 2], [1, 0])], [(0, [1], []), (0, [2], [])], []):
        with pytest.raises(rig.tsb.TsbError):
            s.step(bad)
    with pytest.raises(rig.tsb.TsbError):  # beyond the context window
        s.step([(1, [1] * (CONTEXT + 1), [])])
    s.close()


def test_a_token_outside_the_vocabulary_is_reported(rig):
    s = rig.session("odd", F32, streams=1)
    with pytest.raises(rig.tsb.TsbError):
        s.step([(0, [nm.CONFIGS["odd"]["vocab"]], [0])])
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_cursors_go_back_as_far_as_the_shift_state_reaches(rig, type_):
    s = rig.session("odd", type_, streams=1, max_rows=6)
    t, u = rig.tokens("odd", 90, 6), rig.tokens("odd", 90, 7)
    for i in range(60):
        s.produce(t[i], i)
    s.verify(t[60:66], 60)
    s.rollback_retaining(60, 2)  # two of the six rows stay
    mixed = t[:62] + u[:20]
    got = [s.produce(tok, 62 + i) for i, tok in enumerate(u[:20])]
    check(np.stack(got), rig.logits("odd", mixed)[62:], type_)
    with pytest.raises(rig.tsb.TsbError, match="state"):
        s.rollback_retaining(40, 0)
    # prefix reuse: from where the state reaches, else from the start; both give the right logits
    assert s.try_reuse_prefix(mixed + [5]) == 82
    assert s.try_reuse_prefix(mixed[:30] + [5]) == 0
    check(s.step([(0, mixed[:31], [30])]), rig.logits("odd", mixed[:31])[30:], type_)
    with pytest.raises(rig.tsb.TsbError, match="chains"):
        s.verify_tree([1, 2, 3], [-1, 0, 0], 31)
    s.close()


# ------------------------------------------------------------------ generation
def greedy(rig, name, prompt, n):
    """Oracle greedy continuation; None behind a step whose two best logits are closer than rounding could tell."""
    toks, out = list(prompt), []
    for _ in range(n):
        l = rig.logits(name, toks)[-1]
        top = np.sort(l)[-2:]
        if top[1] - top[0] < 1e-3:
            break
        out.append(int(l.argmax()))
        toks.append(out[-1])
    return out


@pytest.mark.parametrize("name", ["one_kv", "mixed_layers"])
def test_greedy_generation_one_request_many_requests_and_speculation(rig, name):
    tsb = rig.tsb
    s = rig.session(name, F32, streams=3, pool=640, rows=64)
    prompts = [rig.tokens(name, n, 40 + i) for i, n in enumerate([5, 90, 1, 33, 64, 150, 12])]
    budgets = [24, 10, 30, 1, 16, 20, 8]
    want = [greedy(rig, name, p, b) for p, b in zip(prompts, budgets)]
    assert sum(map(len, want)) > 0.8 * sum(budgets)
    rc = tsb.run_config(tsb.shaping(temperature=0.0), max(budgets), 3)
    out, reasons, stats = s.serve(prompts, budgets, rc, prefill_chunk=40)
    assert [len(o) for o in out] == budgets and not reasons.any()
    assert stats.most_live == 3 and stats.prompt_rows == sum(map(len, prompts)) and stats.decode_rows == sum(budgets) - len(budgets)
    for o, w in zip(out, want):
        assert o[:len(w)].tolist() == w
    # the single-request loop gives the same tokens; a stop token ends a request in both
    for i in (0, 3, 4):
        rc1 = tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 3)
        _, seq, res = s.sequential_run(prompts[i], rc1, stream=1)
        assert np.array_equal(seq, out[i])
    stop = int(out[0][5])
    rcs = tsb.run_config(tsb.shaping(temperature=0.0), 24, 3, stop_tokens=[stop])
    o2, r2, _ = s.serve(prompts[:2], budgets[:2], rcs)
    first = out[0].tolist().index(stop) + 1
    assert o2[0].tolist() == out[0][:first].tolist() and r2[0] == 1
    _, seq, res = s.sequential_run(prompts[0], rcs)
    assert np.array_equal(seq, o2[0]) and res.reason == 1
    s.close()
    # speculation with the model's first layers as the drafter commits the same greedy tokens
    cfg = nm.CONFIGS[name]
    small = dict(cfg, layers=cfg["layers"][:1])
    draft = nigenex.build(rig.ctx, small, rig.weights[name].__getitem__, CONTEXT, F32)
    s = rig.session(name, F32, streams=2, max_rows=6, draft=draft)
    for i in (0, 4, 5):
        rc1 = tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 4)
        _, spec, res = s.spec_run(prompts[i], rc1, stream=i % 2)
        assert np.array_equal(spec, out[i]) and res.rounds > 0
    rct = tsb.run_config(tsb.shaping(temperature=0.0), 8, 2, tree_nodes=4, tree_branching=(2, 1))
    with pytest.raises(tsb.TsbError, match="chains"):
        s.spec_run(prompts[0], rct)
    s.close(), draft.close()


def test_speculative_rounds_of_several_streams_replay_as_a_graph(rig):
    """Lockstep rounds (a CUDA graph after the first) leave the tokens that the streams decode alone."""
    tsb, name = rig.tsb, "one_kv"
    small = dict(nm.CONFIGS[name], layers=nm.CONFIGS[name]["layers"][:1])
    draft = nigenex.build(rig.ctx, small, rig.weights[name].__getitem__, CONTEXT, F32)
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


def test_sampling_settings_reach_the_batch(rig):
    tsb, name = rig.tsb, "one_kv"
    s = rig.session(name, F32, streams=3)
    prompts = [rig.tokens(name, n, 70 + n) for n in (4, 20, 9, 30)]
    b = [12] * 4

    def serve(**kw):
        return [o.tolist() for o in s.serve(prompts, b, tsb.run_config(tsb.shaping(**kw), 12, 1))[0]]

    a = serve(temperature=1.0, seed=5)
    assert a == serve(temperature=1.0, seed=5) and a != serve(temperature=1.0, seed=6)
    assert serve(temperature=1.0, top_k=1, seed=5) == serve(temperature=0.0)
    pen = serve(temperature=1.0, top_k=1, repetition_penalty=1e6, seed=5)
    assert all(len(set(o)) == len(o) for o in pen) and all(not set(o) & set(p) or min(o) >= 0 for o, p in zip(pen, prompts))
    # a request's draws depend on its number and seed, not on its company
    rc = tsb.run_config(tsb.shaping(temperature=1.0, seed=5), 12, 1)
    assert s.serve(prompts[:1], b[:1], rc)[0][0].tolist() == a[0]
    _, seq, _ = s.sequential_run(prompts[0], rc)
    assert seq.tolist() == a[0]
    with pytest.raises(tsb.TsbError):
        s.serve([[1] * 600], [4], rc)
    s.close()


# ------------------------------------------------------------------ entry points
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_and_command_line(rig, tmp_path, dtype):
    name = "odd"
    type_ = F32 if dtype == "float32" else BF16
    folder = str(tmp_path / "model")
    nm.write_folder(folder, nm.CONFIGS[name], rig.weights[name])
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
    V = nm.CONFIGS[name]["vocab"]
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


def test_steps_of_a_block_quantised_model_equal_its_producer_calls(rig):
    tsb, ctx = rig.tsb, rig.ctx
    m = tsb.Model(ctx, tsb.ModelConfig(2, 256, 4, 2, 64, 512, 1024, 128, 1e-6, 1e4))
    m.fill_synthetic(tsb.Q4_K, seed=3)
    s = tsb.Session(ctx, m, None, 2, 4)
    t, u = list(range(3, 14)), list(range(50, 55))
    got = s.step([(1, t, [0, 5, 10]), (0, u, [4])])
    s2 = tsb.Session(ctx, m, None, 2, 4)
    a = [s2.produce(x, i, stream=0) for i, x in enumerate(t)]
    b = [s2.produce(x, i, stream=1) for i, x in enumerate(u)]
    assert got.dtype == np.uint16 and np.array_equal(got, np.stack([a[0], a[5], a[10], b[4]]))
    with pytest.raises(tsb.TsbError):
        s.serve([[1]], [1], tsb.run_config(tsb.shaping(temperature=0.0), 1, 1))
    with pytest.raises(tsb.TsbError):
        tsb.Session(ctx, m, None, 2, 4, step_rows=100)
    s.close(), s2.close(), m.close()


def test_a_model_with_a_missing_tensor_or_an_unsupported_size_is_refused(rig):
    tsb = rig.tsb
    cfg, layers = nigenex.parse_config(nm.CONFIGS["single"], 64)
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    w = dict(rig.weights["single"])
    nigenex.load_tensors(m, w.__getitem__)
    with pytest.raises(tsb.TsbError, match="must be"):
        m.set(5, np.zeros((3, 3), dtype=np.float32), layer=0)
    m.close()
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    with pytest.raises(tsb.TsbError, match="missing"):
        tsb.Session(rig.ctx, m, None, 1, 1)
    m.close()
    big = nm.config(64, 40, [nm.layer(1, 1, 300, 9, 16)])
    with pytest.raises(tsb.TsbError, match="head size"):
        tsb.PlainModel(rig.ctx, *nigenex.parse_config(big, 64))
