"""Ronelorn models through the framework's own sessions, steps, loops and entry points, against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import ronelorn_oracle as ro
from tests import ronelorn_models as rm
from turbospark_b200 import ronelorn
from turbospark_b200.plain import BF16, F32

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {F32: 5e-5, BF16: 4e-2}
CONTEXT = 512


@pytest.fixture(scope="module")
def rig():
    """Models by (configuration, type) and oracle logits by (configuration, tokens), made once."""
    import turbospark_b200 as tsb
    ctx = tsb.Ctx(0)
    weights = {n: rm.random_weights(c, i) for i, (n, c) in enumerate(rm.CONFIGS.items())}
    models, logits = {}, {}

    class Rig:
        def model(self, name, type_):
            if (name, type_) not in models:
                models[name, type_] = ronelorn.build(ctx, rm.CONFIGS[name], weights[name].__getitem__, CONTEXT, type_)
            return models[name, type_]

        def logits(self, name, tokens):
            key = (name, tuple(tokens))
            if key not in logits:
                logits[key] = ro.forward(weights[name], rm.CONFIGS[name], list(tokens))
            return logits[key]

        def tokens(self, name, n, seed):
            return np.random.default_rng(seed).integers(0, rm.CONFIGS[name]["vocab"], size=n).tolist()

        def session(self, name, type_, streams=3, max_rows=1, pool=0, rows=700, draft=None, page=64):
            return tsb.Session(ctx, self.model(name, type_), draft, streams, max_rows, page_tokens=page, pool_tokens=pool, step_rows=rows)

    r = Rig()
    r.ctx, r.tsb, r.weights = ctx, tsb, weights
    yield r
    for m in models.values():
        m.close()
    ctx.close()


def check(got, want, type_, at=""):
    e = rm.logit_error(got, want)
    assert e.max() <= LIMIT[type_], (at, int(e.argmax()), float(e.max()))


NAMES = list(rm.CONFIGS)


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(rig, name, type_):
    """Lengths on both sides of windows, blocks, kept tokens, key tiles and pages, and of where recurrences go by runs."""
    s = rig.session(name, type_)
    t = rig.tokens(name, 300, 7)
    for i, n in enumerate([1, 2, 3, 31, 32, 41, 63, 64, 65, 128, 129, 300]):
        check(s.step([(i % 3, t[:n], list(range(n)))]), rig.logits(name, t)[:n], type_, n)
        s.reset(i % 3)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_equals_the_whole_prompt(rig, name, type_):
    s = rig.session(name, type_, streams=1)
    t = rig.tokens(name, 300, 7)
    got = np.stack([s.produce(tok, i) for i, tok in enumerate(t[:180])])
    check(got, rig.logits(name, t)[:180], type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("size", [2, 3, 7, 33, 64, 65, 100])
def test_portions(rig, name, type_, size):
    s = rig.session(name, type_, streams=2, page=16 if size == 33 else 64)
    t = rig.tokens(name, 300, 7)
    got = [s.step([(1, t[i:i + size], list(range(len(t[i:i + size]))))]) for i in range(0, len(t), size)]
    check(np.concatenate(got), rig.logits(name, t), type_)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
def test_a_step_larger_than_a_pass_and_than_the_logit_rows(rig, type_):
    """Steps are cut where they exceed what a pass holds; the answer stays the same."""
    t, u = rig.tokens("odd", 300, 7), rig.tokens("odd", 40, 3)
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
    equals the request alone, whatever pages, blocks, states and streams it got."""
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
@pytest.mark.parametrize("name", ["odd", "even", "large"])
def test_long_decoding(rig, name, type_):
    s = rig.session(name, type_, streams=2)
    t = rig.tokens(name, 420, 4)
    got = [s.step([(0, t[:20], [19])])]
    for i in range(20, 420):
        got.append(s.step([(0, t[i:i + 1], [0])]))
    check(np.concatenate(got), rig.logits(name, t)[19:], type_)
    s.close()


def test_many_rows(rig):
    """A batch of long portions, on the kernels for many queries and many tokens."""
    name = "even"
    s = rig.session(name, BF16, streams=4, rows=2048)
    reqs = [rig.tokens(name, n, 50 + i) for i, n in enumerate([500, 411, 77, 330])]
    got, r = s.step([(i, t, list(range(0, len(t), 7))) for i, t in enumerate(reqs)]), 0
    for t in reqs:
        n = len(range(0, len(t), 7))
        check(got[r:r + n], rig.logits(name, t)[::7], BF16)
        r += n
    s.close()


def test_the_bfloat16_residual_and_recurrence_stay_in_32_bits(rig):
    """A stream a thousand times larger than what the sublayers add to it, and gates that keep the state over hundreds of tokens: 16-bit sums would lose both."""
    cfg = rm.config(64, 48, [rm.mingru(32)] * 1 + [rm.kept(2, 1, 16, 16, 40, 3, None, rot=4)], mult=1.0, embed=1.0)
    w = rm.random_weights(cfg, 2)
    w["embed"][:, 0] = 4096.0  # one coordinate dominates every norm
    w["l0.mix.z.b"][:] = -6.0
    w["l0.mix.o"] = w["l0.mix.o"] * 64
    w["final.norm"][0], w["head"][:, 0] = -1.0, 0.0  # and is not read
    w["head"] = w["head"] * 256
    w = rm.rounded(w)
    model = ronelorn.build(rig.ctx, cfg, w.__getitem__, CONTEXT, BF16)
    s = rig.tsb.Session(rig.ctx, model, None, 1, 1, step_rows=512)
    t = np.random.default_rng(3).integers(0, 48, size=400).tolist()
    want = ro.forward(w, cfg, t)
    got = np.concatenate([s.step([(0, t[:300], list(range(300)))])] + [s.step([(0, [x], [0])]) for x in t[300:]])
    check(got, want, BF16)
    s.close(), model.close()


# ------------------------------------------------------------------ a far token that decides, the edges of windows, blocks and kept tokens
def sharp_model(entry, seed):
    """One attention layer in which the marked token's key answers the query of the asking token far above all others."""
    cfg = rm.config(64, 48, [entry], mult=1.0, embed=1.0)
    w = rm.random_weights(cfg, seed)
    m, mark, ask = entry["mixer"], 5, 7
    e = w["embed"]
    e[:, :2] = 0.0
    e[mark, 0], e[ask, 1] = 24.0, 24.0  # coordinate 0: "I am marked", coordinate 1: "I am asking"
    w["l0.norm1"][:2] = 0.0
    D = m["dim"]
    for name, heads, coordinate in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        x = w["l0.mix." + name] = w["l0.mix." + name] * 0.05
        x[:, :2] = 0.0
        x.reshape(heads, D, 64)[:, D - 1] = 0.0
        x.reshape(heads, D, 64)[:, D - 1, coordinate] = 1.0  # a column that does not turn
        w["l0.mix.%s.norm" % name][:] = 1.0
    w["l0.mix.o"] = w["l0.mix.o"] * 3
    return cfg, rm.rounded(w), mark, ask


def visible(entry, i, j):
    mask = entry["mixer"]["mask"]
    if i - j < mask["size"] or j < mask.get("keep_first", 0):
        return True
    pool = mask.get("pool", 0)
    return pool > 0 and j // pool * pool + pool - 1 <= i - mask["size"]


SHARP = [rm.pooled(4, 2, 16, 16, 70, 4, None, rot=8, cap=60.0, scale=3.0), rm.pooled(2, 1, 64, 64, 64, 3, None, rot=32, factor=2.0, cap=60.0, scale=0.7),
         rm.pooled(4, 1, 16, 8, 129, 5, None, rot=2, cap=60.0, scale=3.0), rm.kept(4, 2, 16, 16, 70, 4, None, rot=8, scale=1.0), rm.kept(2, 1, 64, 64, 128, 65, None, rot=32, scale=0.25),
         rm.kept(4, 4, 16, 24, 1, 1, None, rot=8, scale=1.0)]


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("at", range(len(SHARP)))
def test_a_far_key_and_both_sides_of_every_edge(rig, at, type_):
    entry = SHARP[at]
    cfg, w, mark, ask = sharp_model(entry, 3)
    mask, last = entry["mixer"]["mask"], 299
    model = ronelorn.build(rig.ctx, cfg, w.__getitem__, CONTEXT, type_)
    s = rig.tsb.Session(rig.ctx, model, None, 2, 1, step_rows=512)
    base = np.random.default_rng(1).integers(10, 48, size=last + 1).tolist()
    edge = last - mask["size"] + 1  # the first position of the window
    places = [edge, edge + 1, edge - 1, last - 1, 63, 64]
    if "pool" in mask:
        end = edge // mask["pool"] * mask["pool"]  # the first position of the first block that is not seen yet
        places += [end - 1, end - mask["pool"], end, end + mask["pool"] - 1, 0, 2]
    else:
        places += [mask["keep_first"] - 1, mask["keep_first"], 0]
    states = set()
    for n, place in enumerate(sorted({p for p in places if 0 <= p < last})):
        t = list(base)
        t[place], t[last] = mark, ask
        plain = list(base)
        plain[last] = ask
        want = ro.forward(w, cfg, t)[last:]
        shows = rm.logit_error(ro.forward(w, cfg, plain)[last:], want).max()
        seen = visible(entry, last, place)
        assert shows > 2.5 * LIMIT[BF16] if seen else shows < 1e-9, (place, shows)
        states.add(seen)
        for cut in ([last + 1], [last, 1], [200, last - 200, 1], [edge or 1, last + 1 - (edge or 1)], [place + 1, last - place]):
            at_, got = 0, None
            for m in cut:
                got = s.step([(n % 2, t[at_:at_ + m], [m - 1])])
                at_ += m
            s.reset(n % 2)
            check(got, want, type_, (place, cut))
    assert states == {True, False} or mask["size"] + mask.get("keep_first", 0) > last
    s.close(), model.close()


# ------------------------------------------------------------------ pool, refusals, rewinding
def test_a_step_that_does_not_fit_is_refused_and_changes_nothing(rig):
    s = rig.session("odd", F32, streams=3, pool=192)
    t = rig.tokens("odd", 300, 7)[:130]
    s.step([(0, t[:100], [])])
    with pytest.raises(rig.tsb.TsbError, match="pages"):
        s.step([(1, t[:70], [0]), (0, t[100:], [0])])
    check(s.step([(0, t[100:], list(range(30)))]), rig.logits("odd", rig.tokens("odd", 300, 7))[100:130], F32)
    s.close()


@pytest.mark.parametrize("type_", [F32, BF16])
@pytest.mark.parametrize("name", ["odd", "ones", "even"])
def test_cursors_go_back_as_far_as_the_states(rig, name, type_):
    """Rejected rows of a verify pass leave no trace - in blocks, states or rows; a state that is gone is not used."""
    s = rig.session(name, type_, streams=1, max_rows=6)
    t, u = rig.tokens(name, 90, 6), rig.tokens(name, 150, 7)
    s.step([(0, t[:57], [])])
    for i in range(57, 60):
        s.produce(t[i], i)
    mixed = t[:60]
    for keep in (2, 0, 5, 1, 3, 4):  # rounds of six rows of which some are kept
        base = s.checkpoint()
        s.verify(t[60:66], base)
        s.rollback_retaining(base, keep)
        mixed = mixed + t[60:60 + keep]
    assert s.checkpoint() == len(mixed)
    got = [s.produce(tok, len(mixed) + i) for i, tok in enumerate(u[:120])]
    check(np.stack(got), rig.logits(name, mixed + u[:120])[len(mixed):], type_)
    # a prefix that ends where no state is kept: the stream starts over
    assert s.try_reuse_prefix(mixed[:30] + [5, 6]) == 0
    fresh = mixed[:30] + [5, 6]
    check(s.step([(0, fresh, list(range(32)))]), rig.logits(name, fresh), type_)
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


@pytest.mark.parametrize("name", ["odd", "near"])
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
    # speculation with the model's first layers as the drafter, sharing their tensors, commits the same greedy tokens
    small = dict(rm.CONFIGS[name], layers=rm.CONFIGS[name]["layers"][:2])
    draft = ronelorn.build(rig.ctx, small, rig.weights[name].__getitem__, CONTEXT, F32)
    s = rig.session(name, F32, streams=2, max_rows=6, draft=draft)
    for i in (0, 4, 5):
        _, spec, res = s.spec_run(prompts[i], tsb.run_config(tsb.shaping(temperature=0.0), budgets[i], 4), stream=i % 2)
        assert np.array_equal(spec, out[i]) and res.rounds > 0
    s.close(), draft.close()


def test_speculative_rounds_of_several_streams_replay_as_a_graph(rig):
    """Lockstep rounds (a CUDA graph after the first) leave the tokens that the streams decode alone."""
    tsb, name = rig.tsb, "odd"
    small = dict(rm.CONFIGS[name], layers=rm.CONFIGS[name]["layers"][:2])
    cfg, layers = ronelorn.parse_config(small, CONTEXT, F32)
    draft = tsb.PlainModel(rig.ctx, cfg, layers)
    target = rig.model(name, F32)
    draft.share(-1, target, -1), draft.share(0, target, 3), draft.share(1, target, 1)  # a layer that itself uses another's tensors shares those
    s = rig.session(name, F32, streams=2, max_rows=5, draft=draft)
    prompts = [rig.tokens(name, 77, 60), rig.tokens(name, 77, 61)]
    rc = tsb.run_config(tsb.shaping(temperature=0.0), 1 << 20, 4)
    nxt = np.zeros(2, dtype=np.int32)
    for q, p in enumerate(prompts):
        s.step([(q, p[:-1], [])])
        nxt[q] = int(s.produce(p[-1], 76, stream=q).argmax())
        s.prime_drafter(p[-1], 75, stream=q)
    out = [[int(nxt[0])], [int(nxt[1])]]
    ctr = np.zeros(2, dtype=np.uint64)
    for _ in range(8):
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
    rm.write_folder(folder, rm.CONFIGS[name], rig.weights[name])
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
    V = rm.CONFIGS[name]["vocab"]
    read = lambda n: np.fromfile(out / ("%d.f32" % n), dtype="<f4").reshape(-1, V)
    whole = rig.logits(name, rig.tokens(name, 300, 7))
    check(read(0), whole[[0, 69]], type_)
    check(read(1)[:1], rig.logits(name, u)[8:9], type_)
    check(read(1)[1:], whole[99:100], type_)
    assert not (out / "2.f32").exists()
    if type_ == F32:
        r = subprocess.run([sys.executable, "-m", "turbospark_b200.generate", "--model", folder, "--dtype", dtype, "--max-new-tokens", "6", "--prompt",
                            " ".join(map(str, u)), "--prompt", "1,2"], capture_output=True, text=True, timeout=240, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        lines = [json.loads(l) for l in r.stdout.splitlines()]
        want = greedy(rig, name, u, 6)
        assert lines[0]["tokens"][:len(want)] == want and lines[0]["reason"] == "length" and len(lines[1]["tokens"]) == 6


def test_a_model_with_a_missing_tensor_or_an_unsupported_size_is_refused(rig):
    tsb, name = rig.tsb, "odd"
    cfg, layers = ronelorn.parse_config(rm.CONFIGS[name], 64)
    m = tsb.PlainModel(rig.ctx, cfg, layers)
    ronelorn.load_tensors(m, rig.weights[name].__getitem__)
    for which, shape, layer, match in ((tsb.plain.P_Q, (3, 3), 0, "must be"), (tsb.plain.P_FF_GATE, (88, 200), 0, "no tensor"), (tsb.plain.P_SINK, (6,), 2, "no tensor"),
                                       (tsb.plain.P_REC_NORM, (136,), 1, "no tensor"), (tsb.plain.P_Q, (240, 200), 3, "uses the tensors")):
        with pytest.raises(tsb.TsbError, match=match):
            m.set(which, np.zeros(shape, dtype=np.float32), layer=layer)
    m.close()
    for missing in ("l1.mix.z.b", "l2.mix.k.norm", "l4.mlp.up", "l0.norm2"):
        m = tsb.PlainModel(rig.ctx, cfg, layers)
        real = m.set
        lost = {"l1.mix.z.b": (tsb.plain.P_REC_F_BIAS, 1), "l2.mix.k.norm": (tsb.plain.P_K_NORM, 2), "l4.mlp.up": (tsb.plain.P_FF_UP, 4), "l0.norm2": (tsb.plain.P_NORM2, 0)}[missing]
        m.set = lambda which, a, layer=-1: None if (which, layer) == lost else real(which, a, layer=layer)
        ronelorn.load_tensors(m, rig.weights[name].__getitem__)
        with pytest.raises(tsb.TsbError, match="missing"):
            tsb.Session(rig.ctx, m, None, 1, 1)
        m.close()
    for bad in (rm.pooled(3, 2, 8, 8, 4, 2, None, rot=2), rm.kept(2, 1, 600, 8, 4, 2, None, rot=2), rm.kept(2, 1, 8, 300, 4, 2, None, rot=2)):
        with pytest.raises(tsb.TsbError):
            tsb.PlainModel(rig.ctx, *ronelorn.parse_config(rm.config(64, 40, [bad]), 64))
    good = ronelorn.parse_config(rm.config(64, 40, [rm.pooled(2, 1, 8, 8, 4, 2, 16, rot=2)]), 64)
    for change in (dict(window=0), dict(keep_first=3), dict(rot_dim=10), dict(rot_dim=3), dict(recurrence=tsb.plain.REC_MINGRU, rec_heads=1, rec_dim=1, rec_vdim=8), dict(sink=3),
                   dict(token_shift=1), dict(weights_of=7), dict(act=9), dict(qk_norm=0), dict(pool=-1)):
        layer = tsb.PlainLayer.from_buffer_copy(good[1][0])
        for k, v in change.items():
            setattr(layer, k, v)
        with pytest.raises(tsb.TsbError):
            tsb.PlainModel(rig.ctx, good[0], [layer])
