"""Layer-described models on the GPU against the plain implementation in oracle/layered.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered as L
from tests import layered_util as U

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 3e-5, "bfloat16": 2e-2}
DTYPES = list(TOL)


def agree(got, ref, dtype, what=None):
    """Every row within the tolerance.  In bf16 one row in fifty may be up to six times off: where the memory's
    normaliser almost cancels, rounding alone moves the logits that far."""
    err = U.rel(got, ref)
    over = int((err > TOL[dtype]).sum())
    allowed = err.size // 50 if dtype == "bfloat16" else 0
    assert over <= allowed and err.max() < 6 * TOL[dtype], (what, over, int(err.argmax()), float(err.max()))


@pytest.fixture(scope="module")
def load(cuda, mglib, tmp_path_factory):
    """load(cfg, weights, dtype, max_seq) -> engine of a model folder, closed at the end."""
    from mongoose_b200 import registry
    made = []

    def make(cfg, w, dtype="float32", max_seq=320):
        path = tmp_path_factory.mktemp("model")
        U.write_folder(str(path), cfg, w)
        made.append(registry.load_model(str(path), dtype=dtype, max_seq=max_seq))
        return made[-1]

    yield make
    for e in made:
        e.close()


def portions(engine, toks, sizes):
    rows, p, i = [], 0, 0
    while p < len(toks):
        k = min(sizes[i % len(sizes)], len(toks) - p)
        rows.append(engine.Forward(toks[p:p + k], p, range(k)))
        p += k
        i += 1
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_prompt_portions_and_decoding(load, name, dtype):
    """A whole prompt, portions of several sizes, and one token at a time give the oracle's logits."""
    cfg = U.CONFIGS[name]
    w = U.weights(cfg, seed=3)
    toks = U.tokens(cfg, 203)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in ([203], [2], [64], [65, 3], [1], [1, 128, 2, 1, 63]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("branch", ["attention", "memory"])
def test_each_branch_alone(load, branch, dtype):
    """The other branch's output norm weight is zero, so only one mechanism reaches the logits."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=5)
    for i in range(len(cfg["layers"])):
        w[f"l{i}.mix.{'right' if branch == 'attention' else 'left'}.out"][:] = 0
    toks = U.tokens(cfg, 150)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in ([150], [1], [33, 2, 70]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


@pytest.mark.parametrize("f_bias,i_bias", [(-6.0, 0.0), (8.0, -6.0), (0.0, 6.0), (8.0, 4.0)])
def test_memory_gates_at_their_ends(load, f_bias, i_bias):
    """Fast forgetting, long memory, and input gates that push the running maximum."""
    cfg = U.config(48, 40, 1e-5, [U.layer(2, 2, 16, 0.2, 0.1, 10, 2, 20, 36, 7.0, 0)])
    w = U.weights(cfg, seed=7)
    w["l0.mix.left.out"][:] = 0
    w["l0.mix.right.f"] *= 4
    w["l0.mix.right.i"] *= 4
    w["l0.mix.right.f.b"][:] = f_bias
    w["l0.mix.right.i.b"][:] = i_bias
    toks = U.tokens(cfg, 260)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w)
    for sizes in ([260], [1], [64, 1, 2, 31]):
        assert U.rel(portions(e, toks, sizes), ref).max() < TOL["float32"]


def planted(cfg, w):
    """Weights under which one token's query meets only the key of another: the embedding's first half
    makes keys, its second half queries, through one matrix, so a token whose second half is another's
    first half finds that one.  The embedding drowns the position vector, other weights are near zero, and
    the mixer's output dominates the residual."""
    W, d = cfg["width"], cfg["layers"][0]["mixer"]["left"]["dim"]
    m = w["l0.mix.left.k"][:, :W // 2].copy()
    w["l0.mix.left.k"] = np.concatenate([m, 0 * m], axis=1)
    w["l0.mix.left.q"] = np.concatenate([0 * m, m], axis=1)
    w["l0.mix.left.q.norm"][:] = 1
    w["l0.mix.left.k.norm"][:] = 1
    w["l0.mix.left.pb"][:] = U.bf16(-0.85 * d)
    w["l0.mix.right.out"][:] = 0
    w["l0.norm1"][:] = 30
    w["embed"] = U.bf16(w["embed"] * 8)
    w["embed"][FINDER, W // 2:] = w["embed"][FOUND, :W // 2]
    return w


FINDER, FOUND, STAND_IN = 0, 1, 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys(load, dtype):
    """One far key decides the logits of one query, in a prompt, in a portion of two, and in decoding."""
    cfg = U.config(64, 400, 1e-5, [U.layer(4, 4, 24, 1.0, 0.0, 1, 1, 8, 8, 5.0, 0)])
    w = planted(cfg, U.weights(cfg, seed=11))
    e = load(cfg, w, dtype)
    at = 259
    for distance in (1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 200, 258, 259):
        toks = (3 + np.random.default_rng(2).permutation(397)[:260]).tolist()
        toks[at], toks[at - distance] = FINDER, FOUND
        ref = U.want(cfg, w, toks)[at]
        other = list(toks)
        other[at - distance] = STAND_IN
        lost = U.rel(U.want(cfg, w, other)[at][None], ref[None]).max()
        assert lost > 5 * TOL[dtype], "losing the key would not show"
        whole = e.Forward(toks, 0, [at])
        e.Forward(toks[:at], 0)
        decoded = e.Forward(toks[at:], at, [0])
        e.Forward(toks[:at - 1], 0)
        pair = e.Forward(toks[at - 1:], at - 1, [1])
        for got in (whole, decoded, pair):
            assert U.rel(got, ref[None]).max() < TOL[dtype], distance


def test_the_oracle_is_sensitive_to_each_mechanism():
    """A mistake planted in the oracle moves its logits far beyond the float32 tolerance."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=3)
    toks = U.tokens(cfg, 60)
    ref = U.want(cfg, w, toks)

    def moved(**changes):
        saved = {k: getattr(L, k) for k in changes}
        try:
            for k, v in changes.items():
                setattr(L, k, v)
            return U.rel(L.forward(cfg, w, toks), ref).max()
        finally:
            for k, v in saved.items():
                setattr(L, k, v)

    slopes = L.distance_slopes
    assert moved(query_temperature=lambda p, c, e: 1.0) > 1e-3
    assert moved(query_temperature=lambda p, c, e: 1.0 + c * np.log(p // e + 1)) > 1e-3
    assert moved(distance_slopes=lambda n: 0.5 * slopes(n)) > 1e-3
    assert moved(sinusoid=lambda p, n, base=10000.0: np.zeros(n)) > 1e-3
    step = L.mlstm_step
    assert moved(mlstm_step=lambda S, n, m, *r: step(S, n, -1e30, *r)) > 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
def test_query_temperature_steps(load, dtype):
    """Positions around every step of the temperature, a large coefficient."""
    cfg = U.config(64, 60, 1e-5, [U.layer(3, 3, 16, 0.3, 2.0, 13, 1, 8, 8, 5.0, 0)])
    w = U.weights(cfg, seed=13)
    w["l0.mix.right.out"][:] = 0
    toks = U.tokens(cfg, 70)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in ([70], [1], [13, 12]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_that_reuse_the_cache(load, dtype):
    """A request is independent of what the slot held before, with and without ResetKV, cut at an odd or
    even length."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=17)
    e = load(cfg, w, dtype)
    for seed, n, reset in ((1, 180, True), (2, 3, True), (3, 77, False), (4, 1, False), (5, 2, False), (6, 130, True)):
        toks = U.tokens(cfg, n, seed=seed)
        ref = U.want(cfg, w, toks)
        agree(e.Forward(toks, 0, range(n)), ref, dtype)
        if reset:
            e.ResetKV()
        agree(portions(e, toks, [1, 5]), ref, dtype)


def test_prompts_longer_than_a_block_of_rows(load):
    """One call that the engine cuts into blocks of rows, and attention into blocks of queries, equals
    portions that need no cutting, in 32-bit and (within its rounding) in bf16."""
    cfg = U.config(64, 90, 1e-5, [U.layer(32, 8, 8, 0.35, 0.3, 300, 2, 16, 24, 8.0, 48)])
    w = U.weights(cfg, seed=41)
    n = 2175
    toks = U.tokens(cfg, n)
    places = [0, 700, 1919, 1920, 1921, 2046, 2047, 2048, 2049, 2100, n - 1]
    e = load(cfg, w, max_seq=n)
    parts = portions(e, toks, [640])[places]
    assert U.rel(e.Forward(toks, 0, places), parts).max() < TOL["float32"]
    b = load(cfg, w, "bfloat16", max_seq=n)
    agree(b.Forward(toks, 0, places), parts, "bfloat16")
    short = 300                                     # the oracle on what it can do quickly
    assert U.rel(parts[:1], U.want(cfg, w, toks[:short])[places[:1]]).max() < TOL["float32"]
    agree(portions(b, toks[:short], [short]), U.want(cfg, w, toks[:short]), "bfloat16")


def test_long_decoding(load):
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=19)
    toks = U.tokens(cfg, 640)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, max_seq=640)
    e.Forward(toks[:40], 0)
    got = np.concatenate([e.Forward([t], 40 + i, [0]) for i, t in enumerate(toks[40:])])
    assert U.rel(got, ref[40:]).max() < TOL["float32"]


@pytest.mark.parametrize("name", ["mixed", "one_head"])
def test_greedy_generation(load, name):
    """Generate (prompt portion, captured decode steps, device-side argmax) against the oracle's greedy
    choice; a differing token must be a tie of the oracle's logits."""
    cfg = U.CONFIGS[name]
    w = U.weights(cfg, seed=23)
    e = load(cfg, w)
    for n in (1, 2, 3, 41):
        toks = U.tokens(cfg, n, seed=n)
        new = e.Generate(toks, 24).tolist()
        assert new == e.Generate(toks, 24).tolist()
        ref = U.want(cfg, w, toks + new[:-1])[n - 1:]
        top = ref.max(1)
        picked = ref[np.arange(24), new]
        assert (top - picked <= 1e-4 * np.abs(ref).max()).all()
        assert (ref.argmax(1) == np.array(new)).mean() > 0.9


def test_device_side_greedy_loop_continues_a_portion(load):
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=23)
    e = load(cfg, w)
    toks = U.tokens(cfg, 30)
    new = e.Generate(toks, 12).tolist()
    e.Forward(toks[:29], 0)
    e.SetCursor(toks[29], 29)
    e.EnqueueGreedy(12)
    assert e.GetCursor() == (new[-1], 41)


def test_layer_ranges_and_replay(load):
    """PartialStep over ranges of layers equals whole steps; captured steps equal plain launches."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=29)
    e = load(cfg, w)
    toks = U.tokens(cfg, 9)
    ref = U.want(cfg, w, toks)
    outs = []
    L.forward(cfg, w, toks, outs)
    hidden, logits = np.empty(cfg["width"], np.float32), np.empty(cfg["vocab"], np.float32)
    for p, t in enumerate(toks):
        x = (w["embed"][t] + L.sinusoid(p, cfg["width"])).astype(np.float32)
        e.PartialStep(x, p, 0, 1, hiddenOut=hidden)
        np.testing.assert_allclose(hidden, outs[0][p], atol=3e-5 * np.abs(outs[0]).max())
        e.PartialStepContinue(p, 1, 2, logitsOut=logits)
        assert U.rel(logits[None], ref[p][None]).max() < TOL["float32"]
        np.testing.assert_allclose(e.ExportHidden(), outs[1][p], atol=3e-5 * np.abs(outs[1]).max())
    assert e.ValidateGraphCapture(x, 0, 2) and e.last_validate_diff == 0.0


def test_steps_that_cannot_continue_are_refused(load):
    from mongoose_b200.fused_infer import MongooseError
    cfg = U.CONFIGS["one_head"]
    e = load(cfg, U.weights(cfg), max_seq=16)
    e.Forward([1, 2, 3], 0)
    for tokens, pos in (([1, 2], 2), ([1], 4), ([1] * 14, 3), ([1], -1), ([cfg["vocab"]], 3)):
        with pytest.raises(MongooseError):
            e.Forward(tokens, pos)
    with pytest.raises(MongooseError):
        e.Forward([1, 2], 3, [1, 0])
    e.Forward([1] * 13, 3)
    with pytest.raises(MongooseError):
        e.Forward([1], 16)
    with pytest.raises(MongooseError):
        e.EnqueueGreedy(1)


def test_bf16_weights_read_back_exactly(load):
    from mongoose_b200.layered import LAYER_SLOTS, SLOTS
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=31)
    e = load(cfg, w, "bfloat16")
    for name, slot in (("l1.mix.right.v", LAYER_SLOTS + SLOTS["mem.v"]), ("l0.mix.left.o", SLOTS["at.o"]), ("head", 2 * LAYER_SLOTS + 2)):
        assert np.array_equal(e.DequantRows(slot, 0, *w[name].shape), w[name])


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_and_generation_commands(load, tmp_path, dtype):
    """The two command-line programs on a model folder."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=37)
    model = U.write_folder(str(tmp_path / "m"), cfg, w)
    a, b = U.tokens(cfg, 21, seed=1), U.tokens(cfg, 6, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [16, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[18:], "want": [1, 2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [5]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model, "--dtype", dtype, "--out", str(out), "--max-tokens", "21"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb = U.want(cfg, w, a), U.want(cfg, w, b)
    for step, ref in ((0, ra[[16, 0]]), (2, ra[[19, 20]]), (3, rb[[5]])):
        got = np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert U.rel(got, ref).max() < TOL[dtype]
    assert not (out / "1.f32").exists()
    r = subprocess.run([sys.executable, "-m", "mongoose_b200.generate", "--model", model, "--dtype", dtype, "--prompt",
                        ",".join(map(str, a)), "--new", "5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    e = load(cfg, w, dtype)
    assert [int(t) for t in r.stdout.split(",")] == e.Generate(a, 5).tolist()
