"""Kuzipel models on the GPU against the plain implementation in oracle/layered.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered as L
from tests import kuzipel_util as U

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 3e-5, "bfloat16": 3e-2}
DTYPES = list(TOL)


def agree(got, ref, dtype, what=None):
    err = U.rel(got, ref)
    assert err.max() < TOL[dtype], (what, int(err.argmax()), float(err.max()))


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


CUTS = ([203], [2], [64], [65, 3], [1], [1, 128, 2, 1, 63])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_prompt_portions_and_decoding(load, name, dtype):
    """A whole prompt, portions of several sizes, and one token at a time give the oracle's logits."""
    cfg = U.CONFIGS[name]
    w = U.weights(cfg, seed=3, steady=dtype == "bfloat16")
    toks = U.tokens(cfg, 203)
    assert U.margin(cfg, w, toks) > (0.1 if dtype == "bfloat16" else 1e-5)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in CUTS:
        agree(portions(e, toks, sizes), ref, dtype, sizes)


SINGLE = {
    "latent": U.config(64, 60, 1e-5, [U.layer(U.latent(3, 20, 10, 28, 40, 44)), U.layer(U.latent(4, 12, 4, 8, 24, 72))], 0.9),
    "wkv": U.config(64, 60, 1e-5, [U.layer(U.wkv(3, 20, 12)), U.layer(U.wkv(2, 32, 6))], 0.9),
    "experts": U.config(64, 60, 1e-5, [U.layer(U.wkv(1, 8, 4), U.moe(7, 3, 48, 40)), U.layer(U.wkv(1, 8, 4), U.moe(3, 1, 56, 90))], 0.9),
    "loop": U.config(64, 60, 1e-5, [U.layer(U.wkv(1, 8, 4)), U.layer(U.wkv(1, 8, 4))], 0.9, (1, 2, 3)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_alone(load, name, dtype):
    """What does not belong to the mechanism is scaled to nothing, so that it alone reaches the logits."""
    cfg = SINGLE[name]
    w = U.weights(cfg, seed=5, steady=dtype == "bfloat16" and name == "experts")
    if name in ("experts", "loop"):
        for i in range(2):
            w[f"l{i}.ls1"][:] = 0
    toks = U.tokens(cfg, 150)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in ([150], [1], [33, 2, 70]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


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

    shift, step, route, rot, runs = L.token_shift, L.wkv_step, L.route, L.rotate, L.layer_runs
    assert moved(token_shift=lambda h, mu: h) > 1e-2
    assert moved(token_shift=lambda h, mu: shift(h, 1 - mu)) > 1e-2
    assert moved(wkv_step=lambda S, r, k, v, d, u: step(S, r, k, v, d, 1 + 0 * u)) > 1e-2
    assert moved(wkv_step=lambda S, r, k, v, d, u: step(S, r, k, v, d.max() + 0 * d, u)) > 1e-2
    assert moved(rotate=lambda x, p, base: x) > 1e-2
    assert moved(rotate=lambda x, p, base: rot(x, p + 1, base)) < 1e-9          # only differences of positions matter
    assert moved(rotate=lambda x, p, base: rot(x, p, 2 * base)) > 1e-3
    assert moved(route=lambda z, top: route(z, top - 1)) > 1e-2
    assert moved(route=lambda z, top: route(z, top) / 2) > 1e-2
    assert moved(layer_norm=lambda x, g, eps: L.rms_norm(x, g, eps)) > 1e-2
    assert moved(layer_runs=lambda n, loop: [(i, False) for i, _ in runs(n, loop)]) > 1e-2
    assert moved(sigmoid=lambda z: 0.5 + 0 * z) > 1e-2


FINDER, FOUND, STAND_IN = 0, 1, 2
DISTANCES = (1, 2, 15, 16, 17, 31, 32, 62, 63, 64, 65, 127, 128, 129, 191, 192, 193, 255, 256, 258, 259)


def far_key(heads, dim, rot):
    """One token's query meets only the key of another: channels of the embedding's first half become the latent
    and through it keys and values, channels of its second half the queries, by the same matrix, so a token whose
    second half is another's first half finds that one.  The rotated part is silenced."""
    W, half = 64, 32
    cfg = U.config(W, 400, 1e-6, [U.layer(U.latent(heads, dim, rot, 16, half, half, scale=1.0))], 40.0)
    w = U.weights(cfg, seed=11)
    rng = np.random.default_rng(12)
    # channels +-1 in pairs: every token has mean 0 and the same norm, which both norms then leave alone
    e = rng.choice([-1.0, 1.0], (400, W // 4))
    w["embed"] = np.repeat(e, 4, axis=1) * np.tile([1.0, -1.0], W // 2)
    w["embed"][FINDER, half:] = w["embed"][FOUND, :half]
    w["l0.norm1"][:] = 1
    w["l0.ls1"][:] = 1
    eye = np.eye(half)
    w["l0.mix.dkv"] = np.concatenate([np.concatenate([eye, 0 * eye], 1), np.zeros((rot, W))])
    w["l0.mix.dq"] = np.concatenate([0 * eye, eye], 1)
    w["l0.mix.dq.norm"][:] = 1
    w["l0.mix.dkv.norm"][:] = 1
    k = U.bf16(2.0 * rng.standard_normal((heads * dim, half)) / np.sqrt(dim))
    w["l0.mix.uk"] = k
    w["l0.mix.uq"] = np.concatenate([np.concatenate([k[h * dim:(h + 1) * dim], np.zeros((rot, half))]) for h in range(heads)])
    return cfg, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(3, 24, 8), (6, 40, 4)])
def test_far_keys(load, sizes, dtype):
    """One far key decides the logits of one query: in a prompt, in a portion of two, and in decoding."""
    cfg, w = far_key(*sizes)
    e = load(cfg, w, dtype)
    at = 259
    for distance in DISTANCES:
        toks = (3 + np.random.default_rng(2).permutation(397)[:260]).tolist()
        toks[at], toks[at - distance] = FINDER, FOUND
        ref = U.want(cfg, w, toks)[at]
        other = list(toks)
        other[at - distance] = STAND_IN
        lost = U.rel(U.want(cfg, w, other)[at][None], ref[None]).max()
        assert lost > 5 * TOL[dtype], ("losing the key would not show", distance, lost)
        whole = e.Forward(toks, 0, [at])
        e.Forward(toks[:at], 0)
        decoded = e.Forward(toks[at:], at, [0])
        e.Forward(toks[:at - 1], 0)
        pair = e.Forward(toks[at - 1:], at - 1, [1])
        for got in (whole, decoded, pair):
            assert U.rel(got, ref[None]).max() < TOL[dtype], distance


@pytest.mark.parametrize("dtype", DTYPES)
def test_growing_scores(load, dtype):
    """Scores that grow along the sequence by far more than a row's reference tolerates, then fall again."""
    cfg = U.config(64, 300, 1e-5, [U.layer(U.latent(2, 32, 8, 32, 48, 48, scale=0.6))], 3.0)
    w = U.weights(cfg, seed=21)
    w["l0.mix.dkv.norm"] = U.bf16(np.abs(w["l0.mix.dkv.norm"]) * 2)
    toks = U.tokens(cfg, 280, seed=4)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    tol = {"float32": 1e-4, "bfloat16": 6e-2}[dtype]        # near a hard maximum rounding of a score moves the weights
    for sizes in ([280], [100, 180], [279, 1]):
        assert U.rel(portions(e, toks, sizes), ref).max() < tol, sizes


@pytest.mark.parametrize("w0", [-9.0, -4.0, 0.0, 1.5, 4.0])
def test_decays_at_their_ends(load, w0):
    """Memory over hundreds of tokens, and channels that forget within one, side by side with channels of the
    other kind."""
    cfg = U.config(48, 40, 1e-5, [U.layer(U.wkv(2, 36, 8))], 2.0)
    w = U.weights(cfg, seed=7)
    w["l0.mix.w0"][:] = w0
    w["l0.mix.w0"][::5] = -w0
    toks = U.tokens(cfg, 300)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w)
    for sizes in ([300], [1], [64, 1, 2, 31]):
        assert U.rel(portions(e, toks, sizes), ref).max() < TOL["float32"], sizes


def test_a_far_token_in_the_recurrence(load):
    """With channels that hardly forget, the first token still shows hundreds of tokens later; every cut keeps it."""
    cfg = U.config(48, 40, 1e-5, [U.layer(U.wkv(2, 16, 4))], 2.0)
    w = U.weights(cfg, seed=9)
    w["l0.mix.w0"][:] = -12
    w["l0.mix.w2"][:] = 0
    for t in "rkv":
        w["l0.mix.mu." + t][:] = 0
    w["l0.mix.k"] *= U.bf16(0.25)
    toks = U.tokens(cfg, 260)
    toks[0] = 1
    other = [2] + toks[1:]
    ref = U.want(cfg, w, toks)
    assert U.rel(U.want(cfg, w, other)[-1:], ref[-1:]).max() > 30 * TOL["float32"], "losing the token would not show"
    e = load(cfg, w)
    for sizes in ([260], [1], [2], [129, 2, 64], [259, 1]):
        assert U.rel(portions(e, toks, sizes), ref).max() < TOL["float32"], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_last_token_is_carried_over_every_cut(load, dtype):
    """Mixes that read mostly the token before: a cut that lost it would show at the next position."""
    cfg = U.config(64, 60, 1e-5, [U.layer(U.wkv(2, 24, 6)), U.layer(U.wkv(2, 24, 6))], 2.0, (0, 1, 2))
    w = U.weights(cfg, seed=15)
    for i in range(2):
        for t in "rkvgw":
            w[f"l{i}.mix.mu.{t}"] = U.bf16(1.0 - 0.2 * w[f"l{i}.mix.mu.{t}"])
    toks = U.tokens(cfg, 40)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, dtype)
    for sizes in ([40], [1], [2], [3], [1, 2], [7, 1, 1, 2]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_expert_is_reached(load, dtype):
    """Each token's experts differ, and each expert alone decides the logits of some tokens; one of them, when it is
    silenced, shows."""
    cfg = U.config(64, 90, 1e-5, [U.layer(U.wkv(1, 8, 4), U.moe(10, 2, 24, 16))], 4.0)
    w = U.weights(cfg, seed=25, steady=True)
    w["l0.ls1"][:] = 0
    toks = list(range(90))
    ref = U.want(cfg, w, toks)
    for x in range(10):
        silent = dict(w, **{f"l0.mlp.e{x}.down": 0 * w[f"l0.mlp.e{x}.down"]})
        hit = U.rel(U.want(cfg, silent, toks), ref) > 5 * TOL[dtype]
        assert 1 <= hit.sum() < 60
    e = load(cfg, w, dtype)
    for sizes in ([90], [1], [2, 5]):
        agree(portions(e, toks, sizes), ref, dtype, sizes)


def test_many_tokens_for_one_expert(load):
    """More tokens than a tile of rows choose the same expert, others choose none."""
    cfg = U.config(64, 50, 1e-5, [U.layer(U.wkv(1, 8, 4), U.moe(6, 2, 24, 16))], 2.0)
    w = U.weights(cfg, seed=27)
    w["l0.mlp.router.b"] = U.bf16(np.array([30.0, 0.0, -30.0, 0.1, 0.2, -30.0]))
    toks = U.tokens(cfg, 300)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w)
    for sizes in ([300], [129, 128, 43]):
        agree(portions(e, toks, sizes), ref, "float32", sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_that_reuse_cache_and_state(load, dtype):
    """A request is independent of what the slot held before, with and without ResetKV."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=17, steady=dtype == "bfloat16")
    e = load(cfg, w, dtype)
    for seed, n, reset in ((1, 180, True), (2, 3, True), (3, 77, False), (4, 1, False), (5, 2, False), (6, 130, True)):
        toks = U.tokens(cfg, n, seed=seed)
        ref = U.want(cfg, w, toks)
        agree(e.Forward(toks, 0, range(n)), ref, dtype)
        if reset:
            e.ResetKV()
        agree(portions(e, toks, [1, 5]), ref, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_block_of_rows(load, dtype):
    """One call that the engine cuts into blocks of rows equals portions that need no cutting."""
    cfg = U.config(64, 90, 1e-5, [U.layer(U.latent(4, 24, 8, 24, 32, 40), U.moe(5, 2, 24, 40)), U.layer(U.wkv(4, 16, 8), U.moe(5, 2, 24, 40))], 0.8, (1, 2, 2))
    w = U.weights(cfg, seed=41, steady=dtype == "bfloat16")
    n = 2175
    toks = U.tokens(cfg, n)
    places = [0, 700, 1919, 1920, 2046, 2047, 2048, 2049, 2100, n - 1]
    e = load(cfg, w, max_seq=n)
    parts = portions(e, toks, [640])[places]
    if dtype == "float32":
        assert U.rel(e.Forward(toks, 0, places), parts).max() < TOL["float32"]
        short = 300
        assert U.rel(parts[:1], U.want(cfg, w, toks[:short])[places[:1]]).max() < TOL["float32"]
    else:
        b = load(cfg, w, "bfloat16", max_seq=n)
        agree(b.Forward(toks, 0, places), parts, "bfloat16")
        e.Forward(toks[:-1], 0)
        b.Forward(toks[:-1], 0)
        agree(b.Forward(toks[-1:], n - 1, [0]), e.Forward(toks[-1:], n - 1, [0]), "bfloat16")


def test_long_decoding(load):
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=19)
    toks = U.tokens(cfg, 640)
    ref = U.want(cfg, w, toks)
    e = load(cfg, w, max_seq=640)
    e.Forward(toks[:40], 0)
    got = np.concatenate([e.Forward([t], 40 + i, [0]) for i, t in enumerate(toks[40:])])
    assert U.rel(got, ref[40:]).max() < TOL["float32"]


@pytest.mark.parametrize("name", ["mixed", "loop_first", "loop_all"])
def test_greedy_generation(load, name):
    """Generate (prompt portion, captured decode steps, device-side argmax) against the oracle's greedy choice; a
    differing token must be a tie of the oracle's logits."""
    cfg = U.CONFIGS[name]
    w = U.weights(cfg, seed=23)
    e = load(cfg, w)
    for n in (1, 2, 3, 41):
        toks = U.tokens(cfg, n, seed=n)
        new = e.Generate(toks, 24).tolist()
        assert new == e.Generate(toks, 24).tolist()
        ref = U.want(cfg, w, toks + new[:-1])[n - 1:]
        picked = ref[np.arange(24), new]
        assert (ref.max(1) - picked <= 1e-4 * np.abs(ref).max()).all()
        assert (ref.argmax(1) == np.array(new)).mean() > 0.9


@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_layer_ranges_and_replay(load, name):
    """PartialStep over ranges of layer runs (a looped layer counts every time) equals whole steps; captured steps
    equal plain launches."""
    cfg = U.CONFIGS[name]
    w = U.weights(cfg, seed=29)
    e = load(cfg, w)
    runs = e.cfg.runs()
    toks = U.tokens(cfg, 9)
    outs = []
    ref = L.forward(cfg, w, toks, outs)
    assert len(outs) == len(runs)
    hidden, logits = np.empty(cfg["width"], np.float32), np.empty(cfg["vocab"], np.float32)
    for p, t in enumerate(toks):
        cut = [0, *sorted({1 + p % len(runs), 1 + (3 * p) % len(runs)}), len(runs)]
        x = np.ascontiguousarray(w["embed"][t], np.float32)
        for a, b in zip(cut, cut[1:]):
            if a == b:
                continue
            last = b == len(runs)
            out = {"logitsOut": logits} if last else {"hiddenOut": hidden}
            if a == 0:
                e.PartialStep(x, p, a, b, **out)
            else:
                e.PartialStepContinue(p, a, b, **out)
            if not last:
                np.testing.assert_allclose(hidden, outs[b - 1][p], atol=3e-5 * np.abs(outs[b - 1]).max())
        assert U.rel(logits[None], ref[p][None]).max() < TOL["float32"]
        np.testing.assert_allclose(e.ExportHidden(), outs[-1][p], atol=3e-5 * np.abs(outs[-1]).max())
    assert e.ValidateGraphCapture(x, 0, len(runs)) and e.last_validate_diff == 0.0


def test_bf16_weights_read_back_exactly(load):
    from mongoose_b200.layered import LAYER_SLOTS, SLOTS
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=31)
    e = load(cfg, w, "bfloat16")
    stack = np.concatenate([w[f"l0.mlp.e{x}.down"] for x in range(6)])
    for a, slot in ((w["l0.mix.uq"], SLOTS["la.uq"]), (w["l2.mix.uk"], 2 * LAYER_SLOTS + SLOTS["la.uk"]), (stack, SLOTS["moe.down"]),
                    (w["l1.mix.w2"], LAYER_SLOTS + SLOTS["wkv.w2"]), (w["loop.in"], 4 * LAYER_SLOTS + 3)):
        assert np.array_equal(e.DequantRows(slot, 0, *a.shape), a)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_and_generation_commands(load, tmp_path, dtype):
    """The two command-line programs on a model folder."""
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg, seed=37, steady=dtype == "bfloat16")
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
    r = subprocess.run([sys.executable, "-m", "mongoose_b200.generate", "--model", model, "--dtype", dtype, "--prompt",
                        ",".join(map(str, a)), "--new", "5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    e = load(cfg, w, dtype)
    assert [int(t) for t in r.stdout.split(",")] == e.Generate(a, 5).tolist()
