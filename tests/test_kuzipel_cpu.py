"""Kuzipel models without a GPU: configuration, weight slots, and the oracle's mechanisms against other forms of the
same mathematics."""
import json

import numpy as np
import pytest

from mongoose_b200 import layered, registry
from mongoose_b200.layered import LAYER_SLOTS, LatentAttention, MixtureOfExperts, Wkv, slot_shapes
from mongoose_b200.safetensors import SafeTensors, from_bf16_bits
from oracle import layered as L
from tests import kuzipel_util as U


def read(tmp_path, cfg, w=None):
    U.write_folder(str(tmp_path), cfg, U.weights(cfg) if w is None else w)
    return registry.read_config(str(tmp_path))


def test_config_reader_takes_every_size_from_the_folder(tmp_path):
    arch, c = read(tmp_path, U.CONFIGS["mixed"])
    assert arch.name == "Kuzipel" and arch.family == "layered"
    assert (c.width, c.vocab, c.norm_eps, c.residual_mult, c.n_layers) == (88, 97, 1e-5, 0.7, 4)
    assert (c.norm, c.positions) == (layered.NORM_LAYER, layered.POS_NONE)
    assert c.runs() == (0, 1, 2, 1, 2, 3)
    assert c.layers[0].mixer == LatentAttention(5, 24, 12, 40, 36, 52, 36 ** -0.5, 10000.0)
    assert c.layers[1].mixer == Wkv(3, 24, 10)               # the rank is known from a tensor only
    assert c.layers[0].moe == MixtureOfExperts(6, 2, 40, 72) and c.layers[2].moe is None
    assert registry.kuzipel_config(U.CONFIGS["no_loop"], lambda t: (33, 0)).loop is None


@pytest.mark.parametrize("change", [
    lambda j: j["layers"][0].update(type="unheard"),
    lambda j: j["layers"][0]["mlp"].update(kind="dense"),
    lambda j: j["layers"][0]["mixer"]["rot"].update(dims=6),
    lambda j: j["layers"][0]["mixer"].update(rot_dim=11, rot={"base": 1e4, "dims": 11}),
    lambda j: j["layers"][0]["mixer"].pop("scale"),
    lambda j: j["layers"][0]["mlp"]["router"].update(top=7),
    lambda j: j["loop"].update(stop=5),
    lambda j: j["loop"].update(times=0),
    lambda j: j.pop("width"),
])
def test_config_reader_refuses_what_it_does_not_know(tmp_path, change):
    j = json.loads(json.dumps(U.CONFIGS["mixed"]))
    w = U.weights(j)
    change(j)
    with pytest.raises(registry.ConfigError):
        read(tmp_path, j, w)


def test_a_missing_tensor_is_reported(tmp_path):
    w = U.weights(U.CONFIGS["mixed"])
    del w["l1.mix.w1"]
    with pytest.raises(registry.ConfigError):
        read(tmp_path, U.CONFIGS["mixed"], w)


class Engine:
    def __init__(self, cfg):
        self.cfg, self.got = cfg, {}

    def SetWeightBF16(self, idx, bits):
        self.got[idx] = bits.copy()


@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_every_tensor_reaches_its_slot(tmp_path, name):
    cfg = U.CONFIGS[name]
    w = U.weights(cfg)
    arch, c = read(tmp_path, cfg, w)
    e, seen = Engine(c), set()
    arch.load_weights(e, SafeTensors(str(tmp_path / "model.safetensors")))
    for idx, slot, layer, rows, cols in slot_shapes(c):
        names = registry.kuzipel_tensors(c, slot, layer)
        stack = np.concatenate([w[t].reshape(-1) for t in names])
        assert stack.size == max(rows, 1) * cols
        assert np.array_equal(from_bf16_bits(e.got[idx]).reshape(-1), stack)
        assert idx // LAYER_SLOTS == (layer if layer >= 0 else c.n_layers)
        seen.update(names)
    assert seen == set(w) and len(e.got) == len(list(slot_shapes(c)))


def test_a_tensor_of_the_wrong_shape_is_refused(tmp_path):
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg)
    w["l0.mlp.e3.down"] = w["l0.mlp.e3.down"].T.copy()
    arch, c = read(tmp_path, cfg, w)
    with pytest.raises(registry.ConfigError):
        arch.load_weights(Engine(c), SafeTensors(str(tmp_path / "model.safetensors")))


def test_bytes_and_work_count_every_run_of_a_layer():
    def shape(tensor):
        return (8, 64)

    layers = [U.layer(U.wkv(2, 16, 8), U.moe(4, 1, 16, 8)), U.layer(U.latent(2, 16, 8, 16, 24, 32), None)]
    one = registry.kuzipel_config(U.config(64, 50, 1e-5, layers), shape)
    two = registry.kuzipel_config(U.config(64, 50, 1e-5, layers, loop=(0, 1, 2)), shape)
    wkv = 2 * (64 * (5 * 32 + 8) + 32 * 8 + 64 * (4 + 3 * 16 + 3 * 8 + 1))       # one of four experts
    assert layered.weight_bytes_per_token(two) - layered.weight_bytes_per_token(one) == wkv + 2 * 2 * 64 * 128
    assert layered.state_bytes(two) == 2 * layered.state_bytes(one) == 2 * 4 * (2 * 16 * 16 + 64)
    assert layered.cache_bytes_per_position(one) == 2 * (32 + 8)
    assert layered.prefill_flops(two, 10) > layered.prefill_flops(one, 10) > 0


# ---- the oracle -----------------------------------------------------------------------------------------

def test_oracle_is_causal():
    for name in ("mixed", "once"):
        cfg = U.CONFIGS[name]
        w = U.weights(cfg)
        toks = U.tokens(cfg, 40)
        full = U.want(cfg, w, toks)
        for n in (1, 2, 17):
            np.testing.assert_allclose(U.want(cfg, w, toks[:n]), full[:n], atol=1e-9)


def test_scores_of_folded_queries_equal_scores_of_formed_keys():
    """q . (U_k c) = (U_k^T q) . c, and U_v of the weighted latents equals the weighted values."""
    rng = np.random.default_rng(0)
    p = {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 5, "q_rank": 7, "kv_rank": 8, "scale": 0.4, "rot": {"base": 100.0, "dims": 4}}
    n, W, eps = 9, 12, 1e-5
    w = {k: rng.standard_normal(s) for k, s in {"dq": (7, W), "dq.norm": 7, "uq": (20, 7), "dkv": (12, W), "dkv.norm": 8, "uk": (12, 8),
                                               "uv": (10, 8), "o": (W, 10)}.items()}
    h = rng.standard_normal((n, W))
    got = L.latent_attention(h, w, p, eps)
    c = L.rms_norm(h @ w["dkv"][:8].T, w["dkv.norm"], eps)
    q = L.rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T
    for t in range(n):
        o = []
        for a in range(2):
            qa = w["uk"][6 * a:6 * a + 6].T @ q[t, 10 * a:10 * a + 6]
            s = np.array([qa @ c[j] for j in range(t + 1)])
            for j in range(t + 1):
                u = q[t, 10 * a + 6:10 * a + 8] + 1j * q[t, 10 * a + 8:10 * a + 10]
                kr = h[j] @ w["dkv"][8:].T
                z = (kr[:2] + 1j * kr[2:]) * np.exp(1j * (j - t) * 100.0 ** (-np.arange(2) / 2))
                s[j] += np.real(np.conj(u) @ z)             # the rotation of one against the other
            e = np.exp(p["scale"] * (s - s.max()))
            o.append(w["uv"][5 * a:5 * a + 5] @ (e @ c[:t + 1] / e.sum()))
        np.testing.assert_allclose(got[t], w["o"] @ np.concatenate(o), rtol=1e-9, atol=1e-9)


def test_recurrence_equals_its_sum_form():
    """o_t = sum over s < t of (r_t * k_s * w_(s+1) ... w_(t-1)) v_s, plus the current token with the bonus."""
    rng = np.random.default_rng(1)
    n, D = 12, 5
    r, k, v = (rng.standard_normal((n, D)) for _ in range(3))
    d, u = rng.uniform(0, 1, (n, D)), rng.standard_normal(D)
    S = np.zeros((D, D))
    for t in range(n):
        S, o = L.wkv_step(S, r[t], k[t], v[t], d[t], u)
        want = (r[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (r[t] * k[s] * np.prod(d[s + 1:t], axis=0)).sum() * v[s]
        np.testing.assert_allclose(o, want, rtol=1e-10, atol=1e-12)


def test_pieces():
    x = np.array([[1.0, 2.0, 3.0, 6.0]])                    # mean 3, mean squared deviation 3.5
    np.testing.assert_allclose(L.layer_norm(x, 2 * np.ones(4), 0.5), x - 3)
    np.testing.assert_allclose(L.rotate(np.array([[1.0, 0.0, 0.0, 1.0]]), [3], 100.0),
                               [[np.cos(3), -np.sin(0.3), np.sin(3), np.cos(0.3)]], atol=1e-12)
    np.testing.assert_allclose(L.token_shift(np.array([[1.0], [3.0]]), np.array([0.25])), [[0.75], [2.5]])
    np.testing.assert_allclose(L.channel_decay(np.zeros((1, 2)), np.ones((1, 2)), np.ones((1, 1)), np.array([0.0])), [[np.exp(-1)]])
    g = L.route(np.array([[0.0, 2.0, 1.0, -5.0]]), 2)
    np.testing.assert_allclose(g, [[0, np.e / (1 + np.e), 1 / (1 + np.e), 0]])
    np.testing.assert_allclose(L.silu(np.array([0.0, 1.0])), [0.0, 1 / (1 + np.exp(-1))])
    assert L.layer_runs(4, {"start": 1, "stop": 3, "times": 2}) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
