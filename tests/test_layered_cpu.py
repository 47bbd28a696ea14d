"""Layer-described models without a GPU: configuration, loader, trace replay, and the oracle itself."""
import json

import numpy as np
import pytest

from mongoose_b200 import registry, synthetic
from mongoose_b200.layered import LAYER_SLOTS, slot_shapes, weight_bytes_per_token
from mongoose_b200.safetensors import SafeTensors, from_bf16_bits, to_bf16_bits
from mongoose_b200.trace import Replay
from oracle import layered as L
from tests import layered_util as U


def test_config_reader_takes_every_size_from_the_file(tmp_path):
    cfg = U.CONFIGS["mixed"]
    U.write_folder(str(tmp_path), cfg, U.weights(cfg))
    arch, c = registry.read_config(str(tmp_path))
    assert arch.name == "Mitotar" and arch.family == "layered"
    assert (c.width, c.vocab, c.norm_eps, c.n_layers) == (80, 97, 1e-5, 2)
    a, m = c.layers[0].attn, c.layers[0].mem
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.temp_coef, a.temp_every) == (6, 3, 20, 0.3, 0.9, 7)
    assert (m.heads, m.dim, m.vdim, m.gate_cap) == (3, 24, 40, 5.0)
    assert (c.layers[0].ffn_dim, c.layers[1].ffn_dim) == (112, 0)


@pytest.mark.parametrize("change", [
    lambda j: j.update(architecture="Nothing"),
    lambda j: j["layers"][0].update(type="unheard"),
    lambda j: j["layers"][0]["mlp"].update(kind="routed"),
    lambda j: j["layers"][0]["mixer"]["left"].update(vdim=8),
    lambda j: j["layers"][0]["mixer"]["left"]["q_temp"].update(every=0),
    lambda j: j.pop("width"),
    lambda j: j["layers"][0]["mixer"].pop("right"),
])
def test_config_reader_refuses_what_it_does_not_know(tmp_path, change):
    j = json.loads(json.dumps(U.CONFIGS["mixed"]))
    change(j)
    (tmp_path / "config.json").write_text(json.dumps(j))
    with pytest.raises(registry.ConfigError):
        registry.read_config(str(tmp_path))


def test_every_slot_has_a_tensor_and_every_tensor_a_slot(tmp_path):
    for name, cfg in U.CONFIGS.items():
        w = U.weights(cfg)
        c = registry.mitotar_config(cfg)
        seen = set()
        for idx, slot, layer, rows, cols in slot_shapes(c):
            t = registry.mitotar_tensor(slot, layer)
            assert w[t].size == max(rows, 1) * cols, (name, t)
            assert idx == (layer * LAYER_SLOTS + idx % LAYER_SLOTS if layer >= 0 else c.n_layers * LAYER_SLOTS + idx % LAYER_SLOTS)
            seen.add(t)
        assert seen == set(w)


def test_weights_reach_the_engine_by_slot(tmp_path):
    class Engine:
        def __init__(self, cfg):
            self.cfg, self.got = cfg, {}

        def SetWeightBF16(self, idx, bits):
            self.got[idx] = bits.copy()

    cfg = U.CONFIGS["pairs"]
    w = U.weights(cfg)
    U.write_folder(str(tmp_path), cfg, w)
    arch, c = registry.read_config(str(tmp_path))
    e = Engine(c)
    arch.load_weights(e, SafeTensors(str(tmp_path / "model.safetensors")))
    for idx, slot, layer, rows, cols in slot_shapes(c):
        t = registry.mitotar_tensor(slot, layer)
        assert np.array_equal(from_bf16_bits(e.got[idx]).reshape(w[t].shape), w[t])
    bad = dict(w, head=w["head"][:, :-1])
    U.write_folder(str(tmp_path), cfg, bad)
    with pytest.raises(registry.ConfigError):
        arch.load_weights(Engine(c), SafeTensors(str(tmp_path / "model.safetensors")))


def test_bf16_conversion_rounds_to_nearest_even():
    a = np.array([1.0, 1.0 + 2 ** -8, 1.0 + 3 * 2 ** -8, 1.0 + 2 ** -8 + 2 ** -12, -3.1415927, 0.0, 1e-30], np.float32)
    got = from_bf16_bits(to_bf16_bits(a))
    assert got[0] == 1.0 and got[1] == 1.0 and got[2] == 1.0 + 2 ** -6 and got[3] == 1.0 + 2 ** -7
    assert np.array_equal(got, U.bf16(a))


def test_named_configurations():
    assert registry.named_config("tiny").name == "tiny"
    c = registry.named_config("mitotar-tiny")
    assert weight_bytes_per_token(c) == sum(2 * w.size for _, n, _, w in synthetic.layered_tensors(c) if w.ndim == 2 and n != "embed")
    with pytest.raises(registry.ConfigError):
        registry.named_config("nothing")


class FakeEngine:
    def __init__(self):
        self.cfg = type("C", (), {"vocab": 4})
        self.calls, self.resets = [], 0

    def ResetKV(self):
        self.resets += 1

    def Forward(self, tokens, pos, want):
        self.calls.append((list(tokens), pos, list(want)))
        return np.array([[pos + w] * 4 for w in want], np.float32)


def test_trace_replay_continues_requests_and_keeps_the_order_of_what_is_wanted():
    e = FakeEngine()
    r = Replay(e)
    got = r.step([{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], [])
    assert got[:, 0].tolist() == [2, 0]
    assert r.step([{"id": "a", "tokens": [4], "want": []}], []).shape == (0, 4)
    with pytest.raises(ValueError):
        r.step([{"id": "b", "tokens": [1], "want": []}], [])
    assert r.step([{"id": "a", "tokens": [5, 6], "want": [1]}], ["a"])[:, 0].tolist() == [5]
    assert r.step([{"id": "b", "tokens": [7], "want": [0]}], ["b"])[:, 0].tolist() == [0]
    assert [c[:2] for c in e.calls] == [([1, 2, 3], 0), ([4], 3), ([5, 6], 4), ([7], 0)]
    assert e.resets == 2


# ---- the oracle: its mechanisms against other forms of the same mathematics -------------------------------

def test_oracle_is_causal():
    cfg = U.CONFIGS["mixed"]
    w = U.weights(cfg)
    toks = U.tokens(cfg, 40)
    full = U.want(cfg, w, toks)
    for n in (1, 2, 17):
        np.testing.assert_allclose(U.want(cfg, w, toks[:n]), full[:n], atol=1e-9)


def test_memory_recurrence_equals_its_sum_form():
    """o_t = sum_s exp(F_t - F_s + i_s) (k_s . q_t) v_s over the same normaliser, F the log-forget sum."""
    rng = np.random.default_rng(0)
    n, D, V = 30, 5, 7
    q, k, v = (rng.standard_normal((n, d)) for d in (D, D, V))
    ig, fg = 2 * rng.standard_normal(n), L.log_sigmoid(rng.standard_normal(n))
    S, nrm, m = np.zeros((D, V)), np.zeros(D), 0.0
    F = np.cumsum(fg)
    for t in range(n):
        S, nrm, m, o = L.mlstm_step(S, nrm, m, q[t], k[t], v[t], ig[t], fg[t])
        a = np.exp(F[t] - F[:t + 1] + ig[:t + 1]) * (k[:t + 1] @ q[t])
        mt = max(F[t], (F[t] - F[:t + 1] + ig[:t + 1]).max())
        assert abs(m - mt) < 1e-12
        np.testing.assert_allclose(o, a @ v[:t + 1] * np.exp(-mt) / (max(abs(a.sum()) * np.exp(-mt), np.exp(-mt)) + 1e-6), rtol=1e-9, atol=1e-12)


def test_attention_pieces():
    assert L.query_temperature(6, 0.5, 7) == 1 + 0.5 * np.log(2) and L.query_temperature(5, 0.5, 7) == 1.0
    np.testing.assert_allclose(L.distance_slopes(4), [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    q = k = np.ones((3, 1, 4))
    a = L.gate_weights(q, k, 0.5, np.array([0.25]), np.array([-1.0]))[0]
    np.testing.assert_allclose(a[2], 1 / (1 + np.exp(-(2 - 0.25 * np.array([2, 1, 0]) - 1))))
    assert (a[0, 1:] == 0).all() and (a[1, 2:] == 0).all()
    np.testing.assert_allclose(L.gelu_tanh(np.array([0.0, 1.0])), [0.0, 0.841192], atol=1e-6)
    np.testing.assert_allclose(L.log_sigmoid(np.array([-800.0, 0.0, 800.0])), [-800.0, -np.log(2), 0.0], atol=1e-12)
    np.testing.assert_allclose(L.sinusoid(3, 4), [np.sin(3), np.cos(3), np.sin(0.03), np.cos(0.03)])
