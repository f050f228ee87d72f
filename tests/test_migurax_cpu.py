"""CPU: the plain Migurax statement against its own definition, the model registry and its
configuration checks (which need no GPU)."""
import copy
import os

import numpy as np
import pytest

import plain_migurax as plain
from conftest import package
from migurax_cases import MEMORY, MIXED, MODELS, UNEVEN, weights
from revitar_cases import write_model


def describe(folder):
    return package().backend.describe_model(str(folder))


def test_plain_rotation_by_hand():
    """Neighbouring columns are a pair; the first pair turns by the position itself."""
    x = np.array([[1.0, 0.0, 0.0, 2.0]])
    got = plain.rotate(x, [3], 100.0)[0]
    assert np.allclose(got, [np.cos(3), np.sin(3), -2 * np.sin(0.3), 2 * np.cos(0.3)])
    both = plain.rotate(np.stack([x, -x], 1), [3], 100.0)[0]  # heads turn alike
    assert np.allclose(both, [got, -got])


def test_plain_sink_by_hand():
    """One head, two keys: the sink is one more term of the denominator, unscaled."""
    c, k_rot = np.array([[1.0, 2.0], [0.5, -1.0]]), np.array([[1.0, 0.0], [0.0, 1.0]])
    uk, uv = np.array([[[2.0, 1.0]]]), np.array([[[1.0, 1.0], [0.0, 3.0]]])
    q, q_rot = np.array([[[0.5]]]), np.array([[[0.25, -1.0]]])
    got = plain.latent_attention_core(q, q_rot, c, k_rot, uk, uv, np.array([1]), np.arange(2), 2.0,
                                      np.array([0.7]))
    s0, s1 = 2 * (0.5 * 4 + 0.25), 2 * (0.5 * 0 - 1)
    v0, v1 = np.array([3.0, 6.0]), np.array([-0.5, -3.0])
    den = np.exp(s0) + np.exp(s1) + np.exp(0.7)
    assert np.allclose(got[0, 0], (np.exp(s0) * v0 + np.exp(s1) * v1) / den)


def test_plain_memory_is_a_weighted_sum():
    """The recurrence against its unrolled form: weights exp(sum of later f + i), one scale."""
    rng = np.random.Generator(np.random.PCG64(3))
    T, H, D, V = 12, 2, 5, 3
    q, k, v = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)), rng.standard_normal((T, H, V))
    i, f = rng.standard_normal((T, H)) * 2, plain.log_sigmoid(rng.standard_normal((T, H)) + 1)
    got, _ = plain.mlstm_core(q, k, v, i, f)
    for t in range(T):
        for h in range(H):
            w = np.array([f[j + 1:t + 1, h].sum() + i[j, h] for j in range(t + 1)])
            m = max(0 + f[:t + 1, h].sum(), w.max())
            e = np.exp(w - m)
            s = (q[t, h] * k[:t + 1, h]).sum(1)
            den = max(abs((e * s).sum()), np.exp(-m)) + 1e-6
            assert np.allclose(got[t, h], ((e * s)[:, None] * v[:t + 1, h]).sum(0) / den)


def test_plain_routing_is_a_softmax_over_the_chosen():
    chosen, weight = plain.route(np.eye(2), np.array([[1.0, 0.0], [0.0, 3.0], [2.0, 2.0]]),
                                 np.array([0.0, 0.0, -1.5]), 2)
    assert chosen.tolist() == [[0, 2], [1, 2]]
    e = np.exp([1.0, 0.5])
    assert np.allclose(weight[0], e / e.sum())


@pytest.mark.parametrize("name", sorted(MODELS))
def test_plain_model_is_causal(name):
    cfg = MODELS[name]
    w = weights(cfg, 5)
    rng = np.random.Generator(np.random.PCG64(6))
    tokens = rng.integers(0, cfg["vocab"], 24)
    whole = plain.logits(cfg, w, tokens)
    assert np.allclose(whole[:9], plain.logits(cfg, w, tokens[:9]), atol=1e-8)
    other = tokens.copy()
    other[11] = (other[11] + 1) % cfg["vocab"]
    moved = np.abs(plain.logits(cfg, w, other) - whole).max(axis=1)
    assert moved[:11].max() < 1e-8 and moved[11] > 1e-3 and moved[12:].min() > 1e-6


def test_describe(tmp_path):
    write_model(tmp_path, MIXED, {})
    d = describe(tmp_path)
    assert (d["architecture"], d["layers"], d["vocab"], d["width"]) == ("Migurax", 5, 203, 88)
    assert d["max_window"] == 0
    # cache rows are padded to eight elements: 44 + 10 and 64 + 24
    assert d["kv_bytes_per_token_bf16"] == 2 * (56 + 88)
    # per head and tile of 32 columns: the state, n and m of its own
    rec = lambda dim: dim * 32 + (dim + 3) // 4 * 4 + 4
    assert d["state_bytes_per_sequence"] == 4 * (3 * 2 * rec(24) + 2 * rec(36) + 3 * rec(70))
    write_model(tmp_path, MEMORY, {})
    assert describe(tmp_path)["kv_bytes_per_token_bf16"] == 0


@pytest.mark.parametrize("change, message", [
    (lambda c: c.pop("postln_alpha"), "'postln_alpha'"),
    (lambda c: c["norm"].pop("eps"), "'norm.eps'"),
    (lambda c: c["layers"][0].update(type="attention"), "mixer type 'attention'"),
    (lambda c: c["layers"][0].pop("mixer"), "no 'mixer'"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0), "'gate_cap' is not positive"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "'heads'"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "'q_rank'"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "'scale'"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rotates 8 of 10"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=-1), "'rot.base' is not positive"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "kind 'gated'"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "'ff'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top 8 of 7"),
])
def test_bad_configurations_are_refused(tmp_path, change, message):
    kb = package().backend
    cfg = copy.deepcopy(MIXED)
    change(cfg)
    write_model(tmp_path, cfg, {})
    with pytest.raises(kb.KansoError) as e:
        describe(tmp_path)
    assert e.value.code == kb.ERR_CONFIG and message in e.value.message


def test_library_of_the_class(tmp_path):
    build = package().build
    write_model(tmp_path, UNEVEN, {})
    assert build.model_class(str(tmp_path)) == "Migurax"
    for s in build.CORE + build.MODEL_CLASSES["Migurax"]:
        assert os.path.exists(os.path.join(build.CSRC, s + ".cu")), s
