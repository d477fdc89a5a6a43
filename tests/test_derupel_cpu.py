"""CPU: configuration, registry and the plain implementation of the Derupel model."""
import json

import numpy as np
import pytest

import _derupel as Z
import plain_derupel as P


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_config_round_trip(name):
    cfg = Z.CONFIGS[name]()
    from ytensor_b200.derupel import DerupelConfig
    assert DerupelConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_config_refuses_what_it_does_not_know():
    from ytensor_b200.derupel import DerupelLayer
    d = Z.decayed().to_dict()
    assert DerupelLayer.from_dict(dict(d, mlp=None)).mlp == 0
    for bad in (dict(d, type="something"), dict(d, mlp={"kind": "something"}),
                dict(d, mixer=dict(d["mixer"], decay=[0.5]))):
        with pytest.raises(ValueError):
            DerupelLayer.from_dict(bad)
    t = Z.latent().to_dict()
    with pytest.raises(ValueError):
        DerupelLayer.from_dict(dict(t, mixer=dict(t["mixer"], rot={"base": 10.0, "dims": 14})))


def test_registry_and_sources():
    from ytensor_b200 import registry
    from ytensor_b200.build import CSRC
    m = registry.find_model({"architecture": "Derupel"})
    assert m.dtypes == ("bfloat16", "float32")
    assert all((CSRC / (s + ".cu")).exists() for s in m.sources)


def test_command_line_lists_the_model(capsys):
    from ytensor_b200.__main__ import main
    assert main(["models"]) == 0
    assert "Derupel bfloat16 float32" in capsys.readouterr().out


# ---------------------------------------------------------------- the plain implementation itself
def test_plain_rotation_turns_neighbouring_pairs():
    x = np.zeros((2, 6))
    x[:, 0], x[:, 2], x[:, 4] = 1.0, 1.0, 1.0
    y = P.rotate(x, [0, 3], 100.0, 4)
    assert np.allclose(y[0], x[0])
    assert np.allclose(y[1], [np.cos(3), np.sin(3), np.cos(0.3), np.sin(0.3), 1.0, 0.0])
    a, b = np.random.default_rng(0).standard_normal((2, 1, 8))
    dots = [float((P.rotate(a, [p], 50.0, 8) @ P.rotate(b, [p + 5], 50.0, 8).T)[0, 0]) for p in (0, 7, 90)]
    assert np.allclose(dots, dots[0])  # only the distance counts


def test_plain_decayed_attention():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((7, 2, 3)), rng.standard_normal((7, 2, 3)), rng.standard_normal((7, 2, 4))
    w = [0.5, 1.0]
    out, state = P.decayed_attention(q, k, v, w)
    for h in range(2):
        for t in range(7):
            want = sum(w[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(out[t, h], want)
    a, mid = P.decayed_attention(q[:4], k[:4], v[:4], w)
    b, end = P.decayed_attention(q[4:], k[4:], v[4:], w, mid)
    assert np.allclose(np.concatenate([a, b]), out) and np.allclose(end, state)


def test_plain_experts():
    assert np.allclose(P.clamped_gate(np.array([9.0]), np.array([-9.0]), 2.0), 2.0 / (1 + np.exp(-3.404)) * -1.0)
    assert np.allclose(P.clamped_gate(np.array([-9.0]), np.array([9.0]), 2.0), -9.0 / (1 + np.exp(9 * 1.702)) * 3.0)
    assert P.route(np.array([0.1, 2.0, -1.0, 2.0]), 2)[0] == [1, 3]
    assert np.allclose(P.route(np.array([0.0, -3.0]), 1)[1], [0.5])
    assert np.allclose(P.squared_relu(np.array([-2.0, 3.0])), [0.0, 9.0])


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_plain_model_is_causal(name):
    cfg = Z.CONFIGS[name]()
    w = Z.floats(Z.weights(cfg, seed=len(name)))
    toks = np.random.default_rng(5).integers(0, cfg.vocab, 24).tolist()
    whole = P.forward(cfg.to_dict(), w, toks)
    assert np.allclose(P.forward(cfg.to_dict(), w, toks[:15]), whole[:15])
