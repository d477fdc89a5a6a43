"""CPU: configuration, registry, weight files and the plain implementation of the Duzozen model."""
import json

import numpy as np
import pytest

import _duzozen as Z
import plain_lm as P


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_config_round_trip(name):
    cfg = Z.CONFIGS[name]()
    from ytensor_b200.duzozen import DuzozenConfig
    assert DuzozenConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_config_defaults_and_unknown_kinds():
    from ytensor_b200.duzozen import MLP_NONE, DuzozenLayer
    d = {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 4, "scale": 0.5, "mask": None}, "mlp": None}
    L = DuzozenLayer.from_dict(d)
    assert (L.window, L.softcap, L.v_mix, L.mlp) == (0, 0.0, False, MLP_NONE)
    with pytest.raises(ValueError):
        DuzozenLayer.from_dict(dict(d, type="something"))
    with pytest.raises(ValueError):
        DuzozenLayer.from_dict(dict(d, mlp={"kind": "something"}))
    r = {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 4, "top": 2}}
    L = DuzozenLayer.from_dict(dict(d, mlp=r))
    assert (L.identity, L.groups, L.keep) == (0, 1, 1)


def test_registry_knows_both_models():
    from ytensor_b200 import registry
    assert registry.find_model({"architecture": "Duzozen"}).dtypes == ("bfloat16", "float32")
    assert registry.find_model({"architectures": ["X", "Qwen3ForCausalLM"]}).name == "Qwen3ForCausalLM"
    with pytest.raises(registry.UnsupportedModel):
        registry.find_model({"architecture": "Nothing"})
    from ytensor_b200.build import CSRC
    for m in registry.MODELS.values():
        assert all((CSRC / (s + ".cu")).exists() for s in m.sources)


def test_command_line_lists_the_models(capsys):
    from ytensor_b200.__main__ import main
    assert main(["models"]) == 0
    assert "Duzozen bfloat16 float32" in capsys.readouterr().out


def test_safetensors_round_trip_and_damage(tmp_path):
    from ytensor_b200.safetensors import SafetensorsError, SafetensorsFile, write_safetensors
    t = {"a": np.arange(6, dtype=np.uint16).reshape(2, 3), "b": np.float32([1.5]), "s": np.uint16(7).reshape(())}
    write_safetensors(tmp_path / "x", t)
    f = SafetensorsFile(tmp_path / "x")
    assert sorted(f.names()) == ["a", "b", "s"] and f.dtype("a") == "BF16" and f.shape("s") == ()
    for n, a in t.items():
        assert np.array_equal(f[n], a)
    with pytest.raises(SafetensorsError):
        f["missing"]
    raw = (tmp_path / "x").read_bytes()
    (tmp_path / "y").write_bytes(raw[:-4])
    with pytest.raises(SafetensorsError):
        SafetensorsFile(tmp_path / "y")


def test_trace_runner_refuses_what_it_cannot_run(tmp_path):
    from ytensor_b200.trace import main
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    assert main(["--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "8"]) == 2
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Qwen3ForCausalLM"}))
    assert main(["--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "8", "--dtype", "float32"]) == 3


class _Fake:
    """Stands in for a model: logits of a position are (sequence length so far, token)."""

    def __init__(self):
        import torch
        self.torch, self.n, self.calls = torch, 0, []

    def reset_kv_cache(self):
        self.n = 0

    def forward(self, ids):
        self.n += ids.shape[1]
        self.calls.append(ids.shape[1])
        return self.torch.tensor([[float(self.n), float(ids[0, -1])]])

    def check_status(self):
        pass


def test_logits_at_places_of_a_model_that_computes_the_last_one_only():
    torch = pytest.importorskip("torch")
    from ytensor_b200.causal_lm import CausalLM
    m = _Fake()
    got = CausalLM.forward_at(m, torch.tensor([[5, 6, 7, 8, 9]], dtype=torch.int32), [1, 2])
    assert got.tolist() == [[2.0, 6.0], [3.0, 7.0]] and m.calls == [2, 1, 2]


# ---------------------------------------------------------------- the plain implementation itself
def test_plain_window_and_mixing():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 1, 4)), rng.standard_normal((6, 1, 3))
    full = P.attention(q, k, v, 0.5, None, None)
    one = P.attention(q, k, v, 0.5, None, 1)
    assert np.allclose(one, np.repeat(v, 2, 1)) and not np.allclose(full[3:], one[3:])
    assert np.allclose(P.attention(q, k, v, 0.5, None, 6), full)
    assert np.allclose(P.attention(q[4:], k, v, 0.5, 3.0, 4), P.attention(q, k, v, 0.5, 3.0, 4)[4:])
    assert np.allclose(P.mix_values(2.0, 6.0, 0.25), 3.0)


def test_plain_router_takes_the_correction_for_the_choice_only():
    z = np.log(np.array([0.4, 0.3, 0.2, 0.1]))
    assert P.route(z, np.zeros(4), 2, 1, 1)[0] == [0, 1]
    chosen, w = P.route(z, np.array([-5.0, 0, 0, -0.2]), 2, 1, 1)
    assert chosen == [1, 2] and np.allclose(w, [0.3, 0.2])
    # groups {0, 1} and {2, 3}: the correction lifts 3, its group wins, and negative choice scores still count
    chosen, w = P.route(z, np.array([-1.0, -1.0, -1.0, 0.5]), 2, 2, 1)
    assert chosen == [3, 2] and np.allclose(w, [0.1, 0.2])


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_plain_model_is_causal(name):
    """A sequence is causal: its prefix has the same logits."""
    cfg = Z.CONFIGS[name]()
    w = Z.floats(Z.weights(cfg, seed=len(name)))
    toks = np.random.default_rng(5).integers(0, cfg.vocab, 30).tolist()
    whole = P.forward(cfg.to_dict(), w, toks)
    assert np.allclose(P.forward(cfg.to_dict(), w, toks[:17]), whole[:17])
