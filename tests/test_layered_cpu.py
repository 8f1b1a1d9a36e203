"""Layered decoders without a GPU: configuration, safetensors files, registry, and the plain statement of the layers itself."""
import json

import numpy as np
import pytest

from oracle import layered_oracle as lo
from tests import layered_util as lu


def test_config_is_read_and_checked():
    from sharpmind_b200 import layered, ops

    cfg = lu.config([lu.latent(), lu.mamba(ff=0)])
    cfg["layers"].append(lu.share(cfg, 1))
    c = layered.read_config(cfg)
    assert c["hidden"] == 96 and c["alpha"] == 2.0 and [x["weights_of"] for x in c["layers"]] == [0, 1, 1] and c["layers"][1]["ffn"] == 0
    assert not any(k.startswith("l2.") for k in layered.tensor_shapes(c))
    cfg["layers"].append(lu.share(cfg, 2))  # shares what layer 2 shares
    assert [x["weights_of"] for x in layered.read_config(cfg)["layers"]] == [0, 1, 1, 1]
    for edit in (lambda d: d["layers"][1].update(weights_of=2), lambda d: d["layers"][0].update(type="retention"), lambda d: d["layers"][2].update(weights_of=0), lambda d: d["layers"][2].update(weights_of=7),
                 lambda d: d["layers"][0]["mlp"].update(kind="experts")):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises((ops.NotSupportedException, ops.ArgumentException)):
            layered.read_config(bad)


def test_safetensors_round_trip(tmp_path):
    import torch

    from sharpmind_b200.safetensors import SafetensorsFile

    cfg = lu.config([lu.latent(), lu.mamba()])
    t16, _ = lu.weights(cfg)
    lu.write_model(tmp_path, cfg, t16)
    f = SafetensorsFile(str(tmp_path / "model.safetensors"))
    assert sorted(f.tensors) == sorted(t16) and all(torch.equal(f[k], v) for k, v in t16.items())
    with pytest.raises(KeyError):
        f["nothing"]
    raw = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "short.safetensors").write_bytes(raw[:-10])
    with pytest.raises(ValueError):
        SafetensorsFile(str(tmp_path / "short.safetensors"))


def test_registry_describes_folders(tmp_path):
    from sharpmind_b200 import ops, registry

    cfg = lu.config([lu.latent(), lu.mamba()])
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    text = registry.describe(str(tmp_path))
    assert "Fitodra" in text and "latent_attention" in text and "mamba2" in text
    (tmp_path / "config.json").write_text(json.dumps(dict(cfg, architecture="Other")))
    with pytest.raises(ops.NotSupportedException):
        registry.describe(str(tmp_path))


def test_oracle_is_causal_and_windowed():
    cfg = lu.config([lu.latent(window=5)])
    _, w = lu.weights(cfg)
    tk = np.arange(30) % 19
    a = lo.forward(cfg, w, tk)
    tk2 = tk.copy()
    tk2[10] = 50
    b = lo.forward(cfg, w, tk2)
    d = np.abs(a - b).max(axis=1)
    assert d[:10].max() == 0 and d[10:15].min() > 1e-6 and d[15:].max() < 1e-12
    assert np.allclose(lo.forward(cfg, w, tk[:12]), a[:12])


def test_oracle_mechanisms_by_hand():
    # a convolution of two taps, a one-state recurrence, a softmax whose sink holds half the weight
    y = lo.causal_conv(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 1.0]]), np.array([0.5]))
    assert np.allclose(y[:, 0], [1.5, 12.5, 24.5])
    dt = np.full((3, 1), 0.5)
    y = lo.state_space(np.array([1.0, 0.0, 0.0]).reshape(3, 1, 1), np.ones((3, 1, 1)), np.full((3, 1, 1), 2.0), dt, np.zeros(1), np.array([3.0]), 1)
    assert np.allclose(y[:, 0, 0], [0.5 * 2 + 3, 0.5 * 2 * np.exp(-0.5), 0.5 * 2 * np.exp(-1.0)])
    o = lo.attend_window_sink(np.zeros((2, 2)), np.array([[2.0], [4.0]]), 0.0, 1)
    assert np.allclose(o[:, 0], [1.0, 2.0])
    f, fac = lo.rotary_frequencies(4, 100.0, None)
    assert np.allclose(f, [1.0, 0.1]) and fac == 1.0
    r = lo.rotate_halves(np.array([[1.0, 0.0, 0.0, 1.0]]), [2], f, 1.0)
    assert np.allclose(r, [[np.cos(2), -np.sin(0.2), np.sin(2), np.cos(0.2)]])
