"""Molopel without a GPU: configuration, registry, and the plain statement of its layers by hand."""
import json
import math

import numpy as np
import pytest

from oracle import layered_oracle as lo
from tests import layered_util as lu


def test_config_is_read_and_checked():
    from sharpmind_b200 import layered, ops

    cfg = lu.molopel([lu.lightning(ff=0), lu.parallel(), lu.lightning()])
    c = layered.read_config(cfg)
    assert (c["norm_place"], c["ffn_act"], c["embed_scale"], c["softcap"]) == (layered.NORM_BEFORE, layered.FFN_GELU_TANH, 0.7, 12.0)
    assert [x["ffn"] for x in c["layers"]] == [0, 72, 72]
    shapes = layered.tensor_shapes(c)
    assert shapes["l1.mix.left.rel"] == (None, 6) and shapes["l1.mix.left.k"] == (48, 96) and shapes["l1.mix.right.o"] == (96, 48)
    assert "l0.norm2" not in shapes and shapes["l0.mix.v"] == (48, 96)
    for edit in (lambda d: d["layers"][0].update(type="latent_attention"), lambda d: d["layers"][1]["mlp"].update(kind="experts"),
                 lambda d: d["layers"][0]["mixer"]["decay"].pop(), lambda d: d["layers"][1]["mixer"]["right"]["decay"].append(0.5),
                 lambda d: d.update(architecture="Fitodra"), lambda d: d.update(architecture="Nothing")):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        with pytest.raises((ops.NotSupportedException, ops.ArgumentException)):
            layered.read_config(bad)


def test_registry_describes_folders(tmp_path):
    from sharpmind_b200 import registry

    cfg = lu.molopel([lu.lightning(), lu.parallel()])
    t16, _ = lu.weights(cfg, buckets=10)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    text = registry.describe(str(tmp_path))
    assert "Molopel" in text and "lightning" in text and "6 + 2 heads" in text
    lu.write_model(tmp_path, cfg, t16)
    assert f"{sum(t.numel() for t in t16.values())} parameters" in registry.describe(str(tmp_path))


def test_distance_buckets():
    rows = [lo.distance_bucket(n, 8, 64) for n in range(200)]
    assert rows[:4] == [0, 1, 2, 3]                                     # one distance each
    assert rows[4] == 4 and rows[7] == 4 and rows[8] == 5 and rows[15] == 5 and rows[16] == 6 and rows[31] == 6  # doubling ranges
    assert rows[33] == 7 and set(rows[64:]) == {7}
    assert lo.distance_bucket(5, 2, 3) == 1 and lo.distance_bucket(0, 2, 3) == 0


def test_oracle_mechanisms_by_hand():
    y = lo.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 1.0]), 0.0)
    assert np.allclose(y, [[-2.0, 1.0]])
    y = lo.layer_norm(np.array([[1.0, 3.0]]), np.ones(2), 3.0)
    assert np.allclose(y, [[-0.5, 0.5]])
    assert lo.gelu_tanh(0.0) == 0 and abs(lo.gelu_tanh(30.0) - 30.0) < 1e-12 and abs(lo.gelu_tanh(-30.0)) < 1e-12
    assert abs(lo.gelu_tanh(1.0) - 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715))) < 1e-15
    one = np.ones((3, 1, 1))
    o = lo.decayed_sum(one, np.array([2.0, 0.0, 0.0]).reshape(3, 1, 1), one, [0.5])
    assert np.allclose(o[:, 0, 0], [2.0, 1.0, 0.5])


def test_oracle_is_causal_windowed_and_remembers():
    """A change at one place: later places see it through the window or the state, earlier ones do not."""
    for layer, far in ((lu.parallel(window=5, right_scale=0.0), False), (lu.parallel(window=5), True), (lu.lightning(), True)):
        cfg = lu.molopel([layer])
        _, w = lu.weights(cfg)
        tk = np.arange(30) % 19
        a = lo.forward(cfg, w, tk)
        tk2 = tk.copy()
        tk2[10] = 50
        d = np.abs(a - lo.forward(cfg, w, tk2)).max(axis=1)
        assert d[:10].max() == 0 and d[10:15].min() > 1e-7
        assert d[15:].min() > 1e-9 if far else d[15:].max() < 1e-12
        assert np.allclose(lo.forward(cfg, w, tk[:12]), a[:12])
