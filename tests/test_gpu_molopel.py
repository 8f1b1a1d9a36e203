"""Molopel (lightning attention, windowed attention beside retention, layer norm before each part) against the plain float64
statement of the same layers."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered_oracle as lo
from tests import layered_util as lu
from tests.test_gpu_layered import BF16, F32, TOL, build, rel_err_max, run, toks

pytestmark = pytest.mark.gpu


def tiny(window=11, **kw):
    return lu.molopel([lu.lightning(ff=0), lu.parallel(window=window), lu.lightning(heads=2, dim=16, vdim=40),
                       lu.parallel(heads=4, kv_heads=4, dim=16, vdim=24, window=window + 2, rot_dims=16, ff=0)], **kw)


def put(t16, name, a):
    import torch

    t16[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16)


def wide(t16):
    return {k: v.double().numpy() for k, v in t16.items()}


# ---------------------------------------------------------------------------------------- operations
@pytest.mark.parametrize("rows", [5, 700])
@pytest.mark.parametrize("n", [8, 97, 1000, 2048, 2052, 4096, 6000, 8200])
def test_layer_norm(dev, n, rows):
    import torch

    rng = np.random.default_rng(n)
    x, w = rng.standard_normal((rows, n)) + 3.0, 1.0 + 0.2 * rng.standard_normal(n)
    xd, wd = (torch.from_numpy(a.astype(np.float32)).cuda() for a in (x, w))
    want = lo.layer_norm(x.astype(np.float32).astype(np.float64), w.astype(np.float32).astype(np.float64), 1e-3)
    got = dev.layernorm(xd, wd, 1e-3)
    assert np.abs(got.cpu().numpy() - want).max() < 1e-5
    assert torch.equal(dev.layernorm(xd, wd, 1e-3, bf16=True), got.to(torch.bfloat16))


# ---------------------------------------------------------------------------------------- one mixer at a time
LIGHTNINGS = [
    dict(), dict(heads=1, dim=8, vdim=8), dict(heads=5, dim=7, vdim=9), dict(heads=2, dim=40, vdim=136), dict(heads=2, dim=136, vdim=24),
    dict(heads=2, dim=64, vdim=64, decay=[1.0, 0.01]), dict(heads=1, dim=264, vdim=16), dict(heads=3, dim=36, vdim=20), dict(heads=1, dim=128, vdim=128),
]
PARALLELS = [
    dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, window=1, right_heads=1, right_dim=8, right_vdim=8, rot_dims=2),
    dict(heads=5, kv_heads=5, dim=7, vdim=9, window=4, right_heads=3, right_dim=6, right_vdim=5, rot_dims=4),
    dict(heads=20, kv_heads=1, dim=16, vdim=40, window=50, right_dim=40, right_vdim=136, rot_dims=40),
    dict(heads=24, kv_heads=2, dim=40, vdim=24, window=33, bias_max=9), dict(heads=4, kv_heads=2, dim=136, vdim=264, window=100, bias_max=500),
    dict(heads=2, kv_heads=1, dim=264, vdim=16, window=7, right_heads=3, right_dim=24, right_vdim=64, rot_dims=8),
    dict(heads=4, kv_heads=1, dim=128, vdim=128, window=70, right_heads=4, right_dim=64, right_vdim=128, rot_dims=64),
    dict(heads=3, kv_heads=1, dim=32, vdim=12, window=19, right_heads=2, right_dim=12, right_vdim=20, rot_dims=12),
]


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("layer", [lu.lightning(**k) for k in LIGHTNINGS] + [lu.parallel(**k) for k in PARALLELS])
def test_one_layer(cuda, layer, act):
    cfg = lu.molopel([layer])
    t16, w = lu.weights(cfg, 3)
    tk = toks(290, cfg["vocab"])
    want = lo.forward(cfg, w, tk)
    m = build(cuda, cfg, t16, act, chunk=200)
    for cuts in ([], [20, 1, 1, 2, 140]):
        err = rel_err_max(run(m, tk, cuts), want)
        assert err < TOL[act], (cuts, err)
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_odd_width_small_cap_large_eps(cuda, act):
    cfg = lu.molopel([lu.parallel(ff=33), lu.lightning(ff=0), lu.parallel(ff=0), lu.lightning(ff=51)], width=52, vocab=77, eps=0.3, scale=3.0, cap=1.5)
    t16, w = lu.weights(cfg, 8, buckets=5)
    tk = toks(60, cfg["vocab"])
    want = lo.forward(cfg, w, tk)
    assert np.abs(want).max() > 0.95 * 1.5  # the cap is felt
    m = build(cuda, cfg, t16, act)
    for cuts in ([], [3] * 19, [40] + [1] * 20):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act]
    m.close()


def test_residual_stream_layer_by_layer(cuda):
    """With an embedding whose elements share an offset, so that the mean matters to every norm."""
    cfg = tiny(eps=1e-2)
    t16, _ = lu.weights(cfg, 1)
    put(t16, "embed", t16["embed"].float().numpy() + 1.5)
    w, tk, want = wide(t16), toks(40, cfg["vocab"]), []
    lo.forward(cfg, w, tk, want)
    for act, tol in ((F32, 2e-5), (BF16, 3e-2)):
        m = build(cuda, cfg, t16, act)
        dump = m.dump_layers()
        run(m, tk)
        for i, x in enumerate(want):
            got = dump[i, :40].cpu().numpy()
            assert np.sqrt(((got - x) ** 2).mean()) < tol * np.sqrt((x ** 2).mean()), (act, i)
        m.close()


# ---------------------------------------------------------------------------------------- cuts, slots, batches
@pytest.mark.parametrize("act", [F32, BF16])
def test_portions(cuda, act):
    cfg = tiny()
    t16, w = lu.weights(cfg, 4)  # (no head whose only score q . k is near zero at the first token: its norm would blow up rounding)
    tk = toks(390, cfg["vocab"], 4)
    want = lo.forward(cfg, w, tk)
    m = build(cuda, cfg, t16, act, chunk=300)
    assert rel_err_max(run(m, tk), want) < TOL[act]
    for cuts in ([1] * 389, [2] * 194, [3] * 129, [31, 32, 33, 34] * 2, [127, 1, 128, 2, 129], [128, 129, 3], [255, 2, 60], [257, 1, 1, 1], [300, 33]):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act], cuts
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_unequal_batch_against_each_alone(cuda, act):
    import torch

    from sharpmind_b200.layered import POS_NEXT
    from sharpmind_b200.session import Session

    cfg = tiny()
    t16, w = lu.weights(cfg, 5)
    m = build(cuda, cfg, t16, act, slots=3)
    seqs = [toks(n, cfg["vocab"], n) for n in (3, 190, 31)]
    s = Session(m)
    for i, q in enumerate(seqs):
        assert s.open(i) == i
        s.feed(i, q[:-2])
    got = []
    for step in (-2, -1):
        batch = torch.tensor([int(q[step]) for q in seqs], dtype=torch.int32, device="cuda")
        got.append(m.step(batch, POS_NEXT)[0].cpu().numpy())
    for i, q in enumerate(seqs):
        assert rel_err_max(np.stack([got[0][i], got[1][i]]), lo.forward(cfg, w, q)[-2:]) < TOL[act], i
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_slots_are_used_again_and_interleave(cuda, act):
    from sharpmind_b200.session import Session

    cfg = tiny()
    t16, w = lu.weights(cfg, 6)
    m = build(cuda, cfg, t16, act, slots=2)
    s = Session(m)
    a, b, c = toks(180, cfg["vocab"], 1), toks(45, cfg["vocab"], 2), toks(73, cfg["vocab"], 3)
    s.open("a"), s.open("b")
    outs = {"a": [], "b": []}
    for lo_, hi in ((0, 20), (20, 22), (22, 45)):
        for name, q in (("a", a), ("b", b)):
            outs[name].append(s.feed(name, q[lo_:hi], range(hi - lo_)).cpu().numpy())
    s.close("b")
    s.open("c")  # the slot that still holds b's ring and states
    got_c = np.concatenate([s.feed("c", c[:1], [0]).cpu().numpy(), s.feed("c", c[1:], range(72)).cpu().numpy()])
    outs["a"].append(s.feed("a", a[45:], range(135)).cpu().numpy())
    for got, q in ((np.concatenate(outs["a"]), a), (np.concatenate(outs["b"]), b), (got_c, c)):
        assert rel_err_max(got, lo.forward(cfg, w, q)) < TOL[act]
    s.close("a"), s.close("c")
    assert rel_err_max(run(m, b), lo.forward(cfg, w, b)) < TOL[act]
    m.close()


# ---------------------------------------------------------------------------------------- things random weights hide
def needle_model(window, heads=4, kv_heads=2):
    """One layer whose attention queries all look for token 1: its key matches them, its value is large, every other key is
    far from both.  Rows of the logits say whether a position still sees the last token 1."""
    cfg = lu.molopel([lu.parallel(heads=heads, kv_heads=kv_heads, dim=16, vdim=16, window=window, scale=1.0, left_scale=1.0, right_scale=0.01, ff=0)],
                     width=64, vocab=96, scale=1.0, cap=100.0)
    t16, _ = lu.weights(cfg, 11)
    rng = np.random.default_rng(4)
    e = 0.3 * rng.standard_normal((96, 64))
    e[:, 1], e[1, 1] = 0.0, 6.0
    p = "l0.mix.left."
    put(t16, "embed", e)
    put(t16, p + "q", 0.01 * rng.standard_normal((16 * heads, 64)))
    b = np.zeros((heads, 16))
    b[:, 0] = 3.0
    put(t16, p + "q.b", b.ravel())
    k = 0.05 * rng.standard_normal((kv_heads, 16, 64))
    k[:, 0] = 0.0
    k[:, 0, 1] = 3.0
    put(t16, p + "k", k.reshape(-1, 64))
    for n in ("k.b", "v.b", "rel"):
        put(t16, p + n, np.zeros(t16[p + n].shape))
    return cfg, t16, wide(t16)


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 37, 64, 65, 100])
def test_window_edges(cuda, window, act):
    """A needle just inside and just outside the window, in prompts, in portions and decoded."""
    cfg, t16, w = needle_model(window)
    n = 180
    tk = toks(n, 94, window) + 2
    tk[[0, 5, 70]] = 1
    want = lo.forward(cfg, w, tk)
    off = json.loads(json.dumps(cfg))
    for delta in (1, -1):  # the oracle itself tells one token apart at the edges
        if window + delta < 1:
            continue
        off["layers"][0]["mixer"]["left"]["mask"]["size"] = window + delta
        diff = lu.rel_err(lo.forward(off, w, tk), want)
        edge = 70 + window - (1 if delta < 0 else 0)
        if edge < n:
            assert diff[edge] > 3 * TOL[act], (delta, diff[edge])
    m = build(cuda, cfg, t16, act, max_seq=200, chunk=48)
    for cuts in ([], [min(69 + window, 100), 1, 1, 1, 1], [1] * 179, [17, 19] * 4, [2] * 90):
        err = lu.rel_err(run(m, tk, cuts), want)
        assert err.max() < TOL[act], (cuts, int(err.argmax()), float(err.max()))
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("buckets,reach,window", [(10, 60, 100), (16, 25, 64), (6, 200, 90), (2, 8, 40)])
def test_distance_bias_edges(cuda, buckets, reach, window, act, monkeypatch):
    """Biases that jump from bucket to bucket over faint keys: a distance counted one off shows."""
    cfg = lu.molopel([lu.parallel(heads=3, kv_heads=1, dim=16, vdim=16, window=window, scale=0.05, bias_max=reach, left_scale=1.0, right_scale=0.01, ff=0)],
                     scale=1.0, cap=50.0)
    t16, _ = lu.weights(cfg, 19, buckets=buckets)
    rng = np.random.default_rng(1)
    rel = np.where(rng.permuted(np.tile(np.arange(buckets) % 2, (3, 1)), axis=1).T == 1, 3.0, -3.0) + rng.standard_normal((buckets, 3))
    put(t16, "l0.mix.left.rel", rel)
    w, tk = wide(t16), toks(150, cfg["vocab"], 2)
    want = lo.forward(cfg, w, tk)
    bucket = lo.distance_bucket
    with monkeypatch.context() as mp:
        mp.setattr(lo, "distance_bucket", lambda n, r, d: bucket(n + 1, r, d))
        assert rel_err_max(lo.forward(cfg, w, tk), want) > 2 * TOL[act]
    m = build(cuda, cfg, t16, act, max_seq=160, chunk=100)
    for cuts in ([], [60] + [1] * 80, [33, 2, 2, 64]):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act], cuts
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("layer", [lu.lightning(heads=2, decay=[0.9999, 0.3], ff=0), lu.parallel(window=3, right_heads=2, decay=[0.9999, 0.5], left_scale=0.1, ff=0)])
def test_state_remembers_far_tokens(cuda, layer, act):
    """Slow decay and a loud first token: the state still shows it hundreds of tokens on, across chunks and portions."""
    cfg = lu.molopel([layer], scale=1.0, cap=50.0)
    t16, _ = lu.weights(cfg, 12)
    e = 0.4 * t16["embed"].float().numpy()
    e[3] *= 60.0
    put(t16, "embed", e)
    for name in ("v", "right.v"):  # the loud token's value stands out
        if "l0.mix." + name in t16:
            u = e[3] / np.linalg.norm(e[3])
            v = t16["l0.mix." + name].float().numpy()
            put(t16, "l0.mix." + name, v + 3.0 * np.outer(np.sign(v[:, 0]), u))
    w, tk = wide(t16), toks(390, cfg["vocab"] - 4, 3) + 4
    tk[0] = 3
    want = lo.forward(cfg, w, tk)
    other = tk.copy()
    other[0] = 9
    assert lu.rel_err(lo.forward(cfg, w, other), want)[-1] > (3 if act == F32 else 0.3) * TOL[act]
    m = build(cuda, cfg, t16, act, chunk=300)
    for cuts in ([], [64] + [1] * 40, [2] * 195, [5, 60, 61, 62, 63, 64], [128, 128, 128], [129, 127]):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act], cuts
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_heads_are_normed_alone_in_retention_and_together_in_lightning(cuda, act, monkeypatch):
    for layer, name in ((lu.parallel(right_heads=3, left_scale=0.05, ff=0), "l0.mix.right.v"), (lu.lightning(ff=0), "l0.mix.v")):
        cfg = lu.molopel([layer])
        t16, _ = lu.weights(cfg, 23)
        v = t16[name].float().numpy()
        v[:v.shape[0] // 3] *= 8.0  # a loud first head
        put(t16, name, v)
        w, tk = wide(t16), toks(70, cfg["vocab"], 6)
        want = lo.forward(cfg, w, tk)
        with monkeypatch.context() as mp:
            if "right" in name:
                mp.setattr(lo, "unit_rms", lambda x, eps: x / np.sqrt(np.mean(x * x, axis=tuple(range(1, x.ndim)), keepdims=True) + eps))
            else:
                plain = lo.unit_rms
                mp.setattr(lo, "norm_plain", lambda x, g, eps: plain(x.reshape(x.shape[0], 3, -1), eps).reshape(x.shape) * g)
            assert rel_err_max(lo.forward(cfg, w, tk), want) > 2 * TOL[act]
        m = build(cuda, cfg, t16, act)
        for cuts in ([], [33, 1, 2, 3]):
            assert rel_err_max(run(m, tk, cuts), want) < TOL[act]
        m.close()


def test_first_tokens(cuda):
    cfg = tiny()
    t16, w = lu.weights(cfg, 13)
    m = build(cuda, cfg, t16, F32)
    for n in (1, 2, 3, 4, 5):
        for cuts in ([], [1], [2]):
            tk = toks(n, cfg["vocab"], n)
            assert rel_err_max(run(m, tk, cuts), lo.forward(cfg, w, tk)) < TOL[F32]
    m.close()


def test_long_decoding_wraps_the_rings(cuda):
    import torch

    from sharpmind_b200.layered import POS_NEXT

    cfg = tiny()
    t16, w = lu.weights(cfg, 14)
    for act in (F32, BF16):
        m = build(cuda, cfg, t16, act, slots=1, max_seq=400, chunk=8)
        tk = toks(380, cfg["vocab"], 7)
        d = torch.from_numpy(tk).cuda()
        m.forward_rows(d[:5], 0)
        got = np.stack([m.step(d[i:i + 1], POS_NEXT)[0][0].cpu().numpy() for i in range(5, 380)])
        assert rel_err_max(got, lo.forward(cfg, w, tk)[5:]) < TOL[act]
        m.close()


# ---------------------------------------------------------------------------------------- the framework's own entry points
def test_greedy_generation(cuda):
    from sharpmind_b200.session import Sampling, generate

    cfg = tiny(scale=1.0)
    t16, w = lu.weights(cfg, 15, gain=2.0)
    m = build(cuda, cfg, t16, F32, slots=3, max_seq=120)
    prompts = [list(map(int, toks(n, cfg["vocab"], n))) for n in (4, 70, 1)]
    want = [lo.greedy(cfg, w, p, 12) for p in prompts]
    assert max(len(set(r)) for r in want) > 3
    assert generate(m, prompts, 12) == want
    assert generate(m, prompts[:1], 12, graph=False) == want[:1]
    assert generate(m, prompts[1:], 3, Sampling(temperature=0.8, top_k=1, seed=4)) == [r[:3] for r in want[1:]]
    m.close()


def test_lock_step_positions_and_passes(cuda):
    import torch

    cfg = tiny()
    t16, w = lu.weights(cfg, 16)
    m = build(cuda, cfg, t16, F32, slots=2, max_seq=100, chunk=32)
    tk = toks(60, cfg["vocab"], 8)
    want = lo.forward(cfg, w, tk)
    d = torch.from_numpy(tk).cuda()
    last, pick = m.forward_last_logits(d[:50], 0, 1)
    assert rel_err_max(last.cpu().numpy()[None], want[49:50]) < TOL[F32] and int(pick) == int(want[49].argmax())
    rows, picks, hidden = m.forward_logits(d[50:], 50, 1, want_hidden=True)
    assert rel_err_max(rows.cpu().numpy(), want[50:]) < TOL[F32] and np.array_equal(picks.cpu().numpy(), want[50:].argmax(1))
    cap = cfg["logit_softcap"]
    assert rel_err_max(cap * np.tanh(hidden.cpu().numpy() @ w["embed"].T / cap), want[50:]) < TOL[F32]
    for pos in range(5):
        got = m.step(d[pos:pos + 1].repeat(2), pos)[0].cpu().numpy()
        assert rel_err_max(got, np.stack([want[pos]] * 2)) < TOL[F32]
    m.close()


def test_folder_command_line_and_trace(cuda, tmp_path):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = tiny()
    t16, w = lu.weights(cfg, 17, gain=2.0)
    lu.write_model(tmp_path, cfg, t16)
    prompt = list(map(int, toks(40, cfg["vocab"], 2)))
    r = subprocess.run([sys.executable, "-m", "sharpmind_b200", "generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, prompt)),
                        "--max-new", "5", "--dtype", "float32"], cwd=root, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, lo.greedy(cfg, w, prompt, 5)))]
    logits = lo.forward(cfg, w, prompt)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:34], "want": [3, 33]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[34:36], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": prompt[36:], "want": [0, 3]}], "end": ["x"]}]
    for act in (F32, BF16):
        out = tmp_path / act
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", act, "--out", str(out), "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), cwd=root, capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (out / "1.f32").exists()
        for step, places in ((0, [3, 33]), (2, [36, 39])):
            got = np.fromfile(out / f"{step}.f32", "<f4").reshape(2, -1)
            assert rel_err_max(got, logits[places]) < TOL[act]


# ---------------------------------------------------------------------------------------- sizes of real models
def test_wide_heads_many_tiles(cuda):
    """Heads of 128, a window of several key tiles per warp, many chunks, matmuls on the tensor cores' tiles."""
    cfg = lu.molopel([lu.lightning(heads=4, dim=128, vdim=128, ff=320),
                      lu.parallel(heads=12, kv_heads=2, dim=128, vdim=128, window=333, scale=0.09, bias_max=256, right_heads=3, right_dim=128, right_vdim=128,
                                  rot_dims=64, ff=256),
                      lu.lightning(heads=2, dim=64, vdim=256, ff=0)], width=128, vocab=128)
    t16, w = lu.weights(cfg, 21, buckets=32)
    tk = toks(700, 128, 5)
    want = lo.forward(cfg, w, tk)
    m = build(cuda, cfg, t16, BF16, slots=2, max_seq=720, chunk=320)
    for cuts in ([], [300, 1, 1, 16, 2, 64, 65], [320, 10, 10, 300]):
        err = lu.rel_err(run(m, tk, cuts), want)
        assert err.max() < TOL[BF16], (cuts, int(err.argmax()), float(err.max()))
    m.close()


@pytest.mark.parametrize("slots", [5, 9, 18, 40])
def test_large_batches_decode_like_one(cuda, slots):
    """One token for each of many sequences: every cluster size of the attention and every width of the matmuls."""
    import torch

    from sharpmind_b200.layered import POS_NEXT
    from sharpmind_b200.session import Session

    cfg = lu.molopel([lu.parallel(heads=20, kv_heads=2, dim=32, vdim=32, window=150, right_heads=4), lu.lightning()], width=64)
    t16, w = lu.weights(cfg, 22)
    seqs = [toks(n, cfg["vocab"], n) for n in (4, 210, 77)]
    want = [lo.forward(cfg, w, q)[-1] for q in seqs]
    m = build(cuda, cfg, t16, BF16, slots=slots, max_seq=256)
    s = Session(m)
    for i in range(slots):
        s.open(i)
        s.feed(i, seqs[i % 3][:-1])
    batch = torch.tensor([int(seqs[i % 3][-1]) for i in range(slots)], dtype=torch.int32, device="cuda")
    got = m.step(batch, POS_NEXT)[0].cpu().numpy()
    assert rel_err_max(got, np.stack([want[i % 3] for i in range(slots)])) < TOL[BF16]
    m.close()
