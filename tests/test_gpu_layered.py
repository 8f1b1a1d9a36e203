"""Layered decoders (latent attention, Mamba-2, norm after the sum) against the plain float64 statement of the same layers."""
import json
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered_oracle as lo
from tests import layered_util as lu

pytestmark = pytest.mark.gpu

F32, BF16 = "float32", "bfloat16"
TOL = {F32: 3e-5, BF16: 7e-2}


def tiny(window=11, **kw):
    cfg = lu.config([lu.latent(window=window), lu.mamba(), lu.latent(window=window + 2, heads=2, kv_rank=24, vdim=24), lu.mamba(groups=3, norm_groups=1)], **kw)
    cfg["layers"] += [lu.share(cfg, 0), lu.share(cfg, 1)]
    return cfg


def build(cuda, cfg, t16, act, slots=2, max_seq=400, chunk=64):
    from sharpmind_b200.layered import LayeredDecoder, read_config

    return LayeredDecoder(cuda, read_config(cfg), t16, max_batch=slots, max_seq=max_seq, max_chunk=chunk, act=act)


def run(model, tokens, cuts=None):
    """Logits of every position, fed in portions of the sizes `cuts` (the rest in one)."""
    from sharpmind_b200.session import Session

    s = Session(model)
    s.open("a")
    out, at = [], 0
    for n in list(cuts or []) + [len(tokens)]:
        part = tokens[at:at + n]
        if len(part):
            out.append(s.feed("a", part, range(len(part))).cpu().numpy())
        at += len(part)
    s.close("a")
    return np.concatenate(out)


def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).astype(np.int32)


# ---------------------------------------------------------------------------------------- operations
@pytest.mark.parametrize("m", [1, 2, 7, 9, 17, 31, 33, 64, 129, 300])
@pytest.mark.parametrize("n,k", [(16, 32), (100, 192), (452, 80), (640, 200), (37, 36), (129, 1000)])
def test_dense_matmul(cuda, dev, m, n, k):
    import torch

    from sharpmind_b200 import ops

    g = torch.Generator().manual_seed(m * 1000 + n + k)
    w = torch.randn((n, k), generator=g).to(torch.bfloat16)
    x = torch.randn((m, k), generator=g)
    h = cuda.register_dev(w.cuda().view(torch.uint8).reshape(-1), ops.QuantDType.BF16, n, k, repack=False)
    want = x.double() @ w.double().T
    got = dev.qmatmul(x.cuda(), h, ops.Mode.ACT_F32).cpu().double()
    assert float((got - want).abs().max()) < 2e-6 * k ** 0.5 * 4
    want = x.to(torch.bfloat16).double() @ w.double().T
    got = dev.qmatmul(x.cuda(), h, ops.Mode.ACT_BF16).cpu().double()
    assert float((got - want).abs().max()) < 1e-5 * k ** 0.5 * 4
    with pytest.raises(ops.NotSupportedException):
        dev.qmatmul(x.cuda(), h, ops.Mode.ACT_Q8)
    cuda.release(h)


def test_dense_matmul_many_tiles(cuda, dev):
    """More tiles than CTAs, ragged edges: the persistent loop, both accumulators and every ring slot go round."""
    import torch

    from sharpmind_b200 import ops

    g = torch.Generator(device="cuda").manual_seed(5)
    m, n, k = 2100, 5000, 328
    w = torch.randn((n, k), generator=g, device="cuda").to(torch.bfloat16)
    x = torch.randn((m, k), generator=g, device="cuda")
    h = cuda.register_dev(w.view(torch.uint8).reshape(-1), ops.QuantDType.BF16, n, k, repack=False)
    got = dev.qmatmul(x, h, ops.Mode.ACT_BF16)
    want = x.to(torch.bfloat16).double() @ w.double().T
    assert float((got.double() - want).abs().max()) < 2e-4
    cuda.release(h)


@pytest.mark.parametrize("n", [8, 96, 1000])
@pytest.mark.parametrize("offset", [0.0, 1.0])
def test_scaled_add_rmsnorm(dev, n, offset):
    import torch

    rng = np.random.default_rng(n)
    x, y, w = rng.standard_normal((5, n)), rng.standard_normal((5, n)), 0.2 * rng.standard_normal(n)
    xd, x16 = torch.from_numpy(x.astype(np.float32)).cuda(), torch.empty((5, n), dtype=torch.bfloat16, device="cuda")
    dev.scaled_add_rmsnorm_(xd, torch.from_numpy(y.astype(np.float32)).cuda(), torch.from_numpy(w.astype(np.float32)).cuda(), 2.5, 1e-3, offset, x16)
    v = 2.5 * x + y
    want = lo.unit_rms(v, 1e-3) * (offset + w)
    assert np.abs(xd.cpu().numpy() - want).max() < 1e-5
    assert torch.equal(x16, xd.to(torch.bfloat16))


@pytest.mark.parametrize("rot", [lu.yarn(), lu.yarn(base=500.0, dims=24, factor=8.0, original=16, fast=32.0, slow=1.0),
                                 lu.yarn(dims=2), lu.yarn(dims=16, fast=1.0, slow=1.0), {"base": 777.0, "dims": 12}])
def test_yarn_tables(cuda, rot):
    import ctypes as C

    import torch

    from sharpmind_b200.layered import rotation

    n, half = 300, rot["dims"] // 2
    c, s = torch.empty((n, half), device="cuda"), torch.empty((n, half), device="cuda")
    r = rotation(rot)
    cuda.check(cuda.lib.smc_rope_tables_yarn(cuda.h, C.byref(r), n, c.data_ptr(), s.data_ptr()))
    f, fac = lo.rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    a = np.arange(n)[:, None] * f[None]
    assert np.abs(c.cpu().numpy() - np.cos(a) * fac).max() < 1e-6 and np.abs(s.cpu().numpy() - np.sin(a) * fac).max() < 1e-6


def test_embed_bf16(cuda, dev):
    import torch

    from sharpmind_b200 import ops

    w = torch.randn(50, 33).to(torch.bfloat16)
    h = cuda.register_dev(w.cuda().view(torch.uint8).reshape(-1), ops.QuantDType.BF16, 50, 33, repack=False)
    ids = torch.tensor([0, 49, 7, 7], dtype=torch.int32, device="cuda")
    assert torch.equal(dev.embed_bf16(h, ids).cpu(), w[ids.cpu().long()].float())
    cuda.release(h)


# ---------------------------------------------------------------------------------------- one mixer at a time
LATENTS = [
    dict(), dict(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, q_rank=8, window=1), dict(heads=5, dim=7, rot_dim=6, vdim=9, kv_rank=33, q_rank=21, window=4),
    dict(heads=2, dim=40, rot_dim=24, vdim=56, kv_rank=136, q_rank=24, window=50), dict(heads=4, dim=16, rot_dim=16, vdim=136, kv_rank=264, q_rank=16, window=7),
    dict(heads=17, dim=8, rot_dim=8, vdim=8, kv_rank=16, q_rank=64, window=100), dict(heads=2, dim=64, rot_dim=32, vdim=64, kv_rank=520, q_rank=40, window=33),
]
MAMBAS = [
    dict(), dict(heads=1, vdim=4, state=3, groups=1, conv=1, norm_groups=1), dict(heads=4, vdim=20, state=40, groups=4, conv=2, norm_groups=4),
    dict(heads=2, vdim=33, state=130, groups=1, conv=6, norm_groups=2), dict(heads=8, vdim=16, state=64, groups=2, conv=4, norm_groups=8),
    dict(heads=3, vdim=64, state=128, groups=3, conv=3, norm_groups=1), dict(heads=2, vdim=16, state=300, groups=2, conv=4, norm_groups=1),
]


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("layer", [lu.latent(**k) for k in LATENTS] + [lu.mamba(**k) for k in MAMBAS])
def test_one_layer(cuda, layer, act):
    cfg = lu.config([layer])
    t16, w = lu.weights(cfg, 3)
    tk = toks(150, cfg["vocab"])
    want = lo.forward(cfg, w, tk)
    m = build(cuda, cfg, t16, act, chunk=70)
    for cuts in ([], [20, 1, 1, 2, 40]):
        err = rel_err_max(run(m, tk, cuts), want)
        assert err < TOL[act], (cuts, err)
    m.close()


def rel_err_max(got, want):
    return float(lu.rel_err(got, want).max())


@pytest.mark.parametrize("act", [F32, BF16])
def test_no_feed_forward_and_odd_width(cuda, act):
    cfg = lu.config([lu.latent(ff=0), lu.mamba(ff=33), lu.latent(ff=51)], width=52, vocab=77, alpha=0.7, eps=1e-2)
    t16, w = lu.weights(cfg, 8)
    tk = toks(60, cfg["vocab"])
    m = build(cuda, cfg, t16, act)
    assert rel_err_max(run(m, tk), lo.forward(cfg, w, tk)) < TOL[act]
    assert rel_err_max(run(m, tk, [3] * 19), lo.forward(cfg, w, tk)) < TOL[act]
    m.close()


def test_residual_stream_layer_by_layer(cuda):
    cfg = tiny()
    t16, w = lu.weights(cfg, 1)
    tk, want = toks(40, cfg["vocab"]), []
    lo.forward(cfg, w, tk, want)
    for act, tol in ((F32, 2e-5), (BF16, 4e-2)):
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
    t16, w = lu.weights(cfg, 2)
    tk = toks(230, cfg["vocab"], 4)
    want = lo.forward(cfg, w, tk)
    m = build(cuda, cfg, t16, act)
    whole = run(m, tk)
    assert rel_err_max(whole, want) < TOL[act]
    for cuts in ([1] * 229, [2] * 114, [3] * 76, [16, 17, 18, 15] * 3, [64, 1, 63, 2, 62], [65, 66, 3], [100], [10, 11, 12, 13, 1, 2, 3]):
        got = run(m, tk, cuts)
        assert rel_err_max(got, want) < TOL[act], cuts
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_unequal_batch_against_each_alone(cuda, act):
    """Three sequences of different lengths decoded together (positions advanced on the device) and each alone."""
    import torch

    from sharpmind_b200.layered import POS_NEXT
    from sharpmind_b200.session import Session

    cfg = tiny()
    t16, w = lu.weights(cfg, 5)
    m = build(cuda, cfg, t16, act, slots=3)
    seqs = [toks(n, cfg["vocab"], n) for n in (3, 90, 31)]
    s = Session(m)
    for i, q in enumerate(seqs):
        assert s.open(i) == i
        s.feed(i, q[:-2] if len(q) > 2 else q)
    got = []
    for step in (-2, -1):
        batch = torch.tensor([int(q[step]) for q in seqs], dtype=torch.int32, device="cuda")
        got.append(m.step(batch, POS_NEXT)[0].cpu().numpy())
    for i, q in enumerate(seqs):
        want = lo.forward(cfg, w, q)[-2:]
        assert rel_err_max(np.stack([got[0][i], got[1][i]]), want) < TOL[act], i
    m.close()


def test_slots_are_used_again_and_interleave(cuda):
    cfg = tiny()
    t16, w = lu.weights(cfg, 6)
    m = build(cuda, cfg, t16, F32, slots=2)
    from sharpmind_b200.session import Session

    s = Session(m)
    a, b, c = toks(120, cfg["vocab"], 1), toks(45, cfg["vocab"], 2), toks(33, cfg["vocab"], 3)
    s.open("a"), s.open("b")
    outs = {"a": [], "b": []}
    for lo_, hi in ((0, 20), (20, 22), (22, 45)):
        for name, q in (("a", a), ("b", b)):
            outs[name].append(s.feed(name, q[lo_:hi], range(hi - lo_)).cpu().numpy())
    s.close("b")
    s.open("c")  # the slot that still holds b's state
    got_c = s.feed("c", c, range(33)).cpu().numpy()
    outs["a"].append(s.feed("a", a[45:], range(75)).cpu().numpy())
    assert rel_err_max(np.concatenate(outs["a"]), lo.forward(cfg, w, a)) < TOL[F32]
    assert rel_err_max(np.concatenate(outs["b"]), lo.forward(cfg, w, b)) < TOL[F32]
    assert rel_err_max(got_c, lo.forward(cfg, w, c)) < TOL[F32]
    s.close("a"), s.close("c")
    assert rel_err_max(run(m, b), lo.forward(cfg, w, b)) < TOL[F32]
    m.close()


def test_a_recurrence_is_not_continued_elsewhere(cuda):
    import torch

    from sharpmind_b200 import ops

    cfg = tiny()
    t16, _ = lu.weights(cfg, 6)
    m = build(cuda, cfg, t16, F32, max_seq=50)
    d = torch.from_numpy(toks(10, cfg["vocab"])).cuda()
    m.forward_rows(d, 0)
    assert m.sequence_length(0) == 10 and m.sequence_length(1) == 0
    for pos in (9, 11):
        with pytest.raises(ops.ArgumentOutOfRangeException):
            m.forward_rows(d, pos)
    with pytest.raises(ops.ArgumentOutOfRangeException):
        m.forward_rows(d, 45)
    with pytest.raises(ops.NotSupportedException):
        m.forward_rows(d, 10, mode=ops.Mode.ACT_Q8)
    m.forward_rows(d, 10)
    m.reset_sequence(0)
    m.forward_rows(d, 0)
    m.close()


# ---------------------------------------------------------------------------------------- things random weights hide
def needle_model(window, sink=None, scale=1.0):
    """One attention layer in which every query looks for one token: token 1's key matches all queries, its value is large.
    Rows of the logits say whether position i still sees the last token 1."""
    cfg = lu.config([lu.latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=32, q_rank=32, window=window, scale=scale, ff=0)], width=64, vocab=96, alpha=0.5)
    t16, _ = lu.weights(cfg, 11)
    import torch

    rng = np.random.default_rng(4)
    e = 0.3 * rng.standard_normal((96, 64))
    e[:, 0], e[:, 1] = 1.0, 0.0
    e[1, 1] = 6.0
    p = "l0.mix."

    def setw(name, a):
        t16[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16)

    setw("embed", e)
    dq = 0.02 * rng.standard_normal((32, 64))
    dq[0, 0] = 4.0                       # every query latent points along axis 0
    uq = 0.02 * rng.standard_normal((48, 32))
    uq[0, 0], uq[24, 0] = 1.0, 1.0       # first unrotated element of both heads
    dkv = 0.05 * rng.standard_normal((40, 64))
    dkv[:32, 2:] += 0.2 * rng.standard_normal((32, 62))
    dkv[0, 1] = 5.0                      # token 1's latent points along axis 0
    uk = 0.02 * rng.standard_normal((32, 32))
    uk[0, 0], uk[16, 0] = 0.5, 0.5
    setw(p + "dq", dq), setw(p + "uq", uq), setw(p + "dkv", dkv), setw(p + "uk", uk)
    if sink is not None:
        setw(p + "sink", np.full(2, sink))
    return cfg, t16, {k: v.double().numpy() for k, v in t16.items()}


@pytest.mark.parametrize("act", [F32, BF16])
@pytest.mark.parametrize("window", [1, 2, 16, 37, 64, 65, 100])
def test_window_edges(cuda, window, act):
    """A needle that is just inside and just outside the window, in prompts, in portions and decoded."""
    cfg, t16, w = needle_model(window, sink=0.0)
    n = 180
    tk = toks(n, 94, window) + 2
    tk[[0, 5, 70]] = 1
    want = lo.forward(cfg, w, tk)
    off = dict(cfg, layers=[json.loads(json.dumps(cfg["layers"][0]))])
    for delta in (1, -1):  # the oracle itself tells one token apart at the edges
        if window + delta < 1:
            continue
        off["layers"][0]["mixer"]["mask"]["size"] = window + delta
        diff = lu.rel_err(lo.forward(off, w, tk), want)
        edge = 70 + window - (1 if delta < 0 else 0)
        if edge < n:
            assert diff[edge] > 3 * TOL[act], (delta, diff[edge])
    m = build(cuda, cfg, t16, act, max_seq=200, chunk=48)
    for cuts in ([], [71 + window - 2 if 71 + window - 2 < n else 100, 1, 1, 1, 1], [1] * 179, [17, 19] * 4):
        err = lu.rel_err(run(m, tk, cuts), want)
        assert err.max() < TOL[act], (cuts, int(err.argmax()), float(err.max()))
    m.close()


@pytest.mark.parametrize("act", [F32, BF16])
def test_sink(cuda, act):
    outs = []
    for sink in (-30.0, 3.0, 6.0):
        cfg, t16, w = needle_model(20, sink=sink, scale=0.3)
        tk = toks(90, 94, 9) + 2
        tk[[0, 40]] = 1
        want = lo.forward(cfg, w, tk)
        m = build(cuda, cfg, t16, act, max_seq=100)
        for cuts in ([], [50] + [1] * 39):
            assert rel_err_max(run(m, tk, cuts), want) < TOL[act], sink
        outs.append(want)
        m.close()
    assert min(rel_err_max(outs[0], outs[1]), rel_err_max(outs[1], outs[2])) > 3 * TOL[act]


@pytest.mark.parametrize("act", [F32, BF16])
def test_state_remembers_far_tokens(cuda, act):
    """Slow decay and a loud first token: the state still shows it hundreds of tokens on."""
    import torch

    cfg = lu.config([lu.mamba(ff=0)], alpha=0.5)
    t16, _ = lu.weights(cfg, 12)
    t16["l0.mix.A_log"] = torch.full((6,), -7.0).to(torch.bfloat16)
    t16["l0.mix.dt_bias"] = torch.full((6,), -1.0).to(torch.bfloat16)
    w = {k: v.double().numpy() for k, v in t16.items()}
    tk = toks(390, cfg["vocab"], 3)
    other = tk.copy()
    other[0] = (tk[0] + 1) % cfg["vocab"]
    want = lo.forward(cfg, w, tk)
    assert lu.rel_err(lo.forward(cfg, w, other), want)[-1] > 3e-3
    m = build(cuda, cfg, t16, act)
    for cuts in ([], [64] + [1] * 40, [2] * 195, [5, 60, 61, 62, 63, 64]):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act], cuts
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

    cfg = tiny(alpha=0.4)
    t16, w = lu.weights(cfg, 15)
    m = build(cuda, cfg, t16, F32, slots=3, max_seq=120)
    prompts = [list(map(int, toks(n, cfg["vocab"], n))) for n in (4, 70, 1)]
    want = [lo.greedy(cfg, w, p, 12) for p in prompts]
    assert max(len(set(r)) for r in want) > 3
    assert generate(m, prompts, 12) == want
    assert generate(m, prompts[:1], 12, graph=False) == want[:1]
    assert generate(m, prompts[1:], 3, Sampling(temperature=0.8, top_k=1, seed=4)) == [r[:3] for r in want[1:]]
    m.close()


def test_lock_step_positions_and_passes(cuda):
    """smc_decode_step with a named position, ForwardLastLogits, Forward with hidden states: the entry points other models have."""
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
    assert rel_err_max(hidden.cpu().numpy() @ w["embed"].T, want[50:]) < TOL[F32]
    for pos in range(5):
        got = m.step(d[pos:pos + 1].repeat(2), pos)[0].cpu().numpy()
        assert rel_err_max(got, np.stack([want[pos]] * 2)) < TOL[F32]
    m.close()


def test_folder_command_line_and_trace(cuda, tmp_path):
    """A model folder through the registry, the command line and the trace replay, as child processes."""
    import os

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = tiny()
    t16, w = lu.weights(cfg, 17)
    lu.write_model(tmp_path, cfg, t16)
    prompt = list(map(int, toks(30, cfg["vocab"], 2)))
    want = lo.greedy(cfg, w, prompt, 5)
    r = subprocess.run([sys.executable, "-m", "sharpmind_b200", "generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, prompt)),
                        "--max-new", "5", "--dtype", "float32"], cwd=root, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, want))]
    logits = lo.forward(cfg, w, prompt)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[20:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": prompt[22:], "want": [0, 7]}], "end": ["x"]}]
    for act in (F32, BF16):
        out = tmp_path / act
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", act, "--out", str(out), "--max-tokens", "64"],
                           input="".join(json.dumps(s) + "\n" for s in steps), cwd=root, capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert not (out / "1.f32").exists()
        for step, places in ((0, [3, 19]), (2, [22, 29])):
            got = np.fromfile(out / f"{step}.f32", "<f4").reshape(2, -1)
            assert rel_err_max(got, logits[places]) < TOL[act]


# ---------------------------------------------------------------------------------------- head sizes of real models
def test_wide_heads_many_tiles(cuda):
    """Large heads and latents, several key tiles per CTA, two head groups, several chunks of states."""
    cfg = lu.config([lu.latent(heads=18, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96, window=333, scale=0.09, rot=lu.yarn(dims=64)),
                     lu.mamba(heads=4, vdim=64, state=128, groups=2, norm_groups=2), lu.mamba(heads=3, vdim=40, state=64, groups=1, norm_groups=5)],
                    width=128, vocab=128)
    t16, w = lu.weights(cfg, 21)
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

    cfg = lu.config([lu.latent(heads=20, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=48, window=150, rot=lu.yarn(dims=16)), lu.mamba()], width=64)
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


@pytest.mark.parametrize("act", [F32, BF16])
def test_norm_parts_differ_from_groups_and_gate_precedes_norm(cuda, act):
    """A loud gate in one part must not leak into the others' root mean square."""
    import torch

    cfg = lu.config([lu.mamba(heads=4, vdim=16, state=16, groups=4, norm_groups=2, ff=0)], alpha=0.3)
    t16, _ = lu.weights(cfg, 23)
    big = t16["l0.mix.in"].float()
    big[:32] *= 30.0  # z of the first two heads: the first part of the norm
    t16["l0.mix.in"] = big.to(torch.bfloat16)
    w = {k: v.double().numpy() for k, v in t16.items()}
    tk = toks(70, cfg["vocab"], 6)
    want = lo.forward(cfg, w, tk)
    other = json.loads(json.dumps(cfg))
    for parts in (1, 4):
        other["layers"][0]["mixer"]["norm_groups"] = parts
        assert rel_err_max(lo.forward(other, w, tk), want) > 2 * TOL[act]
    m = build(cuda, cfg, t16, act)
    for cuts in ([], [33, 1, 2, 3]):
        assert rel_err_max(run(m, tk, cuts), want) < TOL[act]
    m.close()
