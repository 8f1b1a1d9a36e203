"""Small random layered decoders for the tests: configurations, bfloat16 weights and their float64 twins."""
import copy

import numpy as np


def yarn(base=10000.0, dims=8, factor=2.5, original=64, fast=4.0, slow=1.0):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}


def latent(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, q_rank=56, window=11, scale=0.35, ff=72, rot=None):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": window}, "scale": scale, "rot": rot or yarn(dims=rot_dim)}}


def mamba(heads=6, vdim=8, state=24, groups=2, conv=4, norm_groups=3, ff=72):
    return {"type": "mamba2", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def lightning(heads=3, dim=24, vdim=16, decay=None, ff=72):
    return {"type": "lightning", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 0.6 / 4 ** i for i in range(heads)]}}


def parallel(heads=6, kv_heads=2, dim=24, vdim=16, window=11, scale=0.3, bias_max=40, right_heads=2, right_dim=16, right_vdim=24, rot_dims=12, base=500.0,
             decay=None, left_scale=0.8, right_scale=0.7, ff=72):
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale, "bias_max": bias_max},
                      "right": {"heads": right_heads, "dim": right_dim, "vdim": right_vdim, "rot": {"base": base, "dims": rot_dims},
                                "decay": decay or [1.0 - 2.0 ** (-2 - 3 * i) for i in range(right_heads)]},
                      "left_scale": left_scale, "right_scale": right_scale}}


def molopel(layers, width=96, vocab=160, eps=1e-5, scale=0.7, cap=12.0):
    return {"architecture": "Molopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "logit_softcap": cap,
            "layers": list(layers)}


def share(cfg, j):
    """A copy of layer j that uses layer j's weights."""
    return dict(copy.deepcopy(cfg["layers"][j]), weights_of=j)


def config(layers, width=96, vocab=160, eps=1e-5, alpha=2.0):
    return {"architecture": "Fitodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": list(layers)}


def weights(cfg, seed=0, gain=1.0, buckets=12):
    """name -> torch bfloat16 tensor, and the same numbers in float64.  `buckets`: rows of the distance tables."""
    import torch

    from sharpmind_b200 import layered

    rng = np.random.default_rng(seed)
    t16 = {}
    for name, shape in layered.tensor_shapes(layered.read_config(cfg)).items():
        last = name.split(".", 1)[-1]
        shape = tuple(buckets if n is None else n for n in shape)
        x = rng.standard_normal(shape)
        if last == "mix.left.rel":
            pass
        elif cfg["architecture"] == "Molopel" and last.endswith(("norm", "norm1", "norm2")):
            x = 1.0 + 0.2 * x
        elif len(shape) == 2 and not last.endswith("conv"):
            x *= 1.0 if name == "embed" else gain / np.sqrt(shape[1])
        elif last.endswith("conv"):
            x *= 0.5
        elif last in ("norm1", "norm2", "norm") and ".mix" not in name:
            x *= 0.1
        elif last in ("mix.dq.norm", "mix.dkv.norm", "mix.norm"):
            x = 1.0 + 0.1 * x
        elif last == "mix.A_log":
            x = rng.uniform(-3.0, 1.5, shape)
        elif last == "mix.dt_bias":
            x = rng.uniform(-4.0, 0.0, shape)
        elif last == "mix.sink":
            x = 1.0 + 0.5 * x
        else:
            x *= 0.3
        t16[name] = torch.from_numpy(np.asarray(x, np.float32)).to(torch.bfloat16)
    return t16, {k: v.to(torch.float64).numpy() for k, v in t16.items()}


def rel_err(got, want):
    """Per row: root mean square of the difference (mean taken off) over that of the wanted rows."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1)) / np.sqrt((w ** 2).mean())


def write_model(folder, cfg, t16):
    """config.json and model.safetensors."""
    import json

    import torch

    header, blobs, off = {}, [], 0
    for name, t in t16.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    (folder / "config.json").write_text(json.dumps(cfg))
    (folder / "model.safetensors").write_bytes(len(h).to_bytes(8, "little") + h + b"".join(blobs))
