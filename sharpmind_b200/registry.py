"""Model registry: from a file or folder to a device model.

A GGUF file is a Llama / Qwen-shaped decoder (gguf.load_decoder).  A folder holds config.json, whose 'architecture' picks
the entry of ARCHITECTURES, and model.safetensors.  Every loader returns a decoder.StepModel.
"""
from __future__ import annotations

import json
import os

from . import ops


def _layered(ctx, folder, raw, max_seq, max_batch, act, max_chunk):
    from .layered import LayeredDecoder, read_config
    from .safetensors import SafetensorsFile

    return LayeredDecoder(ctx, read_config(raw), SafetensorsFile(os.path.join(folder, "model.safetensors")), max_batch=max_batch,
                          max_seq=max_seq, max_chunk=max_chunk, act=act)


# architecture name of config.json -> loader(ctx, folder, config, max_seq, max_batch, act, max_chunk)
ARCHITECTURES = {
    "Fitodra": _layered,
    "Molopel": _layered,
}


def load_model(ctx: ops.CudaContext, path: str, max_seq: int, max_batch: int = 1, act: str = "bfloat16", max_chunk: int = 2048):
    """`act`: "bfloat16", the form a model is served in (a GGUF model's quantised activations), or "float32"."""
    if act not in ("bfloat16", "float32"):
        raise ops.ArgumentException(f"activations in '{act}'")
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            raw = json.load(f)
        arch = raw.get("architecture")
        if arch not in ARCHITECTURES:
            raise ops.NotSupportedException(f"architecture '{arch}' ({', '.join(sorted(ARCHITECTURES))} are known)")
        return ARCHITECTURES[arch](ctx, path, raw, max_seq, max_batch, act, max_chunk)
    from .gguf import load_decoder

    model, _ = load_decoder(ctx, path, max_seq, max_batch)
    model.default_mode = ops.Mode.ACT_Q8 if act == "bfloat16" else ops.Mode.ACT_F32
    model.max_chunk = max_chunk
    return model


def describe(path: str) -> str:
    """One line per layer of a model folder, or the architecture of a GGUF file's folderless form."""
    if not os.path.isdir(path):
        return f"{path}: GGUF file"
    from .layered import read_config, tensor_shapes
    from .safetensors import SafetensorsFile

    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    if raw.get("architecture") not in ARCHITECTURES:
        raise ops.NotSupportedException(f"architecture '{raw.get('architecture')}'")
    cfg = read_config(raw)
    weights = os.path.join(path, "model.safetensors")
    held = SafetensorsFile(weights).tensors if os.path.exists(weights) else {}
    params = 0
    for name, shape in tensor_shapes(cfg).items():
        n = 1
        for i, d in enumerate(shape):  # a size the configuration leaves open is the file's
            n *= d if d is not None else (held[name]["shape"][i] if name in held else 0)
        params += n
    lines = [f"{raw['architecture']}: {len(cfg['layers'])} layers, width {cfg['hidden']}, vocabulary {cfg['vocab']}, {params} parameters"]
    for i, L in enumerate(cfg["layers"]):
        shared = f" (weights of layer {L['weights_of']})" if L["weights_of"] != i else ""
        m = L["mixer"]
        heads = " + ".join(str(m[k]["heads"]) for k in ("left", "right")) if L["type"] == "parallel" else m["heads"]
        lines.append(f"  {i}: {L['type']}, {heads} heads, ffn {L['ffn']}{shared}")
    return "\n".join(lines)
