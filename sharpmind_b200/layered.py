"""Decoders described layer by layer: configuration, weight loading and the device model (smc_model_create_layered).

A configuration names for every layer its sequence mixer, the mixer's sizes and its feed-forward; `read_config` turns the
JSON form into the plain description `LayeredDecoder` takes.  Matrices stay bfloat16 on the device; projections that read the
same rows are joined (smc_weight_concat_rows), output projections that are summed lie side by side in one matrix, gate and up
rows are woven (smc_weight_interleave_rows).  A layer with 'weights_of' shares another layer's handles and has a state of its
own.

Architectures:  Fitodra  'latent_attention' and 'mamba2' mixers, an RMS norm after each sum, SiLU feed-forward
                Molopel  'lightning' and 'parallel' (windowed attention beside retention) mixers, a layer norm before each
                         part, GELU feed-forward, scaled embedding, soft-capped logits
"""
from __future__ import annotations

import ctypes as C

from . import ops
from .decoder import StepModel

MIX_LATENT, MIX_MAMBA2, MIX_HEADS = 1, 2, 3
NORM_AFTER, NORM_BEFORE = 0, 1
FFN_SILU, FFN_GELU_TANH = 0, 1
GATE_SILU, GATE_SIGMOID = 0, 1
POS_NEXT = -1  # StepModel.step: every slot's next position, taken from the device


class _Rotation(C.Structure):
    _fields_ = [("dims", C.c_int), ("base", C.c_double), ("factor", C.c_double), ("original", C.c_double), ("fast", C.c_double),
                ("slow", C.c_double)]


class _Attention(C.Structure):
    _fields_ = [("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("window", C.c_int), ("scale", C.c_float),
                ("out_scale", C.c_float), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("bias", C.c_void_p), ("buckets", C.c_int),
                ("bias_max", C.c_double)]


class _Linear(C.Structure):
    _fields_ = [("heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("silu", C.c_int), ("norm_parts", C.c_int), ("gate", C.c_int),
                ("k_scale", C.c_float), ("out_scale", C.c_float), ("rot", _Rotation), ("decay", C.POINTER(C.c_double)), ("mix_norm", C.c_void_p)]


class _Layer(C.Structure):
    _fields_ = [
        ("mixer", C.c_int), ("heads", C.c_int), ("vdim", C.c_int),
        ("dim", C.c_int), ("rot_dim", C.c_int), ("q_rank", C.c_int), ("kv_rank", C.c_int), ("window", C.c_int),
        ("scale", C.c_float), ("rot", _Rotation), ("w_down", C.c_void_p), ("w_uq", C.c_void_p), ("w_ukv", C.c_void_p),
        ("q_norm", C.c_void_p), ("kv_norm", C.c_void_p), ("sink", C.c_void_p),
        ("state", C.c_int), ("groups", C.c_int), ("conv", C.c_int), ("norm_groups", C.c_int), ("w_in", C.c_void_p),
        ("conv_w", C.c_void_p), ("conv_b", C.c_void_p), ("dt_bias", C.c_void_p), ("a_log", C.c_void_p), ("d_skip", C.c_void_p),
        ("mix_norm", C.c_void_p), ("w_out", C.c_void_p),
        ("attn", _Attention), ("linear", _Linear), ("b_in", C.c_void_p),
        ("ffn", C.c_int), ("w_gu", C.c_void_p), ("w_ffn_down", C.c_void_p), ("norm1", C.c_void_p), ("norm2", C.c_void_p),
    ]


class _Desc(C.Structure):
    _fields_ = [
        ("n_layers", C.c_int), ("hidden", C.c_int), ("vocab", C.c_int), ("max_seq", C.c_int), ("max_chunk", C.c_int),
        ("act_dtype", C.c_int), ("eps", C.c_float), ("alpha", C.c_float), ("layers", C.POINTER(_Layer)), ("embedding", C.c_void_p),
        ("final_norm", C.c_void_p), ("norm_place", C.c_int), ("ffn_act", C.c_int), ("embed_scale", C.c_float), ("softcap", C.c_float),
    ]


def rotation(rot: dict) -> _Rotation:
    s = rot.get("scaling") or {}
    return _Rotation(int(rot["dims"]), float(rot["base"]), float(s.get("factor", 0.0)), float(s.get("original", 0.0)),
                     float(s.get("fast", 0.0)), float(s.get("slow", 0.0)))


MIXERS = {"Fitodra": ("latent_attention", "mamba2"), "Molopel": ("lightning", "parallel")}


def read_config(raw: dict) -> dict:
    """The JSON configuration of a layered decoder, checked: {"vocab", "hidden", "eps", "layers": [...]} and what the
    architecture adds ("alpha" or "norm_place", "ffn_act", "embed_scale", "softcap")."""
    arch = raw["architecture"]
    if arch not in MIXERS:
        raise ops.NotSupportedException(f"architecture '{arch}'")
    layers = []
    for i, e in enumerate(raw["layers"]):
        kind, src = e["type"], e.get("weights_of", i)
        if kind not in MIXERS[arch]:
            raise ops.NotSupportedException(f"layer {i}: mixer '{kind}'")
        mlp = e.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ops.NotSupportedException(f"layer {i}: feed-forward '{mlp['kind']}'")
        for _ in range(len(raw["layers"])):  # a shared layer may name one that shares in turn
            if not 0 <= src < len(raw["layers"]):
                raise ops.ArgumentException(f"layer {i}: weights of layer {src}")
            if raw["layers"][src].get("weights_of", src) == src:
                break
            src = raw["layers"][src]["weights_of"]
        else:
            raise ops.ArgumentException(f"layer {i}: no layer owns its weights")
        if raw["layers"][src]["type"] != kind:
            raise ops.ArgumentException(f"layer {i} ({kind}) cannot use the weights of layer {src} ({raw['layers'][src]['type']})")
        m = e["mixer"]
        for part in [m] if kind == "lightning" else ([m["right"]] if kind == "parallel" else []):
            if len(part["decay"]) != part["heads"]:
                raise ops.ArgumentException(f"layer {i}: {len(part['decay'])} decays for {part['heads']} heads")
        layers.append({"type": kind, "weights_of": src, "mixer": dict(m), "ffn": int(mlp["ff"]) if mlp else 0})
    cfg = {"vocab": int(raw["vocab"]), "hidden": int(raw["width"]), "eps": float(raw["norm"]["eps"]), "layers": layers}
    if arch == "Fitodra":
        cfg["alpha"] = float(raw["postln_alpha"])
    else:
        cfg.update(norm_place=NORM_BEFORE, ffn_act=FFN_GELU_TANH, embed_scale=float(raw["embedding"]["scale"]),
                   softcap=float(raw["logit_softcap"] or 0.0))
    return cfg


def tensor_shapes(cfg: dict) -> dict:
    """Name -> shape of every tensor of a configuration; None where the file decides (the rows of a distance table)."""
    H = cfg["hidden"]
    out = {"embed": (cfg["vocab"], H), "final.norm": (H,)}
    for i, L in enumerate(cfg["layers"]):
        if L["weights_of"] != i:
            continue
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"] = (H,)
        if L["type"] == "latent_attention":
            h, dn, dr, dv, qr, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            out.update({p + "mix.dq": (qr, H), p + "mix.dq.norm": (qr,), p + "mix.uq": (h * (dn + dr), qr), p + "mix.dkv": (rk + dr, H),
                        p + "mix.dkv.norm": (rk,), p + "mix.uk": (h * dn, rk), p + "mix.uv": (h * dv, rk), p + "mix.sink": (h,),
                        p + "mix.o": (H, h * dv)})
        elif L["type"] == "lightning":
            n, inner = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({p + "mix.q": (n, H), p + "mix.k": (n, H), p + "mix.v": (inner, H), p + "mix.g": (inner, H), p + "mix.norm": (inner,),
                        p + "mix.o": (H, inner)})
        elif L["type"] == "parallel":
            a, r, pl, pr = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            n, inner = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({pl + "q": (q, H), pl + "q.b": (q,), pl + "k": (k, H), pl + "k.b": (k,), pl + "v": (v, H), pl + "v.b": (v,),
                        pl + "q.norm": (a["dim"],), pl + "k.norm": (a["dim"],), pl + "rel": (None, a["heads"]), pl + "o": (H, a["heads"] * a["vdim"]),
                        pr + "q": (n, H), pr + "k": (n, H), pr + "v": (inner, H), pr + "g": (inner, H), pr + "o": (H, inner)})
        else:
            h, inner, bc = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            ch = inner + 2 * bc
            out.update({p + "mix.in": (inner + ch + h, H), p + "mix.conv": (ch, m["conv"]), p + "mix.conv.b": (ch,), p + "mix.dt_bias": (h,),
                        p + "mix.A_log": (h,), p + "mix.D": (h,), p + "mix.norm": (inner,), p + "mix.o": (H, inner)})
        if L["ffn"]:
            out.update({p + "norm2": (H,), p + "mlp.gate": (L["ffn"], H), p + "mlp.up": (L["ffn"], H), p + "mlp.down": (H, L["ffn"])})
    return out


class LayeredDecoder(StepModel):
    """`tensors`: a mapping from tensor name to a torch tensor (CPU or CUDA), matrices in bfloat16.  `act`: "bfloat16"
    (activations and latent cache in bfloat16, the serving form) or "float32" (everything in fp32)."""

    def __init__(self, ctx: ops.CudaContext, cfg: dict, tensors, max_batch: int, max_seq: int, max_chunk: int = 2048, act: str = "bfloat16"):
        import torch

        self.torch, self.ctx, self.max_batch = torch, ctx, max_batch
        self.cfg = dict(cfg, max_seq=max_seq)
        self.act = act
        self.default_mode = {"bfloat16": ops.Mode.ACT_BF16, "float32": ops.Mode.ACT_F32}[act]
        self.max_chunk = min(max_chunk, max_seq)
        self._keep, self.weights = [], []
        self._dev = ops.DeviceOps(ctx)
        self.h = None
        shapes = tensor_shapes(cfg)

        def fetch(name):
            t = tensors[name]
            if len(t.shape) != len(shapes[name]) or any(w is not None and n != w for n, w in zip(t.shape, shapes[name])):
                raise ops.InvalidOperationException(f"tensor '{name}' is {tuple(t.shape)}, the configuration needs {shapes[name]}")
            return t

        def matrix(name):
            t = fetch(name)
            if t.dtype != torch.bfloat16:
                raise ops.NotSupportedException(f"tensor '{name}' is {t.dtype}; matrices are bfloat16")
            return t

        def mat(*names):
            """One matrix, or several side by side (their products are summed)."""
            t = torch.cat([matrix(n) for n in names], dim=1).contiguous().cuda()
            return ctx.register_dev(t.view(torch.uint8).reshape(-1), ops.QuantDType.BF16, t.shape[0], t.shape[1], repack=False)

        def own(w):
            self.weights.append(w)
            return w.handle

        def joined(*names):
            parts = [mat(n) for n in names]
            w = ctx.concat_rows(parts)
            for p in parts:
                ctx.release(p)
            return own(w)

        def woven(gate, up):
            a, b = mat(gate), mat(up)
            w = self._dev.interleave_rows(a, b)
            ctx.release(a), ctx.release(b)
            return own(w)

        def vec(name):
            t = fetch(name).to(torch.float32).contiguous().cuda()
            self._keep.append(t)
            return t.data_ptr()

        descs = (_Layer * len(cfg["layers"]))()
        for i, L in enumerate(cfg["layers"]):
            d, m, p = descs[i], L["mixer"], f"l{L['weights_of']}."
            if L["weights_of"] != i:
                continue
            d.ffn, d.norm1 = L["ffn"], vec(p + "norm1")
            if L["type"] in ("lightning", "parallel"):
                d.mixer = MIX_HEADS
            else:
                d.heads, d.vdim, d.w_out = m["heads"], m["vdim"], own(mat(p + "mix.o"))
            if L["type"] == "latent_attention":
                d.mixer = MIX_LATENT
                d.dim, d.rot_dim, d.q_rank, d.kv_rank = m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"]
                d.window, d.scale, d.rot = int((m.get("mask") or {}).get("size", 0)), m["scale"], rotation(m["rot"])
                d.w_down, d.w_uq = joined(p + "mix.dq", p + "mix.dkv"), own(mat(p + "mix.uq"))
                d.w_ukv = joined(p + "mix.uk", p + "mix.uv")
                d.q_norm, d.kv_norm, d.sink = vec(p + "mix.dq.norm"), vec(p + "mix.dkv.norm"), vec(p + "mix.sink")
            elif L["type"] == "lightning":
                self._linear(d.linear, m, silu=1, norm_parts=1, gate=GATE_SIGMOID, k_scale=1.0, out_scale=1.0)
                d.linear.mix_norm = vec(p + "mix.norm")
                d.w_in, d.w_out = joined(*(p + "mix." + n for n in "qkvg")), own(mat(p + "mix.o"))
            elif L["type"] == "parallel":
                a, r, pl, pr = m["left"], m["right"], p + "mix.left.", p + "mix.right."
                rel = fetch(pl + "rel")
                d.attn = _Attention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], int((a.get("mask") or {}).get("size", 0)), a["scale"], m["left_scale"],
                                    vec(pl + "q.norm"), vec(pl + "k.norm"), vec(pl + "rel"), rel.shape[0], float(a["bias_max"]))
                self._linear(d.linear, r, silu=0, norm_parts=r["heads"], gate=GATE_SILU, k_scale=r["dim"] ** -0.5, out_scale=m["right_scale"])
                d.w_in = joined(*(pl + n for n in "qkv"), *(pr + n for n in "qkvg"))
                biases = [fetch(pl + n + ".b").to(torch.float32).cuda() for n in "qkv"]
                biases.append(torch.zeros(2 * r["heads"] * (r["dim"] + r["vdim"]), device="cuda"))
                self._keep.append(torch.cat(biases))
                d.b_in, d.w_out = self._keep[-1].data_ptr(), own(mat(pl + "o", pr + "o"))
            else:
                d.mixer = MIX_MAMBA2
                d.state, d.groups, d.conv, d.norm_groups = m["state"], m["groups"], m["conv"], m["norm_groups"]
                d.w_in = own(mat(p + "mix.in"))
                d.conv_w, d.conv_b, d.dt_bias = vec(p + "mix.conv"), vec(p + "mix.conv.b"), vec(p + "mix.dt_bias")
                d.a_log, d.d_skip, d.mix_norm = vec(p + "mix.A_log"), vec(p + "mix.D"), vec(p + "mix.norm")
            if L["ffn"]:
                d.w_gu, d.w_ffn_down, d.norm2 = woven(p + "mlp.gate", p + "mlp.up"), own(mat(p + "mlp.down")), vec(p + "norm2")
        for i, L in enumerate(cfg["layers"]):
            if L["weights_of"] != i:
                C.memmove(C.byref(descs[i]), C.byref(descs[L["weights_of"]]), C.sizeof(_Layer))
        desc = _Desc(len(cfg["layers"]), cfg["hidden"], cfg["vocab"], max_seq, max_chunk,
                     int(ops.QuantDType.BF16) if act == "bfloat16" else 0, cfg["eps"], cfg.get("alpha", 1.0), descs, own(mat("embed")), vec("final.norm"),
                     cfg.get("norm_place", NORM_AFTER), cfg.get("ffn_act", FFN_SILU), cfg.get("embed_scale", 1.0), cfg.get("softcap", 0.0))
        h = C.c_void_p()
        torch.cuda.synchronize()
        ctx.check(ctx.lib.smc_model_create_layered(ctx.h, C.byref(desc), max_batch, C.byref(h)))
        self.h = h

    def _linear(self, d: _Linear, m: dict, **constants):
        d.heads, d.dim, d.vdim = m["heads"], m["dim"], m["vdim"]
        for name, value in constants.items():
            setattr(d, name, value)
        if m.get("rot"):
            d.rot = rotation(m["rot"])
        decay = (C.c_double * m["heads"])(*m["decay"])
        self._keep.append(decay)
        d.decay = C.cast(decay, C.POINTER(C.c_double))

    def sequence_length(self, seq: int) -> int:
        n = C.c_int()
        self.ctx.check(self.ctx.lib.smc_model_seq_length(self.ctx.h, self.h, seq, C.byref(n)))
        return n.value

    def dump_layers(self, on: bool = True):
        """The residual stream after every layer of the following passes: [n_layers, max_chunk, hidden] (None to stop)."""
        t = self.torch
        self._dump = t.zeros((len(self.cfg["layers"]), self.max_chunk, self.cfg["hidden"]), device="cuda") if on else None
        self.ctx.check(self.ctx.lib.smc_model_dump_layers(self.ctx.h, self.h, self._dump.data_ptr() if on else None))
        return self._dump

    def close(self):
        super().close()
        for w in self.weights:
            self.ctx.release(w)
        self.weights = []
