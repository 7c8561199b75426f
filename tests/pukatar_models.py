"""Small Pukatar configurations for the tests, and random weights for them.

The configurations differ from one another in every size and option: widths that are no multiples of four or
eight, grouped, ungrouped and single heads in both mixers, key and value widths that differ and that agree, rotations
over a part of a head and over all of it and none, windows shorter than a page and over several, kept first keys fewer
than a page, more than a page and more than the window, attention without a mask, convolutions of one to five taps,
low-rank projections of different ranks, states whose key widths fill the kernels' row groups and that do not,
routers that choose one, some and all experts, with and without a shared expert whose size and clamp differ from the
experts', dense feed-forwards, layers without one, loops over the start, the middle, the end and the whole of the
layers, one pass, several passes, no loop.  Weights are drawn so that activations are of order one and a lost key, a
lost state or a wrong constant moves the logits by far more than rounding.  This file does not import the engine.
"""
from __future__ import annotations

from typing import Dict

import numpy as np
import torch


def _attn(heads, kv, dim, vdim, scale, window=None, keep=None, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def _delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _config(vocab, width, eps, layers, loop=None):
    d = {"architecture": "Pukatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# A: a loop over the middle, three passes; grouped key heads in both mixers; a window shorter than a page with three kept keys
PUK_A = _config(103, 48, 1e-5, [
    _layer("channel_delta", _delta(4, 2, 12, 20, 3), _dense(56)),
    _layer("attention", _attn(4, 2, 16, 24, 0.3, window=9, keep=3, rot=(500.0, 8)), _moe(5, 2, 16, 1.1, shared=(24, 0.7))),
    _layer("channel_delta", _delta(3, 3, 32, 16, 4), _moe(4, 1, 24, 2.5)),
    _layer("attention", _attn(6, 2, 8, 8, 0.4, window=30, keep=20, rot=(1.0e4, 8)), None),
], loop=(1, 3, 3))
PUK_A_PAGE = 16

# B: pages of 4, the loop starts with the first layer, widths that are no multiple of 4, one tap (no convolution over time),
# two taps, no mask and no rotation, every expert chosen
PUK_B = _config(127, 30, 3e-6, [
    _layer("channel_delta", _delta(2, 1, 6, 10, 1), _moe(3, 3, 20, 0.9, shared=(10, 1.7))),
    _layer("attention", _attn(3, 3, 8, 8, 0.4, window=5, rot=(50.0, 4)), _dense(44)),
    _layer("attention", _attn(2, 1, 12, 6, 0.3), None),
    _layer("channel_delta", _delta(5, 5, 9, 7, 2), _moe(6, 3, 12, 1.4)),
], loop=(0, 2, 2))
PUK_B_PAGE = 4

# C: longer sequences; attention heads of 64 (the tensor-core kernels of the 16-bit mode), a window over several pages with
# more kept keys than a page holds, key widths of 64 and 40, the loop ends with the last layer
PUK_C = _config(211, 64, 1e-5, [
    _layer("attention", _attn(4, 2, 64, 64, 0.125, window=130, keep=21, rot=(2.0e4, 32)), _dense(96)),
    _layer("channel_delta", _delta(2, 1, 64, 48, 4), _moe(9, 3, 32, 1.2, shared=(48, 0.8))),
    _layer("attention", _attn(2, 2, 64, 64, 0.2, window=70, rot=(300.0, 64)), _moe(8, 2, 24, 3.0, shared=(24, 3.0))),
    _layer("channel_delta", _delta(3, 3, 40, 36, 5), _dense(88)),
], loop=(2, 4, 2))
PUK_C_PAGE = 16

# D: no loop; odd sizes throughout, single heads, more kept keys than the window is wide, a window of one key
PUK_D = _config(89, 36, 1e-6, [
    _layer("attention", _attn(1, 1, 20, 12, 0.4, window=3, keep=7, rot=(100.0, 6)), _moe(7, 2, 10, 0.6)),
    _layer("channel_delta", _delta(1, 1, 24, 20, 3), _dense(22)),
    _layer("attention", _attn(6, 3, 4, 12, 1.0, window=1, keep=1, rot=(10.0, 4)), _dense(26)),
    _layer("channel_delta", _delta(6, 2, 5, 3, 4), None),
])
PUK_D_PAGE = 8

# E: attention heads of 128 in groups of two and of one, key widths of 128 and 160 with several columns' blocks, the loop
# over all layers; more experts than a short step has choices
PUK_E = _config(113, 64, 1e-5, [
    _layer("attention", _attn(4, 2, 128, 128, 0.09, window=140, keep=6, rot=(1.0e4, 64)), _moe(12, 2, 40, 1.6, shared=(56, 1.2))),
    _layer("channel_delta", _delta(2, 2, 128, 70, 4), _dense(80)),
    _layer("attention", _attn(2, 2, 128, 128, 0.08, window=33, keep=0, rot=(1.0e4, 128)), None),
    _layer("channel_delta", _delta(2, 1, 160, 33, 4), _dense(72)),
], loop=(0, 4, 2))
PUK_E_PAGE = 16

DECAY_RANK, GATE_RANK = 5, 7          # of the low-rank projections; only the tensors know them


def _norm_shapes(name, W):
    return {name: (W,), name + ".b": (W,)}


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Names and shapes of a model's tensors, written out from the design's naming rules."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W)}
    out.update(_norm_shapes("final.norm", W))
    out.update(_norm_shapes("embed.norm", W))
    if cfg.get("loop"):
        out.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", e["mixer"]
        out.update(_norm_shapes(f"l{i}.norm1", W))
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if e["type"] == "attention":
            out.update({f"{p}.q": (H * D, W), f"{p}.k": (G * D, W), f"{p}.v": (G * V, W), f"{p}.o": (W, H * V), f"{p}.sink": (H,)})
        else:
            n = m["conv"]
            out.update({f"{p}.q": (G * D, W), f"{p}.k": (G * D, W), f"{p}.v": (H * V, W), f"{p}.q.conv": (G * D, n),
                        f"{p}.k.conv": (G * D, n), f"{p}.v.conv": (H * V, n), f"{p}.b": (H, W), f"{p}.A_log": (H,),
                        f"{p}.norm": (V,), f"{p}.a1": (DECAY_RANK, W), f"{p}.a2": (H * D, DECAY_RANK), f"{p}.dt_bias": (H * D,),
                        f"{p}.g1": (GATE_RANK, W), f"{p}.g2": (H * V, GATE_RANK), f"{p}.o": (W, H * V)})
        mlp = e.get("mlp")
        if not mlp:
            continue
        f = f"l{i}.mlp"
        if mlp["kind"] == "dense":
            out.update({f"{f}.gate": (mlp["ff"], W), f"{f}.up": (mlp["ff"], W), f"{f}.down": (W, mlp["ff"])})
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        out.update({f"{f}.router": (E, W), f"{f}.router.b": (E,)})
        for x in range(E):
            out.update({f"{f}.e{x}.gate": (ff, W), f"{f}.e{x}.up": (ff, W), f"{f}.e{x}.down": (W, ff)})
        if mlp.get("shared"):
            s = mlp["shared"]["ff"]
            out.update({f"{f}.shared.gate": (s, W), f"{f}.shared.up": (s, W), f"{f}.shared.down": (W, s), f"{f}.shared.sg": (1, W)})
    return out


def random_weights(cfg: dict, seed: int, sharp: float = 2.5) -> Dict[str, torch.Tensor]:
    """float32 tensors whose values are exactly representable in bfloat16 (so a 16-bit run and a 32-bit run hold the
    same model).  Matrices N(0, 1/fan_in); attention queries times `sharp` so that softmax is peaked and single keys
    matter; routers times 3 with biases N(0, 0.7), so that the bias changes choices and few calls are close; the decays'
    biases N(-2, 2) and A_log N(0, 0.7), so that channels forget at very different rates; sinks N(1, 1.5); norms'
    biases N(0, 0.1), vectors that multiply 1 + N(0, 0.1)."""
    rng = np.random.RandomState(seed)
    w = {}
    kinds = {f"l{i}.mix.q": e["type"] for i, e in enumerate(cfg["layers"])}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith(".dt_bias"):
            t = rng.normal(-2.0, 2.0, shape)
        elif name.endswith(".A_log"):
            t = rng.normal(0.0, 0.7, shape)
        elif name.endswith(".sink"):
            t = rng.normal(1.0, 1.5, shape)
        elif name.endswith(".router.b"):
            t = rng.normal(0.0, 0.7, shape)
        elif name.endswith(".b") and len(shape) == 1:
            t = rng.normal(0.0, 0.1, shape)
        elif name == "loop.step":
            t = rng.normal(0.0, 0.5, shape)
        elif name.endswith(".conv"):
            t = rng.normal(0.0, shape[1] ** -0.5, shape)
        elif len(shape) == 1:
            t = 1.0 + rng.normal(0.0, 0.1, shape)
        elif name == "embed":
            t = rng.normal(0.3, 1.0, shape)
        else:
            t = rng.normal(0.0, shape[1] ** -0.5, shape)
            if kinds.get(name) == "attention":
                t = t * sharp
            if name.endswith(".router"):
                t = t * 3.0
            if name.endswith(".a2") or name.endswith(".shared.sg"):
                t = t * 2.0
        w[name] = torch.from_numpy(np.asarray(t, dtype=np.float32)).to(torch.bfloat16).to(torch.float32)
    return w


def random_tokens(cfg: dict, n: int, seed: int) -> list:
    return np.random.RandomState(seed).randint(0, cfg["vocab"], size=n).tolist()
