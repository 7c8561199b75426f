"""Small Purivik configurations for the tests, and random weights for them.

The configurations differ from one another in every size and option: widths that are no multiples of four or eight,
grouped, ungrouped and single heads, key and value widths that differ and that agree, rotations over a part of a head, over
all of it and none, frequencies with and without scaling whose wavelengths fall on both sides of the ramp and on it, chunks
shorter than a page, no multiple of a page and over several, attention without a mask, chunk sizes that differ between
layers, dense feed-forwards with different limits, routers that choose one, some and all experts, layers without a
feed-forward, loops over the start, the middle, the end and the whole of the layers, one pass, several passes, no loop,
embedding scales and residual factors below and above one (a table that is the output head too would hide the layers behind
a token's own row if its scale were large in every model).  Weights are drawn so that activations are of order one
and a lost key, a chunk off by one or a wrong constant moves the logits by far more than rounding.  This file does not
import the engine.
"""
from __future__ import annotations

from typing import Dict

import numpy as np
import torch


def _attn(heads, kv, dim, vdim, scale, chunk=None, rot=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _config(vocab, width, eps, scale, mult, layers, loop=None):
    d = {"architecture": "Purivik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "residual_mult": mult, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# A: a loop over the middle, three passes; grouped heads, values wider than keys; chunks of 9 and 37 with pages of 16
PUR_A = _config(103, 48, 1e-5, 0.3, 0.7, [
    _layer(_attn(4, 2, 16, 24, 0.3, chunk=37, rot=(500.0, 8), scaling=(3.0, 1.0, 5.0, 60)), _moe(5, 2, 16)),
    _layer(_attn(6, 2, 8, 8, 0.4, chunk=9, rot=(1.0e4, 8)), _dense(56, 0.9)),
    _layer(_attn(3, 3, 24, 8, 0.25, chunk=37, rot=(200.0, 6), scaling=(2.0, 1.0, 2.0, 40)), _moe(4, 1, 24)),
    _layer(_attn(4, 1, 16, 16, 0.3, chunk=50), None),
], loop=(1, 3, 3))
PUR_A_PAGE = 16

# B: pages of 4, the loop starts with the first layer, widths that are no multiple of 4, no mask, no rotation, every expert
# chosen, a residual factor of one
PUR_B = _config(127, 30, 3e-6, 0.3, 1.0, [
    _layer(_attn(3, 3, 8, 10, 0.4, chunk=5, rot=(50.0, 4)), _moe(3, 3, 20)),
    _layer(_attn(2, 1, 12, 6, 0.3), _dense(44, 2.2)),
    _layer(_attn(5, 5, 6, 6, 0.5, chunk=4, rot=(30.0, 6), scaling=(4.0, 0.5, 4.0, 25)), None),
    _layer(_attn(4, 2, 10, 7, 0.4, chunk=11), _moe(6, 3, 12)),
], loop=(0, 2, 2))
PUR_B_PAGE = 4

# C: longer sequences; heads of 64 with equal key and value widths and of 32 / 48, chunks of 130 and 70, the loop ends with
# the last layer
PUR_C = _config(211, 64, 1e-5, 0.6, 0.35, [
    _layer(_attn(4, 2, 64, 64, 0.125, chunk=130, rot=(2.0e4, 32), scaling=(8.0, 1.0, 4.0, 256)), _dense(96, 1.3)),
    _layer(_attn(4, 4, 32, 48, 0.2, chunk=130, rot=(2.0e3, 16)), _moe(9, 3, 32)),
    _layer(_attn(2, 2, 64, 64, 0.2, chunk=70, rot=(300.0, 64), scaling=(2.0, 2.0, 8.0, 100)), _moe(8, 2, 24)),
    _layer(_attn(4, 1, 48, 80, 0.15, chunk=200, rot=(1.0e4, 24)), _dense(88, 0.6)),
], loop=(2, 4, 2))
PUR_C_PAGE = 16

# D: no loop; odd sizes throughout, single heads, chunks of one, two and three keys
PUR_D = _config(89, 36, 1e-6, 1.3, 1.5, [
    _layer(_attn(1, 1, 20, 12, 0.4, chunk=3, rot=(100.0, 6), scaling=(5.0, 1.0, 1.5, 30)), _moe(7, 2, 10)),
    _layer(_attn(6, 3, 4, 12, 1.0, chunk=1, rot=(10.0, 4)), _dense(26, 0.4)),
    _layer(_attn(3, 1, 5, 3, 0.5, chunk=2, rot=(10.0, 2)), _dense(22, 5.0)),
    _layer(_attn(1, 1, 7, 9, 0.6), None),
])
PUR_D_PAGE = 8

# E: heads of 128 in groups of two, four and one, heads of 96 / 160, the loop over all layers; more experts than a short step
# has choices
PUR_E = _config(113, 64, 1e-5, 0.8, 0.5, [
    _layer(_attn(4, 2, 128, 128, 0.09, chunk=140, rot=(1.0e4, 64), scaling=(4.0, 1.0, 4.0, 128)), _moe(12, 2, 40)),
    _layer(_attn(4, 1, 96, 160, 0.1, chunk=33, rot=(1.0e4, 96)), _dense(80, 1.1)),
    _layer(_attn(2, 2, 128, 128, 0.08, chunk=64, rot=(1.0e4, 128)), None),
    _layer(_attn(8, 2, 128, 128, 0.1, chunk=300), _moe(16, 1, 32)),
], loop=(0, 4, 2))
PUR_E_PAGE = 16


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Names and shapes of a model's tensors, written out from the design's naming rules."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", e["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({f"{p}.q": (H * D, W), f"{p}.k": (G * D, W), f"{p}.v": (G * V, W), f"{p}.o": (W, H * V),
                    f"l{i}.norm1": (W,), f"l{i}.norm1b": (W,), f"l{i}.ls1": (W,)})
        mlp = e.get("mlp")
        if not mlp:
            continue
        f = f"l{i}.mlp"
        out.update({f"l{i}.norm2": (W,), f"l{i}.norm2b": (W,), f"l{i}.ls2": (W,)})
        if mlp["kind"] == "dense":
            out.update({f"{f}.gate": (mlp["ff"], W), f"{f}.up": (mlp["ff"], W), f"{f}.down": (W, mlp["ff"])})
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[f"{f}.router"] = (E, W)
        for x in range(E):
            out.update({f"{f}.e{x}.gate": (ff, W), f"{f}.e{x}.up": (ff, W), f"{f}.e{x}.down": (W, ff)})
    return out


def random_weights(cfg: dict, seed: int, sharp: float = 2.5) -> Dict[str, torch.Tensor]:
    """float32 tensors whose values are exactly representable in bfloat16 (so a 16-bit run and a 32-bit run hold the same
    model).  Matrices N(0, 1/fan_in); queries times `sharp` so that softmax is peaked and single keys matter; gate and up
    matrices of dense feed-forwards times 2, so that the clamps bite; routers times 3, so that few calls are close; norms'
    weights 1 + N(0, 0.1), layer scales 0.9 + N(0, 0.4), some of them negative."""
    rng = np.random.RandomState(seed)
    dense = {f"l{i}.mlp" for i, e in enumerate(cfg["layers"]) if e.get("mlp") and e["mlp"]["kind"] == "dense"}
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith((".ls1", ".ls2")):
            t = 0.9 + rng.normal(0.0, 0.4, shape)
        elif len(shape) == 1:
            t = 1.0 + rng.normal(0.0, 0.1, shape)
        elif name == "embed":
            t = rng.normal(0.0, 1.0, shape)
        else:
            t = rng.normal(0.0, shape[1] ** -0.5, shape)
            if name.endswith(".mix.q"):
                t = t * sharp
            if name.endswith(".router"):
                t = t * 3.0
            if name.rsplit(".", 1)[0] in dense and not name.endswith(".down"):
                t = t * 2.0
        w[name] = torch.from_numpy(np.asarray(t, dtype=np.float32)).to(torch.bfloat16).to(torch.float32)
    return w


def random_tokens(cfg: dict, n: int, seed: int) -> list:
    return np.random.RandomState(seed).randint(0, cfg["vocab"], size=n).tolist()
