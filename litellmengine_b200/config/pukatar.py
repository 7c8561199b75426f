"""Typed configuration of the Pukatar design, read from its config.json.

The file names the design with `"architecture": "Pukatar"` and gives `vocab`, `width`, `norm.eps`, optionally `loop`
({"start", "stop", "times"}: layers start .. stop-1 run `times` times in a row with the same tensors, each pass with a
cache and state of its own) and a list `layers`.  A layer entry has `type` ('attention' or 'channel_delta'), the sizes
and constants of its mixer under `mixer`, and its feed-forward under `mlp` ({"kind": "dense", "ff": n}, {"kind": "moe",
...}, or null for a layer without one).  Tensors of layer i start with `l<i>.`; linear weights are [out, in].

What the design fixes, and therefore lives here and in the parts rather than in the file:
  * norms are layer norms with a weight and a bias ('<norm>' and '<norm>.b'); one follows the embedding ('embed.norm'),
    one precedes the output head, which is a tensor of its own, and a layer has ONE, which its mixer and its feed-forward
    both read: x += mixer(norm1(x)) + ff(norm1(x));
  * in front of every pass of the looped span the stream becomes W [x; x0] + step[pass], x0 the normed embedding
    ('loop.in', 'loop.step');
  * 'attention' = grouped-query softmax attention without biases, a rotation of the pairs (i, i + dims/2) of the first
    `rot.dims` entries of a head, scores times `scale`, a sliding window (`mask.size`) that keeps the sequence's first
    `mask.keep_first` keys, and a learned score per head in the softmax's denominator ('.sink');
  * 'channel_delta' = the gated delta rule with a decay per key channel, behind short convolutions of `conv` taps with
    silu, on unit queries and keys; the ranks of its two low-rank projections are the stored tensors' inner sizes;
  * the dense feed-forward is down(silu(gate x) * (up x)); an expert is down(g * sigmoid(1.702 g) * (u + 1)) with
    g = min(gate x, limit), u = clamp(up x, -limit, limit); the router has a bias and weighs the `top` largest logits by
    their softmax; a shared expert (`mlp.shared`, sizes and limit of its own) runs for every token, times a sigmoid gate.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .registry import ConfigError, register_architecture
from .specs import BlockSpec, FeedForwardSpec, MixerSpec, ModelPlan, NormSpec, PositionSpec, RejoinSpec, StageSpec
from .tobovik import _FF_NAMES, _freeze, _need, _thaw

MAX_POSITION = 1 << 20        # nothing of the design is tabulated by absolute position

_ATTN_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("sink", "sink"))
_DELTA_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_conv", "q.conv"), ("k_conv", "k.conv"), ("v_conv", "v.conv"),
                ("b", "b"), ("a1", "a1"), ("a2", "a2"), ("dt", "dt_bias"), ("A", "A_log"), ("g1", "g1"), ("g2", "g2"),
                ("norm", "norm"))


def _heads(m: Dict[str, Any], where: str) -> Tuple[int, int]:
    heads, kv = _need(m, "heads", int, where), _need(m, "kv_heads", int, where)
    if heads % kv:
        raise ConfigError(f"config field {where}heads must be a multiple of {where}kv_heads")
    return heads, kv


def _attention_spec(m: Dict[str, Any], where: str) -> MixerSpec:
    heads, kv = _heads(m, where)
    dim = _need(m, "dim", int, where)
    window, keep = None, 0
    if m.get("mask") is not None:
        window = _need(m["mask"], "size", int, where + "mask.")
        k = m["mask"].get("keep_first", 0)
        if isinstance(k, bool) or not isinstance(k, int) or k < 0:
            raise ConfigError(f"config field {where}mask.keep_first must be a non-negative integer")
        keep = k
    position = PositionSpec(kind="none")
    if m.get("rot") is not None:
        base, dims = _need(m["rot"], "base", float, where + "rot."), _need(m["rot"], "dims", int, where + "rot.")
        if dims % 2 or dims > dim or not base > 0.0:
            raise ConfigError(f"config field {where}rot: dims must be even and at most {where}dim, base positive")
        position = PositionSpec(kind="rope_half", theta=base, rotary_dim=dims)
    return MixerSpec(kind="gated_attention", num_heads=heads, num_kv_heads=kv, head_dim=dim, value_dim=_need(m, "vdim", int, where),
                     position=position, window=window, keep_first=keep, learned_sink=True, scale=_need(m, "scale", float, where),
                     weight_prefix="mix", tensor_names=_ATTN_NAMES)


def _rank(m: Dict[str, Any], key: str, where: str) -> Optional[int]:
    """An inner size that only the stored tensors know; a configuration for random weights may give it."""
    return None if m.get(key) is None else _need(m, key, int, where)


def _delta_spec(m: Dict[str, Any], where: str, eps: float) -> MixerSpec:
    heads, kv = _heads(m, where)
    return MixerSpec(kind="delta_rule", num_heads=heads, num_kv_heads=kv, head_dim=_need(m, "dim", int, where),
                     value_dim=_need(m, "vdim", int, where), weight_prefix="mix", tensor_names=_DELTA_NAMES,
                     params=(("taps", _need(m, "conv", int, where)), ("eps", eps), ("decay_rank", _rank(m, "decay_rank", where)),
                             ("gate_rank", _rank(m, "gate_rank", where))))


def _limit(d: Dict[str, Any], where: str) -> float:
    limit = _need(d, "limit", float, where)
    if not limit > 0:
        raise ConfigError(f"config field {where}limit must be positive")
    return limit


def _feed_forward_spec(mlp: Dict[str, Any], where: str) -> FeedForwardSpec:
    kind = _need(mlp, "kind", str, where)
    if kind == "dense":
        return FeedForwardSpec(kind="swiglu", intermediate_size=_need(mlp, "ff", int, where), weight_prefix="mlp",
                               tensor_names=_FF_NAMES)
    if kind != "moe":
        raise ConfigError(f"{where}kind={kind!r} is not a feed-forward of this design ('dense', 'moe')")
    router, ex, sh = mlp.get("router"), mlp.get("expert"), mlp.get("shared")
    experts, top = _need(router, "experts", int, where + "router."), _need(router, "top", int, where + "router.")
    if top > experts:
        raise ConfigError(f"config field {where}router.top exceeds {where}router.experts")
    params = [("experts", experts), ("top", top), ("groups", None), ("route_scale", 1.0), ("score", "softmax"), ("router_bias", True),
              ("activation", "clamped_swish"), ("limit", _limit(ex, where + "expert.")), ("expert_prefix", "e")]
    if sh is not None:
        params += [("shared", _need(sh, "ff", int, where + "shared.")), ("shared_activation", "clamped_swish"),
                   ("shared_limit", _limit(sh, where + "shared.")), ("shared_gate", True)]
    return FeedForwardSpec(kind="moe", intermediate_size=_need(ex, "ff", int, where + "expert."), weight_prefix="mlp",
                           params=tuple(params))


@register_architecture("Pukatar")
@dataclass(frozen=True)
class PukatarConfig:
    vocab: int
    width: int
    eps: float
    loop: Optional[Tuple[int, int, int]]   # (start, stop, times); None when the file has none
    layers: Tuple[Any, ...]                # the file's layer entries, kept as read (nested tuples of pairs)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PukatarConfig":
        vocab, width = _need(d, "vocab", int, ""), _need(d, "width", int, "")
        eps = _need(d.get("norm"), "eps", float, "norm.")
        if not eps > 0:
            raise ConfigError("config field norm.eps must be positive")
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("Missing required config field: layers")
        loop = None
        if d.get("loop") is not None:
            lp = d["loop"]
            for key in ("start", "stop"):
                if isinstance(lp.get(key), bool) or not isinstance(lp.get(key), int):
                    raise ConfigError(f"config field loop.{key} must be an integer")
            loop = (lp["start"], lp["stop"], _need(lp, "times", int, "loop."))
            if not 0 <= loop[0] < loop[1] <= len(layers):
                raise ConfigError("config field loop: 0 <= start < stop <= number of layers does not hold")
        cfg = cls(vocab=vocab, width=width, eps=eps, loop=loop, layers=tuple(_freeze(x) for x in layers))
        cfg.plan()                    # every other check is the plan's
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": [_thaw(x) for x in self.layers]}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    # what the engine's entry points ask of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def torch_dtype(self) -> str:
        return "bfloat16"

    def run_order(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass that starts in front of it or None) in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop
        order = [(i, None) for i in range(a)]
        for t in range(times):
            order += [(i, t if i == a else None) for i in range(a, b)]
        return order + [(i, None) for i in range(b, n)]

    def plan(self) -> ModelPlan:
        norm = NormSpec(kind="layernorm", eps=self.eps, weight_name="", bias=True)
        blocks = []
        for i, frozen in enumerate(self.layers):
            e, where = _thaw(frozen), f"layers[{i}]."
            kind, m = _need(e, "type", str, where), e.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"Missing required config field: {where}mixer")
            if kind == "attention":
                mixer = _attention_spec(m, where + "mixer.")
            elif kind == "channel_delta":
                mixer = _delta_spec(m, where + "mixer.", self.eps)
            else:
                raise ConfigError(f"{where}type={kind!r} is not a mixer of this design ('attention', 'channel_delta')")
            ffn = None if e.get("mlp") is None else _feed_forward_spec(e["mlp"], where + "mlp.")
            blocks.append(BlockSpec(arrangement="parallel_pre_norm", mixer=mixer, feed_forward=ffn, mixer_norm=norm,
                                    feed_forward_norm=None, weight_prefix=f"l{i}", mixer_norm_name="norm1"))
        plan = ModelPlan(
            hidden_size=self.width, vocab_size=self.vocab, blocks=tuple(blocks),
            order=tuple(StageSpec(block=i, starts_pass=t) for i, t in self.run_order()), final_norm=norm,
            tie_word_embeddings=False, max_position=MAX_POSITION, embedding_name="embed", final_norm_name="final.norm",
            output_name="head", embedding_norm=norm, embedding_norm_name="embed.norm",
            rejoin=RejoinSpec(passes=self.loop[2]) if self.loop is not None else None)
        plan.validate()
        return plan
