"""Typed configuration of the Purivik design, read from its config.json.

The file names the design with `"architecture": "Purivik"` and gives `vocab`, `width`, `embedding.scale`, `norm.eps`,
`residual_mult`, optionally `loop` ({"start", "stop", "times"}: layers start .. stop-1 run `times` times in a row with the
same tensors, each pass with a cache of its own) and a list `layers`.  A layer entry has `type` ('attention'), the sizes
and constants of its mixer under `mixer`, and its feed-forward under `mlp` ({"kind": "dense", ...}, {"kind": "moe", ...},
or null for a layer without one).  Tensors of layer i start with `l<i>.`; linear weights are [out, in].

What the design fixes, and therefore lives here and in the parts rather than in the file:
  * the norm is an RMS norm; a layer has one in front of each sublayer and one on its output, and the normed output is
    multiplied by a learned factor per channel and by `residual_mult` before it joins the stream:
    x += mult * ls1 * norm1b(mixer(norm1(x))), x += mult * ls2 * norm2b(ff(norm2(x)));
  * the embedding is the token's row times `embedding.scale`; the output head is the embedding table, without that scale;
  * in front of every pass of the looped span but the first the embedding output joins the stream;
  * 'attention' = grouped-query softmax attention without biases, values of their own width, a rotation of the pairs
    (i, i + dims/2) of the first `rot.dims` entries of a head whose frequencies `rot.scaling` stretches by wavelength,
    scores times `scale`, within chunks of `mask.size` positions (no `mask`: over all earlier ones);
  * the dense feed-forward is down(g * sigmoid(1.702 g) * (u + 1)) with g = min(gate x, limit), u = clamp(up x, -limit,
    limit); the routed one takes the `top` largest sigmoid scores as weights as they are, and an expert
    down(silu(gate y) * (up y)) runs on y = weight * x.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .pukatar import _heads, _limit
from .registry import ConfigError, register_architecture
from .specs import BlockSpec, FeedForwardSpec, MixerSpec, ModelPlan, NormSpec, PositionSpec, RejoinSpec, StageSpec
from .tobovik import _FF_NAMES, _freeze, _need, _thaw

MAX_POSITION = 1 << 20        # nothing of the design is tabulated by absolute position

_ATTN_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"))


def _rotation(rot: Optional[Dict[str, Any]], where: str, dim: int) -> PositionSpec:
    if rot is None:
        return PositionSpec(kind="none")
    base, dims = _need(rot, "base", float, where), _need(rot, "dims", int, where)
    if dims % 2 or dims > dim or not base > 0.0:
        raise ConfigError(f"config field {where}dims must be even and at most {dim}, {where}base positive")
    params = ()
    if rot.get("scaling") is not None:
        factor, low, high, original = (_need(rot["scaling"], k, float, where + "scaling.") for k in ("factor", "low", "high", "original"))
        if not (factor > 0 and original > 0 and 0 < low <= high):
            raise ConfigError(f"config field {where}scaling: factor, low, high and original must be positive, low at most high")
        params = (("wavelengths", (factor, low, high, original)),)
    return PositionSpec(kind="rope_half", theta=base, rotary_dim=dims, params=params)


def _attention_spec(m: Dict[str, Any], where: str) -> MixerSpec:
    heads, kv = _heads(m, where)
    dim = _need(m, "dim", int, where)
    chunk = None if m.get("mask") is None else _need(m["mask"], "size", int, where + "mask.")
    return MixerSpec(kind="gated_attention", num_heads=heads, num_kv_heads=kv, head_dim=dim, value_dim=_need(m, "vdim", int, where),
                     position=_rotation(m.get("rot"), where + "rot.", dim), chunk=chunk, scale=_need(m, "scale", float, where),
                     weight_prefix="mix", tensor_names=_ATTN_NAMES)


def _feed_forward_spec(mlp: Dict[str, Any], where: str) -> FeedForwardSpec:
    kind = _need(mlp, "kind", str, where)
    if kind == "dense":
        return FeedForwardSpec(kind="swiglu", intermediate_size=_need(mlp, "ff", int, where), weight_prefix="mlp",
                               params=(("activation", "clamped_swish"), ("limit", _limit(mlp, where))), tensor_names=_FF_NAMES)
    if kind != "moe":
        raise ConfigError(f"{where}kind={kind!r} is not a feed-forward of this design ('dense', 'moe')")
    router = mlp.get("router")
    experts, top = _need(router, "experts", int, where + "router."), _need(router, "top", int, where + "router.")
    if top > experts:
        raise ConfigError(f"config field {where}router.top exceeds {where}router.experts")
    return FeedForwardSpec(kind="moe", intermediate_size=_need(mlp.get("expert"), "ff", int, where + "expert."), weight_prefix="mlp",
                           params=(("experts", experts), ("top", top), ("groups", None), ("route_scale", 1.0), ("score", "sigmoid"),
                                   ("normalize", False), ("weight_on_input", True), ("activation", "silu"), ("expert_prefix", "e")))


@register_architecture("Purivik")
@dataclass(frozen=True)
class PurivikConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    residual_mult: float
    loop: Optional[Tuple[int, int, int]]   # (start, stop, times); None when the file has none
    layers: Tuple[Any, ...]                # the file's layer entries, kept as read (nested tuples of pairs)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PurivikConfig":
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
        cfg = cls(vocab=vocab, width=width, embedding_scale=_need(d.get("embedding"), "scale", float, "embedding."), eps=eps,
                  residual_mult=_need(d, "residual_mult", float, ""), loop=loop, layers=tuple(_freeze(x) for x in layers))
        cfg.plan()                    # every other check is the plan's
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
             "norm": {"eps": self.eps}, "residual_mult": self.residual_mult, "layers": [_thaw(x) for x in self.layers]}
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
        norm = NormSpec(kind="rmsnorm", eps=self.eps, weight_name="")
        blocks = []
        for i, frozen in enumerate(self.layers):
            e, where = _thaw(frozen), f"layers[{i}]."
            kind, m = _need(e, "type", str, where), e.get("mixer")
            if kind != "attention":
                raise ConfigError(f"{where}type={kind!r} is not a mixer of this design ('attention')")
            if not isinstance(m, dict):
                raise ConfigError(f"Missing required config field: {where}mixer")
            ffn = None if e.get("mlp") is None else _feed_forward_spec(e["mlp"], where + "mlp.")
            blocks.append(BlockSpec(
                arrangement="sandwich_norm", mixer=_attention_spec(m, where + "mixer."), feed_forward=ffn, mixer_norm=norm,
                feed_forward_norm=norm, weight_prefix=f"l{i}", mixer_norm_name="norm1", feed_forward_norm_name="norm2",
                mixer_post_norm=norm, feed_forward_post_norm=norm, mixer_post_norm_name="norm1b", feed_forward_post_norm_name="norm2b",
                layer_scale_names=("ls1", "ls2"), branch_scale=self.residual_mult))
        plan = ModelPlan(
            hidden_size=self.width, vocab_size=self.vocab, blocks=tuple(blocks),
            order=tuple(StageSpec(block=i, starts_pass=t) for i, t in self.run_order()), final_norm=norm,
            tie_word_embeddings=True, max_position=MAX_POSITION, embedding_name="embed", final_norm_name="final.norm",
            output_name="head", embedding_scale=self.embedding_scale,
            rejoin=RejoinSpec(passes=self.loop[2], kind="add") if self.loop is not None else None)
        plan.validate()
        return plan
