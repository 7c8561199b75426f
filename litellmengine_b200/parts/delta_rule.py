"""The gated delta rule: a recurrent mixer whose state forgets per key channel and is corrected towards each value."""
from __future__ import annotations

from typing import Dict

import torch

from ..cache import StateNeed
from ..config.specs import MixerSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .attention import BranchMixer
from .context import StageContext
from .registry import register_mixer


@register_mixer("delta_rule")
class DeltaRuleMixer(BranchMixer):
    """Per head a state S [D, V] (32-bit, one per request and stage, zero at admission):

        S <- diag(g_t) S,   u = beta_t (v_t - S^T k_t),   S <- S + k_t u^T,   o_t = S^T q_t

    q and k have `num_kv_heads` heads (head h reads number h // (num_heads / num_kv_heads)), v has `num_heads`.  Each of
    the three projections passes a causal convolution over time, channel by channel (`taps` taps, the last one on the
    token itself, zeros before the sequence's start), and silu; q and k become unit vectors per head, x / sqrt(sum(x^2) +
    1e-6), and q is multiplied by D^-1/2.  beta = sigmoid(W_b x) per head; the decay of key channel d of head h is
    g = exp(-exp(A_h) * softplus(z)), z = W_a2 (W_a1 x) + dt.  Each head's o is RMS-normed over V with one weight [V]
    shared by the heads and multiplied by sigmoid(W_g2 (W_g1 x)); W_o follows.  One product yields [q | k | v | b | a1 |
    g1] per token in float32, and nothing of the recurrence is rounded after it.  A request's slot holds the states and
    the convolutions' last inputs in one row of floats (the kernels' layout, see csrc/delta_rule.cu)."""

    graph_safe = True            # kernels on the current stream only; their grids follow the step's entries
    any_division_safe = False

    PADDED = (32, 64, 128, 256)  # what the kernels are instantiated for

    _DEFAULT_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight",
                      "q_conv": "q_conv.weight", "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "b": "b_proj.weight",
                      "a1": "a_proj.0.weight", "a2": "a_proj.1.weight", "dt": "dt_bias", "A": "A_log", "g1": "g_proj.0.weight",
                      "g2": "g_proj.1.weight", "norm": "o_norm.weight"}

    def __init__(self, spec: MixerSpec, hidden_size: int, compute_dtype: torch.dtype, device):
        p = dict(spec.params)
        self.H, self.G, self.D = spec.num_heads, spec.num_kv_heads or spec.num_heads, spec.head_dim
        self.V = spec.value_dim or spec.head_dim
        self.taps = int(p.get("taps", 1))
        if min(self.H, self.G, self.D, self.V, self.taps) <= 0 or self.H % self.G:
            raise ValueError("the delta rule needs positive sizes and heads that are a multiple of its key heads")
        self.eps = float(p.get("eps", 1e-6))                    # of the per-head output norm
        self.ranks = (p.get("decay_rank"), p.get("gate_rank"))  # None: read from the stored tensors
        self.spec, self.hidden, self.dtype, self.device = spec, hidden_size, compute_dtype, torch.device(device)
        self.names = dict(self._DEFAULT_NAMES, **dict(spec.tensor_names))
        self.channels = 2 * self.G * self.D + self.H * self.V    # what passes the convolutions
        self.out_width = self.H * self.V
        self.conv_w = self.w_decay = self.w_gate = self.dt_bias = self.a_log = self.norm_w = None
        # rows of a head's state as the kernels keep them
        self.padded = next((n for n in self.PADDED if self.D <= n), 0)
        if not self.padded or (self.device.type == "cuda" and not ops.delta_supported(self.D, self.V)):
            raise ValueError(f"the delta rule: a state of {self.D} x {self.V} per head is more than its kernels take")

    def parameters(self) -> Dict[str, ParamSpec]:
        n, W = self.names, self.hidden
        gd, hd, hv = self.G * self.D, self.H * self.D, self.H * self.V
        ra, rg = (r if r is not None else -1 for r in self.ranks)
        conv = lambda c: ParamSpec((c, self.taps), role="scale", init=("normal", 0.5))
        return {n["q"]: ParamSpec((gd, W)), n["k"]: ParamSpec((gd, W)), n["v"]: ParamSpec((hv, W)), n["o"]: ParamSpec((W, hv)),
                n["q_conv"]: conv(gd), n["k_conv"]: conv(gd), n["v_conv"]: conv(hv), n["b"]: ParamSpec((self.H, W)),
                n["a1"]: ParamSpec((ra, W)), n["a2"]: ParamSpec((hd, ra)),
                n["dt"]: ParamSpec((hd,), role="scale", init=("normal", 1.0)),
                n["A"]: ParamSpec((self.H,), role="scale", init=("normal", 0.5)),
                n["g1"]: ParamSpec((rg, W)), n["g2"]: ParamSpec((hv, rg)),
                n["norm"]: ParamSpec((self.V,), role="scale", init=("one_plus_normal", 0.01))}

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        n = self.names
        rows = [t[n[k]] for k in ("q", "k", "v", "b", "a1", "g1")]
        self.ranks = (t[n["a1"]].shape[0], t[n["g1"]].shape[0])
        if t[n["a2"]].shape[1] != self.ranks[0] or t[n["g2"]].shape[1] != self.ranks[1]:
            raise ValueError("the two halves of a low-rank projection disagree on their rank")
        dt = torch.float32 if any(x.dtype == torch.float32 for x in rows) else rows[0].dtype
        self.b_off = self.channels
        self.a_off = self.b_off + self.H
        self.g_off = self.a_off + self.ranks[0]
        self.w_in = torch.cat([x.to(dt) for x in rows], dim=0).contiguous()
        self.in_width = self.w_in.shape[0]
        self.w_o = t[n["o"]].contiguous()
        self.conv_w = torch.cat([t[n[k]].float() for k in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        # the second halves of the low-rank projections are read transposed, [rank, channels], by kernels that add in 32-bit
        low = torch.bfloat16 if t[n["a2"]].dtype == t[n["g2"]].dtype == torch.bfloat16 else torch.float32
        self.w_decay, self.w_gate = (t[n[k]].to(low).t().contiguous() for k in ("a2", "g2"))
        self.dt_bias, self.a_log = t[n["dt"]].float().contiguous(), t[n["A"]].float().contiguous()
        self.norm_w = t[n["norm"]].float().contiguous()
        ops.prepare_streaming(self.w_in)
        ops.prepare_streaming(self.w_o)

    def cache_need(self):
        floats = self.H * self.V * self.padded + self.taps * self.channels
        return StateNeed(((floats + 3) // 4 * 4,), "float32")

    def mix(self, proj, col0, ctx: StageContext, out, out_col0, out_scale):
        if ctx.state is None:
            raise RuntimeError("the delta rule was given no state")
        ops.delta_rule(proj, (col0, col0 + self.b_off, col0 + self.a_off, col0 + self.g_off), self.ranks, self.conv_w, self.w_decay,
                       self.w_gate, self.dt_bias, self.a_log, self.norm_w, self.eps, out_scale, out, out_col0, ctx.state, ctx.batch,
                       self.H, self.G, self.D, self.V, single=ctx.batch.max_q_len == 1)
