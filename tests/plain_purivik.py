"""A plain, slow restatement of the Purivik design: whole sequences, no cache, nothing carried between calls, one
function per mechanism.  It shares no code with the engine; the tests compare the engine with it.

Notation.  x [T, W] is the residual stream, u a sublayer's (normed) input, p the position of a token in its sequence
(from 0), `w` a dict of tensors by name, `pre` a name prefix, `m` a mixer's entry of the configuration.  `act` rounds
activations the way a run mode would (identity for the 32-bit mode); what the design keeps in 32-bit stays unrounded.
Everything runs in float64 unless `act` rounds it.
"""
import math

import torch

F64 = torch.float64


def identity(x):
    return x


def bf16_round(x):
    """What a 16-bit run mode does to an activation between two kernels."""
    return x.to(torch.bfloat16).to(x.dtype)


def bf16_round_jittered(seed):
    """The same rounding after a relative nudge of up to half a unit in the last place: another implementation's
    rounding of the same exact value."""
    g = torch.Generator().manual_seed(seed)

    def act(x):
        nudge = (torch.rand(x.shape, generator=g, dtype=F64) - 0.5) * 2.0 ** -8
        return (x * (1.0 + nudge.to(x.dtype))).to(torch.bfloat16).to(x.dtype)
    return act


def silu(z):
    return z * torch.sigmoid(z)


def rms_norm(x, weight, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * weight.to(F64)


def embed(ids, w, scale):
    """The embedding output: the token's row times a constant."""
    return w["embed"][torch.as_tensor(ids, dtype=torch.long)].to(F64) * float(scale)


def frequencies(rot):
    """One frequency per rotated pair, f_i = base^(-2i/dims).  With scaling, by the wavelength l = 2 pi / f_i against
    the context `original`: shorter than original/high, unchanged; longer than original/low, divided by factor; between
    the two a mean of both, weighted by how far original/l has come from low to high."""
    dims = int(rot["dims"])
    out = [float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
        for i, f in enumerate(out):
            length = 2.0 * math.pi / f
            if length > original / low:
                out[i] = f / factor
            elif length >= original / high:
                keep = (original / length - low) / (high - low)
                out[i] = keep * f + (1.0 - keep) * f / factor
    return torch.tensor(out, dtype=F64)


def rotate_half(t, positions, rot):
    """t [T, heads, n]: of the first rot.dims entries, entry i pairs with entry i + dims/2; the pair (a, b) at position p
    becomes (a cos - b sin, b cos + a sin) of the angle p * f_i.  The rest passes."""
    if not rot:
        return t
    dims = int(rot["dims"])
    half = dims // 2
    ang = torch.as_tensor(positions, dtype=F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = t[..., :half], t[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, t[..., dims:]], dim=-1)


def visible_keys(T, mask):
    """[T, T] bool: query i sees key j if j <= i and both lie in the same chunk of mask.size positions, counted from the
    sequence's start; without a mask every j <= i."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    vis = j <= i
    if mask:
        n = int(mask["size"])
        vis = vis & (torch.div(i, n, rounding_mode="floor") == torch.div(j, n, rounding_mode="floor"))
    return vis


def attention(u, w, pre, m, act=identity):
    """Grouped-query softmax attention: query head h reads key/value head h // (heads / kv_heads)."""
    T = u.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda n: w[pre + n].to(F64)
    pos = list(range(T))
    q = act(rotate_half((u @ g("q").T).view(T, H, D), pos, m.get("rot")))
    k = act(rotate_half((u @ g("k").T).view(T, G, D), pos, m.get("rot")))
    v = act((u @ g("v").T).view(T, G, V))
    rep = H // G
    kh = k.permute(1, 0, 2).repeat_interleave(rep, dim=0)
    vh = v.permute(1, 0, 2).repeat_interleave(rep, dim=0)
    scores = (q.permute(1, 0, 2) @ kh.transpose(1, 2)) * float(m["scale"])
    scores = scores.masked_fill(~visible_keys(T, m.get("mask"))[None], float("-inf"))
    o = torch.softmax(scores, dim=-1) @ vh                                                # [H, T, V]
    return act(o.permute(1, 0, 2).reshape(T, H * V)) @ g("o").T


def dense_ff(u, w, pre, limit, act=identity):
    """The clamped feed-forward: the gate is clamped from above, the up value on both sides;
    down(a * sigmoid(1.702 a) * (b + 1))."""
    g = lambda n: w[pre + n].to(F64)
    a = torch.clamp(u @ g("gate").T, max=float(limit))
    b = torch.clamp(u @ g("up").T, min=-float(limit), max=float(limit))
    return act(a * torch.sigmoid(1.702 * a) * (b + 1.0)) @ g("down").T


def expert(u, w, pre, act=identity):
    g = lambda n: w[pre + n].to(F64)
    return act(silu(u @ g("gate").T) * (u @ g("up").T)) @ g("down").T


def route(u, w, pre, top):
    """The experts with the largest scores sigmoid(W_r u), and those scores as they are."""
    s = torch.sigmoid(u @ w[pre + "router"].to(F64).T)
    pick = torch.topk(s, int(top), dim=-1)
    return pick.indices, pick.values


def routed_ff(u, w, pre, mlp, act=identity):
    """The sum over a token's chosen experts of expert(weight * u): the weight is on what goes IN."""
    pick, weight = route(u, w, pre, mlp["router"]["top"])
    out = torch.zeros(u.shape[0], u.shape[1], dtype=F64)
    for t in range(u.shape[0]):
        for e, a in zip(pick[t].tolist(), weight[t].tolist()):
            out[t] += expert(a * u[t:t + 1], w, f"{pre}e{e}.", act)[0]
    return out


def run_order(cfg):
    """(layer, does the embedding output join the stream in front of it) in the order the layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = int(lp["start"]), int(lp["stop"])
    order = [(i, False) for i in range(a)]
    for t in range(int(lp["times"])):
        order += [(i, t > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def sublayer(x, y, w, pre, sub, mult, eps):
    """x + mult * ls * norm(y): a norm on the sublayer's output, then a learned factor per channel."""
    return x + float(mult) * (rms_norm(y, w[f"{pre}norm{sub}b"], eps) * w[f"{pre}ls{sub}"].to(F64))


def forward(cfg, w, ids, act=identity, collect=None):
    """Logits [T, vocab] of one whole sequence.  `collect`, a list, receives the stream after every layer run."""
    eps, mult = float(cfg["norm"]["eps"]), cfg["residual_mult"]
    x0 = x = embed(ids, w, cfg["embedding"]["scale"])
    for i, joins in run_order(cfg):
        e, pre = cfg["layers"][i], f"l{i}."
        if e["type"] != "attention":
            raise ValueError(e["type"])
        if joins:
            x = x + x0
        y = attention(act(rms_norm(x, w[pre + "norm1"], eps)), w, pre + "mix.", e["mixer"], act)
        x = sublayer(x, y, w, pre, 1, mult, eps)
        mlp = e.get("mlp")
        if mlp is not None:
            u = act(rms_norm(x, w[pre + "norm2"], eps))
            if mlp["kind"] == "dense":
                y = dense_ff(u, w, pre + "mlp.", mlp["limit"], act)
            else:
                y = routed_ff(u, w, pre + "mlp.", mlp, act)
            x = sublayer(x, y, w, pre, 2, mult, eps)
        if collect is not None:
            collect.append(x.clone())
    return act(rms_norm(x, w["final.norm"], eps)) @ w["embed"].to(F64).T
