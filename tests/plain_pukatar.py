"""A plain, slow restatement of the Pukatar design: whole sequences, no cache, no state carried
between calls, one function per mechanism.  It shares no code with the engine; the tests compare
the engine with it.

Notation.  x [T, W] is the residual stream, u a layer's (normed) input, p the position of a token
in its sequence (from 0), `w` a dict of tensors by name, `pre` a name prefix, `m` a mixer's entry of
the configuration.  `act` rounds activations the way a run mode would (identity for the 32-bit mode);
what the design keeps in 32-bit stays unrounded.  Everything runs in float64 unless `act` rounds it.
"""
import torch

F64 = torch.float64
UNIT_EPS = 1e-6          # inside the root of the unit norm of queries and keys


def identity(x):
    return x


def bf16_round(x):
    """What a 16-bit run mode does to an activation between two kernels."""
    return x.to(torch.bfloat16).to(x.dtype)


def bf16_round_jittered(seed):
    """The same rounding after a relative nudge of up to half a unit in the last place: another
    implementation's rounding of the same exact value."""
    g = torch.Generator().manual_seed(seed)

    def act(x):
        nudge = (torch.rand(x.shape, generator=g, dtype=torch.float64) - 0.5) * 2.0 ** -8
        return (x * (1.0 + nudge.to(x.dtype))).to(torch.bfloat16).to(x.dtype)
    return act


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros((), dtype=z.dtype))


def rms_unit(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, name, eps):
    """(x - mean) / sqrt(mean of the squared deviations + eps) * weight + bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d * torch.rsqrt(d.pow(2).mean(dim=-1, keepdim=True) + eps) * w[name].to(F64) + w[name + ".b"].to(F64)


def embed(ids, w, eps):
    """The token's row, then the model's norm: the embedding output."""
    return layer_norm(w["embed"][torch.as_tensor(ids, dtype=torch.long)].to(F64), w, "embed.norm", eps)


def start_pass(x, x0, w, t, act=identity):
    """What happens to the stream in front of pass t of the looped span: it is joined with the embedding output by
    a matrix over both, and pass t's vector is added."""
    return torch.cat([act(x), act(x0)], dim=-1) @ w["loop.in"].to(F64).T + w["loop.step"][t].to(F64)


def rotate_half(t, positions, rot):
    """t [T, heads, n]: of the first rot.dims entries, entry i pairs with entry i + dims/2; the pair (a, b) at
    position p becomes (a cos - b sin, b cos + a sin) of the angle p * base^(-2i/dims).  The rest passes."""
    if not rot:
        return t
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = torch.as_tensor(positions, dtype=F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = t[..., :half], t[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, t[..., dims:]], dim=-1)


def visible_keys(T, mask):
    """[T, T] bool: query i sees key j if j <= i and (i - j < size or j < keep_first); without a mask every j <= i."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    vis = j <= i
    if mask:
        vis = vis & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return vis


def softmax_with_sinks(scores, v, visible, sinks):
    """scores [H, T, S], visible [T, S] bool, v [H, S, V], sinks [H]: head h's denominator has one more term
    exp(sinks[h]) that carries no value and is not scaled."""
    scores = scores.masked_fill(~visible[None], float("-inf"))
    z = sinks.to(F64)[:, None, None]
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, z)
    e = torch.exp(scores - top)
    return (e / (e.sum(dim=-1, keepdim=True) + torch.exp(z - top))) @ v


def attention(u, w, pre, m, act=identity):
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
    o = softmax_with_sinks(scores, vh, visible_keys(T, m.get("mask")), g("sink"))       # [H, T, V]
    return act(o.permute(1, 0, 2).reshape(T, H * V)) @ g("o").T


def short_conv(x, taps):
    """Causal, per channel: x [T, C], taps [C, n], the last tap on the token itself, zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += x[:T - back] * taps[:, j]
    return out


def unit(x):
    return x * torch.rsqrt(x.pow(2).sum(dim=-1, keepdim=True) + UNIT_EPS)


def delta_inputs(u, w, pre, m):
    """What the recurrence reads: q, k [T, H, D] (already per head), v [T, H, V], the step sizes beta [T, H] and the
    decays [T, H, D] per key channel."""
    T = u.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda n: w[pre + n].to(F64)
    mixed = {n: silu(short_conv(u @ g(n).T, g(n + ".conv"))) for n in ("q", "k", "v")}
    q = unit(mixed["q"].view(T, G, D)) * D ** -0.5
    k = unit(mixed["k"].view(T, G, D))
    rep = H // G
    beta = torch.sigmoid(u @ g("b").T)
    z = (u @ g("a1").T) @ g("a2").T + g("dt_bias")
    decay = torch.exp(-torch.exp(g("A_log"))[None, :, None] * softplus(z).view(T, H, D))
    return q.repeat_interleave(rep, dim=1), k.repeat_interleave(rep, dim=1), mixed["v"].view(T, H, V), beta, decay


def delta_rule(q, k, v, beta, decay, state=None):
    """Token by token, per head: S <- decay * S (by rows), u = beta (v - S^T k), S <- S + k u^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64) if state is None else state
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = decay[t][:, :, None] * S
        write = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * write[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def channel_delta(u, w, pre, m, eps, act=identity):
    T = u.shape[0]
    H, V = int(m["heads"]), int(m["vdim"])
    g = lambda n: w[pre + n].to(F64)
    o, S = delta_rule(*delta_inputs(u, w, pre, m))
    o = rms_unit(o, eps) * g("norm")
    gate = torch.sigmoid((u @ g("g1").T) @ g("g2").T)
    return act(o.reshape(T, H * V) * gate) @ g("o").T, S


def dense_ff(u, w, pre, act=identity):
    g = lambda n: w[pre + n].to(F64)
    return act(silu(u @ g("gate").T) * (u @ g("up").T)) @ g("down").T


def expert(u, w, pre, limit, act=identity):
    """down(g * sigmoid(1.702 g) * (u + 1)) with the gate clamped from above and the up value on both sides."""
    g = lambda n: w[pre + n].to(F64)
    a = torch.clamp(u @ g("gate").T, max=limit)
    b = torch.clamp(u @ g("up").T, min=-limit, max=limit)
    return act(a * torch.sigmoid(1.702 * a) * (b + 1.0)) @ g("down").T


def route(u, w, pre, top):
    """The experts with the largest logits z = W_r u + b, and the softmax over the chosen logits only."""
    z = u @ w[pre + "router"].to(F64).T + w[pre + "router.b"].to(F64)
    pick = torch.topk(z, int(top), dim=-1)
    return pick.indices, torch.softmax(pick.values, dim=-1)


def routed_ff(u, w, pre, mlp, act=identity):
    pick, weight = route(u, w, pre, mlp["router"]["top"])
    limit = float(mlp["expert"]["limit"])
    out = torch.zeros(u.shape[0], u.shape[1], dtype=F64)
    for t in range(u.shape[0]):
        for e, a in zip(pick[t].tolist(), weight[t].tolist()):
            out[t] += a * expert(u[t:t + 1], w, f"{pre}e{e}.", limit, act)[0]
    if mlp.get("shared") is not None:
        share = torch.sigmoid(u @ w[pre + "shared.sg"].to(F64).T)                        # one number a token
        out = out + share * expert(u, w, pre + "shared.", float(mlp["shared"]["limit"]), act)
    return out


def run_order(cfg):
    """(layer, pass that starts in front of it or None) in the order the layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = int(lp["start"]), int(lp["stop"])
    order = [(i, None) for i in range(a)]
    for t in range(int(lp["times"])):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg, w, ids, act=identity, collect=None):
    """Logits [T, vocab] of one whole sequence.  `collect`, a list, receives the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x0 = x = embed(ids, w, eps)
    for i, starts in run_order(cfg):
        e, pre = cfg["layers"][i], f"l{i}."
        if starts is not None:
            x = start_pass(x, x0, w, starts, act)
        u = act(layer_norm(x, w, pre + "norm1", eps))
        if e["type"] == "attention":
            y = attention(u, w, pre + "mix.", e["mixer"], act)
        elif e["type"] == "channel_delta":
            y, _ = channel_delta(u, w, pre + "mix.", e["mixer"], eps, act)
        else:
            raise ValueError(e["type"])
        if e.get("mlp") is not None:
            if e["mlp"]["kind"] == "dense":
                y = y + dense_ff(u, w, pre + "mlp.", act)
            else:
                y = y + routed_ff(u, w, pre + "mlp.", e["mlp"], act)
        x = x + y
        if collect is not None:
            collect.append(x.clone())
    return act(layer_norm(x, w, "final.norm", eps)) @ w["head"].to(F64).T
