"""The Pukatar design in the engine against the plain implementation of `plain_pukatar.py`: every mechanism's
kernel alone (with inputs made so that a lost key, a wrong edge, a lost sink or a lost state shows), then whole models
in every way of cutting a request into steps, mixed batches with pages and state slots used again, long decoding under
CUDA graphs, and greedy generation through the engine's own entry point and scheduler."""
import types

import numpy as np
import pytest
import torch

import plain_pukatar as pp
import pukatar_models as pm
import replay_helpers as rh

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

CASES = {"A": (pm.PUK_A, pm.PUK_A_PAGE, 3), "B": (pm.PUK_B, pm.PUK_B_PAGE, 5), "C": (pm.PUK_C, pm.PUK_C_PAGE, 9),
         "D": (pm.PUK_D, pm.PUK_D_PAGE, 11), "E": (pm.PUK_E, pm.PUK_E_PAGE, 13)}
# root mean square over the vocabulary of (difference minus its mean), as a fraction of the reference logits'
# spread; the float32 run is measured against the plain code in double precision
LIMIT = {"float32": 1e-4, "bfloat16": 0.12}


def model_of(case):
    cfg, page, seed = CASES[case]
    return cfg, page, pm.random_weights(cfg, seed)


def _spread_error(row, ref_row, spread):
    d = np.asarray(row, dtype=np.float64) - ref_row
    return float(np.sqrt(np.mean((d - d.mean()) ** 2))) / spread


class Reference:
    """Whole-sequence logits of the plain code in double precision, and for each position the error that rounding
    activations to bfloat16 alone causes there (the plain code run again with that rounding, and with the rounding
    jittered): a close call between two experts that a 16-bit run decides the other way is a jump that no
    implementation can avoid, and none can be held to more than a few times its own rounding."""

    def __init__(self, cfg, w, reqs, dtype):
        w64 = {k: v.double() for k, v in w.items()}
        self.rows = {r: pp.forward(cfg, w64, t).numpy() for r, t in reqs.items()}
        self.spread = float(np.sqrt(np.mean([np.var(v) for v in self.rows.values()])))
        self.dtype = dtype
        self.own = {}
        if dtype == "bfloat16":
            for r, t in reqs.items():
                runs = [pp.forward(cfg, w64, t, act=pp.bf16_round).numpy()]
                runs += [pp.forward(cfg, w64, t, act=pp.bf16_round_jittered(seed)).numpy() for seed in (1, 2)]
                self.own[r] = [max(_spread_error(x[p], self.rows[r][p], self.spread) for x in runs) for p in range(len(t))]

    def limit(self, r, pos):
        return max(LIMIT[self.dtype], 3.0 * self.own[r][pos]) if self.own else LIMIT[self.dtype]

    def error(self, row, r, pos):
        return _spread_error(row, self.rows[r][pos], self.spread)


def assert_close(got, ref, dtype, what):
    """float32: every position within the limit.  bfloat16: 3 positions in 100 may exceed theirs."""
    assert got, "nothing was compared"
    held, over = 0, []
    for (r, pos) in sorted(got):
        err, limit = ref.error(got[(r, pos)], r, pos), ref.limit(r, pos)
        if err > limit:
            over.append(f"{what}: request {r} position {pos}: {err:.3e} > {limit:.1e}")
        held += limit <= 2 * LIMIT[dtype]
    allowed = 0 if dtype == "float32" else max(1, int(0.03 * len(got)))
    assert len(over) <= allowed, "; ".join(over[:5])
    assert held >= 0.6 * len(got), "too few positions are well conditioned for this to be a test"


def requests(cfg, lengths, seed):
    return {f"r{i}": pm.random_tokens(cfg, n, seed * 100 + i) for i, n in enumerate(lengths)}


# ---- whole models, every cutting ------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["A", "B", "C", "D", "E"])
def test_every_cutting_matches_plain(case, dtype):
    cfg, page, w = model_of(case)
    reqs = requests(cfg, [1, 2, 3, 37, 90, 150], seed=1)
    ref = Reference(cfg, w, reqs, dtype)
    for name, steps in (("whole", rh.trace_whole(reqs)), ("decode", rh.trace_tail_decode(reqs, tail=33)),
                        ("portions", rh.trace_portions(reqs, seed=2)),
                        ("mixed", rh.trace_mixed(reqs, seed=3, max_live=3))):
        # a pool just large enough, and three slots for six requests: pages and slots are used again
        runner = rh.make_runner(cfg, w, dtype, page, rh.peak_tokens(steps, round_to=page), max_requests=3)
        assert_close(rh.run_trace(runner, steps), ref, dtype, f"{case} {name}")
        runner.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompt_window_and_kept_keys_over_pages(dtype):
    """600 tokens: the window of 130 keys passes over page borders in one step, in portions of many sizes and in 140
    decoded tokens, while the first 21 keys (a page and a third) stay; pages between them go back to the pool on the way."""
    cfg, page, w = model_of("C")
    reqs = requests(cfg, [600, 300], seed=4)
    ref = Reference(cfg, w, reqs, dtype)
    for name, steps in (("whole", rh.trace_whole(reqs)), ("decode", rh.trace_tail_decode(reqs, tail=140)),
                        ("portions", rh.trace_portions(reqs, seed=5, sizes=(2, 61, 64, 65, 128, 257, 300)))):
        runner = rh.make_runner(cfg, w, dtype, page, rh.peak_tokens(steps, round_to=page), max_requests=2)
        assert_close(rh.run_trace(runner, steps), ref, dtype, name)


def test_long_prompt_with_attention_heads_of_128():
    """350 tokens in the 16-bit mode with attention heads of 128: portions that start in the middle of a page, a window
    of 140 keys with six kept ones, decoded tokens after them."""
    cfg, page, w = model_of("E")
    reqs = requests(cfg, [350, 160], seed=8)
    ref = Reference(cfg, w, reqs, "bfloat16")
    for name, steps in (("whole", rh.trace_whole(reqs)), ("decode", rh.trace_tail_decode(reqs, tail=40)),
                        ("portions", rh.trace_portions(reqs, seed=9, sizes=(2, 61, 127, 128, 129, 257)))):
        runner = rh.make_runner(cfg, w, "bfloat16", page, rh.peak_tokens(steps, round_to=page), max_requests=2)
        assert_close(rh.run_trace(runner, steps), ref, "bfloat16", name)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_under_graphs(dtype):
    """Two prompt tokens, then 200 single-token steps of two requests side by side: steps of one shape are replayed as
    a captured graph, the recurrent states and the convolutions' last inputs move on once per replay, in every pass of
    the loop, and the windows slide past the kept keys."""
    cfg, page, w = model_of("A")
    reqs = requests(cfg, [202, 180], seed=6)
    ref = Reference(cfg, w, reqs, dtype)
    steps = [{"step": 0, "entries": [{"id": r, "tokens": t[:2], "want": [0, 1]} for r, t in reqs.items()], "end": []}]
    for k in range(2, 202):
        live = [(r, t) for r, t in reqs.items() if k < len(t)]
        steps.append({"step": len(steps), "entries": [{"id": r, "tokens": [t[k]], "want": [0]} for r, t in live],
                      "end": [r for r, t in live if k == len(t) - 1]})
    runner = rh.make_runner(cfg, w, dtype, page, rh.peak_tokens(steps, round_to=page), max_requests=2)
    assert_close(rh.run_trace(runner, steps), ref, dtype, "long decoding")
    assert runner.graph_replays > 100


def test_batch_does_not_change_a_request():
    """The same request alone and beside others of other lengths: float32 logits agree to rounding."""
    cfg, page, w = model_of("B")
    reqs = requests(cfg, [64, 5, 33], seed=7)
    alone = {}
    for r, t in reqs.items():
        runner = rh.make_runner(cfg, w, "float32", page, 256, max_requests=3)
        alone.update(rh.run_trace(runner, rh.trace_whole({r: t})))
    runner = rh.make_runner(cfg, w, "float32", page, 256, max_requests=3)
    steps = [{"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()],
              "end": list(reqs)}]
    together = rh.run_trace(runner, steps)
    for key, row in alone.items():
        assert np.abs(row - together[key]).max() <= 2e-5 * max(1.0, np.abs(row).max()), key


def test_greedy_generation_through_the_engine_and_scheduler():
    """`PagedGenerateEngine.generate`: chunked prompts, decode batches, more requests than slots, a pool that forces
    preemption; the tokens are the plain code's greedy tokens."""
    from litellmengine_b200.engine import PagedGenerateEngine
    cfg, page, w = model_of("B")
    w64 = {k: v.double() for k, v in w.items()}
    prompts = [pm.random_tokens(cfg, n, 50 + i) for i, n in enumerate([9, 30, 3, 17, 22])]
    new = 12
    want = []
    for p in prompts:
        ids = list(p)
        for _ in range(new):
            ids.append(int(pp.forward(cfg, w64, ids)[-1].argmax()))
        want.append(ids[len(p):])
    runner = rh.make_runner(cfg, w, "float32", page, 64, max_requests=3, max_tokens_per_step=32)
    engine = PagedGenerateEngine(runner, chunk=8)
    got = engine.generate(prompts, new)
    assert got == want
    assert engine.scheduler.num_preemptions > 0
    runner.cache.check_invariants()


def test_trace_replay_and_prompt_command_on_a_model_folder(tmp_path):
    """`bin/trace_run` and `bin/run_prompt` on a folder written in the design's own format."""
    import json
    import os
    import subprocess
    import sys
    from litellmengine_b200.weights.safetensors_io import write_safetensors
    cfg, page, w = model_of("A")
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    toks = pm.random_tokens(cfg, 40, 8)
    w64 = {k: v.double() for k, v in w.items()}
    ref = pp.forward(cfg, w64, toks).numpy()
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:25], "want": [3, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[25:], "want": [14]}], "end": ["a"]}]
    out = tmp_path / "out"
    res = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32",
                          "--out", str(out), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    spread = float(np.std(ref))
    got0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    got1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    for row, pos in ((got0[0], 3), (got0[1], 24), (got1[0], 39)):
        assert _spread_error(row, ref[pos], spread) < 1e-4
    prompt = toks[:17]
    ids = list(prompt)
    for _ in range(6):
        ids.append(int(pp.forward(cfg, w64, ids)[-1].argmax()))
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "run_prompt"), "--model", str(folder), "--input-ids",
                           ",".join(map(str, prompt)), "--max-tokens", "6", "--dtype", "float32"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stdout[-2000:] + proc.stderr[-2000:]
    assert proc.stdout.strip().split("\n")[-1] == ",".join(map(str, ids[len(prompt):]))


# ---- mechanisms alone -------------------------------------------------------------------------------
def _ops():
    from litellmengine_b200.csrc import ops
    return ops


def _i32(x):
    return torch.as_tensor(x, dtype=torch.int32, device=DEV)


def _f32(t):
    return t.float().to(DEV).contiguous()


def _batch(portions):
    """What the kernels read of a step: `portions` = [(slot, first position, tokens)] in batch order."""
    pos, ent, slots, starts, lens = [], [], [], [], []
    for e, (slot, p0, n) in enumerate(portions):
        starts.append(len(pos))
        lens.append(n)
        slots.append(slot)
        pos += list(range(p0, p0 + n))
        ent += [e] * n
    return types.SimpleNamespace(positions=_i32(pos), token_entry=_i32(ent), entry_slot=_i32(slots), entry_q_start=_i32(starts),
                                 entry_q_len=_i32(lens), num_tokens=len(pos),
                                 num_entries=len(portions))


def _paged(T, page, nkv, dk, dv, dtype, shuffle_seed=0):
    """One request of T tokens in slot 1 of 3, its pages scattered over a pool."""
    n = -(-T // page)
    pool = n + 5
    order = np.random.RandomState(shuffle_seed).permutation(pool)[:n]
    table = torch.full((3, n + 2), -1, dtype=torch.int32)
    table[1, :n] = torch.as_tensor(order, dtype=torch.int32)
    keys = torch.zeros(pool, nkv, page, dk, dtype=dtype, device=DEV)
    values = torch.zeros(pool, nkv, page, dv, dtype=dtype, device=DEV) if dv else None
    return keys, values, table.to(DEV), order


def _pairs(H, seed):
    g = torch.Generator().manual_seed(seed)
    return {"n": 1 + 0.2 * torch.randn(H, generator=g, dtype=F64), "n.b": 0.3 * torch.randn(H, generator=g, dtype=F64)}


@pytest.mark.parametrize("H", [40, 30, 1024, 4100])
def test_layer_norm_with_a_bias_and_what_joins_on_the_way(H):
    """out = LN(h + y + y2) * w + b with h written back: two sublayers' outputs as matrices and as the k-splits of
    products, one of them absent; the start of a pass (another source, one row for all tokens, an output); picked rows;
    the new stream itself without a norm.  Row lengths that take sixteen-byte accesses and that do not; a mean far from
    zero."""
    ops = _ops()
    T, eps = 11, 1e-5
    g = torch.Generator().manual_seed(H)
    h0 = torch.randn(T, H, generator=g, dtype=F64) + 5.0
    y, y2 = torch.randn(3, T, H, generator=g, dtype=F64), torch.randn(2, T, H, generator=g, dtype=F64)
    w = _pairs(H, 3)
    nw, nb = _f32(w["n"]), _f32(w["n.b"])
    run = lambda h, y, **k: ops.stream_norm(h, y, None, None, None, nw, eps, True, k.pop("dtype", torch.float32), bias=nb, **k)
    plain = lambda x: pp.layer_norm(x, w, "n", eps)
    h = _f32(h0)
    assert (run(h, None).double().cpu() - plain(h0)).abs().max() < 2e-5 and torch.equal(h.cpu(), h0.float())
    want_h = h0 + y.sum(0) + y2.sum(0)
    for form in ("matrices", "splits", "bf16 out"):
        h = _f32(h0)
        a, b = (ops.PartialSum(_f32(y)), ops.PartialSum(_f32(y2))) if form == "splits" else (_f32(y.sum(0)), _f32(y2.sum(0)))
        out = run(h, a, y2=b, dtype=torch.bfloat16 if form == "bf16 out" else torch.float32)
        assert (h.double().cpu() - want_h).abs().max() < 1e-5
        assert (out.double().cpu() - plain(want_h)).abs().max() < (4e-2 if form == "bf16 out" else 2e-5)
    # the start of a pass: the stream is replaced
    base, row = torch.randn(T, H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64)
    h, src = _f32(h0), _f32(base)
    out = run(h, ops.PartialSum(_f32(y)), source=src, add=_f32(row))
    want = base + row + y.sum(0)
    assert (h.double().cpu() - want).abs().max() < 1e-5 and (out.double().cpu() - plain(want)).abs().max() < 2e-5
    assert torch.equal(src.cpu(), base.float())
    # picked rows leave the stream alone; no norm: the stream itself, written back or not
    h, rows = _f32(h0), [7, 0, 7, 10]
    out = run(h, _f32(y.sum(0)), y2=ops.PartialSum(_f32(y2)), rows=_i32(rows))
    assert (out.double().cpu() - plain(want_h)[rows]).abs().max() < 2e-5 and torch.equal(h.cpu(), h0.float())
    out = ops.stream_norm(h, _f32(y.sum(0)), None, None, None, None, 0.0, False, torch.bfloat16, write_back=False, y2=_f32(y2.sum(0)))
    assert (out.double().cpu() - want_h).abs().max() < 0.1 and torch.equal(h.cpu(), h0.float())
    ops.stream_norm(h, _f32(y[0]), None, None, None, None, 0.0, False, None, source=src, add=_f32(row))
    assert (h.double().cpu() - (base + row + y[0])).abs().max() < 1e-5


@pytest.mark.parametrize("H,dtype", [(40, "bfloat16"), (30, "float32"), (2048, "bfloat16")])
def test_embedding_with_the_models_norm(H, dtype):
    ops = _ops()
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    g = torch.Generator().manual_seed(H)
    table = (torch.randn(50, H, generator=g, dtype=F64) + 1.0).to(tdt)
    w = dict(_pairs(H, 5), embed=table.double())
    w = {k.replace("n", "embed.norm", 1) if k[0] == "n" else k: v for k, v in w.items()}
    ids = [3, 0, 49, 3, 17, -2]                                  # the last one is the token in place 1 of the feedback buffer
    status = torch.zeros(2, dtype=torch.int32, device=DEV)
    out, copy = ops.embedding_norm(_i32(ids), table.to(DEV), _f32(w["embed.norm"]), _f32(w["embed.norm.b"]), 1e-5, True, status,
                                   feedback=_i32([1, 44]), copy_dtype=tdt)
    ref = pp.embed(ids[:-1] + [44], w, 1e-5)
    assert status.tolist() == [0, 0]
    assert (out.double().cpu() - ref).abs().max() < 1e-5
    assert (copy.double().cpu() - ref).abs().max() < (4e-2 if dtype == "bfloat16" else 1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_start_of_a_pass_joins_the_embedding(dtype):
    """x <- W [x; x0] + step[t] for every pass, with outputs still pending on x; one half of W is applied once."""
    from litellmengine_b200.config.specs import NormSpec, RejoinSpec
    from litellmengine_b200.parts.norms import LayerNorm, PendingSum
    from litellmengine_b200.parts.rejoin import EmbeddingRejoin
    ops, W, T, times = _ops(), 48, 9, 3
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    g = torch.Generator().manual_seed(1)
    bf = lambda t: t.to(torch.bfloat16).double()
    w = {"loop.in": bf(torch.randn(W, 2 * W, generator=g, dtype=F64) * W ** -0.5), "loop.step": bf(torch.randn(times, W, generator=g, dtype=F64)),
         "n": torch.ones(W, dtype=F64), "n.b": torch.zeros(W, dtype=F64)}
    part = EmbeddingRejoin(RejoinSpec(passes=times), W, tdt)
    part.load({"loop.in": w["loop.in"].to(tdt).to(DEV), "loop.step": _f32(w["loop.step"])})
    norm = LayerNorm(NormSpec("layernorm", 1e-5, "", True), W)
    norm.load({"": _f32(w["n"]), "b": _f32(w["n.b"])})
    x, x0, y, y2 = (torch.randn(T, W, generator=g, dtype=F64) for _ in range(4))
    base = part.begin(x0.to(tdt).to(DEV))
    act = pp.bf16_round if dtype == "bfloat16" else pp.identity
    for t in (1, 0, 2):
        h = _f32(x)
        u = norm.forward(h, torch.float32, delta=part.start(h, None, PendingSum(_f32(y), _f32(y2)), base, t), write_sum=True)
        want = pp.start_pass(x + y + y2, x0, w, t, act)
        assert (h.double().cpu() - want).abs().max() < (2e-5 if dtype == "float32" else 5e-2)
        assert (u.double().cpu() - pp.layer_norm(want, w, "n", 1e-5)).abs().max() < (2e-5 if dtype == "float32" else 5e-2)
        h2 = _f32(x)                                          # for norms that do not take it: the new stream written plainly
        part.start(h2, None, PendingSum(_f32(y), _f32(y2)), base, t).settle_into(h2)
        assert (h2 - h).abs().max() < 1e-5


@pytest.mark.parametrize("window,keep,dims", [(None, 0, 8), (1, 0, 12), (7, 3, 4), (64, 17, 12), (65, 16, 0), (5, 40, 6)])
def test_attention_half_rotation_window_kept_keys_and_learned_sinks(window, keep, dims):
    """The kernels between the projections of an attention layer, on projections given as numbers: the rotation of the
    pairs (i, i + dims/2), the page write, then attention with a window, kept first keys and a learned score per head in the
    denominator.  One key is turned towards a late query so that it would win by far, and placed just inside and just
    outside that query's window, just inside and just outside the kept keys, at a page's last and first place and at the
    sequence's first token.  The last query's own scores are made very negative, so that the sinks take nearly all of its
    weight.  Prompt rows and single tokens against the plain functions."""
    ops = _ops()
    T, page, H, G, D, V, scale = 150, 16, 6, 2, 12, 20, 0.3
    g = torch.Generator().manual_seed(5)
    proj = torch.randn(T, H * D + G * D + G * V, generator=g, dtype=F64)
    sinks = torch.tensor([0.0, 3.0, -2.0, 8.0, 1.0, -50.0], dtype=F64)
    rot = {"base": 300.0, "dims": dims} if dims else None
    mask = {"size": window, "keep_first": keep} if window else None
    ko, vo = H * D, H * D + G * D

    def plain(p, sinks=sinks):
        pos = list(range(T))
        q, k = pp.rotate_half(p[:, :ko].view(T, H, D), pos, rot), pp.rotate_half(p[:, ko:vo].view(T, G, D), pos, rot)
        s = (q.permute(1, 0, 2) @ k.permute(1, 0, 2).repeat_interleave(H // G, 0).transpose(1, 2)) * scale
        vh = p[:, vo:].view(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, 0)
        return pp.softmax_with_sinks(s, vh, pp.visible_keys(T, mask), sinks).permute(1, 0, 2).reshape(T, H * V)

    def unrotate(x, i, j):              # a key at j that a query x at i meets as x itself: x turned by the angle of j - i
        return pp.rotate_half(x[None, None], [i - j], rot)[0, 0] if rot else x

    probes = [(149, (window or 150) - 1), (148, window or 148), (130, (window or 131) - 1), (141, 141 - 16), (140, 140 - 15), (120, 120),
              (147, 147 - max(keep - 1, 0)), (146, 146 - keep)]
    for i, back in probes:
        j = i - back
        if 0 <= j < i:
            proj[j, ko:ko + D] = unrotate(proj[i, :D], i, j) * 6.0
    seen = [j for j in range(T - 1) if pp.visible_keys(T, mask)[T - 1, j]] + [T - 1]
    for gr in range(G):                                     # the last query looks away from everything it sees
        proj[T - 1, gr * (ko // G):gr * (ko // G) + ko // G] = proj[T - 1, :D].repeat(H // G)
        for j in seen:
            proj[j, ko + gr * D:ko + gr * D + D] = unrotate(proj[T - 1, :D], T - 1, j) * -3.0 if window and window < 9 else proj[j, ko + gr * D:ko + gr * D + D]
    ref = plain(proj)
    assert (ref - plain(proj, sinks * 0 - 60.0)).abs().max() > 0.05          # the sinks matter
    assert (ref - plain(proj, sinks.roll(1))).abs().max() > 0.05             # and each belongs to its head
    from litellmengine_b200.config.specs import PositionSpec
    from litellmengine_b200.parts.registry import lookup
    import litellmengine_b200.parts.position  # noqa: F401  (registers the kinds)
    rotation = lookup("position", "rope_half")(PositionSpec("rope_half", 300.0, dims), D, DEV).kernel_args() if dims else None
    for dtype, tol in ((torch.float32, 5e-5), (torch.bfloat16, 0.08)):
        for portions in ([(1, 0, T)], [(1, 0, 70), (1, 70, 2), (1, 72, 77), (1, 149, 1)]):
            keys, values, block_table, order = _paged(T, page, G, D, V, dtype, 2)
            out = torch.zeros(T, H * V, dtype=dtype, device=DEV)
            status = torch.zeros(2, dtype=torch.int32, device=DEV)
            for slot, p0, n in portions:                        # step by step, as a request would run
                b = _batch([(slot, p0, n)])
                rows = _f32(proj[p0:p0 + n])
                q = ops.attention_prepare(rows, 0, ko, vo, None, None, None, None, 0.0, None, keys, values, b.positions,
                                          b.token_entry, b.entry_slot, block_table, H, G, D, V, page, status, dtype, rotation=rotation)
                o = torch.zeros(n, H * V, dtype=dtype, device=DEV)
                ops.paged_attention_generic_kv(q, keys, values, b.positions, b.token_entry, b.entry_slot, block_table, H, G, D, V,
                                               page, window, scale, status, o, keep_first=keep, sink=_f32(sinks))
                out[p0:p0 + n] = o
            assert status.tolist() == [0, 0]
            assert (out.double().cpu() - ref).abs().max() < tol, (window, keep, dims, dtype, len(portions))
    if window:                      # the edges matter: one key further out, or one more kept, and the result is another
        mask = {"size": window + 1, "keep_first": keep}
        assert (ref - plain(proj)).abs().max() > 0.02
        mask = {"size": window, "keep_first": keep + 1}
        assert (ref - plain(proj)).abs().max() > 0.02


@pytest.mark.parametrize("d,group,window,keep", [(64, 3, 100, 5), (128, 1, 64, 70), (128, 2, 140, 6), (128, 8, None, 0), (64, 4, 30, 0)])
def test_tensor_core_attention_with_kept_keys_and_learned_sinks(d, group, window, keep):
    """The kernels that a 16-bit run takes at head sizes 64 and 128: a prompt portion that starts in the middle of a page
    with keys before it, and single tokens in the split-key decode kernel with one and several splits; a score per head in
    the denominator, some far below and some above the keys' scores.  Keys that would win by far sit among the kept ones,
    just behind them, and at the window's first and just before it."""
    ops = _ops()
    N, past, page, G, scale = 420, 37, 16, 2, 0.2
    H, T = G * group, N - past
    g = torch.Generator().manual_seed(d + group)
    q, k, v = (torch.randn(N, n, d, generator=g, dtype=F64) for n in (H, G, G))
    sinks = torch.tensor([10.0 - 4.0 * (h % 3) for h in range(H)], dtype=F64)
    w = window or N
    for i, j in ((419, max(keep - 1, 0)), (418, keep), (417, 417 - w + 1), (416, 416 - w), (300, 3), (299, max(299 - w, 0))):
        k[j] = q[i, ::group] * (40.0 / d)          # a score of about eight
    q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
    mask = {"size": window, "keep_first": keep} if window else None
    vis = pp.visible_keys(N, mask)[past:]
    kh, vh = (t.permute(1, 0, 2).repeat_interleave(group, 0) for t in (k, v))
    scores = (q[past:].permute(1, 0, 2) @ kh.transpose(1, 2)) * scale
    ref = pp.softmax_with_sinks(scores, vh, vis, sinks).permute(1, 0, 2)
    order = np.random.RandomState(2).permutation(N // page + 6)[:-(-N // page)]
    block_table = torch.full((3, len(order) + 2), -1, dtype=torch.int32)
    block_table[1, :len(order)] = torch.as_tensor(order, dtype=torch.int32)
    block_table = block_table.to(DEV)
    cache = torch.zeros(N // page + 6, 2, G, page, d, dtype=torch.bfloat16, device=DEV)
    for j in range(N):
        cache[order[j // page], 0, :, j % page] = k[j].to(torch.bfloat16).to(DEV)
        cache[order[j // page], 1, :, j % page] = v[j].to(torch.bfloat16).to(DEV)
    qd = q[past:].reshape(T, -1).to(torch.bfloat16).to(DEV)
    out = torch.zeros(T, H * d, dtype=torch.bfloat16, device=DEV)
    status = torch.zeros(2, dtype=torch.int32, device=DEV)
    tiles = _i32([(0, r0) for r0 in range(0, T, ops.PREFILL_TILE_ROWS)])
    ops.paged_attention_prefill_biased(qd, out, 0, cache, tiles, tiles.shape[0], _i32([1]), _i32([0]), _i32([T]), _i32([N]),
                                       block_table, H, G, d, page, window, scale, status, keep_first=keep, sink=_f32(sinks))
    assert status.tolist() == [0, 0]
    assert (out.double().cpu().view(T, H, d) - ref).abs().max() < 0.06
    assert ops.fast_attention_supported(d, group)
    for splits in (1, 3):
        a = torch.zeros(T, H * d, dtype=torch.bfloat16, device=DEV)
        picked = [T - 1, T - 2, T - 3, T - 4, 5, 263, 262]
        ops.paged_attention_decode(qd, a, cache, _i32(picked + [-1]), len(picked) + 1, _i32(list(range(past, N))), _i32([0] * T),
                                   _i32([1]), block_table, H, G, d, page, window, scale, splits, status, keep_first=keep, sink=_f32(sinks))
        assert status.tolist() == [0, 0]
        assert (a.double().cpu().view(T, H, d)[picked] - ref[picked]).abs().max() < 0.06, splits
    # the edges and the sinks matter
    if window and keep:
        other = pp.softmax_with_sinks(scores, vh, pp.visible_keys(N, {"size": window})[past:], sinks).permute(1, 0, 2)
        assert (other - ref).abs().max() > 0.05
    for other in (sinks * 0 - 60.0, sinks.roll(1)):
        assert (pp.softmax_with_sinks(scores, vh, vis, other).permute(1, 0, 2) - ref).abs().max() > 0.1


def _delta_weights(H, G, D, V, taps, Wd, ranks, seed):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    w = {"q": n(G * D, Wd) * Wd ** -0.5, "k": n(G * D, Wd) * Wd ** -0.5, "v": n(H * V, Wd) * Wd ** -0.5, "b": n(H, Wd) * Wd ** -0.5,
         "q.conv": n(G * D, taps) * 0.7, "k.conv": n(G * D, taps) * 0.7, "v.conv": n(H * V, taps) * 0.7,
         "a1": n(ranks[0], Wd) * Wd ** -0.5, "a2": n(H * D, ranks[0]), "dt_bias": n(H * D) * 2 - 2, "A_log": n(H) * 0.7,
         "g1": n(ranks[1], Wd) * Wd ** -0.5, "g2": n(H * V, ranks[1]), "norm": 1 + 0.1 * n(V), "o": torch.eye(H * V, dtype=F64)}
    return w


@pytest.mark.parametrize("H,G,D,V,taps", [(2, 2, 8, 16, 3), (6, 2, 5, 3, 4), (1, 1, 48, 64, 1), (4, 2, 32, 20, 5), (2, 1, 128, 130, 4),
                                          (2, 2, 160, 33, 2), (3, 1, 64, 7, 4)])
def test_delta_rule_in_one_pass_in_portions_and_token_by_token(H, G, D, V, taps):
    """The recurrent mixer's kernels on projections made from given weights, against the plain token-by-token function:
    convolutions with silu, unit norms, decays, step sizes, the recurrence and the gated norm in one pass, in portions that
    carry the state and the convolutions' last inputs in the request's slot (down to two tokens and one: shorter than the
    taps), and through the kernel of decode steps; two requests side by side in one step; a channel that never forgets
    carries an impulse from the first tokens to the last, one that forgets at once loses it.  Other slots stay untouched,
    and the projection may sit anywhere in a wider one."""
    ops = _ops()
    T, Wd, ranks, eps, slots, off = 150, 24, (5, 3), 1e-5, 4, 3
    w = _delta_weights(H, G, D, V, taps, Wd, ranks, H * 100 + D)
    w["a2"][0], w["dt_bias"][0] = 0.0, -60.0            # never forgets
    w["a2"][1], w["dt_bias"][1] = 0.0, 200.0            # forgets at once
    w["k.conv"][0] *= 0.1
    g = torch.Generator().manual_seed(7)
    u = torch.randn(T, Wd, generator=g, dtype=F64)
    u[0] *= 4.0
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V}
    ref, s_ref = pp.channel_delta(u, w, "", m, eps)
    proj = torch.cat([u @ w[n].T for n in ("q", "k", "v", "b", "a1", "g1")], dim=1)
    C = 2 * G * D + H * V
    offs = (off, off + C, off + C + H, off + C + H + ranks[0])
    wide = torch.full((T, proj.shape[1] + off + 2), 9.0, dtype=torch.float32, device=DEV)
    wide[:, off:off + proj.shape[1]] = _f32(proj)
    conv = _f32(torch.cat([w["q.conv"], w["k.conv"], w["v.conv"]]))
    DP = ops.delta_padded(D)
    ring0, total = H * V * DP, (H * V * DP + taps * C + 3) // 4 * 4

    def step(state, out, portions, single, dtype=torch.float32):
        """portions = [(slot, first position, tokens)], the rows of the projection are the tokens' positions."""
        b = _batch(portions)
        rows = torch.cat([wide[p0:p0 + n] for _, p0, n in portions]).contiguous()
        o = torch.full((rows.shape[0], H * V + 5), -3.0, dtype=dtype, device=DEV)
        ops.delta_rule(rows, offs, ranks, conv, _f32(w["a2"].T), _f32(w["g2"].T), _f32(w["dt_bias"]), _f32(w["A_log"]), _f32(w["norm"]),
                       eps, 1.0, o, 2, state, b, H, G, D, V, single=single)
        assert float((o[:, :2] + 3).abs().max()) == 0 and float((o[:, 2 + H * V:] + 3).abs().max()) == 0
        at = 0
        for i, (_, p0, n) in enumerate(portions):
            out[i][p0:p0 + n] = o[at:at + n, 2:2 + H * V].float()
            at += n

    def check(state, slot, out, what, upto=T):
        assert (out[:upto].double().cpu() - ref[:upto]).abs().max() < 3e-5 * max(1.0, float(ref.abs().max())), what
        if upto == T:
            S = state[slot, :ring0].view(H, V, DP).double().cpu()
            assert (S[:, :, :D].transpose(1, 2) - s_ref).abs().max() < 3e-5 * max(1.0, float(s_ref.abs().max())), what
            assert D == DP or float(S[:, :, D:].abs().max()) == 0

    def fresh():
        state = torch.zeros((slots, total), dtype=torch.float32, device=DEV)
        state[1] = 7.0                                            # another request's state stays untouched
        return state, [torch.zeros((T, H * V), dtype=torch.float32, device=DEV) for _ in range(2)]

    for what, cuts in (("one pass", [T]), ("portions", [2, 1, 16, 17, 2, 64, 3, 45]), ("a portion, then token by token", [33] + [1] * (T - 33)),
                       ("token by token from the start", [1] * 12 + [T - 12])):
        state, outs = fresh()
        at = 0
        for n in cuts:
            step(state, outs, [(2, at, n)], single=n == 1 and "token" in what)
            at += n
        assert at == T and float((state[1] - 7.0).abs().max()) == 0 and float(state[0].abs().max()) == 0
        check(state, 2, outs[0], what)
    # two requests in one step: portions beside single tokens, then both in the decode kernel
    state, outs = fresh()
    step(state, outs, [(3, 0, 50), (0, 0, 1)], False)
    step(state, outs, [(3, 50, 1), (0, 1, 70)], False)
    for k in range(T - 71):
        step(state, outs, [(3, 51 + k, 1), (0, 71 + k, 1)], True)
    check(state, 3, outs[0], "beside another", upto=T - 20)
    check(state, 0, outs[1], "beside another")
    # 16-bit output
    state, outs = fresh()
    step(state, outs, [(2, 0, T)], False, dtype=torch.bfloat16)
    assert (outs[0].double().cpu() - ref).abs().max() < 2e-2 * max(1.0, float(ref.abs().max()))
    # the two channels are what they are meant to be
    decay = pp.delta_inputs(u, w, "", m)[4].reshape(T, H * D)
    assert decay[:, 0].min() > 1 - 1e-9 and decay[:, 1].max() < 1e-9


def test_delta_rule_with_16_bit_low_rank_weights():
    """The second halves of the low-rank projections as a 16-bit run holds them, in the scan and in the decode kernel."""
    ops = _ops()
    H, G, D, V, taps, T, ranks, eps = 4, 2, 32, 24, 4, 40, (16, 9), 1e-5
    w = _delta_weights(H, G, D, V, taps, 24, ranks, 3)
    w["a2"], w["g2"] = (w[n].to(torch.bfloat16).double() for n in ("a2", "g2"))
    u = torch.randn(T, 24, generator=torch.Generator().manual_seed(2), dtype=F64)
    ref, _ = pp.channel_delta(u, w, "", {"heads": H, "kv_heads": G, "dim": D, "vdim": V}, eps)
    proj = _f32(torch.cat([u @ w[n].T for n in ("q", "k", "v", "b", "a1", "g1")], dim=1))
    C = 2 * G * D + H * V
    conv = _f32(torch.cat([w["q.conv"], w["k.conv"], w["v.conv"]]))
    low = [w[n].T.to(torch.bfloat16).to(DEV).contiguous() for n in ("a2", "g2")]
    state = torch.zeros((2, (H * V * ops.delta_padded(D) + taps * C + 3) // 4 * 4), dtype=torch.float32, device=DEV)
    out = torch.zeros((T, H * V), dtype=torch.float32, device=DEV)
    for p0, n in [(0, 30)] + [(p, 1) for p in range(30, T)]:
        ops.delta_rule(proj[p0:p0 + n].contiguous(), (0, C, C + H, C + H + ranks[0]), ranks, conv, *low, _f32(w["dt_bias"]), _f32(w["A_log"]),
                       _f32(w["norm"]), eps, 1.0, out[p0:p0 + n], 0, state, _batch([(1, p0, n)]), H, G, D, V, single=n == 1)
    assert (out.double().cpu() - ref).abs().max() < 3e-5 * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("E,top,W,shared", [(5, 2, 40, True), (3, 3, 30, False), (8, 1, 64, True), (40, 6, 48, True), (2, 2, 36, False)])
def test_router_bias_softmax_over_the_chosen_and_the_shared_gate(E, top, W, shared):
    """The router against the plain rule: logits with a bias that changes choices, the largest are chosen, their weights are
    the softmax over the chosen logits only; the shared expert's gate comes out of the same kernel."""
    ops = _ops()
    T = 53
    g = torch.Generator().manual_seed(E * 10 + top)
    x = torch.randn(T, W, generator=g, dtype=F64)
    w = {"router": torch.randn(E, W, generator=g, dtype=F64) * W ** -0.5 * 2, "router.b": torch.randn(E, generator=g, dtype=F64),
         "shared.sg": torch.randn(1, W, generator=g, dtype=F64) * W ** -0.5 * 2}
    pick, weight = pp.route(x, w, "", top)
    plain_pick, _ = pp.route(x, dict(w, **{"router.b": w["router.b"] * 0}), "", top)
    assert (pick.sort(1).values != plain_pick.sort(1).values).any() or top == E          # the bias matters
    got = ops.moe_route(_f32(x), _f32(w["router"]), top, None, 1.0, lists=True, score="softmax", bias=_f32(w["router.b"]),
                        shared_gate=_f32(w["shared.sg"].reshape(-1)) if shared else None)
    dense, ids, wts = got[:3]
    want = torch.zeros(T, E, dtype=F64).scatter_(1, pick, weight)
    assert (dense.double().cpu() - want).abs().max() < 1e-6
    for t in range(T):
        mine = {int(e): float(a) for e, a in zip(ids[t].tolist(), wts[t].tolist())}
        assert set(mine) == set(pick[t].tolist()) and all(abs(mine[e] - float(want[t, e])) < 1e-6 for e in mine)
    if shared:
        assert (got[3].double().cpu() - torch.sigmoid(x @ w["shared.sg"].T)[:, 0]).abs().max() < 1e-6


@pytest.mark.parametrize("dtype,T", [("float32", 3), ("float32", 50), ("bfloat16", 2), ("bfloat16", 20), ("bfloat16", 70)])
@pytest.mark.parametrize("shared", [24, None])
def test_routed_feed_forward_every_way_it_runs(dtype, T, shared):
    """The routed feed-forward part (few tokens: only the chosen experts are read; prompt portions in 16 bits: tokens
    sorted by expert; else all experts, the shared one among them, in one product), with a gated shared expert of another
    size and clamp and without, against the plain function; activations large enough that every clamp bites."""
    from litellmengine_b200.config.specs import FeedForwardSpec
    from litellmengine_b200.parts.feed_forward import RoutedExperts
    W, E, top, ff, limit, limit_s = 48, 12, 3, 16, 0.9, 1.6
    g = torch.Generator().manual_seed(T)
    bf = lambda t: t.to(torch.bfloat16).double()
    x = bf(torch.randn(T, W, generator=g, dtype=F64) * 2)
    w = {"router": bf(torch.randn(E, W, generator=g, dtype=F64) * W ** -0.5 * 3), "router.b": bf(torch.randn(E, generator=g, dtype=F64)),
         "shared.sg": bf(torch.randn(1, W, generator=g, dtype=F64) * W ** -0.5 * 3)}
    for name, n in [(f"e{e}.", ff) for e in range(E)] + [("shared.", 24)]:
        w[name + "gate"], w[name + "up"] = (bf(torch.randn(n, W, generator=g, dtype=F64) * W ** -0.5) for _ in range(2))
        w[name + "down"] = bf(torch.randn(W, n, generator=g, dtype=F64) * n ** -0.5)
    mlp = {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}
    params = [("experts", E), ("top", top), ("groups", None), ("score", "softmax"), ("router_bias", True), ("activation", "clamped_swish"),
              ("limit", limit)]
    if shared:
        mlp["shared"] = {"ff": shared, "limit": limit_s}
        params += [("shared", shared), ("shared_activation", "clamped_swish"), ("shared_limit", limit_s), ("shared_gate", True)]
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    act = pp.bf16_round if dtype == "bfloat16" else pp.identity
    ref = pp.routed_ff(x, w, "", mlp, act=act)
    part = RoutedExperts(FeedForwardSpec(kind="moe", intermediate_size=ff, params=tuple(params)), W, tdt, DEV)
    part.load({k: (v.float() if k in ("router", "router.b", "shared.sg") else v.to(tdt)).to(DEV) for k, v in w.items()
               if k in part.parameters()})
    got = _ops().as_tensor(part.forward(x.to(tdt).to(DEV)))
    tol = (3e-5 if dtype == "float32" else 0.05) * max(1.0, float(ref.abs().max()))
    assert (got.double().cpu() - ref).abs().max() < tol
    if shared:                                                    # its own clamp, its gate: another result without
        assert (pp.routed_ff(x, w, "", dict(mlp, shared={"limit": limit}), act=act) - ref).abs().max() > 2 * tol
        assert (pp.routed_ff(x, dict(w, **{"shared.sg": w["shared.sg"] * 0}), "", mlp, act=act) - ref).abs().max() > 2 * tol
