"""The Purivik design in the engine against the plain implementation of `plain_purivik.py`: every mechanism's kernel alone
(with inputs made so that a lost key, a wrong edge or a lost summand shows), then whole models in every way of cutting a
request into steps, mixed batches with pages and slots used again, long decoding under CUDA graphs, and greedy generation
through the engine's own entry point and scheduler."""
import types

import numpy as np
import pytest
import torch

import plain_purivik as pp
import purivik_models as pm
import replay_helpers as rh

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

CASES = {"A": (pm.PUR_A, pm.PUR_A_PAGE, 3), "B": (pm.PUR_B, pm.PUR_B_PAGE, 5), "C": (pm.PUR_C, pm.PUR_C_PAGE, 9),
         "D": (pm.PUR_D, pm.PUR_D_PAGE, 11), "E": (pm.PUR_E, pm.PUR_E_PAGE, 13)}
# root mean square over the vocabulary of (difference minus its mean), as a fraction of the reference logits'
# spread; the float32 run is measured against the plain code in double precision
LIMIT = {"float32": 1e-4, "bfloat16": 0.06}


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
        held += limit <= 4 * LIMIT[dtype]
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


@pytest.mark.parametrize("case", ["C", "E"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_over_many_chunks(case, dtype):
    """600 and 300 tokens, heads of 64, 96 and 128 with equal and unequal value widths: chunks' edges inside pages, inside
    the kernels' tiles of query rows and between portions, in 140 decoded tokens, and pages of passed chunks that go back
    to the pool on the way."""
    cfg, page, w = model_of(case)
    reqs = requests(cfg, [600, 300], seed=4)
    ref = Reference(cfg, w, reqs, dtype)
    for name, steps in (("whole", rh.trace_whole(reqs)), ("decode", rh.trace_tail_decode(reqs, tail=140)),
                        ("portions", rh.trace_portions(reqs, seed=5, sizes=(2, 61, 64, 65, 128, 257, 300)))):
        runner = rh.make_runner(cfg, w, dtype, page, rh.peak_tokens(steps, round_to=page), max_requests=2)
        assert_close(rh.run_trace(runner, steps), ref, dtype, f"{case} {name}")
        runner.check_status()


@pytest.mark.parametrize("case,dtype", [("A", "float32"), ("A", "bfloat16"), ("E", "bfloat16")])
def test_long_decoding_under_graphs(case, dtype):
    """Two prompt tokens, then 200 single-token steps of two requests side by side: steps of one shape are replayed as a
    captured graph, and the chunks of several sizes come and go, in every pass of the loop."""
    cfg, page, w = model_of(case)
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


def _status():
    return torch.zeros(2, dtype=torch.int32, device=DEV)


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
                                 entry_q_len=_i32(lens), num_tokens=len(pos), num_entries=len(portions))


def _table(N, page, seed):
    """Pages of one request of N tokens in slot 1 of 3, scattered over a pool: (pool size, table on the device, order)."""
    n = -(-N // page)
    order = np.random.RandomState(seed).permutation(n + 5)[:n]
    table = torch.full((3, n + 2), -1, dtype=torch.int32)
    table[1, :n] = torch.as_tensor(order, dtype=torch.int32)
    return n + 5, table.to(DEV), order


@pytest.mark.parametrize("H", [40, 30, 1024, 4104, 8200])
def test_norms_around_the_residual_add_with_what_joins_there(H):
    """v = h + rms(y) w_post (+ join), written back; rms(v) w_pre returned: y as a matrix in either dtype and as the k-splits
    of a product, absent, or joined without a norm; picked rows; different eps on the two sides; rows that stay in
    registers, rows too long for that and rows without sixteen-byte accesses."""
    ops = _ops()
    T, e1, e2 = 9, 1e-3, 1e-5
    g = torch.Generator().manual_seed(H)
    h0, join = (torch.randn(T, H, generator=g, dtype=F64) for _ in range(2))
    y = torch.randn(3, T, H, generator=g, dtype=F64) * 0.05            # so small that its eps matters
    w1, w2 = (1 + 0.3 * torch.randn(H, generator=g, dtype=F64) for _ in range(2))
    post, pre = (_f32(w1), e1), (_f32(w2), e2)
    plain_v = lambda y, j: h0 + pp.rms_norm(y, w1, e1) + (join if j else 0)
    for form, j in (("matrix", False), ("splits", True), ("bf16 out", True), ("bf16 y", False)):
        h, ys = _f32(h0), y.sum(0)
        a = ops.PartialSum(_f32(y)) if form == "splits" else _f32(ys)
        if form == "bf16 y":
            a = a.to(torch.bfloat16)
            ys = a.double().cpu()
        out = ops.rmsnorm_sandwich(h, a, post, pre, torch.bfloat16 if form == "bf16 out" else torch.float32, join=_f32(join) if j else None)
        want = plain_v(ys, j)
        assert (h.double().cpu() - want).abs().max() < 1e-5, form
        assert (out.double().cpu() - pp.rms_norm(want, w2, e2)).abs().max() < (4e-2 if form == "bf16 out" else 2e-5), form
    # no norm on the way; nothing but what joins; nothing at all (the stream stays)
    h = _f32(h0)
    out = ops.rmsnorm_sandwich(h, _f32(y[0]), None, pre, torch.float32)
    assert (h.double().cpu() - (h0 + y[0])).abs().max() < 1e-5
    h = _f32(h0)
    out = ops.rmsnorm_sandwich(h, None, None, pre, torch.float32, join=_f32(join))
    assert (h.double().cpu() - (h0 + join)).abs().max() < 1e-5
    assert (out.double().cpu() - pp.rms_norm(h0 + join, w2, e2)).abs().max() < 2e-5
    h = _f32(h0)
    out = ops.rmsnorm_sandwich(h, None, None, pre, torch.float32)
    assert torch.equal(h.cpu(), h0.float()) and (out.double().cpu() - pp.rms_norm(h0, w2, e2)).abs().max() < 2e-5
    # picked rows leave the stream alone
    rows = [7, 0, 7, 8]
    out = ops.rmsnorm_sandwich(h, ops.PartialSum(_f32(y)), post, pre, torch.float32, rows=_i32(rows), join=_f32(join))
    assert torch.equal(h.cpu(), h0.float())
    assert (out.double().cpu() - pp.rms_norm(plain_v(y.sum(0), True), w2, e2)[rows]).abs().max() < 2e-5


@pytest.mark.parametrize("H,dtype", [(40, "bfloat16"), (30, "float32"), (2048, "bfloat16")])
def test_scaled_embedding_written_twice(H, dtype):
    ops = _ops()
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    table = torch.randn(50, H, generator=torch.Generator().manual_seed(H), dtype=F64).to(tdt)
    ids, status = [3, 0, 49, 3, 17, -2], _status()                # the last one is the token in place 1 of the feedback buffer
    keep = torch.full((6, H), 9.0, device=DEV)
    out = ops.embedding(_i32(ids), table.to(DEV), status, feedback=_i32([1, 44]), scale=2.7, keep=keep)
    ref = pp.embed(ids[:-1] + [44], {"embed": table.double()}, 2.7)
    assert status.tolist() == [0, 0] and torch.equal(out, keep)
    assert (out.double().cpu() - ref).abs().max() < 1e-5
    ops.embedding(_i32([1, 50]), table.to(DEV), status, scale=2.7, keep=keep[:2])       # an id past the table: a zero row, and a record of it
    assert status.tolist() == [1, 1] and float(keep[1].abs().max()) == 0.0


def test_start_of_a_pass_adds_the_embedding():
    """In front of every pass but the first x0 joins, with an output still pending on the stream: in the kernel of an RMS
    norm, and beside norms that do not take it."""
    from litellmengine_b200.config.specs import NormSpec, RejoinSpec
    from litellmengine_b200.parts.norms import PendingNormed, RMSNorm, TanhNorm
    from litellmengine_b200.parts.rejoin import AddedEmbedding
    W, T, eps = 48, 9, 1e-5
    g = torch.Generator().manual_seed(1)
    part = AddedEmbedding(RejoinSpec(passes=3, kind="add"), W, torch.float32)
    norm, post = (RMSNorm(NormSpec("rmsnorm", eps, ""), W) for _ in range(2))
    ws = [1 + 0.2 * torch.randn(W, generator=g, dtype=F64) for _ in range(2)]
    for n, w in zip((norm, post), ws):
        n.load({"": _f32(w)})
    x, x0, y = (torch.randn(T, W, generator=g, dtype=F64) for _ in range(3))
    for t in (0, 1, 2):
        h = _f32(x)
        u = norm.forward(h, torch.float32, delta=part.start(h, PendingNormed(_f32(y), post), _f32(x0), t, norm), write_sum=True)
        want = x + pp.rms_norm(y, ws[1], eps) + (x0 if t else 0)
        assert (h.double().cpu() - want).abs().max() < 1e-5
        assert (u.double().cpu() - pp.rms_norm(want, ws[0], eps)).abs().max() < 2e-5
    tanh = TanhNorm(NormSpec("tanh", eps, ""), W)
    h, pending = _f32(x), PendingNormed(_f32(y), None)
    assert part.start(h, pending, _f32(x0), 1, tanh) is pending and (h.double().cpu() - (x + x0)).abs().max() < 1e-5


def _chunk_probes(N, chunk):
    """(query, key) pairs: the chunk's first key and the last of the chunk before, seen from the chunk's last query, its
    first and one in the middle; the query itself; the sequence's first key."""
    out = []
    for c0 in range(chunk, N - chunk, max(chunk, 40)):
        c0 = c0 // chunk * chunk
        for i in (c0 + chunk - 1, c0, c0 + chunk // 2):
            out += [(i, c0), (i, c0 - 1)]
    return out + [(N - 1, N - 1), (N - 1, 0), (N - 1, (N - 1) // chunk * chunk)]


@pytest.mark.parametrize("chunk,dims,H,G,D,V", [(1, 12, 6, 2, 12, 20), (7, 4, 3, 3, 5, 3), (16, 0, 6, 2, 12, 20), (50, 12, 4, 1, 16, 8),
                                                (64, 16, 2, 2, 32, 48), (65, 6, 4, 2, 16, 16), (None, 8, 6, 3, 8, 24)])
def test_attention_rotation_and_chunks(chunk, dims, H, G, D, V):
    """The kernels between the projections of an attention layer, on projections given as numbers: the rotation with
    stretched frequencies, the page write, attention within chunks.  Keys that a query would follow by far are placed at
    the chunk's first position and just before it, so that an edge off by one is another result.  One step, portions and
    single tokens, against the plain functions."""
    ops = _ops()
    from litellmengine_b200.config.specs import PositionSpec
    from litellmengine_b200.parts.registry import lookup
    import litellmengine_b200.parts.position  # noqa: F401  (registers the kinds)
    T, page, scale = 150, 16, 0.3
    g = torch.Generator().manual_seed(5)
    proj = torch.randn(T, H * D + G * D + G * V, generator=g, dtype=F64)
    scaling = (3.0, 1.0, 5.0, 60)
    rot = {"base": 300.0, "dims": dims, "scaling": dict(zip(("factor", "low", "high", "original"), scaling))} if dims and dims <= D else None
    mask = {"size": chunk} if chunk else None
    ko, vo = H * D, H * D + G * D

    def plain(p, mask, rot=rot):
        pos = list(range(T))
        q, k = pp.rotate_half(p[:, :ko].view(T, H, D), pos, rot), pp.rotate_half(p[:, ko:vo].view(T, G, D), pos, rot)
        s = (q.permute(1, 0, 2) @ k.permute(1, 0, 2).repeat_interleave(H // G, 0).transpose(1, 2)) * scale
        vh = p[:, vo:].view(T, G, V).permute(1, 0, 2).repeat_interleave(H // G, 0)
        s = s.masked_fill(~pp.visible_keys(T, mask)[None], float("-inf"))
        return (torch.softmax(s, -1) @ vh).permute(1, 0, 2).reshape(T, H * V)

    for i, j in _chunk_probes(T, chunk or 60):
        x = proj[i, :D]                    # a key at j that a query x at i meets as x itself: x turned by the angle of i - j
        proj[j, ko:ko + D] = (pp.rotate_half(x[None, None], [i - j], rot)[0, 0] if rot else x) * 6.0
    ref = plain(proj, mask)
    rotation = None
    if rot:
        rotation = lookup("position", "rope_half")(PositionSpec("rope_half", 300.0, dims, (("wavelengths", scaling),)), D, DEV).kernel_args()
    for dtype, tol in ((torch.float32, 5e-5), (torch.bfloat16, 0.12)):
        for portions in ([(1, 0, T)], [(1, 0, 70), (1, 70, 2), (1, 72, 77), (1, 149, 1)]):
            pool, table, order = _table(T, page, 2)
            keys = torch.zeros(pool, G, page, D, dtype=dtype, device=DEV)
            values = torch.zeros(pool, G, page, V, dtype=dtype, device=DEV)
            out, status = torch.zeros(T, H * V, dtype=dtype, device=DEV), _status()
            for slot, p0, n in portions:                        # step by step, as a request would run
                b = _batch([(slot, p0, n)])
                q = ops.attention_prepare(_f32(proj[p0:p0 + n]), 0, ko, vo, None, None, None, None, 0.0, None, keys, values, b.positions,
                                          b.token_entry, b.entry_slot, table, H, G, D, V, page, status, dtype, rotation=rotation)
                o = torch.zeros(n, H * V, dtype=dtype, device=DEV)
                ops.paged_attention_generic_kv(q, keys, values, b.positions, b.token_entry, b.entry_slot, table, H, G, D, V,
                                               page, -chunk if chunk else None, scale, status, o)
                out[p0:p0 + n] = o
            assert status.tolist() == [0, 0]
            assert (out.double().cpu() - ref).abs().max() < tol, (dtype, len(portions))
    if chunk:                       # the edges matter, and so does the scaling
        for other in ({"size": chunk + 1}, None) + (({"size": chunk - 1},) if chunk > 1 else ()):
            assert (ref - plain(proj, other)).abs().max() > 0.1
    if rot and dims > 2 and chunk != 1:
        assert (ref - plain(proj, mask, {k: v for k, v in rot.items() if k != "scaling"})).abs().max() > 0.05


@pytest.mark.parametrize("d,group,chunk", [(64, 3, 100), (64, 4, 30), (128, 1, 64), (128, 2, 140), (128, 8, 300), (128, 3, 128), (128, 4, 1)])
def test_tensor_core_attention_within_chunks(d, group, chunk):
    """The kernels that a 16-bit run takes at head sizes 64 and 128: a prompt portion that starts in the middle of a page
    and of a chunk with keys before it (the tcgen05 kernel at 128, the mma kernel at both), and single tokens in the
    split-key decode kernel with one and several splits.  Keys that would win by far sit at chunks' first positions and
    just before them."""
    ops = _ops()
    N, past, page, G, scale = 420, 37, 16, 2, 0.2
    H, T = G * group, N - past
    g = torch.Generator().manual_seed(d + group)
    q, k, v = (torch.randn(N, n, d, generator=g, dtype=F64) for n in (H, G, G))
    for i, j in _chunk_probes(N, chunk):
        k[j] = q[i, ::group] * (40.0 / d)          # a score of about eight
    q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
    kh, vh = (t.permute(1, 0, 2).repeat_interleave(group, 0) for t in (k, v))
    scores = (q[past:].permute(1, 0, 2) @ kh.transpose(1, 2)) * scale

    def plain(size):
        vis = pp.visible_keys(N, {"size": size})[past:]
        return (torch.softmax(scores.masked_fill(~vis[None], float("-inf")), -1) @ vh).permute(1, 0, 2)
    ref = plain(chunk)
    pool, table, order = _table(N, page, 2)
    cache = torch.zeros(pool, 2, G, page, d, dtype=torch.bfloat16, device=DEV)
    for j in range(N):
        cache[order[j // page], 0, :, j % page] = k[j].to(torch.bfloat16).to(DEV)
        cache[order[j // page], 1, :, j % page] = v[j].to(torch.bfloat16).to(DEV)
    qd = q[past:].reshape(T, -1).to(torch.bfloat16).to(DEV)
    status = _status()
    tiles = _i32([(0, r0) for r0 in range(0, T, ops.PREFILL_TILE_ROWS)])
    kernels = [ops.paged_attention_prefill] + ([ops.paged_attention_prefill_tcgen05] if ops.prefill_tcgen05_supported(d, page) else [])
    assert len(kernels) == (2 if d == 128 else 1)
    for kernel in kernels:
        out = torch.zeros(T, H * d, dtype=torch.bfloat16, device=DEV)
        kernel(qd, out, cache, tiles, tiles.shape[0], _i32([1]), _i32([0]), _i32([T]), _i32([N]), table, H, G, d, page, -chunk, scale, status)
        assert status.tolist() == [0, 0]
        assert (out.double().cpu().view(T, H, d) - ref).abs().max() < 0.06, kernel.__name__
    assert ops.fast_attention_supported(d, group)
    for splits in (1, 3):
        a = torch.zeros(T, H * d, dtype=torch.bfloat16, device=DEV)
        picked = sorted({i - past for i, _ in _chunk_probes(N, chunk) if i >= past} | {5, 263})[:60]
        ops.paged_attention_decode(qd, a, cache, _i32(picked + [-1]), len(picked) + 1, _i32(list(range(past, N))), _i32([0] * T),
                                   _i32([1]), table, H, G, d, page, -chunk, scale, splits, status)
        assert status.tolist() == [0, 0]
        assert (a.double().cpu().view(T, H, d)[picked] - ref[picked]).abs().max() < 0.06, splits
    for other in (chunk + 1,) + ((chunk - 1,) if chunk > 1 else ()):
        assert (plain(other) - ref).abs().max() > 0.3


@pytest.mark.parametrize("H,G,D,V,span,page", [(6, 3, 64, 88, -110, 16), (6, 2, 32, 48, -30, 16), (16, 1, 128, 256, -300, 64), (3, 3, 256, 128, 100, 16),
                                               (8, 2, 8, 8, None, 4), (2, 1, 72, 24, -1, 8), (4, 2, 256, 256, -64, 16), (5, 5, 96, 96, 65, 5),
                                               (4, 2, 40, 192, -128, 16)])
def test_tensor_core_attention_of_any_widths(H, G, D, V, span, page):
    """The 16-bit kernels for keys and values of their own widths, within chunks, windows and over everything: a prompt
    portion that starts in the middle of a page and of a chunk with keys before it, a second request's portion beside it,
    single tokens with one and several splits, the result scaled and in a column of a wider buffer; separate tensors of keys
    and values and the halves of one.  Keys that would win by far sit at the edges."""
    ops = _ops()
    N, past, scale = 330, 37, 0.25
    group, T = H // G, N - past
    g = torch.Generator().manual_seed(D + V)
    q, k, v = (torch.randn(N, n, w, generator=g, dtype=F64) for n, w in ((H, D), (G, D), (G, V)))
    size = abs(span or 60)
    for i, j in _chunk_probes(N, size) + [(N - 1, max(0, N - size)), (N - 2, max(0, N - 2 - size)), (200, max(0, 201 - size))]:
        k[j] = q[i, ::group] * (32.0 / D)          # a score of about eight
    q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
    kh, vh = (t.permute(1, 0, 2).repeat_interleave(group, 0) for t in (k, v))
    scores = (q[past:].permute(1, 0, 2) @ kh.transpose(1, 2)) * scale

    def plain(span):
        vis = pp.visible_keys(N, {"size": -span} if span and span < 0 else None)
        if span and span > 0:
            vis = vis & (torch.arange(N)[:, None] - torch.arange(N)[None, :] < span)
        return (torch.softmax(scores.masked_fill(~vis[past:][None], float("-inf")), -1) @ vh).permute(1, 0, 2)
    ref = plain(span)
    pool, table, order = _table(N, page, 2)
    if D == V:
        kv = torch.zeros(pool, 2, G, page, D, dtype=torch.bfloat16, device=DEV)
        keys, values = kv[:, 0], kv[:, 1]
    else:
        keys, values = (torch.zeros(pool, G, page, w, dtype=torch.bfloat16, device=DEV) for w in (D, V))
    at, inside = torch.as_tensor(order, device=DEV)[torch.arange(N, device=DEV) // page].long(), torch.arange(N, device=DEV) % page
    keys[at, :, inside] = k.to(torch.bfloat16).to(DEV)
    values[at, :, inside] = v.to(torch.bfloat16).to(DEV)
    qd = q[past:].reshape(T, -1).to(torch.bfloat16).to(DEV)
    status, off, by = _status(), 8, 0.5
    R = ops.PREFILL_TILE_ROWS
    # one entry over everything, and the same rows as two entries of which the second has the first's keys behind it
    for cuts in ([T], [70, T - 70]):
        starts = [sum(cuts[:e]) for e in range(len(cuts))]
        tiles = [(e, r0) for e, n in enumerate(cuts) for r0 in range(0, n, R)] + [(-1, -1)]
        out = torch.full((T, H * V + 16), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.wide_attention_prefill(qd, out, off, keys, values, _i32(tiles), len(tiles), _i32([1] * len(cuts)), _i32(starts), _i32(cuts),
                                   _i32([past + s + n for s, n in zip(starts, cuts)]), table, H, G, D, V, page, span, scale, status, out_scale=by)
        assert status.tolist() == [0, 0] and float((out[:, :off] - 7).abs().max()) == 0 and float((out[:, off + H * V:] - 7).abs().max()) == 0
        assert (out[:, off:off + H * V].double().cpu().view(T, H, V) - ref * by).abs().max() < 0.04, cuts
    for splits in (1, 4):
        a = torch.full((T, H * V), 7.0, dtype=torch.bfloat16, device=DEV)
        picked = sorted({i - past for i, _ in _chunk_probes(N, size) if i >= past} | {T - 1, T - 2, 5, 200 - past})[:60]
        ops.wide_attention_decode(qd, a, 0, keys, values, _i32(picked + [-1]), len(picked) + 1, _i32(list(range(past, N))), _i32([0] * T),
                                  _i32([1]), table, H, G, D, V, page, span, scale, splits, status)
        assert status.tolist() == [0, 0]
        assert (a.double().cpu().view(T, H, V)[picked] - ref[picked]).abs().max() < 0.06, splits
        assert float((a[[i for i in range(T) if i not in picked]] - 7).abs().max()) == 0
    if span:
        assert (plain(span + (1 if span > 0 else -1)) - ref).abs().max() > 0.2
    assert not ops.wide_attention_supported(D + 4, V, group) and not ops.wide_attention_supported(264, V, group)


@pytest.mark.parametrize("dtype,T,ff", [("float32", 3, 44), ("float32", 70, 40), ("bfloat16", 2, 40), ("bfloat16", 50, 36), ("bfloat16", 300, 4096)])
def test_clamped_dense_feed_forward_every_way_it_runs(dtype, T, ff):
    """The clamped feed-forward part: few tokens (the streaming product's k-splits), a plain product, and the paired
    tcgen05 product with the activation in its epilogue; activations large enough that every clamp bites."""
    from litellmengine_b200.config.specs import FeedForwardSpec
    from litellmengine_b200.parts.feed_forward import SwiGLU
    ops, W, limit = _ops(), 64, 0.8
    g = torch.Generator().manual_seed(T)
    bf = lambda t: t.to(torch.bfloat16).double()
    x = bf(torch.randn(T, W, generator=g, dtype=F64) * 2)
    w = {"gate": bf(torch.randn(ff, W, generator=g, dtype=F64) * W ** -0.5), "up": bf(torch.randn(ff, W, generator=g, dtype=F64) * W ** -0.5),
         "down": bf(torch.randn(W, ff, generator=g, dtype=F64) * ff ** -0.5)}
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    act = pp.bf16_round if dtype == "bfloat16" else pp.identity
    ref = pp.dense_ff(x, w, "", limit, act)
    spec = FeedForwardSpec(kind="swiglu", intermediate_size=ff, params=(("activation", "clamped_swish"), ("limit", limit)),
                           tensor_names=tuple((n, n) for n in ("gate", "up", "down")))
    part = SwiGLU(spec, W, tdt, DEV)
    part.load({k: v.to(tdt).to(DEV) for k, v in w.items()})
    got = ops.as_tensor(part.forward(x.to(tdt).to(DEV)))
    tol = (3e-5 if dtype == "float32" else 0.03) * max(1.0, float(ref.abs().max()))
    assert (got.double().cpu() - ref).abs().max() < tol
    assert (pp.dense_ff(x, w, "", 2 * limit, act) - ref).abs().max() > 4 * tol
    if dtype == "bfloat16" and T >= ops.PAIR_MIN_ROWS:
        xd, wd = x.to(tdt).to(DEV), torch.cat([w["gate"], w["up"]]).to(tdt).to(DEV)
        paired = ops.linear_pair_silu_mul(xd, wd, activation="clamped_swish", limit=limit)
        plain = ops.silu_and_mul(ops.linear(xd, wd), activation="clamped_swish", limit=limit)
        assert (paired.double() - plain.double()).abs().max() < 0.03
    with pytest.raises(ValueError):
        SwiGLU(FeedForwardSpec(kind="swiglu", intermediate_size=8, params=(("activation", "clamped_swish"), ("limit", 0.0))), W, tdt, DEV)


@pytest.mark.parametrize("E,top,W", [(5, 2, 40), (3, 3, 30), (8, 1, 64), (40, 6, 48), (1, 1, 36)])
def test_router_scores_are_the_weights(E, top, W):
    """The largest sigmoid scores are chosen and are the weights as they are; with `normalize` they would be shares of one."""
    ops, T = _ops(), 53
    g = torch.Generator().manual_seed(E * 10 + top)
    x = torch.randn(T, W, generator=g, dtype=F64)
    w = {"router": torch.randn(E, W, generator=g, dtype=F64) * W ** -0.5 * 2}
    pick, weight = pp.route(x, w, "", top)
    dense, ids, wts = ops.moe_route(_f32(x), _f32(w["router"]), top, None, 1.0, lists=True, normalize=False)
    want = torch.zeros(T, E, dtype=F64).scatter_(1, pick, weight)
    assert (dense.double().cpu() - want).abs().max() < 1e-6
    for t in range(T):
        mine = {int(e): float(a) for e, a in zip(ids[t].tolist(), wts[t].tolist())}
        assert set(mine) == set(pick[t].tolist()) and all(abs(mine[e] - float(want[t, e])) < 1e-6 for e in mine)
    # scores that crowd together just below one: the choice is still the largest
    hot = {"router": w["router"] * 0 + 1.0 / W}
    hot["router"] = hot["router"] * (17.0 + torch.arange(E, dtype=F64)[:, None] / 64)
    ones = torch.ones(T, W, dtype=F64)
    _, ids, _ = ops.moe_route(_f32(ones), _f32(hot["router"]), top, None, 1.0, lists=True, normalize=False)
    assert ids.tolist() == [list(range(E - 1, E - 1 - top, -1))] * T
    shares = ops.moe_route(_f32(x), _f32(w["router"]), top, None, 1.0)
    assert (shares.double().cpu() - want / want.sum(1, keepdim=True)).abs().max() < 1e-6
    assert (shares.double().cpu() - want).abs().max() > 0.05


@pytest.mark.parametrize("dtype,T", [("float32", 3), ("float32", 50), ("bfloat16", 2), ("bfloat16", 20), ("bfloat16", 70)])
@pytest.mark.parametrize("top", [1, 3])
def test_routed_feed_forward_every_way_it_runs(dtype, T, top):
    """The routed feed-forward part with the weight on the experts' input (few tokens: only the chosen experts are read;
    prompt portions in 16 bits: tokens sorted by expert; else all experts in one product), against the plain function."""
    from litellmengine_b200.config.specs import FeedForwardSpec
    from litellmengine_b200.parts.feed_forward import RoutedExperts
    W, E, ff = 48, 12, 16
    g = torch.Generator().manual_seed(T)
    bf = lambda t: t.to(torch.bfloat16).double()
    x = bf(torch.randn(T, W, generator=g, dtype=F64))
    w = {"router": bf(torch.randn(E, W, generator=g, dtype=F64) * W ** -0.5 * 0.6)}        # scores well below one
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = (bf(torch.randn(ff, W, generator=g, dtype=F64) * W ** -0.5) for _ in range(2))
        w[f"e{e}.down"] = bf(torch.randn(W, ff, generator=g, dtype=F64) * ff ** -0.5)
    tdt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    act = pp.bf16_round if dtype == "bfloat16" else pp.identity
    ref = pp.routed_ff(x, w, "", {"router": {"top": top}}, act=act)
    params = (("experts", E), ("top", top), ("groups", None), ("score", "sigmoid"), ("normalize", False), ("weight_on_input", True),
              ("activation", "silu"))
    part = RoutedExperts(FeedForwardSpec(kind="moe", intermediate_size=ff, params=params), W, tdt, DEV)
    part.load({k: (v.float() if k == "router" else v.to(tdt)).to(DEV) for k, v in w.items()})
    got = _ops().as_tensor(part.forward(x.to(tdt).to(DEV)))
    tol = (3e-5 if dtype == "float32" else 0.03) * max(1.0, float(ref.abs().max()))
    assert (got.double().cpu() - ref).abs().max() < tol
    pick, weight = pp.route(x, w, "", top)                        # the weight on the output would be another result
    other = torch.stack([sum(float(a) * pp.expert(x[t:t + 1], w, f"e{int(e)}.")[0] for e, a in zip(pick[t], weight[t])) for t in range(T)])
    assert (other - ref).abs().max() > 2 * tol
