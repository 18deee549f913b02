"""Sovanex on a GPU: each mechanism's kernel alone against the functions of tests/sovanex_oracle.py, then whole models in fp32
and bf16 over portions, mixed batches, captured decode steps and the scheduler."""
import math
from types import SimpleNamespace

import pytest
import torch

import sovanex_cases as S
import sovanex_oracle as O
from fllm_b200.runtime.request import SamplingParams

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {True: 2e-5, False: 6e-2}                     # fp32, bf16


@pytest.fixture(scope="module")
def ops():
    from fllm_b200.ops.native import NativeOps
    return NativeOps(torch.device(DEV))


def gen(seed):
    return torch.Generator(device=DEV).manual_seed(seed)


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-12))


# ------------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,width,ld", [(1, 64, 64), (2, 75, 80), (3, 13, 16), (4, 2048, 2048), (4, 4100, 4104), (8, 96, 96)])
def test_stream_update_read_and_norm(ops, streams, width, ld, dtype):
    g, T = gen(streams), 9
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width))
    table = pad(torch.randn(50, width, device=DEV, generator=g)).to(dtype)
    w, b = (pad(torch.randn(width, device=DEV, generator=g)).to(dtype) for _ in range(2))
    ids = torch.randint(0, 50, (T,), device=DEV, generator=g).int()
    inp, out, nxt = (torch.randn(streams, device=DEV, generator=g) for _ in range(3))
    mix = torch.randn(streams, streams, device=DEV, generator=g)
    y = pad(torch.randn(T, width, device=DEV, generator=g)).to(dtype)
    d = lambda t: t.double().cpu()
    norm = lambda u: O.layer_norm(u[:, :width], d(w)[:width], d(b)[:width], 1e-3)
    tol = 4e-6 if dtype == torch.float32 else 4e-3
    x, h = ops.streams_begin(ids, table, streams, inp, w, b, width, 1e-3)
    xs = [d(table)[ids.cpu().long()] for _ in range(streams)]
    assert rel(h[:, :width], norm(sum(d(inp)[s] * xs[s] for s in range(streams)))) < tol and not h[:, width:].any()
    for step in range(2):                                              # unequal streams from the second update on
        h = ops.streams_step(x, y, mix, out, nxt, w, b, width, 1e-3)
        xs = [sum(d(mix)[s, t] * xs[s] for s in range(streams)) + d(out)[t] * d(y) for t in range(streams)]
        assert rel(h[:, :width], norm(sum(d(nxt)[s] * xs[s] for s in range(streams)))) < tol
        assert max(rel(x[:, t], xs[t]) for t in range(streams)) < 1e-6       # the streams stay in fp32
    before = x.clone()
    rows = torch.tensor([7, 0, 7], dtype=torch.int32, device=DEV)
    h = ops.streams_step(x, y, mix, out, torch.ones(streams, device=DEV), w, b, width, 1e-3, rows=rows, write=False)
    new = sum(sum(d(mix)[s, t] * xs[s] for s in range(streams)) + d(out)[t] * d(y) for t in range(streams))
    assert rel(h[:, :width], norm(new)[rows.cpu().long()]) < tol and torch.equal(before, x)


def test_streams_take_split_k_partial_sums(ops):
    g, T, K, N = gen(1), 8, 4096, 512
    a, w = torch.randn(T, K, device=DEV, generator=g).bfloat16(), (torch.randn(N, K, device=DEV, generator=g) * K ** -0.5).bfloat16()
    x = torch.randn(T, 2, N, device=DEV, generator=g)
    one, mix = torch.ones(2, device=DEV), torch.eye(2, device=DEV)
    nw = torch.ones(N, device=DEV, dtype=torch.bfloat16)
    y = ops.linear(a, w, defer=True)
    assert not isinstance(y, torch.Tensor)
    want = x + (a.float() @ w.float().t())[:, None]
    ops.streams_step(x, y, mix, one, one, nw, None, N, 1e-5)
    assert rel(x, want) < 1e-5


# ------------------------------------------------------------------------------------------------ latent attention
def latent_batch(lens, ctxs, bs=16, seed=0):
    g = torch.Generator().manual_seed(seed)
    B, mb = len(lens), max(-(-c // bs) for c in ctxs)
    tab = torch.randperm(B * mb + 3, generator=g)[:B * mb].view(B, mb).int()
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    pos = torch.cat([torch.arange(c - n, c) for n, c in zip(lens, ctxs)]).int()
    seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).int()
    dev = lambda t: t.to(DEV)
    b = SimpleNamespace(num_seqs=B, max_q_len=max(lens), max_kv_len=max(ctxs), positions=dev(pos), row_seq=dev(seq), block_tables=dev(tab),
                        q_starts=dev(torch.tensor(starts, dtype=torch.int32)))
    return b, tab, B * mb + 3, pos, seq


def dense(q, cache, tab, pos, seq, scale, R, bs=16):
    """Softmax over the visible rows of every token, in fp64."""
    q, cache = q.double().cpu(), cache.double().cpu()
    out = torch.zeros(q.shape[0], q.shape[1], R, dtype=torch.float64)
    for t in range(q.shape[1]):
        n = int(pos[t]) + 1
        rows = torch.stack([cache[tab[seq[t], j // bs], j % bs] for j in range(n)])
        out[:, t] = torch.softmax(q[:, t] @ rows.T * scale, -1) @ rows[:, :R]
    return out


SHAPES = [(4, 37, 6), (1, 8, 2), (3, 96, 16), (16, 512, 64), (20, 512, 64), (5, 130, 30), (40, 256, 32), (2, 600, 8)]
BATCHES = [([1, 1, 1], [1, 40, 129]), ([5, 1, 23], [5, 17, 60]), ([70], [133]), ([1], [700])]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,R,dr", SHAPES)
@pytest.mark.parametrize("lens,ctxs", BATCHES)
def test_latent_attention(ops, H, R, dr, lens, ctxs, dtype):
    from fllm_b200.ops.latent import latent_width
    W, g = latent_width(R, dr), gen(H + R)
    b, tab, nb, pos, seq = latent_batch(lens, ctxs)
    cache = torch.randn(nb, 16, W, device=DEV, generator=g)
    cache[:, :, R + dr:] = 0
    q = torch.randn(H, len(pos), W, device=DEV, generator=g)
    q[:, :, R + dr:] = 0
    cache, q = cache.to(dtype), q.to(dtype)
    scale = 2.0 / math.sqrt(R + dr)
    want = dense(q, cache, tab, pos, seq, scale, R)
    tol = 2e-6 if dtype == torch.float32 else 4e-3
    assert rel(ops.attention_latent(q, cache, b, scale, R), want) < tol
    if dtype == torch.bfloat16:
        assert rel(ops.attention_latent(q, cache, b, scale, R, tensor_cores=False), want) < tol
        for splits in (2, 5):
            assert rel(ops.attention_latent(q, cache, b, scale, R, splits=splits), want) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("lens,ctx", [([1], 200), ([90], 200)])
def test_single_keys_at_every_border(ops, lens, ctx, dtype):
    """One key's score stands far out: the result is that key's latent wherever it lies (first tokens, page and tile borders,
    the query's own position), and the key right behind a query is never seen."""
    R, dr, H = 48, 16, 3
    b, tab, nb, pos, seq = latent_batch(lens, [ctx], seed=4)
    g = gen(3)
    base = torch.randn(nb, 16, 64, device=DEV, generator=g) * 0.1
    q = torch.randn(H, len(pos), 64, device=DEV, generator=g)
    for place in (0, 1, 15, 16, 31, 32, 63, 64, 65, 109, 110, 111, 127, 128, 191, 192, 198, 199):
        cache = base.clone()
        last = len(pos) - 1
        spot = int(tab[0, place // 16]), place % 16
        for t in sorted({0, last // 2, last}):
            cache[spot] = q[1, t] * 3                                   # query t, head 1 points at this key
            c, qq = cache.to(dtype), q.to(dtype)
            got = ops.attention_latent(qq, c, b, 1.0, R)[1, t].float()
            if place <= int(pos[t]):
                assert rel(got, c[spot][:R]) < 1e-2, (place, t)
            else:
                assert float(got @ qq[1, t, :R].float()) < 0.5 * float(c[spot][:R].float() @ qq[1, t, :R].float()), (place, t)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("style", [0, 1])
def test_latent_rows_and_rotation(ops, style, dtype):
    H, R, dr, head, T = 3, 37, 6, 26, 11
    g = gen(style)
    ckv = torch.randn(T, 48, device=DEV, generator=g).to(dtype)
    q = torch.randn(T, 80, device=DEV, generator=g).to(dtype)
    w = torch.randn(R, device=DEV, generator=g).to(dtype)
    pos = torch.tensor([0, 1, 2, 1000, 70000, 5, 6, 7, 8, 9, 0], dtype=torch.int32, device=DEV)
    slots = torch.tensor([3, 17, 4, 60, 33, 32, 31, 48, 0, 16, -1], dtype=torch.int32, device=DEV)
    inv = torch.tensor([50.0 ** (-2.0 * i / dr) for i in range(dr // 2)], device=DEV)
    cache = torch.full((4, 16, 48), 7.0, device=DEV, dtype=dtype)
    ql = torch.zeros(H, T, 48, device=DEV, dtype=dtype)
    ops.latent_prepare(ckv, q, head, 20, pos, slots, inv, 1.0, w, 1e-3, cache, ql, R, style)
    perm = list(range(dr)) if style == 0 else [0, 2, 4, 1, 3, 5]       # neighbours -> halves
    back = [perm.index(i) for i in range(dr)]
    rot = lambda x: O.rotate_half(x[..., perm], pos.cpu().float(), 50.0)[..., back]
    d = lambda t: t.float().cpu()
    want = torch.cat([O.rms_norm(d(ckv)[:, :R], d(w), 1e-3), rot(d(ckv)[:, R:R + dr])], -1)
    tol = 1e-5 if dtype == torch.float32 else 4e-3                     # (angles of 70000 radians in fp32)
    keep = slots[:-1].long().cpu()
    assert rel(cache.view(-1, 48)[keep, :R + dr], want[:-1]) < tol and not cache.view(-1, 48)[keep, R + dr:].any()
    untouched = [i for i in range(64) if i not in keep.tolist()]
    assert bool((cache.view(-1, 48)[untouched] == 7).all())
    for h in range(H):
        assert rel(ql[h, :, R:R + dr], rot(d(q)[:, h * head + 20:h * head + 26])) < tol
    before = cache.clone()
    ops.latent_prepare(None, q, head, 20, pos, slots, inv, 1.0, None, 1e-3, cache, ql, R, style)      # a layer that shares rows
    assert torch.equal(before, cache)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_head_gate_and_products(ops, dtype):
    g = gen(0)
    o = torch.randn(3, 7, 11, device=DEV, generator=g).to(dtype)
    gate = (torch.randn(7, 8, device=DEV, generator=g) * 3).to(dtype)
    y = ops.head_gate(o, gate[:, 2:5], 40)
    want = (o.float() * torch.sigmoid(gate[:, 2:5].float()).t()[:, :, None]).transpose(0, 1).reshape(7, 33)
    assert rel(y[:, :33], want) < (1e-6 if dtype == torch.float32 else 4e-3) and not y[:, 33:].any()
    if dtype == torch.float32:
        for T, N, K in ((1, 8, 8), (70, 203, 75), (129, 65, 300)):
            x, w, bias = (torch.randn(*s, device=DEV, generator=g) for s in ((T, K), (N, K), (N,)))
            assert rel(ops.linear(x, w, bias), x.double() @ w.double().t() + bias.double()) < 1e-6
        a, m = torch.randn(5, 9, 40, device=DEV, generator=g)[:, :, 3:33], torch.randn(5, 30, 21, device=DEV, generator=g)
        assert rel(ops.bmm(a, m), a.double() @ m.double()) < 1e-6


# ------------------------------------------------------------------------------------------------ gated delta rule
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Hk,d,dv", [(4, 2, 20, 13), (1, 1, 8, 8), (6, 3, 16, 40), (4, 1, 64, 24), (2, 2, 128, 128), (2, 1, 256, 20), (3, 3, 100, 300)])
def test_delta_scan(ops, H, Hk, d, dv, dtype):
    """Ragged steps that continue each other: prompts, portions of 2 .. 33 tokens and single tokens, rows of the pool in any order."""
    g = gen(d)
    lens, slots = [45, 70, 3], [2, 0, 4]
    K, V = Hk * d, H * dv
    Kp = (K + 7) // 8 * 8
    rows = [torch.randn(n, 2 * Kp + V + 2 * H, device=DEV, generator=g).to(dtype) for n in lens]
    A = -torch.exp(torch.randn(H, device=DEV, generator=g) * 0.5)
    bias = torch.randn(H, device=DEV, generator=g) - 2
    state = torch.full((6, H, dv, d), 9.0, device=DEV)                 # stale rows of earlier requests
    got = [[] for _ in lens]
    at = [0, 0, 0]
    for take in ([17, 2, 1], [0, 33, 1], [1, 1, 1], [1, 1, 0], [26, 33, 0]):
        part = [(i, n) for i, n in enumerate(take) if n]
        x = torch.cat([rows[i][at[i]:at[i] + n] for i, n in part])
        mk = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        qs = mk([sum(n for _, n in part[:j]) for j in range(len(part) + 1)])
        pos = mk([p for i, n in part for p in range(at[i], at[i] + n)])
        gates = x[:, 2 * Kp + V:]
        y = ops.matrix_state_scan(2, x[:, :K], x[:, Kp:Kp + K], x[:, 2 * Kp:2 * Kp + V], None, None, None, None, gates[:, :H], state, qs,
                                  mk([slots[i] for i, _ in part]), pos, H, d, dv, H // Hk, True, d ** -0.5, gate_raw=gates[:, H:], gate_A=A,
                                  gate_dt_bias=bias)
        for j, (i, n) in enumerate(part):
            got[i].append(y[int(qs[j]):int(qs[j + 1])])
            at[i] += n
    for i, n in enumerate(lens):
        x = rows[i].double().cpu()
        q, k = O.unit(x[:, :K].view(n, Hk, d)) / math.sqrt(d), O.unit(x[:, Kp:Kp + K].view(n, Hk, d))
        beta = torch.sigmoid(x[:, 2 * Kp + V:2 * Kp + V + H])
        decay = torch.exp(A.double().cpu() * torch.nn.functional.softplus(x[:, 2 * Kp + V + H:] + bias.double().cpu()))
        v = x[:, 2 * Kp:2 * Kp + V].view(n, H, dv)
        want = torch.stack([O.delta_rule(q[:, h // (H // Hk)], k[:, h // (H // Hk)], v[:, h], decay[:, h], beta[:, h]) for h in range(H)], 1)
        assert rel(torch.cat(got[i]).view(n, H, dv), want) < (3e-6 if dtype == torch.float32 else 4e-3)
    assert bool((state[[1, 3, 5]] == 9).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [2, 5, 8])
def test_short_convolution(ops, W, dtype):
    g, C, n = gen(W), 40, 150
    x = torch.randn(n, C, device=DEV, generator=g).to(dtype)
    taps = torch.randn(C, W, device=DEV, generator=g)
    state = torch.full((3, W - 1, C), 5.0, device=DEV, dtype=dtype)
    want = O.short_conv_silu(x.double().cpu(), taps.double().cpu())
    out, lo = [], 0
    mk = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    for m in (1, 2, 1, 70, 3, 73):
        out.append(ops.causal_conv1d(x[lo:lo + m], taps, None, state, mk([0, m]), mk([1]), mk(list(range(lo, lo + m))), True, m))
        lo += m
    assert rel(torch.cat(out), want) < (1e-6 if dtype == torch.float32 else 4e-3)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", list(S.CONFIGS))
def test_model_over_schedules(name, f32):
    """One prompt at once, token by token through captured graphs, and in portions around pages and tiles; every request reuses
    the pages and state rows of the one before it."""
    cfg, w, toks, want = S.expected(name, 140, 2)
    eng = S.engine(cfg, w, DEV, f32, blocks=9, max_len=144)
    rp = S.TraceReplay(eng)
    tol = TOL[f32]
    assert S.error(S.feed(rp, "a", toks, []), want) < tol
    assert S.error(S.feed(rp, "b", toks, range(1, 140)), want) < tol
    assert eng.stats.graph_steps > 100
    for cuts in ([2, 4, 6, 15, 31, 33, 63, 64, 66, 128, 129], [100, 101, 102, 120]):
        assert S.error(S.feed(rp, "c", toks, cuts), want) < tol
    assert int(eng.ops.status.item()) == 0


@pytest.mark.parametrize("f32", [True, False])
def test_mixed_batches_match_each_alone(f32):
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, DEV, f32, blocks=14, max_len=96)
    rp = S.TraceReplay(eng)
    g = torch.Generator().manual_seed(8)
    reqs = {f"r{i}": S.prompt(cfg, n, 200 + i) for i, n in enumerate((40, 3, 61, 20, 33, 2, 50, 9))}
    want = {k: O.forward(cfg, w, v, torch.float64) for k, v in reqs.items()}
    at, waiting, live = {k: 0 for k in reqs}, list(reqs), []
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-len(reqs[k]) // 16) for k in live + waiting[:1]) <= 14:
            live.append(waiting.pop(0))
        # some steps are pure decode steps (a request's first entry is a prompt)
        single = all(at[k] for k in live) and int(torch.randint(0, 2, (1,), generator=g)) == 0
        entries = []
        for k in live:
            n = 1 if single else min(int(torch.randint(1, 20, (1,), generator=g)), len(reqs[k]) - at[k])
            entries.append(dict(id=k, tokens=reqs[k][at[k]:at[k] + n], want=list(range(n))))
        ends = [e["id"] for e in entries if at[e["id"]] + len(e["tokens"]) == len(reqs[e["id"]])]
        lg, row = rp.step(entries, ends), 0
        for e in entries:
            n, k = len(e["tokens"]), e["id"]
            assert S.error(lg[row:row + n], want[k][at[k]:at[k] + n]) < TOL[f32], (k, at[k])
            at[k] += n
            row += n
        live = [k for k in live if k not in ends]
    assert eng.stats.graph_steps > 0 and len(eng.blocks.state_free) == 4 and len(eng.blocks.free) == 14


@pytest.mark.parametrize("f32", [True, False])
def test_generation_through_the_scheduler(f32):
    """Greedy text of unequal requests with chunked prompts, graphs and launch-ahead steps: each token is the oracle's best
    one within the precision; long decoding included."""
    cfg = S.CONFIGS["attention-only" if f32 else "odd"]
    w = S.tensors(cfg)
    eng = S.engine(cfg, w, DEV, f32, chunk=32, seqs=3, spare=8, blocks=60, max_len=256)
    prompts = [S.prompt(cfg, n, n) for n in (3, 90, 17, 40)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=60, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 60
        lg = O.forward(cfg, w, p + o)[len(p) - 1:-1]
        gap = (lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]) / (lg.max(-1).values - lg.min(-1).values)
        assert float(gap.max()) < (1e-4 if f32 else 0.05)
    assert eng.stats.graph_steps > 0
    alone = S.engine(cfg, w, DEV, f32, spare=8, blocks=60, max_len=256, graphs=False).generate(prompts[:1], SamplingParams(max_tokens=60, ignore_eos=True))
    assert not f32 or alone[0] == outs[0]


def test_fp32_is_refused_where_kernels_are_missing():
    from fllm_b200.config import EngineConfig, preset
    from fllm_b200.runtime.engine import LLMEngine
    with pytest.raises(ValueError):
        LLMEngine(preset("qwen3-tiny"), EngineConfig(dtype="fp32", num_kv_blocks=8, max_model_len=64), device=DEV)


def test_replay_program(tmp_path):
    """bin/trace_run as a process: steps on standard input, one logits file and one 'done' line per step."""
    import json
    import os
    import subprocess

    import numpy as np
    cfg, w, toks, want = S.expected("odd", 140, 2)
    path = S.write_checkpoint(tmp_path / "m", cfg, w)
    os.mkdir(tmp_path / "out")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    lines = [dict(step=0, entries=[dict(id="x", tokens=toks[:9], want=[8, 2])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=toks[9:10], want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=toks[10:11], want=[0])], end=["x"])]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "64"], input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=280)
    assert r.returncode == 0 and [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"], r.stderr[-500:]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
    assert S.error(read(0), want[[8, 2]]) < 2e-5 and S.error(read(2), want[[10]]) < 2e-5 and not (tmp_path / "out" / "1.f32").exists()
