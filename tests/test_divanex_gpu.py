"""Divanex on a GPU: each mechanism's kernel alone against the functions of tests/divanex_oracle.py, then whole models in fp32
and bf16 over portions, mixed batches, captured decode steps and the scheduler."""
import json
import math
import os
import subprocess
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import divanex_cases as S
import divanex_oracle as O
from fllm_b200.runtime.request import SamplingParams

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {True: 2e-5, False: 1e-1}                     # fp32, bf16
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from fllm_b200.ops.native import NativeOps
    return NativeOps(torch.device(DEV))


def gen(seed):
    return torch.Generator(device=DEV).manual_seed(seed)


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-12))


def ints(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


d64 = lambda t: t.double().cpu()


# ------------------------------------------------------------------------------------------------ residual, token input
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ld", [(64, 64), (75, 80), (13, 16), (2048, 2048), (4100, 4104), (9000, 9000)])
def test_postnorm_steps(ops, width, ld, dtype):
    g, T, eps = gen(width), 9, 1e-3
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width))
    mk = lambda *s: pad(torch.randn(*s, width, device=DEV, generator=g)).to(dtype)
    table, w1, w2, wf, y1, y2 = mk(50), mk(), mk(), mk(), mk(T), mk(T)
    ids = torch.randint(0, 50, (T,), device=DEV, generator=g).int()
    cut = lambda t: d64(t)[..., :width]
    tol = 2e-6 if dtype == torch.float32 else 4e-3
    x, h = ops.postnorm_begin(ids, table, 3.7)
    want = cut(table)[ids.cpu().long()] * 3.7
    assert rel(x[:, :width], want) < 1e-6 and rel(h[:, :width], want) < tol
    h = ops.postnorm_step(x, y1, w1, width, eps, 1.3)                                       # norm behind the sum
    want = O.rms(1.3 * want + cut(y1), eps) * cut(w1)
    assert rel(x[:, :width], want) < 2e-6 and rel(h[:, :width], want) < tol and not x[:, width:].any()
    h = ops.postnorm_step(x, y2, w2, width, eps, 1.0, True)                                 # norm of what is added
    want = want + O.rms(cut(y2), eps) * cut(w2)
    assert rel(x[:, :width], want) < 2e-6 and rel(h[:, :width], want) < tol and not h[:, width:].any()
    rows, before = ints([7, 0, 7]), x.clone()
    for add in (True, False):                                                               # with the final norm, chosen rows
        h = ops.postnorm_step(x, y1, w1, width, eps, 0.9, add, wf, 0.25, rows)
        last = want + O.rms(cut(y1), eps) * cut(w1) if add else O.rms(0.9 * want + cut(y1), eps) * cut(w1)
        assert rel(h[:, :width], (O.rms(last, eps) * cut(wf) * 0.25)[rows.cpu().long()]) < tol and torch.equal(before, x)


@pytest.mark.parametrize("dtype", DTYPES)
def test_side_gate(ops, dtype):
    g = gen(3)
    table, gate = torch.randn(30, 77, device=DEV, generator=g).to(dtype), (torch.randn(7, 16, device=DEV, generator=g) * 2).to(dtype)
    ids = ints([0, 29, 3, 3, 11, 5, 8])
    y = ops.side_gate(gate, ids, table, 33, 11)
    want = O.gelu_tanh(d64(gate)[:, :11]) * d64(table)[ids.cpu().long(), 33:44]
    assert rel(y[:, :11], want) < (1e-6 if dtype == torch.float32 else 4e-3) and not y[:, 11:].any()


def test_consumers_take_split_k_partial_sums(ops):
    """A projection whose split-K reduction is left to the kernel behind it."""
    g, T, K, N = gen(1), 8, 4096, 512
    a = torch.randn(T, K, device=DEV, generator=g).bfloat16()
    w = (torch.randn(N, K, device=DEV, generator=g) * K ** -0.5).bfloat16()
    y = d64(a) @ d64(w).t()

    def deferred():
        p = ops.linear(a, w, defer=True)
        assert not isinstance(p, torch.Tensor)
        return p
    nw = torch.ones(N, device=DEV, dtype=torch.bfloat16)
    x = torch.randn(T, N, device=DEV, generator=g)
    want = O.rms(1.5 * d64(x) + y, 1e-5)
    ops.postnorm_step(x, deferred(), nw, N, 1e-5, 1.5)
    assert rel(x, want) < 1e-5
    table, ids = torch.randn(9, N, device=DEV, generator=g).bfloat16(), ints(list(range(8)))
    assert rel(ops.side_gate(deferred(), ids, table, 0, N), O.gelu_tanh(y) * d64(table)[:8]) < 4e-3
    cache, factor = torch.zeros(2, 2, 16, 128, device=DEV, dtype=torch.bfloat16), torch.zeros(2, 2, 16, device=DEV)
    q, qf = ops.tied_prepare(deferred(), 256, 2, 128, ints(list(range(8))), ints(list(range(16, 24))), 1e-5, 1.0, 0.0, 1.0, cache, factor)
    assert rel(q, y[:, :256]) < 4e-3 and rel(cache[1, :, :8].transpose(0, 1).reshape(T, 256), y[:, 256:]) < 4e-3
    assert rel(qf, 1 / torch.sqrt(y[:, :256].view(T, 2, 128).pow(2).mean(-1) + 1e-5)) < 4e-3


@pytest.mark.parametrize("kind", [0, 1, 2])
def test_gated_activation_in_fp32(ops, kind):
    x = torch.randn(5, 2 * 37, device=DEV, generator=gen(kind)) * 2
    g, u = (d64(x)[:, 0::2], d64(x)[:, 1::2]) if kind == 2 else (d64(x)[:, :37], d64(x)[:, 37:])
    want = O.clamped_glu(g, u, 0.7) if kind == 2 else (O.silu(g) if kind == 0 else O.gelu_tanh(g)) * u
    assert rel(ops.glu(x, kind, 1.702, 0.7), want) < 1e-6


# ------------------------------------------------------------------------------------------------ tied attention
def batch(lens, ctxs, bs=16, seed=0):
    g = torch.Generator().manual_seed(seed)
    B, mb = len(lens), max(-(-c // bs) for c in ctxs)
    tab = torch.randperm(B * mb + 3, generator=g)[:B * mb].view(B, mb).int()
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    pos = torch.cat([torch.arange(c - n, c) for n, c in zip(lens, ctxs)]).int()
    seq = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).int()
    dev = lambda t: t.to(DEV)
    b = SimpleNamespace(num_seqs=B, max_q_len=max(lens), min_q_len=min(lens), max_kv_len=max(ctxs), positions=dev(pos), row_seq=dev(seq),
                        block_tables=dev(tab), q_starts=dev(torch.tensor(starts, dtype=torch.int32)))
    return b, tab, B * mb + 3, starts


def dense(q, qf, cache, kf, tab, starts, lens, ctxs, H, G, dim, cap, bs=16):
    """Softmax over the visible rows of every token, in fp64."""
    q, qf, cache, kf = (d64(t) for t in (q, qf, cache, kf))
    out = torch.zeros(q.shape[0], H * dim, dtype=torch.float64)
    for i, (n, c) in enumerate(zip(lens, ctxs)):
        idx, off = tab[i][torch.arange(c) // bs].long(), torch.arange(c) % bs
        for h in range(H):
            k, f = cache[idx, h // (H // G), off, :dim], kf[idx, h // (H // G), off]
            rows = slice(starts[i], starts[i] + n)
            qq = q[rows, h * dim:(h + 1) * dim] * qf[rows, h:h + 1]
            out[rows, h * dim:(h + 1) * dim] = O.attend(qq, k * f[:, None], k, 1.0, cap)
    return out


SHAPES = [(8, 2, 64), (80, 1, 64), (12, 1, 128), (3, 3, 24), (40, 2, 128), (5, 1, 80), (6, 2, 20), (4, 4, 136), (1, 1, 8)]
BATCHES = [([1, 1, 1], [1, 40, 129]), ([5, 1, 23], [5, 17, 60]), ([70], [133]), ([1], [700]), ([150, 1, 130], [150, 300, 400])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim", SHAPES)
@pytest.mark.parametrize("lens,ctxs", BATCHES)
def test_tied_attention(ops, H, G, dim, lens, ctxs, dtype):
    from fllm_b200.ops.tied import tied_width
    W, g = tied_width(dim), gen(H + dim)
    b, tab, nb, starts = batch(lens, ctxs)
    T = starts[-1]
    cache = torch.nn.functional.pad(torch.randn(nb, G, 16, dim, device=DEV, generator=g), (0, W - dim)).to(dtype)
    kf = torch.rand(nb, G, 16, device=DEV, generator=g) + 0.5
    q = torch.randn(T, H * dim + 5, device=DEV, generator=g).to(dtype)[:, :H * dim]
    qf = (torch.rand(T, H, device=DEV, generator=g) + 0.5) * 3 / math.sqrt(dim)
    for cap in ((20.0, None, 100.0) if len(lens) < 3 or dtype == torch.bfloat16 else (20.0,)):
        want = dense(q, qf, cache, kf, tab, starts, lens, ctxs, H, G, dim, cap)
        tol = 3e-6 if dtype == torch.float32 else 4e-3
        assert rel(ops.attention_tied(q, qf, cache, kf, dim, b, cap or 0.0), want) < tol, cap
        if dtype == torch.bfloat16:
            assert rel(ops.attention_tied(q, qf, cache, kf, dim, b, cap or 0.0, tensor_cores=False), want) < tol, cap
            for splits in (2, 5):
                assert rel(ops.attention_tied(q, qf, cache, kf, dim, b, cap or 0.0, splits=splits), want) < tol, (cap, splits)
    y = ops.attention_tied(q, qf, cache, kf, dim, b, 20.0, H * dim + 8)                     # padded columns are zero
    assert y.shape[1] == H * dim + 8 and not y[:, H * dim:].any()
    assert int(ops.status.item()) == 0


@pytest.mark.parametrize("block_size", [32, 48])
def test_tied_attention_with_larger_blocks(ops, block_size):
    H, G, dim, lens, ctxs = 8, 2, 64, [100, 1], [130, 200]
    g = gen(5)
    b, tab, nb, starts = batch(lens, ctxs, block_size)
    cache = torch.randn(nb, G, block_size, dim, device=DEV, generator=g).bfloat16()
    kf = torch.rand(nb, G, block_size, device=DEV, generator=g) + 0.5
    q, qf = torch.randn(101, H * dim, device=DEV, generator=g).bfloat16(), torch.full((101, H), 0.3, device=DEV)
    assert rel(ops.attention_tied(q, qf, cache, kf, dim, b, 20.0), dense(q, qf, cache, kf, tab, starts, lens, ctxs, H, G, dim, 20.0, block_size)) < 4e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens,ctx", [([1], 400), ([200], 400)])
def test_single_keys_at_every_border(ops, lens, ctx, dtype):
    """One key's score stands far out: the result is that key wherever it lies (first tokens, page and tile borders, the query's
    own position), and the key right behind a query is never seen."""
    H, G, dim = 4, 2, 64
    b, tab, nb, starts = batch(lens, [ctx], seed=4)
    g, n = gen(3), lens[0]
    base = torch.randn(nb, G, 16, dim, device=DEV, generator=g) * 0.1
    q = torch.randn(n, H * dim, device=DEV, generator=g)
    kf, qf = torch.ones(nb, G, 16, device=DEV), torch.ones(n, H, device=DEV)
    for place in (0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 129, 199, 200, 201, 255, 256, 383, 384, 398, 399):
        for t in sorted({0, n // 2, n - 1}):
            key = q[t, 3 * dim:] * 3                                    # query t, head 3 points at this key of head 1
            cache = base.clone()
            cache[int(tab[0, place // 16]), 1, place % 16] = key
            got = ops.attention_tied(q.to(dtype), qf, cache.to(dtype), kf, dim, b, 50.0)[t, 3 * dim:].float()
            if place <= ctx - n + t:
                assert rel(got, key) < 1e-2, (place, t)
            else:
                assert float(got @ key) < 0.5 * float(key @ key), (place, t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,dim", [(2, 20), (1, 128)])
def test_factors_and_cache_rows(ops, G, dim, dtype):
    from fllm_b200.ops.tied import tied_width
    H, T, W, off, g = 4, 8, tied_width(dim), 4 * dim + 8, gen(dim)
    x = torch.randn(T, off + G * dim + 3, device=DEV, generator=g).to(dtype)
    pos = ints([0, 98, 99, 100, 198, 199, 70000, 0])
    slots = [3, 17, 4, 60, 33, 32, 31, -1]
    cache, factor = torch.full((4, G, 16, W), 7.0, device=DEV, dtype=dtype), torch.full((4, G, 16), 7.0, device=DEV)
    q, qf = ops.tied_prepare(x, off, H, dim, pos, ints(slots), 1e-3, 0.7, 0.4, 100.0, cache, factor)
    v = d64(x)
    inv = lambda t: 1 / torch.sqrt(t.pow(2).mean(-1) + 1e-3)
    temp = 1 + 0.4 * torch.tensor([math.log((p + 1) // 100 + 1) for p in pos.tolist()], dtype=torch.float64)
    assert torch.equal(q, x[:, :H * dim]) and rel(qf, 0.7 * temp[:, None] * inv(v[:, :H * dim].view(T, H, dim))) < 1e-6
    for t, s in enumerate(slots[:-1]):
        for h in range(G):
            k = x[t, off + h * dim:off + (h + 1) * dim]
            assert torch.equal(cache[s // 16, h, s % 16, :dim], k) and not cache[s // 16, h, s % 16, dim:].any()
            assert abs(float(factor[s // 16, h, s % 16]) / float(inv(d64(k))) - 1) < 1e-6
    assert int((factor == 7).sum()) == (64 - 7) * G


# ------------------------------------------------------------------------------------------------ Mamba-2
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,P,N,G", [(4, 13, 20, 2), (1, 8, 8, 1), (6, 40, 16, 3), (4, 24, 64, 1), (2, 64, 128, 2), (2, 20, 256, 1), (3, 300, 100, 3), (2, 64, 48, 1),
                                     (2, 7, 32, 2)])
def test_ssd_scan(ops, H, P, N, G, dtype):
    """Ragged steps that continue each other: prompts, portions of 2 .. 33 tokens and single tokens, rows of the pool in any order."""
    g = gen(N)
    lens, slots = [45, 70, 3], [2, 0, 4]
    p8 = lambda n: (n + 7) // 8 * 8
    oB, oC, oD = p8(H * P), p8(H * P) + p8(G * N), p8(H * P) + 2 * p8(G * N)
    rows = [torch.randn(n, p8(oD + H), device=DEV, generator=g).to(dtype) for n in lens]
    A = -torch.exp(torch.randn(H, device=DEV, generator=g))
    A[-1] *= 30                                                        # a head that forgets within a token or two
    D, bias = torch.randn(H, device=DEV, generator=g), torch.randn(H, device=DEV, generator=g) - 2
    state = torch.full((6, H, P, N), 9.0, device=DEV)                  # stale rows of earlier requests
    got, at = [[] for _ in lens], [0, 0, 0]
    for take in ([17, 2, 1], [0, 33, 1], [1, 1, 1], [1, 1, 0], [26, 33, 0]):
        part = [(i, n) for i, n in enumerate(take) if n]
        x = torch.cat([rows[i][at[i]:at[i] + n] for i, n in part])
        qs = ints([sum(n for _, n in part[:j]) for j in range(len(part) + 1)])
        pos = ints([p for i, n in part for p in range(at[i], at[i] + n)])
        y = ops.mamba2_scan(x[:, :H * P], x[:, oD:oD + H], x[:, oB:oB + G * N], x[:, oC:oC + G * N], A, D, bias, state, qs, ints([slots[i] for i, _ in part]), pos,
                            H, P, G, N)
        for j, (i, n) in enumerate(part):
            got[i].append(y[int(qs[j]):int(qs[j + 1])])
            at[i] += n
    for i, n in enumerate(lens):
        x = d64(rows[i])
        dt = O.softplus(x[:, oD:oD + H] + d64(bias))
        B, C = x[:, oB:oB + G * N].view(n, G, N), x[:, oC:oC + G * N].view(n, G, N)
        want = [O.ssd(x[:, h * P:(h + 1) * P], dt[:, h], B[:, h // (H // G)], C[:, h // (H // G)], -d64(A)[h], d64(D)[h]) for h in range(H)]
        assert rel(torch.cat(got[i]), torch.cat([y for y, _ in want], 1)) < (2e-6 if dtype == torch.float32 else 4e-3)
        assert rel(state[slots[i]], torch.stack([s.t() for _, s in want])) < 2e-6                # fp32 in both modes
    assert bool((state[[1, 3, 5]] == 9).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_ssd_state_over_long_decoding(ops, dtype):
    """600 single tokens after a prompt: the state keeps its precision."""
    H, P, N, g = 2, 16, 24, gen(7)
    n = 640
    x = torch.randn(n, H * P + 2 * N + 8, device=DEV, generator=g).to(dtype)
    A, bias = -torch.tensor([0.01, 0.5], device=DEV), torch.tensor([-3.0, -1.0], device=DEV)
    state, out, lo = torch.zeros(1, H, P, N, device=DEV), [], 0
    for m in [40] + [1] * 600:
        r = x[lo:lo + m]
        out.append(ops.mamba2_scan(r[:, :H * P], r[:, H * P + 2 * N:H * P + 2 * N + H], r[:, H * P:H * P + N], r[:, H * P + N:H * P + 2 * N], A, None, bias, state,
                                   ints([0, m]), ints([0]), ints(list(range(lo, lo + m))), H, P, 1, N))
        lo += m
    v = d64(x)
    dt = O.softplus(v[:, H * P + 2 * N:H * P + 2 * N + H] + d64(bias))
    want = torch.cat([O.ssd(v[:, h * P:(h + 1) * P], dt[:, h], v[:, H * P:H * P + N], v[:, H * P + N:H * P + 2 * N], -d64(A)[h], 0.0)[0] for h in range(H)], 1)
    assert rel(torch.cat(out), want) < (3e-6 if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,groups,width", [(36, 3, 40), (2048, 1, 2048), (13, 1, 16), (96, 96, 96)])
def test_grouped_gated_norm(ops, inner, groups, width, dtype):
    g = gen(inner)
    y, z, w = (torch.randn(*s, device=DEV, generator=g).to(dtype) for s in ((6, inner), (6, inner + 4), (inner,)))
    got = ops.gated_rmsnorm(y, z[:, :inner], w, 1e-3, inner // groups, False, width)
    assert rel(got[:, :inner], O.grouped_gated_norm(d64(y), d64(z)[:, :inner], d64(w), groups, 1e-3)) < (1e-6 if dtype == torch.float32 else 4e-3)
    assert not got[:, inner:].any()


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
def test_long_prompt_and_long_decoding(f32):
    """600 tokens at once, then 200 of them one by one behind a long prompt."""
    cfg, w, toks, want = S.expected("odd", 600, 5)
    rp = S.TraceReplay(S.engine(cfg, w, DEV, f32, blocks=38, max_len=608, chunk=608))
    assert S.error(S.feed(rp, "a", toks, []), want) < TOL[f32]
    assert S.error(S.feed(rp, "b", toks, range(400, 600)), want) < TOL[f32]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", ["odd", "attention-only"])
def test_mixed_batches_match_each_alone(name, f32):
    cfg = S.CONFIGS[name]
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
    assert eng.stats.graph_steps > 0 and len(eng.blocks.free) == 14


@pytest.mark.parametrize("f32", [True, False])
def test_generation_through_the_scheduler(f32):
    """Greedy text of unequal requests with chunked prompts, graphs and launch-ahead steps: each token is the oracle's best one
    within the precision; long decoding included."""
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


def test_replay_program(tmp_path):
    """bin/trace_run as a process: steps on standard input, one logits file and one 'done' line per step."""
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
