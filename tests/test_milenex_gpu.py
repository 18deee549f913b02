"""Milenex on a GPU: each mechanism's kernel alone against the functions of tests/milenex_oracle.py, then whole models in fp32 and
bf16 over portions, mixed batches, captured decode steps and the scheduler."""
import json
import math
import os
import subprocess
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import milenex_cases as S
import milenex_oracle as O
from fllm_b200.config import MoeSpec
from fllm_b200.models.decoder import Decoder
from fllm_b200.models.weights import LayerWeights
from fllm_b200.ops.maps import ConvWindow, maps_width, spread_width
from fllm_b200.ops.prenorm import TokenShift
from fllm_b200.runtime.request import SamplingParams

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {True: 2e-5, False: 8e-2}                     # fp32, bf16
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
pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))


# ------------------------------------------------------------------------------------------------ residual, norm, token shift
def step_batch(lens, starts, slots):
    """The sequences of a step: their tokens, their first positions and their state rows."""
    qs = [0]
    for n in lens:
        qs.append(qs[-1] + n)
    return SimpleNamespace(q_starts=ints(qs), seq_state=ints(slots), row_seq=ints([i for i, n in enumerate(lens) for _ in range(n)]),
                           positions=ints([p for n, p0 in zip(lens, starts) for p in range(p0, p0 + n)]), max_q_len=max(lens))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ld", [(64, 64), (75, 80), (13, 16), (2048, 2048), (4100, 4104), (9000, 9000)])
def test_norm_in_front_and_embeddings_added_again(ops, width, ld, dtype):
    g, T, eps = gen(width), 9, 1e-3
    mk = lambda *s: pad(torch.randn(*s, width, device=DEV, generator=g), ld).to(dtype)
    table, w, y = mk(30), (mk() * 0.3).to(dtype), mk(T)
    ids = ints([3, 29, 0, 7, 7, 1, 2, 4, 28])
    cut, tol = (lambda t: d64(t)[..., :width]), 2e-6 if dtype == torch.float32 else 4e-3
    x, h = ops.prenorm_step(None, None, w, width, eps, ids=ids, table=table)
    want = cut(table)[ids.long().cpu()]
    assert rel(x[:, :width], want) < 1e-7 and rel(h[:, :width], O.norm(want, cut(w), eps)) < tol and not h[:, width:].any() and not x[:, width:].any()
    x2, h = ops.prenorm_step(x, y, w, width, eps)
    want = want + cut(y)
    assert x2 is x and rel(x[:, :width], want) < 2e-7 and rel(h[:, :width], O.norm(want, cut(w), eps)) < tol
    x, h = ops.prenorm_step(x, y, w, width, eps, ids=ids, table=table)
    want = want + cut(y) + cut(table)[ids.long().cpu()]
    assert rel(x[:, :width], want) < 2e-7 and rel(h[:, :width], O.norm(want, cut(w), eps)) < tol
    before = x.clone()
    _, h = ops.prenorm_step(x, y, w, width, eps, offset=0.5, rows=ints([8, 0, 3]))
    assert torch.equal(before, x) and rel(h[:, :width], (O.rms(want + cut(y), eps) * (0.5 + cut(w)))[[8, 0, 3]]) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ld", [(75, 80), (2048, 2048), (4100, 4104)])
def test_token_shift_over_portions(ops, width, ld, dtype):
    """Ragged steps that continue each other, among them steps long enough for several rows per CTA, with state rows in any order;
    every portion's first token meets the last one of the portion before, exactly as in one piece."""
    g, eps, slots = gen(width), 1e-3, [2, 0, 4]
    lens = [1900, 1100, 3]
    rows = [pad(torch.randn(n, width, device=DEV, generator=g), ld).to(dtype) for n in lens]
    w, mu = (pad(torch.randn(width, device=DEV, generator=g) * 0.3, ld).to(dtype) for _ in range(2))
    state = torch.full((6, ld), 9.0, device=DEV)                   # stale rows of earlier requests
    got, at = [[] for _ in lens], [0, 0, 0]
    for take in ([17, 2, 1], [0, 33, 1], [1, 1, 1], [1, 1, 0], [2, 0, 0], [1750, 1000, 0], [128, 62, 0], [1, 1, 0]):
        part = [(i, n) for i, n in enumerate(take) if n]
        y = torch.cat([rows[i][at[i]:at[i] + n] for i, n in part])
        b = step_batch([n for _, n in part], [at[i] for i, _ in part], [slots[i] for i, _ in part])
        x = torch.zeros(y.shape[0], ld, device=DEV)
        new, h = ops.prenorm_step(x, y, w, width, eps, shift=TokenShift(mu, state, b))
        assert new is not x and not x.any() and torch.equal(new, y.float())
        for j, (i, n) in enumerate(part):
            got[i].append(h[int(b.q_starts[j]):int(b.q_starts[j + 1])])
            at[i] += n
    for i in range(3):
        n = at[i]
        normed = O.norm(d64(rows[i])[:n, :width], d64(w)[:width], eps)
        assert rel(torch.cat(got[i])[:, :width], O.token_shift(normed, d64(mu)[:width])) < (2e-6 if dtype == torch.float32 else 4e-3)
        assert rel(state[slots[i], :width], normed[-1]) < 2e-6                               # fp32 in both modes
    assert bool((state[[1, 3, 5]] == 9).all())


def test_consumers_take_split_k_partial_sums(ops):
    """A projection whose split-K reduction is left to the kernel behind it: the residual, and the attention inputs with their
    convolution and their gate columns."""
    g, T, K, N = gen(1), 8, 4096, 512
    h = torch.randn(T, K, device=DEV, generator=g).bfloat16()
    w = (torch.randn(N, K, device=DEV, generator=g) * K ** -0.5).bfloat16()
    y = d64(h) @ d64(w).t()

    def deferred():
        p = ops.linear(h, w, defer=True)
        assert not isinstance(p, torch.Tensor)
        return p
    zero, x = torch.zeros(N, device=DEV, dtype=torch.bfloat16), torch.randn(T, N, device=DEV, generator=g)
    want = d64(x) + y
    b = step_batch([1] * T, list(range(T)), list(range(T)))
    new, out = ops.prenorm_step(x, deferred(), zero, N, 1e-5, shift=TokenShift(zero, torch.zeros(T, N, device=DEV), b))
    assert rel(new, want) < 1e-5 and rel(out, O.rms(want, 1e-5)) < 4e-3
    kc, vc = torch.zeros(2, 2, 16, 64, device=DEV, dtype=torch.bfloat16), torch.zeros(2, 1, 16, 64, device=DEV, dtype=torch.bfloat16)
    conv_w, state = torch.randn(448, 4, device=DEV, generator=g), torch.randn(T, 3, 448, device=DEV, generator=g).bfloat16()
    u = torch.cat([d64(state), y[:, None, :448]], 1)
    want, gate = (u * d64(conv_w).t()).sum(1), torch.empty(T, 5, device=DEV)
    q = ops.maps_prepare(deferred(), (0, 256, 384), 4, 64, 60, ints(list(range(5, 13))), ints(list(range(16, 24))), torch.zeros(8, device=DEV), 1.0, None, None, False,
                         1e-5, kc, vc, conv=ConvWindow(conv_w, state, ints(list(range(T)))), extra_out=gate, extra_offset=450)
    unit = lambda t: O.rms(t.reshape(T, -1, 64), 1e-5).view(T, -1)
    assert rel(q.view(T, 256), unit(want[:, :256])) < 4e-3 and rel(kc[1, :, :8].transpose(0, 1).reshape(T, 128), unit(want[:, 256:384])) < 4e-3
    assert rel(vc[1, 0, :8, :60], want[:, 384:444]) < 4e-3 and rel(gate, y[:, 450:455]) < 1e-5 and rel(state[:, :, :444], u[:, 1:, :444]) < 4e-3


# ------------------------------------------------------------------------------------------------ queries and cache rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", ["unit", "none"])
@pytest.mark.parametrize("H,G,dim,v_dim,rot,conv", [(4, 2, 20, 28, 10, 0), (3, 1, 64, 128, 64, 4), (2, 2, 96, 64, 32, 2), (1, 1, 7, 5, 2, 8), (2, 1, 140, 9, 140, 3),
                                                    (16, 4, 128, 128, 0, 4), (4, 4, 40, 12, 6, 5)])
def test_queries_and_cache_rows(ops, H, G, dim, v_dim, rot, conv, norm, dtype):
    """Neighbouring values turn together, norms without weights or none, the convolution of single tokens, further columns."""
    g, T, eps, E = gen(dim), 8, 1e-3, 3
    inv = torch.tensor([700.0 ** (-2 * i / rot) for i in range(rot // 2)], device=DEV)
    p8 = lambda n: (n + 7) // 8 * 8
    nq, nk, nv = p8(H * dim), p8(G * dim), p8(G * v_dim)
    x = torch.randn(T, nq + nk + nv + E, device=DEV, generator=g).to(dtype)
    if dim % 4 == 0 and v_dim % 4 == 0:
        x = pad(x, nq + nk + nv + 8).contiguous()
    pos, slots = [0, 1, 98, 99, 100, 5000, 3, 0], [3, 17, 4, 60, 33, 32, 31, -1]
    Wk, Wv = maps_width(dim), maps_width(v_dim)
    kc, vc = torch.full((4, G, 16, Wk), 7.0, device=DEV, dtype=dtype), torch.full((4, G, 16, Wv), 7.0, device=DEV, dtype=dtype)
    extra, window, u = torch.empty(T, E, device=DEV), None, d64(x)
    if conv:
        C, order = nq + nk + nv, [5, 0, 3, 9, 1, 7, 2, 8]
        cw, state = torch.randn(C, conv, device=DEV, generator=g), torch.randn(10, conv - 1, C, device=DEV, generator=g).to(dtype)
        old = d64(state)
        window = ConvWindow(cw, state, ints(order))
        u = torch.stack([O.causal_conv(torch.cat([old[order[t]] * (pos[t] > 0), u[t:t + 1, :C]]), d64(cw))[-1] for t in range(T)])
    q = ops.maps_prepare(x, (0, nq, nq + nk), H, dim, v_dim, ints(pos), ints(slots), inv, 1.0, None, None, False, eps if norm == "unit" else -1.0, kc, vc, pairs=True,
                         conv=window, extra_out=extra, extra_offset=nq + nk + nv)

    def want(off, n):
        t = u[:, off:off + n * dim].reshape(T, n, dim)
        t = torch.stack([torch.cat([O.rotate(t[i:i + 1, j], rot, 700.0, pos[i]) for j in range(n)]) for i in range(T)]) if rot else t
        return O.rms(t, eps) if norm == "unit" else t
    tol = 5e-5 if dtype == torch.float32 else 4e-3                  # (an fp32 angle of some thousand radians)
    assert rel(q[:, :, :dim], want(0, H)) < tol and not q[:, :, dim:].any() and torch.equal(extra, x[:, nq + nk + nv:nq + nk + nv + E].float())
    k, v = want(nq, G), u[:, nq + nk:nq + nk + G * v_dim].reshape(T, G, v_dim)
    for t, s in enumerate(slots[:-1]):
        assert rel(kc[s // 16, :, s % 16, :dim], k[t]) < tol and not kc[s // 16, :, s % 16, dim:].any()
        assert rel(vc[s // 16, :, s % 16, :v_dim], v[t]) < tol and not vc[s // 16, :, s % 16, v_dim:].any()
    assert int((kc == 7).all(-1).sum()) == (64 - 7) * G and int((vc == 7).all(-1).sum()) == (64 - 7) * G
    if conv:
        live = [c for o, n in ((0, H * dim), (nq, G * dim), (nq + nk, G * v_dim)) for c in range(o, o + n)]
        for t in range(T - 1):                                       # (the last row has no place in the cache: a padding row)
            seen = torch.cat([old[order[t]] * (pos[t] > 0), d64(x)[t:t + 1, :C]])[1:]
            assert torch.equal(d64(state)[order[t]][:, live], seen[:, live])
        assert torch.equal(d64(state)[[4, 6]], old[[4, 6]])


# ------------------------------------------------------------------------------------------------ attention
def batch(lens, ctxs, bs=16, seed=0):
    g = torch.Generator().manual_seed(seed)
    B, mb = len(lens), max(-(-c // bs) for c in ctxs)
    tab = torch.randperm(B * mb + 3, generator=g)[:B * mb].view(B, mb).int()
    b = step_batch(lens, [c - n for n, c in zip(lens, ctxs)], list(range(B)))
    b.num_seqs, b.min_q_len, b.max_kv_len, b.block_tables = B, min(lens), max(ctxs), tab.to(DEV)
    return b, tab, B * mb + 3, b.q_starts.tolist()


def dense(q, kc, vc, tab, starts, lens, ctxs, H, G, dim, v_dim, scale, window, sink, r1=None, r2=None, mix=None, gate=None, bs=16):
    """Plain attention over the visible rows of every sequence, in fp64. ``mix``: talking heads over value rows of all heads."""
    q, kc, vc, sink = (d64(t) for t in (q, kc, vc, sink))
    out = torch.zeros(q.shape[0], H * v_dim, dtype=torch.float64)
    for i, (n, c) in enumerate(zip(lens, ctxs)):
        idx, off = tab[i][torch.arange(c) // bs].long(), torch.arange(c) % bs
        rows = slice(starts[i], starts[i] + n)
        bias = lambda h: (None, None) if r1 is None else (d64(r1)[h], d64(r2)[h])
        per = [O.weights(q[rows, h, :dim], kc[idx, h // (H // G), off, :dim], scale, window or c, sink[h], *bias(h)) for h in range(H)]
        per = O.talk(per, d64(mix)) if mix is not None else per
        for h in range(H):
            g = h // (H // G)
            v = vc[idx, 0, off, g * v_dim:(g + 1) * v_dim] if mix is not None else vc[idx, g, off, :v_dim]
            a = per[h] @ v
            out[rows, h * v_dim:(h + 1) * v_dim] = a if gate is None else a * O.sigmoid(d64(gate)[rows, h])[:, None]
    return out


BATCHES = [([1, 1, 1], [1, 40, 129]), ([5, 1, 23], [5, 17, 60]), ([70], [133]), ([1], [700]), ([150, 1, 130], [150, 300, 290])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,v_dim", [(8, 2, 64, 128), (12, 4, 96, 64), (3, 3, 24, 20), (20, 1, 40, 96), (4, 2, 136, 200), (1, 1, 8, 1)])
@pytest.mark.parametrize("lens,ctxs", BATCHES)
def test_attention_with_sinks(ops, H, G, dim, v_dim, lens, ctxs, dtype):
    g = gen(H + dim)
    b, tab, nb, starts = batch(lens, ctxs)
    mk = lambda n, d: pad(torch.randn(nb, n, 16, d, device=DEV, generator=g), maps_width(d)).to(dtype)
    kc, vc = mk(G, dim), mk(G, v_dim)
    q = pad(torch.randn(starts[-1], H, dim, device=DEV, generator=g), maps_width(dim)).to(dtype)
    scale, sink = 2 / math.sqrt(dim), torch.randn(H, device=DEV, generator=g) * 4 + 2
    for window in (0, 17, 50):
        want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, dim, v_dim, scale, window, sink)
        tol = 5e-6 if dtype == torch.float32 else 4e-3
        assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, sink=sink), want) < tol, window
        if dtype == torch.bfloat16:
            assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, tensor_cores=False, sink=sink), want) < tol, window
            if max(lens) * (H // G) <= 64:
                assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, splits=5, sink=sink), want) < tol, window
    assert int(ops.status.item()) == 0


SHAPES = [(8, 2, 64, 32), (12, 4, 96, 64), (6, 3, 20, 13), (16, 2, 128, 128), (7, 1, 64, 100), (20, 1, 100, 48), (4, 4, 50, 60), (24, 1, 16, 40), (5, 5, 128, 128), (4, 2, 136, 72),
          (1, 1, 8, 1), (6, 2, 200, 300)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,v_dim", SHAPES)
@pytest.mark.parametrize("lens,ctxs", BATCHES)
def test_talking_heads(ops, H, G, dim, v_dim, lens, ctxs, dtype):
    g = gen(H + dim)
    b, tab, nb, starts = batch(lens, ctxs)
    kc = pad(torch.randn(nb, G, 16, dim, device=DEV, generator=g), maps_width(dim)).to(dtype)
    vc = pad(torch.randn(nb, 1, 16, G * v_dim, device=DEV, generator=g), spread_width(G * v_dim)).to(dtype)
    q = pad(torch.randn(starts[-1], H, dim, device=DEV, generator=g), maps_width(dim)).to(dtype)
    scale, sink, mix = 2 / math.sqrt(dim), torch.randn(H, device=DEV, generator=g) * 3, torch.randn(H, H, device=DEV, generator=g)
    r1, r2 = torch.rand(H, device=DEV, generator=g) * 1.5, torch.rand(H, device=DEV, generator=g) * 2
    gate = torch.randn(starts[-1], H + 2, device=DEV, generator=g)[:, :H]
    for window in (0, 17, 50, 128) if H < 16 else (50,):
        want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, dim, v_dim, scale, window, sink, r1, r2, mix, gate)
        tol = 1e-5 if dtype == torch.float32 else 4e-3
        run = lambda **k: ops.attention_talk(q, kc, vc, dim, v_dim, b, scale, mix, window, sink, r1, r2, gate, H * v_dim + 8, **k)
        y = run()
        assert rel(y[:, :H * v_dim], want) < tol and not y[:, H * v_dim:].any(), window
        if dtype == torch.bfloat16:
            assert rel(run(tensor_cores=False)[:, :H * v_dim], want) < tol, window
            if max(lens) * (H // G) <= 64:
                assert rel(run(splits=3)[:, :H * v_dim], want) < tol, window
    assert int(ops.status.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_talking_heads_without_bias_sink_and_gate(ops, dtype):
    """The terms are optional; larger blocks."""
    H, G, dim, v_dim, lens, ctxs, g = 8, 2, 64, 64, [100, 1], [130, 200], gen(5)
    b, tab, nb, starts = batch(lens, ctxs, 32)
    kc, vc = torch.randn(nb, G, 32, dim, device=DEV, generator=g).to(dtype), torch.randn(nb, 1, 32, G * v_dim, device=DEV, generator=g).to(dtype)
    q, mix = torch.randn(101, H, dim, device=DEV, generator=g).to(dtype), torch.randn(H, H, device=DEV, generator=g)
    none = torch.full((H,), -1e4)
    want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, dim, v_dim, 0.3, 70, none, mix=mix, bs=32)
    assert rel(ops.attention_talk(q, kc, vc, dim, v_dim, b, 0.3, mix, 70), want) < (1e-5 if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_strong_distance_bias(ops, dtype):
    """A bias that falls by dozens of powers of two inside one tile, against far keys whose scores stand out as much."""
    H, G, dim, v_dim, lens, ctxs, g = 4, 2, 64, 32, [300, 1], [300, 290], gen(6)
    b, tab, nb, starts = batch(lens, ctxs)
    kc, vc = torch.randn(nb, G, 16, dim, device=DEV, generator=g).to(dtype), torch.randn(nb, 1, 16, G * v_dim, device=DEV, generator=g).to(dtype)
    q, mix, sink = torch.randn(301, H, dim, device=DEV, generator=g).to(dtype), torch.randn(H, H, device=DEV, generator=g), torch.zeros(H, device=DEV)
    kc[:, :, ::5] *= 6
    r1, r2 = torch.tensor([6.0, 9.0, 3.0, 0.0], device=DEV), torch.tensor([0.5, 4.0, 0.01, 1.0], device=DEV)
    want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, dim, v_dim, 0.5, 0, sink, r1, r2, mix)
    assert rel(ops.attention_talk(q, kc, vc, dim, v_dim, b, 0.5, mix, 0, sink, r1, r2), want) < (1e-5 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("talk", [False, True])
@pytest.mark.parametrize("lens,ctx", [([1], 400), ([200], 400)])
def test_single_keys_at_every_border(ops, lens, ctx, talk, dtype):
    """One key's score stands far out: the head's output is the key's value wherever it lies inside the window (first tokens, page and
    tile borders, the query's own position, the window's first token), and not one token outside it. With a sink above every other
    score the output outside is nearly zero."""
    H, G, dim, v_dim, n = 4, 2, 64, 64, lens[0]
    b, tab, nb, starts = batch(lens, [ctx], seed=4)
    g = gen(3)
    kc = torch.randn(nb, G, 16, dim, device=DEV, generator=g) * 0.1
    vc, q = torch.randn(nb, G, 16, v_dim, device=DEV, generator=g), torch.randn(n, H, dim, device=DEV, generator=g)
    sink, one = torch.full((H,), 20.0, device=DEV), torch.full((H,), 0.5, device=DEV)
    joint = vc.transpose(1, 2).reshape(nb, 1, 16, G * v_dim).to(dtype)
    mix = torch.zeros(H, H, device=DEV)
    mix[1, 3] = 1.0                                                # head 1, of the other group, speaks with head 3's weights
    seen = 0
    for window in (0, 1, 16, 33, 128, 200):
        for t in sorted({0, n // 2, n - 1}):
            i = ctx - n + t
            places = {0, 1, 15, 16, 127, 128, 129, i, i + 1, i - window, i - window + 1, i - window - 1, i - window + 2, (i - window + 1) // 16 * 16}
            for place in sorted(x for x in places if 0 <= x < ctx):
                key, block, at = q[t, 3] * 3, int(tab[0, place // 16]), place % 16          # query t, head 3
                cache = kc.clone()
                cache[block, 1, at] = key
                if talk:
                    got = ops.attention_talk(q.to(dtype), cache.to(dtype), joint, dim, v_dim, b, 1.0, mix, window, sink, one, one)[t].view(H, v_dim).float()
                    assert not got[[0, 2, 3]].any()
                    got, value = got[1], vc[block, 0, at]
                else:
                    got, value = ops.attention_maps(q.to(dtype), cache.to(dtype), vc.to(dtype), dim, v_dim, b, 1.0, window, sink=sink)[t, 3 * v_dim:].float(), vc[block, 1, at]
                inside = place <= i and (window == 0 or i - place < window)
                seen += inside
                assert rel(got, value) < 1e-2 if inside else float(got.norm()) < 0.05 * float(value.norm()), (window, t, place)
    assert seen >= 20


# ------------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,shared,groups", [(1, 64, 6, 2, 32, 48, (3, 2)), (37, 200, 12, 3, 48, 0, (4, 2)), (300, 256, 8, 8, 16, 32, None), (64, 128, 40, 5, 32, 64, (10, 4)),
                                                        (5, 24, 1, 1, 16, 16, None), (6, 64, 300, 9, 16, 32, (30, 3)), (50, 128, 256, 8, 16, 16, (256, 20))])
def test_routed_experts(ops, T, W, E, top, ff, shared, groups, dtype):
    g = gen(E)
    mk = lambda *s, gain=1.0: (torch.randn(*s, device=DEV, generator=g) * gain * s[-1] ** -0.5).to(dtype)
    h = torch.randn(T, W, device=DEV, generator=g).to(dtype)
    pairs = lambda a, b: torch.stack([a, b], -2).reshape(*a.shape[:-2], -1, a.shape[-1])       # gate and up rows of a feature side by side
    eg, eu, ed = mk(E, ff, W, gain=2.0), mk(E, ff, W, gain=2.0), mk(E, W, ff)
    corr = torch.randn(E, device=DEV, generator=g) * 0.3 - 0.5
    lw = LayerWeights(None, None, None, None, router_w=mk(E, W, gain=1.5), router_select_b=corr, exp_gate_up=pairs(eg, eu).contiguous(), exp_down=ed,
                      moe=MoeSpec(E, top, "deepseek_v2", groups=groups[0] if groups else 1, topk_groups=groups[1] if groups else 1, act="swiglu_oai", fp32_router=True,
                                  masked=float("-inf"), limit=0.8, shared_limit=1.3))
    w = {"router": d64(lw.router_w), "correction": d64(corr)}
    for e in range(E):
        w.update({f"e{e}.gate": d64(eg[e]), f"e{e}.up": d64(eu[e]), f"e{e}.down": d64(ed[e])})
    spec = dict(router=dict(top=top), expert=dict(limit=0.8))
    if groups:
        spec["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        sg, su = mk(shared, W, gain=2.0), mk(shared, W, gain=2.0)
        lw.shared_gate_up, lw.shared_down, lw.shared_gate_w = pairs(sg, su).contiguous(), mk(W, shared), mk(1, W, gain=2.0)
        w.update({"shared.gate": d64(sg), "shared.up": d64(su), "shared.down": d64(lw.shared_down), "shared.sg": d64(lw.shared_gate_w)})
        spec["shared"] = dict(limit=1.3)
    cfg = SimpleNamespace(mlp_kind="glu", swiglu_alpha=1.702, swiglu_limit=7.0)
    dec = SimpleNamespace(cfg=cfg, ops=ops, spec=SimpleNamespace(expert_parallel=False), ep_a2a=None)
    got = Decoder._ffn_block(dec, lw, h)
    assert rel(got, O.routed_mlp(d64(h), w, "", spec)) < (5e-6 if dtype == torch.float32 else 1e-2)      # every choice is the oracle's: the logits are fp32 sums


@pytest.mark.parametrize("dtype", DTYPES)
def test_dense_network(ops, dtype):
    g = gen(2)
    h, up, down = (torch.randn(*s, device=DEV, generator=g).to(dtype) for s in ((33, 80), (48, 80), (80, 48)))
    lw = LayerWeights(None, None, None, None, w_gate_up=up, w_down=down, plain_act="gelu")
    dec = SimpleNamespace(cfg=SimpleNamespace(mlp_kind="glu"), ops=ops, defer_to_residual=False)
    want = O.gelu(d64(h) @ d64(up).t()) @ d64(down).t()
    assert rel(Decoder._ffn_block(dec, lw, h), want) < (2e-6 if dtype == torch.float32 else 6e-3)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", list(S.CONFIGS))
def test_model_over_schedules(name, f32):
    """One prompt at once, token by token through captured graphs, and in portions around pages, windows and tiles; every request
    reuses the pages and state rows of the one before it."""
    cfg, w, toks, want = S.expected(name, 140, 2, not f32)
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
    cfg, w, toks, want = S.expected("odd", 600, 5, not f32)
    rp = S.TraceReplay(S.engine(cfg, w, DEV, f32, blocks=38, max_len=608, chunk=608))
    assert S.error(S.feed(rp, "a", toks, []), want) < TOL[f32]
    assert S.error(S.feed(rp, "b", toks, range(400, 600)), want) < TOL[f32]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("name", ["odd", "tensor-cores"])
def test_mixed_batches_match_each_alone(name, f32):
    cfg = S.CONFIGS[name]
    w = S.tensors(cfg, 0, not f32)
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
    """Greedy text of unequal requests with chunked prompts, graphs and launch-ahead steps, in a pool whose pages behind the
    windows come free on the way: each token is the oracle's best one within the precision; long decoding included."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg, 0, not f32)
    eng = S.engine(cfg, w, DEV, f32, chunk=32, seqs=3, spare=8, blocks=24, max_len=256)
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


@pytest.mark.parametrize("f32", [True, False])
def test_captured_steps_with_padding_rows(f32):
    """Requests that end one after another behind their windows: the captured steps of four rows hold more and more padding, whose
    results stay finite and leave the other rows alone."""
    cfg = S.CONFIGS["odd"]
    w = S.tensors(cfg, 0, not f32)
    eng = S.engine(cfg, w, DEV, f32, chunk=64, seqs=4, spare=8, blocks=40, max_len=256, graph_buckets=[4])
    build, widths = eng._build_batch, []

    def watched(step, pad_to=0, slot=0):
        b = build(step, pad_to=pad_to, slot=slot)
        if pad_to:
            widths.append(len(step.seqs))
            assert b.block_tables[len(step.seqs):, 0].tolist() == [0] * (pad_to - len(step.seqs))
        return b

    eng._build_batch = watched
    prompts = [S.prompt(cfg, n, n) for n in (40, 90, 50, 70)]
    reqs = [eng.requests[eng.add_request(p, SamplingParams(max_tokens=12 + 9 * k, ignore_eos=True))] for k, p in enumerate(prompts)]
    while not all(r.finish_reason for r in reqs):
        eng.step()
        for g in eng._graphs.values():
            assert torch.isfinite(g.logits).all()
    assert set(widths) >= {1, 2, 3, 4} and eng.ops.check_status() == 0
    for p, r in zip(prompts, reqs):
        lg = O.forward(cfg, w, p + list(r.output))[len(p) - 1:-1]
        gap = (lg.max(-1).values - lg.gather(1, torch.tensor(list(r.output))[:, None])[:, 0]) / (lg.max(-1).values - lg.min(-1).values)
        assert float(gap.max()) < (1e-4 if f32 else 0.05)


@pytest.mark.parametrize("E,k", [(5, 3), (8, 8), (60, 6), (256, 8)])
def test_routes_of_rows_that_are_not_numbers(ops, E, k):
    """Scores that are NaN or infinite still give k different experts of the layer, and the other rows do not notice."""
    z = torch.randn(9, E, device=DEV, generator=gen(E))
    clean = z.clone()
    z[1], z[3], z[5, : E // 2], z[7] = float("nan"), float("-inf"), float("nan"), float("inf")
    bad = [1, 3, 5, 7]
    good = [i for i in range(9) if i not in bad]

    def run(call, x):
        ids, wts = torch.empty(9, k, dtype=torch.int32, device=DEV), torch.empty(9, k, device=DEV)
        call(x, ids, wts)
        return ids, wts

    calls = [lambda x, i, w: ops.k.moe_route(x.bfloat16(), None, k, False, i, w), lambda x, i, w: ops.k.moe_route(x.bfloat16(), None, k, True, i, w),
             lambda x, i, w: ops.k.moe_route_scored(x.bfloat16(), None, k, 1, True, 1.0, i, w),
             lambda x, i, w: ops.k.moe_route_scored(x.bfloat16(), None, k, 2, True, 1.0, i, w),
             lambda x, i, w: ops.k.moe_route_fp32(x, None, 0, E, E, k, 1, False, 1.0, i, w, None, 1, 1, float("-inf"), None)]
    for call in calls:
        (ids, wts), (ids0, wts0) = run(call, z), run(call, clean)
        assert int(ids.min()) >= 0 and int(ids.max()) < E and all(len(set(r)) == k for r in ids.tolist())
        assert torch.equal(ids[good], ids0[good]) and torch.equal(wts[good], wts0[good])


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
