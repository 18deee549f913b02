"""Dorevik on a GPU: each mechanism's kernel alone against the functions of tests/dorevik_oracle.py, then whole models in fp32
and bf16 over portions, mixed batches, captured decode steps and the scheduler."""
import json
import math
import os
import subprocess
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import dorevik_cases as S
import dorevik_oracle as O
from fllm_b200.config import MoeSpec
from fllm_b200.ops.maps import Combine, NormedPair, maps_width
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


# ------------------------------------------------------------------------------------------------ residual
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ld", [(64, 64), (75, 80), (13, 16), (2048, 2048), (4100, 4104), (9000, 9000)])
def test_residual_of_a_normed_pair(ops, width, ld, dtype):
    g, T, eps = gen(width), 9, 1e-3
    mk = lambda *s: pad(torch.randn(*s, width, device=DEV, generator=g), ld).to(dtype)
    a, b, wa, wb, w, wf = mk(T), mk(T) * 5, mk(), mk(), mk(), mk()
    cut = lambda t: d64(t)[..., :width]
    x = pad(torch.randn(T, width, device=DEV, generator=g), ld)
    y = (O.rms(cut(a), eps) * cut(wa) + O.rms(cut(b), eps) * cut(wb)) / 2
    for add in (True, False):
        want = cut(x) + O.rms(y, eps) * cut(w) if add else O.rms(1.5 * cut(x) + y, eps) * cut(w)
        before = x.clone()
        h = ops.postnorm_step(x, NormedPair(a, b, wa, wb), w, width, eps, 1.5, add, wf, 0.5, ints([8, 0, 3]))
        assert rel(h[:, :width], (O.rms(want, eps) * cut(wf) * 0.5)[[8, 0, 3]]) < (2e-6 if dtype == torch.float32 else 4e-3) and torch.equal(before, x)
        h = ops.postnorm_step(x, NormedPair(a, b, wa, wb), w, width, eps, 1.5, add)
        assert rel(x[:, :width], want) < 2e-6 and rel(h[:, :width], want) < (2e-6 if dtype == torch.float32 else 4e-3) and not x[:, width:].any()


def test_consumers_take_split_k_partial_sums(ops):
    """A projection whose split-K reduction is left to the kernel behind it: the pair's second half, and the attention inputs."""
    g, T, K, N = gen(1), 8, 4096, 512
    h = torch.randn(T, K, device=DEV, generator=g).bfloat16()
    w = (torch.randn(N, K, device=DEV, generator=g) * K ** -0.5).bfloat16()
    bias = torch.randn(N, device=DEV, generator=g).bfloat16()
    y = d64(h) @ d64(w).t()

    def deferred(b=None):
        p = ops.linear(h, w, b, defer=True)
        assert not isinstance(p, torch.Tensor)
        return p
    one, a, x = torch.ones(N, device=DEV, dtype=torch.bfloat16), torch.randn(T, N, device=DEV, generator=g).bfloat16(), torch.randn(T, N, device=DEV, generator=g)
    want = d64(x) + O.rms((O.rms(d64(a), 1e-5) + O.rms(y, 1e-5)) / 2, 1e-5)
    ops.postnorm_step(x, NormedPair(a, deferred(), one, one), one, N, 1e-5, 1.0, True)
    assert rel(x, want) < 1e-5
    kc, vc = torch.zeros(2, 2, 16, 64, device=DEV, dtype=torch.bfloat16), torch.zeros(2, 1, 16, 128, device=DEV, dtype=torch.bfloat16)
    qn, inv = torch.ones(64, device=DEV, dtype=torch.bfloat16), torch.zeros(8, device=DEV)
    yb = y + d64(bias)
    for full in (False, True):
        norms = [torch.ones(n, device=DEV, dtype=torch.bfloat16) for n in ((256, 128) if full else (64, 64))]
        q = ops.maps_prepare(deferred(bias), (0, 256, 384), 4, 64, 100, ints(list(range(8))), ints(list(range(16, 24))), inv, 1.0, *norms, full, 1e-5, kc, vc)
        group = (lambda t: O.rms(t, 1e-5)) if full else (lambda t: O.rms(t.view(T, -1, 64), 1e-5).view(T, -1))
        assert rel(q.view(T, 256), group(yb[:, :256])) < 4e-3 and rel(kc[1, :, :8].transpose(0, 1).reshape(T, 128), group(yb[:, 256:384])) < 4e-3
        assert rel(vc[1, 0, :8, :100], yb[:, 384:484]) < 4e-3 and not vc[1, 0, :, 100:].any()


# ------------------------------------------------------------------------------------------------ attention of one or two maps
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("full", [False, True])
@pytest.mark.parametrize("H,G,M,dim,v_dim,rot", [(4, 2, 2, 20, 28, 10), (3, 1, 1, 64, 128, 64), (2, 2, 2, 128, 64, 32), (1, 1, 1, 7, 5, 2), (2, 1, 2, 140, 9, 140), (16, 4, 1, 128, 128, 128)])
def test_queries_and_cache_rows(ops, H, G, M, dim, v_dim, rot, full, dtype):
    from fllm_b200.config import RopeScaling, scaled_inv_freq
    g, T, eps = gen(dim), 8, 1e-3
    spec = dict(base=700.0, dims=rot, scaling=dict(factor=3.0, original=90, fast=4.0, slow=0.5))
    inv, factor = scaled_inv_freq(rot, 700.0, RopeScaling("yarn", 3.0, original_max_position=90, beta_fast=4.0, beta_slow=0.5))
    p8 = lambda n: (n + 7) // 8 * 8
    nq, nk = p8(H * M * dim), p8(G * M * dim)
    x = torch.randn(T, nq + nk + G * v_dim + 3, device=DEV, generator=g).to(dtype)
    if G * v_dim % 8 == 0:
        x = x[:, :nq + nk + G * v_dim].contiguous()
    pos, slots = [0, 1, 98, 99, 100, 5000, 3, 0], [3, 17, 4, 60, 33, 32, 31, -1]
    Wk, Wv = maps_width(dim), maps_width(v_dim)
    kc, vc = torch.full((4, G * M, 16, Wk), 7.0, device=DEV, dtype=dtype), torch.full((4, G, 16, Wv), 7.0, device=DEV, dtype=dtype)
    wq, wk = ((torch.randn(n * dim if full else dim, device=DEV, generator=g) * 0.3 + 1).to(dtype) for n in (H * M, G * M))
    q = ops.maps_prepare(x, (0, nq, nq + nk), H * M, dim, v_dim, ints(pos), ints(slots), torch.tensor(inv, device=DEV), factor, wq, wk, full, eps, kc, vc)

    def want(off, n, w):
        t = d64(x)[:, off:off + n * dim]
        t = (O.rms(t, eps) * d64(w)).view(T, n, dim) if full else O.rms(t.view(T, n, dim), eps) * d64(w)
        return torch.stack([torch.cat([O.rotate(t[i:i + 1, j], spec, pos[i]) for j in range(n)]) for i in range(T)])
    tol = 5e-5 if dtype == torch.float32 else 4e-3                  # (an fp32 angle of some thousand radians)
    assert rel(q[:, :, :dim], want(0, H * M, wq)) < tol and not q[:, :, dim:].any()
    k = want(nq, G * M, wk)
    for t, s in enumerate(slots[:-1]):
        assert rel(kc[s // 16, :, s % 16, :dim], k[t]) < tol and not kc[s // 16, :, s % 16, dim:].any()
        assert torch.equal(vc[s // 16, :, s % 16, :v_dim].flatten(), x[t, nq + nk:nq + nk + G * v_dim]) and not vc[s // 16, :, s % 16, v_dim:].any()
    assert int((kc == 7).all(-1).sum()) == (64 - 7) * G * M and int((vc == 7).all(-1).sum()) == (64 - 7) * G


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


def dense(q, kc, vc, tab, starts, lens, ctxs, H, G, M, dim, v_dim, scale, window, combine, bs=16):
    """Softmax over the visible rows of every token, in fp64."""
    q, kc, vc = (d64(t) for t in (q, kc, vc))
    out = torch.zeros(q.shape[0], H * v_dim, dtype=torch.float64)
    for i, (n, c) in enumerate(zip(lens, ctxs)):
        idx, off = tab[i][torch.arange(c) // bs].long(), torch.arange(c) % bs
        rows = slice(starts[i], starts[i] + n)
        for h in range(H):
            g = h // (H // G)
            v = vc[idx, g, off, :v_dim]
            a = [O.attend(q[rows, h * M + m, :dim], kc[idx, g * M + m, off, :dim], v, scale, window or c) for m in range(M)]
            out[rows, h * v_dim:(h + 1) * v_dim] = O.differential(a[0], a[1], combine.lam, 1 - combine.out_scale, combine.eps) if M == 2 else a[0]
    return out


SHAPES = [(8, 2, 2, 64, 128), (8, 2, 1, 128, 64), (12, 1, 2, 128, 128), (3, 3, 1, 24, 20), (4, 4, 2, 50, 60), (20, 1, 2, 40, 96), (40, 2, 1, 64, 64), (5, 1, 1, 128, 100),
          (2, 1, 2, 136, 72), (4, 2, 1, 16, 200), (1, 1, 2, 8, 1)]
BATCHES = [([1, 1, 1], [1, 40, 129]), ([5, 1, 23], [5, 17, 60]), ([70], [133]), ([1], [700]), ([150, 1, 130], [150, 300, 400])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,M,dim,v_dim", SHAPES)
@pytest.mark.parametrize("lens,ctxs", BATCHES)
def test_attention(ops, H, G, M, dim, v_dim, lens, ctxs, dtype):
    g = gen(H + dim)
    b, tab, nb, starts = batch(lens, ctxs)
    mk = lambda n, d: pad(torch.randn(nb, n, 16, d, device=DEV, generator=g), maps_width(d)).to(dtype)
    kc, vc = mk(G * M, dim), mk(G, v_dim)
    q = pad(torch.randn(starts[-1], H * M, dim, device=DEV, generator=g), maps_width(dim)).to(dtype)
    scale, c = 2 / math.sqrt(dim), Combine(0.37, 0.6, 1e-4)
    for window in (0, 17, 50, 128) if dtype == torch.bfloat16 else (0, 50):
        want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, M, dim, v_dim, scale, window, c)
        tol = 5e-6 if dtype == torch.float32 else 4e-3
        assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, c), want) < tol, window
        if dtype == torch.bfloat16:
            assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, c, tensor_cores=False), want) < tol, window
            for splits in (2, 5):
                assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, window, c, splits=splits), want) < tol, (window, splits)
    y = ops.attention_maps(q, kc, vc, dim, v_dim, b, scale, 17, c, H * v_dim + 8)           # padded columns are zero
    assert y.shape[1] == H * v_dim + 8 and not y[:, H * v_dim:].any()
    assert int(ops.status.item()) == 0


@pytest.mark.parametrize("M", [1, 2])
@pytest.mark.parametrize("block_size", [32, 48])
def test_attention_with_larger_blocks(ops, block_size, M):
    H, G, dim, v_dim, lens, ctxs, g = 8, 2, 64, 128, [100, 1], [130, 200], gen(5)
    b, tab, nb, starts = batch(lens, ctxs, block_size)
    kc, vc = (torch.randn(nb, n, block_size, d, device=DEV, generator=g).bfloat16() for n, d in ((G * M, dim), (G, v_dim)))
    q, c = torch.randn(101, H * M, dim, device=DEV, generator=g).bfloat16(), Combine(0.5, 0.5, 1e-5)
    for window in (0, 70):
        want = dense(q, kc, vc, tab, starts, lens, ctxs, H, G, M, dim, v_dim, 0.3, window, c, block_size)
        assert rel(ops.attention_maps(q, kc, vc, dim, v_dim, b, 0.3, window, c), want) < 4e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 2])
@pytest.mark.parametrize("lens,ctx", [([1], 400), ([200], 400)])
def test_single_keys_at_every_border(ops, lens, ctx, M, dtype):
    """One key's score stands far out in one map: that map's output is the key's value wherever it lies inside the window (first
    tokens, page and tile borders, the query's own position, the window's first token), and not one token outside it."""
    H, G, dim, v_dim, n = 4, 2, 64, 64, lens[0]
    b, tab, nb, starts = batch(lens, [ctx], seed=4)
    g = gen(3)
    kc = torch.randn(nb, G * M, 16, dim, device=DEV, generator=g) * 0.1
    vc, q = torch.randn(nb, G, 16, v_dim, device=DEV, generator=g), torch.randn(n, H * M, dim, device=DEV, generator=g)
    seen = 0
    for window in (0, 1, 16, 33, 128, 200):
        for t in sorted({0, n // 2, n - 1}):
            i = ctx - n + t
            places = {0, 1, 15, 16, 127, 128, 129, i, i + 1, i - window, i - window + 1, i - window - 1, i - window + 2, (i - window + 1) // 16 * 16}
            for place in sorted(x for x in places if 0 <= x < ctx):
                for m in range(M):
                    key, block, at = q[t, 3 * M + m] * 3, int(tab[0, place // 16]), place % 16          # query t, head 3, map m
                    cache = kc.clone()
                    cache[block, M + m, at] = key
                    got = ops.attention_maps(q.to(dtype), cache.to(dtype), vc.to(dtype), dim, v_dim, b, 1.0, window, Combine(1e-6 if m == 0 else 1e6, 1.0, 0.0))
                    got, value = got[t, 3 * v_dim:].float(), vc[block, 1, at] * (1 - 2 * m)
                    near = float(torch.nn.functional.cosine_similarity(got, value, 0))
                    inside = place <= i and (window == 0 or i - place < window)
                    seen += inside
                    assert near > 0.999 if inside else near < 0.9, (window, t, place, m)
    assert seen >= 20


# ------------------------------------------------------------------------------------------------ lightning attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V,K", [(4, 13, 20), (1, 8, 8), (3, 40, 16), (4, 24, 64), (2, 64, 128), (2, 20, 256), (3, 300, 100), (16, 128, 128), (2, 7, 32), (1, 1, 1), (2, 64, 32), (60, 40, 72)])
@pytest.mark.parametrize("chunks", [0, 32, 2])
def test_decay_scan(ops, H, V, K, dtype, chunks):
    """Ragged steps that continue each other: prompts, portions of 2 .. 130 tokens and single tokens, rows of the pool in any order;
    token by token, in matrix form from 32 tokens on, and in matrix form down to portions of two tokens."""
    if chunks and (dtype == torch.float32 or K % 8 or V % 8 or K > 128):
        pytest.skip("sizes and types of the token-by-token form")
    g = gen(K)
    lens, slots = [245, 170, 3], [2, 0, 4]
    p8 = lambda n: (n + 7) // 8 * 8
    ok, ov = p8(H * K), 2 * p8(H * K)
    rows = [torch.randn(n, ov + p8(H * V), device=DEV, generator=g).to(dtype) for n in lens]
    decay = torch.tensor([0.999, 0.004, 0.6, 1.0, 0.03][:H] + [0.97] * (H - 5), device=DEV)
    state = torch.full((6, H, V, K), 9.0, device=DEV)                  # stale rows of earlier requests
    got, at = [[] for _ in lens], [0, 0, 0]
    for take in ([17, 2, 1], [0, 33, 1], [1, 1, 1], [1, 1, 0], [96, 133, 0], [130, 0, 0]):
        part = [(i, n) for i, n in enumerate(take) if n]
        x = torch.cat([rows[i][at[i]:at[i] + n] for i, n in part])
        qs = ints([sum(n for _, n in part[:j]) for j in range(len(part) + 1)])
        pos = ints([p for i, n in part for p in range(at[i], at[i] + n)])
        many = [n for _, n in part] if chunks else [0]
        y = ops.decay_scan(x[:, :H * K], x[:, ok:ok + H * K], x[:, ov:ov + H * V], decay, state, qs, ints([slots[i] for i, _ in part]), pos, H, K, V, H * V + 4,
                           max(many), min(many), chunks)
        assert not y[:, H * V:].any()
        for j, (i, n) in enumerate(part):
            got[i].append(y[int(qs[j]):int(qs[j + 1]), :H * V])
            at[i] += n
    for i, n in enumerate(lens):
        x = O.silu(d64(rows[i]))
        cut = lambda o, w, h: x[:, o + h * w:o + (h + 1) * w]
        want = [O.decayed_sum(cut(0, K, h), cut(ok, K, h), cut(ov, V, h), d64(decay)[h]) for h in range(H)]
        assert rel(torch.cat(got[i]), torch.cat([y for y, _ in want], 1)) < (2e-6 if dtype == torch.float32 else 4e-3)
        # fp32 in both modes (in matrix form the activations are bf16 operands)
        assert rel(state[slots[i]], torch.stack([s.t() for _, s in want])) < (4e-3 if chunks else 2e-6)
    assert bool((state[[1, 3, 5]] == 9).all())


def test_chunks_keep_the_precision_of_the_state(ops):
    """1000 tokens in matrix form against the recurrence on the same bf16 activations: the state has fp32 precision, the outputs
    that of their own rounding; decays from hardly to at once."""
    H, V, K, n, g = 5, 40, 72, 1000, gen(9)
    x = torch.randn(n, 2 * H * K + H * V, device=DEV, generator=g).bfloat16()
    decay, state = torch.tensor([0.9999, 0.99, 0.7, 0.01, 1.0], device=DEV), torch.zeros(2, H, V, K, device=DEV)
    q, k, v = x[:, :H * K], x[:, H * K:2 * H * K], x[:, 2 * H * K:]
    for t0, t1 in ((0, 500), (500, 502), (502, 1000)):
        y = ops.decay_scan(q[t0:t1], k[t0:t1], v[t0:t1], decay, state, ints([0, t1 - t0]), ints([1]), ints(list(range(t0, t1))), H, K, V, 0, t1 - t0, t1 - t0, 2)
        x[t0:t1, :H * V] = y                                            # (the activations replaced q, k and v; the outputs go over q)
    f = d64(torch.cat([k, v], 1))                                       # bf16 activations
    for h in range(H):
        kh, vh = f[:, h * K:(h + 1) * K], f[:, H * K + h * V:H * K + (h + 1) * V]
        _, S = O.decayed_sum(torch.zeros_like(kh), kh, vh, d64(decay)[h])
        assert rel(state[1, h], S.t()) < 3e-6, h
    assert not state[0].any()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decayed_state_over_long_decoding(ops, dtype):
    """600 single tokens after a prompt: the state keeps its precision."""
    H, V, K, g = 2, 16, 24, gen(7)
    x = torch.randn(640, 2 * H * K + H * V, device=DEV, generator=g).to(dtype)
    decay, state, out, lo = torch.tensor([0.9995, 0.7], device=DEV), torch.zeros(1, H, V, K, device=DEV), [], 0
    for m in [40] + [1] * 600:
        r = x[lo:lo + m]
        out.append(ops.decay_scan(r[:, :H * K], r[:, H * K:2 * H * K], r[:, 2 * H * K:], decay, state, ints([0, m]), ints([0]), ints(list(range(lo, lo + m))), H, K, V))
        lo += m
    v = O.silu(d64(x))
    want = torch.cat([O.decayed_sum(v[:, h * K:(h + 1) * K], v[:, (H + h) * K:(H + h + 1) * K], v[:, 2 * H * K + h * V:2 * H * K + (h + 1) * V], d64(decay)[h])[0]
                      for h in range(H)], 1)
    assert rel(torch.cat(out), want) < (3e-6 if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,width", [(36, 40), (2048, 2048), (13, 16), (600, 600)])
def test_norm_before_a_sigmoid_gate(ops, D, width, dtype):
    g = gen(D)
    y, z, w = (torch.randn(*s, device=DEV, generator=g).to(dtype) for s in ((6, D), (6, D + 4), (D,)))
    got = ops.gated_rmsnorm(y, z[:, :D], w, 1e-3, D, True, width, "sigmoid")
    assert rel(got[:, :D], O.rms(d64(y), 1e-3) * d64(w) * O.sigmoid(d64(z)[:, :D])) < (1e-6 if dtype == torch.float32 else 4e-3) and not got[:, D:].any()


# ------------------------------------------------------------------------------------------------ feed-forward, head
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,shared", [(1, 64, 6, 2, 32, 48), (37, 200, 12, 1, 48, 0), (300, 256, 7, 7, 16, 32), (64, 128, 40, 5, 32, 64), (5, 24, 1, 1, 16, 16), (6, 64, 300, 9, 16, 0)])
def test_routed_experts_weigh_their_input(ops, T, W, E, top, ff, shared, dtype):
    from fllm_b200.models.decoder import Decoder
    from fllm_b200.models.weights import LayerWeights
    g = gen(E)
    mk = lambda *s, gain=1.0: (torch.randn(*s, device=DEV, generator=g) * gain * s[-1] ** -0.5).to(dtype)
    h = torch.randn(T, W, device=DEV, generator=g).to(dtype)
    lw = LayerWeights(None, None, None, None, router_w=mk(E, W, gain=1.5), exp_gate_up=mk(E, 2 * ff, W), exp_down=mk(E, W, ff),
                      moe=MoeSpec(E, top, "deepseek_v3", weigh_input=True, fp32_router=True))
    w = {"router": d64(lw.router_w)}
    for e in range(E):
        w.update({f"e{e}.gate": d64(lw.exp_gate_up[e, :ff]), f"e{e}.up": d64(lw.exp_gate_up[e, ff:]), f"e{e}.down": d64(lw.exp_down[e])})
    if shared:
        lw.shared_gate_up, lw.shared_down = mk(2 * shared, W), mk(W, shared)
        w.update({"shared.gate": d64(lw.shared_gate_up[:shared]), "shared.up": d64(lw.shared_gate_up[shared:]), "shared.down": d64(lw.shared_down)})
    cfg = SimpleNamespace(mlp_kind="glu", swiglu_alpha=1.0, swiglu_limit=0.0)
    dec = SimpleNamespace(cfg=cfg, ops=ops, spec=SimpleNamespace(expert_parallel=False), ep_a2a=None)
    got = Decoder._ffn_block(dec, lw, h)
    want = O.routed_mlp(d64(h), w, "", dict(router=dict(top=top), shared=shared or None))
    assert rel(got, want) < (3e-6 if dtype == torch.float32 else 8e-3)       # every choice is the oracle's: the logits are fp32 sums


@pytest.mark.parametrize("dtype", DTYPES)
def test_softcap(ops, dtype):
    x = (torch.randn(5, 203, device=DEV, generator=gen(2)) * 20).to(dtype)
    want = 7 * torch.tanh(d64(x) / 7)
    y = pad(x, 204)
    assert rel(ops.softcap_(y, 7.0)[:, :203], want) < (1e-6 if dtype == torch.float32 else 4e-3)


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
