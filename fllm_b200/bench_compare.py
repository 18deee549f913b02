"""Throughput of a design beside the framework's closest other model at equal size (``bench.py --compare
sovanex|divanex|dorevik|milenex``).

The closest other model of Sovanex is a hybrid of the layer kinds it shares with other families: the gated delta rule
(Qwen3-Next) and 512 + 64 wide latent attention (DeepSeek), with the same layer order, heads, widths and squared-ReLU
networks, but RMSNorm around one bf16 residual, no gate on the attention heads and no shared rows. That of Divanex is a
hybrid of Mamba-2 and grouped-query attention with normalised queries and keys and capped scores (Bamba, Gemma-2), the same
layer order, sizes and clamped SwiGLU networks (gpt-oss), but separate values, norms in front of the blocks around one bf16
residual, and no token input. That of Dorevik is a hybrid of windowed grouped-query attention with normalised queries and keys,
of that attention beside Mamba-2 (Falcon-H1) and of routed experts beside a shared one (DeepSeek-V3's router), with the same
layer order and as many weights and products, but one softmax per head, weights on the experts' outputs, and norms in front of
the blocks around one bf16 residual. That of Milenex is a stack of windowed grouped-query attention with sinks and of clamped SwiGLU
networks and experts (gpt-oss) with a shared expert, as many layers as Milenex runs and as many weights in each, but no
convolution, no mixing of heads, no token shift, and one bf16 residual. Both models run random weights through the engine: prompts of 1024 tokens in 2048-token
steps, then captured decode steps. ``--kernels`` times the kernels that differ, each beside its like kernel on the same sizes.
"""
from __future__ import annotations

import dataclasses
import statistics
from typing import Dict, List

import torch

from .config import EngineConfig, ModelConfig, divanex_from_config, dorevik_from_config, milenex_from_config, sovanex_from_config

# name -> width, layers, feed-forward width, value heads / key heads of the delta rule, attention heads
SIZES = {"1b": (2048, 12, 8192, 32, 16, 16), "3b": (3072, 24, 12288, 48, 24, 24), "7b": (4096, 32, 16384, 64, 32, 32)}
VOCAB = 65536


def sovanex_config(size: str) -> ModelConfig:
    W, L, ff, Hv, Hk, Ha = SIZES[size]
    layers = []
    for i in range(L):
        if i % 4 < 3:
            mixer = dict(heads=Hv, kv_heads=Hk, dim=128, vdim=128, conv=4)
        else:
            mixer = dict(heads=Ha, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot=dict(base=1e6, dims=64))
            if i % 8 == 7:
                mixer["kv_from"] = i - 4
        layers.append(dict(type="delta" if i % 4 < 3 else "latent_attention", mixer=mixer, mlp=dict(kind="dense", ff=ff)))
    return sovanex_from_config(ModelConfig, dict(architecture="Sovanex", name=f"sovanex-{size}", layers=layers, norm=dict(eps=1e-5),
                                                 residual_mult=0.25, streams=4, vocab=VOCAB, width=W))


def twin_config(size: str) -> ModelConfig:
    W, L, ff, Hv, Hk, Ha = SIZES[size]
    return ModelConfig(arch="hybrid", name=f"delta-mla-hybrid-{size}", vocab_size=VOCAB, hidden_size=W, num_layers=L, num_heads=Ha, num_kv_heads=1,
                       head_dim=192, rotary_dim=64, rope_style="pair", intermediate_size=ff, mlp_kind="plain", act="relu2", tie_embeddings=True,
                       layer_kinds=["gated_delta" if i % 4 < 3 else "mla" for i in range(L)],
                       ssm=dict(num_k_heads=Hk, num_v_heads=Hv, head_k_dim=128, head_v_dim=128, d_conv=4),
                       mla=dict(q_lora_rank=0, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128))


# name -> width, layers, feed-forward width, Mamba-2 heads (of 64, state 128, 8 groups), query / key heads (of 128), token input
DIVANEX_SIZES = {"1b": (2048, 24, 8192, 64, 16, 4, 256), "3b": (3072, 32, 12288, 96, 24, 6, 256), "7b": (4096, 40, 16384, 128, 32, 8, 256)}


def divanex_config(size: str) -> ModelConfig:
    W, L, ff, Hm, H, G, side = DIVANEX_SIZES[size]
    mamba = dict(heads=Hm, vdim=64, state=128, groups=8, norm_groups=8, conv=4)
    attn = dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, q_temp=dict(coef=0.1, every=8192))
    layers = [dict(type="attention", mixer=attn, mlp=dict(kind="dense", ff=ff, limit=7.0)) if i % 4 == 3 else dict(type="mamba2", mixer=mamba, mlp=None)
              for i in range(L)]
    return divanex_from_config(ModelConfig, dict(architecture="Divanex", name=f"divanex-{size}", layers=layers, norm=dict(eps=1e-5), embedding=dict(scale=4.0),
                                                 postln_alpha=2.0, logit_scale=0.5, token_side=dict(dim=side), vocab=VOCAB, width=W))


def divanex_twin_config(size: str) -> ModelConfig:
    W, L, ff, Hm, H, G, _ = DIVANEX_SIZES[size]
    return ModelConfig(arch="hybrid", name=f"mamba2-gqa-hybrid-{size}", vocab_size=VOCAB, hidden_size=W, num_layers=L, num_heads=H, num_kv_heads=G, head_dim=128,
                       use_rope=False, qk_norm=True, attn_softcap=30.0, intermediate_size=ff, act="swiglu_oai", tie_embeddings=False,
                       layer_kinds=["attention" if i % 4 == 3 else "mamba2" for i in range(L)], ffn_kinds=["glu" if i % 4 == 3 else "none" for i in range(L)],
                       ssm=dict(d_inner=Hm * 64, d_state=128, d_conv=4, n_groups=8, head_dim=64, n_heads=Hm, norm_groups=8, conv_bias=True, dt_min=0.0,
                                dt_max=1e30))


# name -> width, layers, feed-forward width, query / key heads (values of 128; differential: two maps of 64), experts, their width, shared
# width, tokens of every window
DOREVIK_SIZES = {"1b": (2048, 16, 6144, 16, 4, 32, 768, 1536, 1024), "3b": (3072, 20, 9216, 24, 6, 32, 1024, 2048, 1024),
                 "7b": (4096, 24, 12288, 32, 8, 32, 1536, 3072, 1024)}
DOREVIK_TOP = 4


def dorevik_config(size: str) -> ModelConfig:
    W, L, ff, H, G, E, fe, fs, window = DOREVIK_SIZES[size]
    rot = lambda n: dict(base=1e6, dims=n)
    diff = dict(heads=H, kv_heads=G, dim=64, vdim=128, scale=64 ** -0.5, diff=0.7, mask=dict(size=window), rot=rot(64))
    left = dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=window), rot=rot(128))
    right = dict(heads=H, dim=128, vdim=128, decay=[1 - 2.0 ** (-3 - 6 * i / H) for i in range(H)])
    moe = dict(kind="moe", expert=dict(ff=fe), router=dict(experts=E, top=DOREVIK_TOP), shared=dict(ff=fs))
    layers = [dict(type="parallel" if i % 4 == 3 else "attention", mixer=dict(left=left, right=right) if i % 4 == 3 else diff,
                   mlp=moe if i % 2 else dict(kind="dense", ff=ff)) for i in range(L)]
    return dorevik_from_config(ModelConfig, dict(architecture="Dorevik", name=f"dorevik-{size}", layers=layers, norm=dict(eps=1e-6), logit_softcap=30.0,
                                                 vocab=VOCAB, width=W))


def dorevik_twin_config(size: str) -> ModelConfig:
    W, L, ff, H, G, E, fe, fs, window = DOREVIK_SIZES[size]
    return ModelConfig(arch="hybrid", name=f"gqa-mamba2-moe-hybrid-{size}", vocab_size=VOCAB, hidden_size=W, num_layers=L, num_heads=H, num_kv_heads=G,
                       head_dim=128, rope_theta=1e6, qk_norm=True, sliding_window=window, intermediate_size=ff, act="swiglu", tie_embeddings=False,
                       logit_softcap=30.0, num_experts=E, experts_per_token=DOREVIK_TOP, moe_intermediate_size=fe, shared_intermediate_size=fs,
                       router_kind="deepseek_v3", layer_kinds=["attention+mamba2" if i % 4 == 3 else "attention" for i in range(L)],
                       ffn_kinds=["moe" if i % 2 else "glu" for i in range(L)],
                       ssm=dict(d_inner=H * 128, d_state=128, d_conv=4, n_groups=H, head_dim=64, n_heads=2 * H, norm_groups=1, conv_bias=True, dt_min=0.0, dt_max=1e30))


# name -> width, layers (the first quarter runs twice), feed-forward width of two matrices, query / key heads (of 128, values of 64 in the
# talking-heads layers), experts (in 8 groups, the best 4 kept), their width, shared width, tokens of every window
MILENEX_SIZES = {"1b": (2048, 12, 9216, 16, 4, 32, 768, 1536, 1024), "3b": (3072, 16, 13824, 24, 6, 32, 1024, 2048, 1024),
                 "7b": (4096, 20, 18432, 32, 8, 32, 1536, 3072, 1024)}
MILENEX_TOP = 4


def milenex_config(size: str) -> ModelConfig:
    W, L, ff, H, G, E, fe, fs, window = MILENEX_SIZES[size]
    heads = dict(heads=H, kv_heads=G, dim=128, scale=128 ** -0.5, mask=dict(size=window))
    rotary, talking = dict(heads, vdim=128, conv=4, rot=dict(base=1e6, dims=128)), dict(heads, vdim=64)
    moe = dict(kind="moe", expert=dict(ff=fe, limit=7.0), router=dict(experts=E, top=MILENEX_TOP, groups=dict(count=8, keep=4)), shared=dict(ff=fs, limit=7.0))
    layers = [dict(type="attention" if i % 4 in (1, 2) else "attention_2", mixer=rotary if i % 4 in (1, 2) else talking, mlp=moe if i % 2 else dict(kind="dense", ff=ff))
              for i in range(L)]
    return milenex_from_config(ModelConfig, dict(architecture="Milenex", name=f"milenex-{size}", layers=layers, loop=dict(start=0, stop=L // 4, times=2),
                                                 norm=dict(eps=1e-6), vocab=VOCAB, width=W))


def milenex_twin_config(size: str) -> ModelConfig:
    W, L, ff, H, G, E, fe, fs, window = MILENEX_SIZES[size]
    order = milenex_config(size).layer_source
    return ModelConfig(arch="hybrid", name=f"gqa-sink-moe-{size}", vocab_size=VOCAB, hidden_size=W, num_layers=len(order), num_heads=H, num_kv_heads=G, head_dim=128,
                       rope_theta=1e6, attn_sinks=True, sliding_window=window, intermediate_size=ff * 2 // 3, act="swiglu_oai", tie_embeddings=False, num_experts=E,
                       experts_per_token=MILENEX_TOP, moe_intermediate_size=fe, shared_intermediate_size=fs, router_kind="deepseek_v2",
                       layer_kinds=["attention"] * len(order), ffn_kinds=["moe" if i % 2 else "glu" for i in order])


def throughput(cfg: ModelConfig, batch: int, prompt_len: int, steps: int, warmup: int, device, graphs: bool = True) -> Dict[str, float]:
    """Device-timed prefill and decode of ``batch`` requests (CUDA events around whole engine steps / graph replays)."""
    from .runtime import LLMEngine, SamplingParams
    # sequences that prefill first decode along while the others are still prefilled
    room = batch * prompt_len // 2048 + warmup + steps + 16
    ec = EngineConfig(max_num_seqs=batch, max_num_batched_tokens=2048, max_model_len=prompt_len + room, enable_prefix_caching=False, use_cuda_graphs=graphs)
    ec.num_kv_blocks = batch * (-(-ec.max_model_len // ec.block_size)) * 11 // 10 + 16
    eng = LLMEngine(cfg, ec, device=device)
    g = torch.Generator().manual_seed(7)
    prompts = [torch.randint(0, cfg.vocab_size, (prompt_len,), generator=g).tolist() for _ in range(batch)]
    sp = SamplingParams(max_tokens=room, ignore_eos=True)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    eng.generate(prompts[:8], dataclasses.replace(sp, max_tokens=2))          # warm-up of both step kinds, and of the allocator
    for p in prompts:
        eng.add_request(p, sp)
    torch.cuda.synchronize()
    e0.record()
    while any(not r.output for r in eng.requests.values()):
        eng.step()
    e1.record()
    torch.cuda.synchronize()
    prefill = batch * prompt_len / (e0.elapsed_time(e1) / 1e3)
    for _ in range(warmup):
        eng.step()
    eng.drain()
    graph = eng._graphs[eng._bucket_for(batch)]
    step = eng.scheduler.schedule()
    eng._build_batch(step, pad_to=graph.bucket)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(steps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    status = eng.ops.check_status()
    launches = graph.launches
    eng.close()
    del eng, graph
    torch.cuda.empty_cache()
    return {"prefill_tok_s": round(prefill, 1), "decode_tok_s": round(batch / (ms / 1e3), 1), "decode_ms": round(ms, 4), "launches_per_step": launches,
            "status": status}


# ------------------------------------------------------------------------------------------------ kernels
def _time(fn, flush, n: int = 15) -> float:
    """Median microseconds with a cold L2 (CUDA events on the launching stream)."""
    for _ in range(3):
        fn()
    out = []
    for _ in range(n):
        flush.zero_()
        torch.cuda._sleep(200000)                  # the host queues the launch while the device is busy
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b) * 1e3)
    return statistics.median(out)


def _batch(lens: List[int], ctxs: List[int], device, bs: int = 16):
    from types import SimpleNamespace
    B, mb = len(lens), max(-(-c // bs) for c in ctxs)
    i32 = lambda t: t.to(device=device, dtype=torch.int32)
    tab = torch.randperm(B * mb).view(B, mb)
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    pos = torch.cat([torch.arange(c - n, c) for n, c in zip(lens, ctxs)])
    slots = torch.cat([tab[i, torch.arange(c - n, c) // bs] * bs + torch.arange(c - n, c) % bs for i, (n, c) in enumerate(zip(lens, ctxs))])
    return SimpleNamespace(num_seqs=B, max_q_len=max(lens), max_kv_len=max(ctxs), positions=i32(pos), slots=i32(slots), blocks=B * mb,
                           row_seq=i32(torch.cat([torch.full((n,), i) for i, n in enumerate(lens)])), block_tables=i32(tab),
                           q_starts=i32(torch.tensor(starts)), seq_state=i32(torch.arange(B)), tokens=starts[-1])


class _Table:
    """Rows of kernels beside their like kernels: microseconds, the floor of each (bytes at the measured copy bandwidth or
    products at the measured GEMM rate, whichever is longer), and the ratio of the two distances."""

    def __init__(self, device):
        import json
        import os
        from .ops.native import NativeOps
        self.ops, self.device, self.rows = NativeOps(device), device, []
        self.gen = torch.Generator(device=device).manual_seed(1)
        self.peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
        path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
        if os.path.exists(path):
            self.peaks.update({k: v for k, v in json.load(open(path)).items() if k in self.peaks})
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=device)

    def rnd(self, *shape, dtype=torch.bfloat16):
        return torch.randn(*shape, device=self.device, generator=self.gen).to(dtype)

    def time(self, fn) -> float:
        return _time(fn, self.flush)

    def floor(self, nbytes, flops=0.0) -> float:
        return max(nbytes / self.peaks["hbm_gbs"] / 1e3, flops / self.peaks["bf16_tflops"] / 1e6)

    def add(self, shape, name, us, fl, like, like_us, like_fl) -> None:
        self.rows.append({"shape": shape, "kernel": name, "us": round(us, 1), "floor_us": round(fl, 2), "like": like, "like_us": round(like_us, 1),
                          "like_floor_us": round(like_fl, 2), "times_as_far": round((us / fl) / (like_us / like_fl), 2)})


def sovanex_kernels(device, size: str = "1b") -> List[dict]:
    tab = _Table(device)
    ops, rnd, floor, add = tab.ops, tab.rnd, tab.floor, tab.add
    bf = torch.bfloat16
    W, _, ff, Hv, Hk, H = SIZES[size]
    R, dr, dn, S = 512, 64, 128, 4
    for shape, lens, ctxs in (("decode 64 x 1152", [1] * 64, [1152] * 64), ("decode 8 x 4096", [1] * 8, [4096] * 8),
                              ("prompt 2048", [2048], [2048]), ("prompt 4 x 512 at 2048", [512] * 4, [2048] * 4)):
        b = _batch(lens, ctxs, device)
        T = b.tokens
        cache, q = rnd(b.blocks, 16, R + dr), rnd(H, T, R + dr)
        qa, qp = q[:, :, :R].contiguous(), q[:, :, R:].transpose(0, 1).contiguous()
        keys = sum(c * n - n * (n - 1) // 2 for n, c in zip(lens, ctxs))
        fl = floor(2 * (sum(ctxs) * (R + dr) + q.numel() + H * T * R), 2.0 * keys * H * (2 * R + dr))
        add(shape, "attention_latent", tab.time(lambda: ops.attention_latent(q, cache, b, 0.07, R)), fl, "attention_mla",
            tab.time(lambda: ops.attention_mla(qa, qp, cache, b.block_tables, b.row_seq, b.positions, 0.07, b.max_kv_len)), fl)
        ckv, qh, inv, nw = rnd(T, R + dr), rnd(T, H * (dn + dr)), torch.rand(dr // 2, device=device), torch.ones(R, device=device, dtype=bf)
        fl = floor(2 * T * (2 * (R + dr) + 2 * H * dr))
        add(shape, "latent_prepare", tab.time(lambda: ops.latent_prepare(ckv, qh, dn + dr, dn, b.positions, b.slots, inv, 1.0, nw, 1e-5, cache, q, R, 0)), fl,
            "mla_prepare", tab.time(lambda: ops.mla_prepare(ckv, qh.view(T, H, dn + dr), dn, b.positions, b.slots, inv, 1.0, nw, 1e-5, cache)), fl)
    for T in (64, 2048):
        shape = f"{T} rows"
        x, y, res = rnd(T, S, W, dtype=torch.float32), rnd(T, W), rnd(T, W)
        mix, vec, w = torch.eye(S, device=device), torch.ones(S, device=device), torch.ones(W, device=device, dtype=bf)
        add(shape, "streams_step (4 fp32 streams, LayerNorm)", tab.time(lambda: ops.streams_step(x, y, mix, vec, vec, w, w, W, 1e-5)),
            floor(T * W * (8 * S + 4)), "residual add + rmsnorm", tab.time(lambda: ops.rmsnorm(res, y, w, 1e-5)), floor(T * W * 8))
        add(shape, "streams_step (4 fp32 streams, LayerNorm)", tab.time(lambda: ops.streams_step(x, y, mix, vec, vec, w, w, W, 1e-5)),
            floor(T * W * (8 * S + 4)), "residual add + layernorm", tab.time(lambda: ops.layernorm(res, y, w, w, 1e-5)), floor(T * W * 8))
        o, gate = rnd(H, T, 128), rnd(T, H)
        add(shape, "head_gate", tab.time(lambda: ops.head_gate(o, gate, H * 128)), floor(T * H * 512), "transposing copy",
            tab.time(lambda: o.transpose(0, 1).reshape(T, H * 128)), floor(T * H * 512))
        D = 128
        b = _batch([1] * T if T == 64 else [T], [1024] * T if T == 64 else [T], device)
        qkv, gates = rnd(T, (2 * Hk + Hv) * D), rnd(T, 2 * Hv)
        st = torch.zeros(b.num_seqs, Hv, D, D, device=device)
        A, db = -torch.rand(Hv, device=device), torch.zeros(Hv, device=device)
        K = Hk * D
        us = tab.time(lambda: ops.matrix_state_scan(2, qkv[:, :K], qkv[:, K:2 * K], qkv[:, 2 * K:], None, None, None, None, gates[:, :Hv], st, b.q_starts,
                                                 b.seq_state, b.positions, Hv, D, D, Hv // Hk, True, D ** -0.5, gate_raw=gates[:, Hv:], gate_A=A,
                                                 gate_dt_bias=db))
        fl = floor(st.numel() * 8 + 2 * T * ((2 * Hk + 2 * Hv) * D))
        add(shape, "gated delta scan", us, fl, "the same kernel", us, fl)
    return tab.rows


def divanex_kernels(device, size: str = "1b") -> List[dict]:
    tab = _Table(device)
    ops, rnd, floor, bf = tab.ops, tab.rnd, tab.floor, torch.bfloat16
    W, _, ff, Hm, H, G, side = DIVANEX_SIZES[size]
    D = 128
    for shape, lens, ctxs in (("decode 64 x 1152", [1] * 64, [1152] * 64), ("decode 8 x 4096", [1] * 8, [4096] * 8), ("prompt 2048", [2048], [2048]),
                              ("prompt 8192", [8192], [8192]), ("prompt 4 x 512 at 2048", [512] * 4, [2048] * 4)):
        b = _batch(lens, ctxs, device)
        T = b.tokens
        b.min_q_len, b.seq_lens = min(lens), torch.tensor(ctxs, dtype=torch.int32, device=device)
        cache, factor = rnd(b.blocks, G, 16, D), torch.rand(b.blocks, G, 16, device=device) + 0.5
        kc, vc = rnd(b.blocks, G, 16, D), rnd(b.blocks, G, 16, D)
        q, qf = rnd(T, H * D), torch.full((T, H), D ** -0.5, device=device)
        flops = 4.0 * sum(c * n - n * (n - 1) // 2 for n, c in zip(lens, ctxs)) * H * D
        tied, split = floor(sum(ctxs) * G * (2 * D + 4) + 4 * T * H * D, flops), floor(sum(ctxs) * G * 4 * D + 4 * T * H * D, flops)
        us = tab.time(lambda: ops.attention_tied(q, qf, cache, factor, D, b, 30.0))
        for cap in (30.0, 0.0):
            like = tab.time(lambda: ops.attention(q, kc, vc, b.block_tables, b.row_seq, b.positions, H, G, D, D ** -0.5, 0, None, cap, meta=b))
            tab.add(shape, "attention_tied", us, tied, "attention" + (", capped" if cap else ""), like, split)
        if len(lens) == 4:
            continue
        x, w, inv = rnd(T, (H + 2 * G) * D), torch.ones(D, device=device, dtype=bf), torch.zeros(D // 2, device=device)
        tab.add(shape, "tied_prepare", tab.time(lambda: ops.tied_prepare(x, H * D, H, D, b.positions, b.slots, 1e-5, 0.1, 0.1, 8192.0, cache, factor)),
                floor(2 * T * (H + 2 * G) * D), "rope_kv_write",
                tab.time(lambda: ops.rope_kv_write(x, b.positions, b.slots, inv, w, w, kc, vc, H, G, D, D, 0, 1e-5)), floor(2 * T * (2 * H + 4 * G) * D))
    for T in (64, 2048):
        shape = f"{T} rows"
        x, y, res, w = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), torch.ones(W, device=device, dtype=bf)
        norm, norm_fl = tab.time(lambda: ops.rmsnorm(res, y, w, 1e-5)), floor(T * W * 8)
        tab.add(shape, "postnorm, norm of the sum", tab.time(lambda: ops.postnorm_step(x, y, w, W, 1e-5, 2.0)), floor(T * W * 12), "residual add + rmsnorm", norm, norm_fl)
        tab.add(shape, "postnorm, norm of what is added", tab.time(lambda: ops.postnorm_step(x, y, w, W, 1e-5, 1.0, True)), floor(T * W * 12),
                "residual add + rmsnorm", norm, norm_fl)
        gate, gu, table = rnd(T, side), rnd(T, 2 * side), rnd(4096, 4 * side)
        ids = torch.randint(0, 4096, (T,), device=device, generator=tab.gen).int()
        tab.add(shape, "side_gate", tab.time(lambda: ops.side_gate(gate, ids, table, side, side)), floor(6 * T * side), "geglu", tab.time(lambda: ops.glu(gu, 1)),
                floor(6 * T * side))
        b = _batch([1] * T if T == 64 else [T], [1024] * T if T == 64 else [T], device)
        P, N, Gm = 64, 128, 8
        xs, bc, dt = rnd(T, Hm * P), rnd(T, 2 * Gm * N), rnd(T, Hm)
        st, A, Dv = torch.zeros(b.num_seqs, Hm, P, N, device=device), -torch.rand(Hm, device=device), torch.ones(Hm, device=device)
        us = tab.time(lambda: ops.mamba2_scan(xs, dt, bc[:, :Gm * N], bc[:, Gm * N:], A, Dv, Dv, st, b.q_starts, b.seq_state, b.positions, Hm, P, Gm, N))
        fl = floor(st.numel() * 8 + 2 * T * (2 * Hm * P + 2 * Gm * N))
        tab.add(shape, "Mamba-2 scan", us, fl, "the same kernel", us, fl)
    return tab.rows


def dorevik_kernels(device, size: str = "1b") -> List[dict]:
    from .ops.maps import Combine, NormedPair
    tab = _Table(device)
    ops, rnd, floor, bf = tab.ops, tab.rnd, tab.floor, torch.bfloat16
    W, _, ff, H, G, E, fe, fs, _ = DOREVIK_SIZES[size]
    D, K = 128, 64
    for shape, lens, ctxs, windows in (("decode 64 x 1152", [1] * 64, [1152] * 64, (0, 512)), ("decode 8 x 4096", [1] * 8, [4096] * 8, (0, 512)),
                                       ("prompt 2048", [2048], [2048], (0, 512)), ("prompt 8192", [8192], [8192], (0, 1024)),
                                       ("prompt 4 x 512 at 2048", [512] * 4, [2048] * 4, (0, 512))):
        b = _batch(lens, ctxs, device)
        T = b.tokens
        b.min_q_len, b.seq_lens = min(lens), torch.tensor(ctxs, dtype=torch.int32, device=device)
        kc, vc, k2 = rnd(b.blocks, G, 16, D), rnd(b.blocks, G, 16, D), rnd(b.blocks, 2 * G, 16, K)
        q, q1, q2 = rnd(T, H * D), rnd(T, H, D), rnd(T, 2 * H, K)
        for window in windows:
            see = lambda i: min(i + 1, window or i + 1)
            keys = sum(see(i) for n, c in zip(lens, ctxs) for i in range(c - n, c))
            rows = sum(min(c, n + (window or c) - 1) for n, c in zip(lens, ctxs))
            fl = floor(rows * G * 4 * D + 4 * T * H * D, 4.0 * keys * H * D)
            fl2 = floor(rows * G * 4 * D + 4 * T * H * D, 2.0 * keys * H * (2 * K + 2 * D))       # two maps: each weighs all values
            like = tab.time(lambda: ops.attention(q, kc, vc, b.block_tables, b.row_seq, b.positions, H, G, D, D ** -0.5, window, None, 0.0, meta=b))
            at = f"{shape}, window {window}" if window else shape
            tab.add(at, "attention_maps, two maps of 64", tab.time(lambda: ops.attention_maps(q2, k2, vc, K, D, b, K ** -0.5, window, Combine(0.5, 0.3, 1e-6))), fl2,
                    "attention", like, fl)
            tab.add(at, "attention_maps, one map of 128", tab.time(lambda: ops.attention_maps(q1, kc, vc, D, D, b, D ** -0.5, window)), fl, "attention", like, fl)
        if len(lens) == 4:
            continue
        x, w, inv = rnd(T, (H + 2 * G) * D), torch.ones(H * D, device=device, dtype=bf), torch.rand(D // 2, device=device)
        fl = floor(2 * T * (2 * H + 4 * G) * D)
        like = tab.time(lambda: ops.rope_kv_write(x, b.positions, b.slots, inv, w[:D], w[:D], kc, vc, H, G, D, D, 0, 1e-5))
        tab.add(shape, "maps_prepare, norm per map", tab.time(lambda: ops.maps_prepare(x, (0, H * D, (H + G) * D), 2 * H, K, D, b.positions, b.slots, inv[:K // 2], 1.0,
                                                                                   w[:K], w[:K], False, 1e-5, k2, vc)), fl, "rope_kv_write", like, fl)
        tab.add(shape, "maps_prepare, norm over all heads", tab.time(lambda: ops.maps_prepare(x, (0, H * D, (H + G) * D), H, D, D, b.positions, b.slots, inv, 1.0,
                                                                                          w, w[:G * D], True, 1e-5, kc, vc)), fl, "rope_kv_write", like, fl)
    for T in (64, 2048):
        shape = f"{T} rows"
        x, y, y2, res, w = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W), torch.ones(W, device=device, dtype=bf)
        norm, norm_fl = tab.time(lambda: ops.rmsnorm(res, y, w, 1e-5)), floor(T * W * 8)
        tab.add(shape, "postnorm, norm of what is added", tab.time(lambda: ops.postnorm_step(x, y, w, W, 1e-5, 1.0, True)), floor(T * W * 12),
                "residual add + rmsnorm", norm, norm_fl)
        tab.add(shape, "postnorm of a normed pair", tab.time(lambda: ops.postnorm_step(x, NormedPair(y2, y, w, w), w, W, 1e-5, 1.0, True)), floor(T * W * 14),
                "residual add + rmsnorm", norm, norm_fl)
        o, z, wn = rnd(T, H * D), rnd(T, H * D), torch.ones(H * D, device=device, dtype=bf)
        fl = floor(6 * T * H * D)
        tab.add(shape, "norm before a sigmoid gate", tab.time(lambda: ops.gated_rmsnorm(o, z, wn, 1e-5, H * D, True, 0, "sigmoid")), fl, "norm behind a silu gate",
                tab.time(lambda: ops.gated_rmsnorm(o, z, wn, 1e-5, H * D)), fl)
        rw, bias = rnd(E, W), torch.zeros(E, device=device)
        ids, wts = torch.empty(T, DOREVIK_TOP, dtype=torch.int32, device=device), torch.empty(T, DOREVIK_TOP, device=device)

        def routed(fp32):
            z = ops.linear(y, rw, force_splits=2 if fp32 else 0, defer=fp32)
            if fp32:
                ops.k.moe_route_fp32(None, ops.workspace, z.splits, E, E, DOREVIK_TOP, 2, False, 1.0, ids, wts)
            else:
                ops.k.moe_route_scored(z, bias, DOREVIK_TOP, 2, False, 1.0, ids, wts)
        fl = floor(2 * (T * W + E * W))
        tab.add(shape, "router, fp32 logits", tab.time(lambda: routed(True)), fl, "router, bf16 logits", tab.time(lambda: routed(False)), fl)
        n = T * DOREVIK_TOP
        token_of, row_w, xp, row_of = torch.arange(n, device=device).int() // DOREVIK_TOP, torch.rand(n, device=device), rnd(n, W), torch.arange(n, device=device).int().view(T, -1)
        fl = floor(2 * (T + n) * W)
        tab.add(shape, "gather of weighed rows", tab.time(lambda: ops.k.moe_gather(y, token_of, xp, row_w)), fl, "gather", tab.time(lambda: ops.k.moe_gather(y, token_of, xp)), fl)
        tab.add(shape, "combine with the shared expert", tab.time(lambda: ops.k.moe_combine(xp, row_of, None, y2, res)), floor(2 * (2 * T + n) * W), "combine",
                tab.time(lambda: ops.k.moe_combine(xp, row_of, wts, y2)), fl)
        b = _batch([1] * T if T == 64 else [T], [1024] * T if T == 64 else [T], device)
        qkv, dt = rnd(T, 3 * H * D), rnd(T, 2 * H)
        st, A, dec = torch.zeros(b.num_seqs, H, D, D, device=device), -torch.rand(2 * H, device=device), torch.full((H,), 0.99, device=device)
        us = tab.time(lambda: ops.decay_scan(qkv[:, :H * D], qkv[:, H * D:2 * H * D], qkv[:, 2 * H * D:], dec, st, b.q_starts, b.seq_state, b.positions, H, D, D, 0,
                                             b.max_q_len, b.max_q_len))
        st2 = st.view(b.num_seqs, 2 * H, 64, D)
        like = tab.time(lambda: ops.mamba2_scan(qkv[:, 2 * H * D:], dt, qkv[:, H * D:2 * H * D], qkv[:, :H * D], A, A, A, st2, b.q_starts, b.seq_state, b.positions,
                                                2 * H, 64, H, D))
        fl = floor(st.numel() * 8 + 2 * T * 4 * H * D)
        tab.add(shape, "constant-decay scan", us, fl, "Mamba-2 scan", like, fl)
    return tab.rows


def milenex_kernels(device, size: str = "1b") -> List[dict]:
    from .ops.maps import ConvWindow
    from .ops.prenorm import TokenShift
    tab = _Table(device)
    ops, rnd, floor, bf = tab.ops, tab.rnd, tab.floor, torch.bfloat16
    W, _, ff, H, G, E, fe, fs, _ = MILENEX_SIZES[size]
    D, V = 128, 64
    per_head = lambda: torch.rand(H, device=device)
    for shape, lens, ctxs, windows in (("decode 64 x 1152", [1] * 64, [1152] * 64, (0, 512)), ("decode 8 x 4096", [1] * 8, [4096] * 8, (0, 512)),
                                       ("prompt 2048", [2048], [2048], (0, 512)), ("prompt 8192", [8192], [8192], (0, 1024)),
                                       ("prompt 4 x 512 at 2048", [512] * 4, [2048] * 4, (0, 512))):
        b = _batch(lens, ctxs, device)
        T = b.tokens
        b.min_q_len, b.seq_lens = min(lens), torch.tensor(ctxs, dtype=torch.int32, device=device)
        kc, vc, joint = rnd(b.blocks, G, 16, D), rnd(b.blocks, G, 16, D), rnd(b.blocks, 1, 16, G * V)
        q, sink, r1, r2, gate = rnd(T, H, D), per_head(), per_head(), per_head(), rnd(T, H, dtype=torch.float32)
        mix, sinks = torch.eye(H, device=device) + 0.1, sink.float()
        for window in windows:
            see = lambda i: min(i + 1, window or i + 1)
            keys = sum(see(i) for n, c in zip(lens, ctxs) for i in range(c - n, c))
            rows = sum(min(c, n + (window or c) - 1) for n, c in zip(lens, ctxs))
            fl = floor(rows * G * 4 * D + 4 * T * H * D, 4.0 * keys * H * D)
            talk_bytes = rows * G * 2 * (D + V) + 2 * T * H * (D + V)
            like = tab.time(lambda: ops.attention(q.view(T, -1), kc, vc, b.block_tables, b.row_seq, b.positions, H, G, D, D ** -0.5, window, sinks, 0.0, meta=b))
            at = f"{shape}, window {window}" if window else shape
            tab.add(at, "attention_maps, sink", tab.time(lambda: ops.attention_maps(q, kc, vc, D, D, b, D ** -0.5, window, sink=sink)), fl, "attention, sink", like, fl)
            us = tab.time(lambda: ops.attention_talk(q, kc, joint, D, V, b, D ** -0.5, mix, window, sink, r1, r2, gate, reach=9.0))
            # products: scores, mixed weights, values once per head; or the values of all key/value heads per head, as one pass over the keys needs
            tab.add(at, "attention_talk", us, floor(talk_bytes, 2.0 * keys * H * (D + V + H)), "attention, sink", like, fl)
            tab.add(at, "attention_talk, products of one pass", us, floor(talk_bytes, 2.0 * keys * H * (D + G * V)), "attention, sink", like, fl)
        if len(lens) == 4:
            continue
        N = (H + 2 * G) * D
        x, w, inv, qs, none = rnd(T, N), torch.ones(D, device=device, dtype=bf), torch.rand(D // 2, device=device), b.q_starts, torch.zeros(0, device=device)
        fl = floor(2 * T * (2 * H + 4 * G) * D)
        like = tab.time(lambda: ops.rope_kv_write(x, b.positions, b.slots, inv, w, w, kc, vc, H, G, D, D, 0, 1e-5))
        prepare = lambda conv=None: ops.maps_prepare(x, (0, H * D, (H + G) * D), H, D, D, b.positions, b.slots, inv, 1.0, None, None, False, 1e-5, kc, vc, pairs=True,
                                                     conv=conv)
        tab.add(shape, "maps_prepare, norms without weights", tab.time(prepare), fl, "rope_kv_write", like, fl)
        cw, state = torch.rand(N, 4, device=device), torch.zeros(b.num_seqs, 3, N, device=device, dtype=bf)
        if lens[0] == 1:
            tab.add(shape, "maps_prepare behind a convolution", tab.time(lambda: prepare(ConvWindow(cw, state, b.seq_state))),
                    floor(2 * T * (2 * H + 4 * G) * D + 12 * T * N + 16 * N), "rope_kv_write", like, fl)
        else:
            us = tab.time(lambda: ops.causal_conv1d(x, cw, None, state, qs, b.seq_state, b.positions, False, b.max_q_len))
            us2 = tab.time(lambda: ops.causal_conv1d(x, cw, None, state, qs, b.seq_state, b.positions, True, b.max_q_len))
            tab.add(shape, "convolution", us, floor(4 * T * N), "the same with an activation", us2, floor(4 * T * N))
        gates, xt = torch.empty(T, H, device=device), rnd(T, H * D + G * (D + V) + H)
        tab.add(shape, "maps_prepare, joint values and gates", tab.time(lambda: ops.maps_prepare(
            xt, (0, H * D, (H + G) * D), H, D, G * V, b.positions, b.slots, none, 1.0, None, None, False, -1.0, kc, joint, extra_out=gates, extra_offset=(H + G) * D + G * V)),
            floor(2 * T * (2 * H * D + 2 * G * (D + V) + 3 * H)), "rope_kv_write", like, fl)
    for T in (64, 2048):
        shape = f"{T} rows"
        b = _batch([1] * T if T == 64 else [T], [1024] * T if T == 64 else [T], device)
        x, y, y2, res, w = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W), torch.ones(W, device=device, dtype=bf)
        state = torch.zeros(b.num_seqs, W, device=device)
        norm, norm_fl = tab.time(lambda: ops.rmsnorm(res, y, w, 1e-5)), floor(T * W * 8)
        tab.add(shape, "prenorm", tab.time(lambda: ops.prenorm_step(x, y, w, W, 1e-5)), floor(T * W * 12), "residual add + rmsnorm", norm, norm_fl)
        tab.add(shape, "prenorm with a token shift", tab.time(lambda: ops.prenorm_step(x, y, w, W, 1e-5, shift=TokenShift(w, state, b))),
                floor(T * W * 12 + state.numel() * 8), "residual add + rmsnorm", norm, norm_fl)
        rw, rw8, bias = rnd(E, W), rnd(E + 8, W), torch.zeros(E, device=device)
        ids, wts, gate = torch.empty(T, MILENEX_TOP, dtype=torch.int32, device=device), torch.empty(T, MILENEX_TOP, device=device), torch.empty(T, device=device)

        def routed(grouped):
            if grouped:
                z = ops.linear(y, rw8, force_splits=2, defer=True)
                ops.k.moe_route_fp32(None, ops.workspace, z.splits, E + 8, E, MILENEX_TOP, 1, False, 1.0, ids, wts, bias, 8, 4, float("-inf"), gate)
            else:
                ops.k.moe_route_scored(ops.linear(y, rw), bias, MILENEX_TOP, 1, False, 1.0, ids, wts)
        fl = floor(2 * (T * W + E * W))
        tab.add(shape, "router, fp32 logits, groups, shared gate", tab.time(lambda: routed(True)), fl, "router, bf16 logits", tab.time(lambda: routed(False)), fl)
        n = T * MILENEX_TOP
        xp, row_of = rnd(n, W), torch.arange(n, device=device).int().view(T, -1)
        tab.add(shape, "combine with the gated shared expert", tab.time(lambda: ops.k.moe_combine(xp, row_of, wts, y2, res, gate)), floor(2 * (2 * T + n) * W), "combine",
                tab.time(lambda: ops.k.moe_combine(xp, row_of, wts, y2)), floor(2 * (T + n) * W))
        u, gu = rnd(T, ff), rnd(T, 2 * ff)
        tab.add(shape, "gelu", tab.time(lambda: ops.act_(u, "gelu")), floor(4 * T * ff), "clamped SwiGLU", tab.time(lambda: ops.glu(gu, 2)), floor(6 * T * ff))
    return tab.rows


DESIGNS = {"milenex": (milenex_config, milenex_twin_config, milenex_kernels), "dorevik": (dorevik_config, dorevik_twin_config, dorevik_kernels), "sovanex": (sovanex_config, twin_config, sovanex_kernels), "divanex": (divanex_config, divanex_twin_config, divanex_kernels)}


def main(args) -> dict:
    """``args``: design, sizes, steps, warmup, batch, prompt_len, kernels (see bench.py)."""
    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    out = {"compare": args.compare, "data": "synthetic (uniform random token ids, random weights)", "prompt_len": args.prompt_len or 1024,
           "steps": args.steps, "warmup": args.warmup, "throughput": []}
    design, twin, kernels = DESIGNS[args.compare]
    for size in args.sizes.split(",") if args.sizes else ():
        for cfg in (design(size), twin(size)):
            for batch in ([args.batch] if args.batch else [8, 64]):
                r = throughput(cfg, batch, out["prompt_len"], args.steps, args.warmup, device)
                out["throughput"].append({"model": cfg.name, "batch": batch, **r})
    if args.kernels:
        out["kernels"] = kernels(device)
    return out
