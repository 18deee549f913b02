"""Small Dorevik configurations and random weights for the tests, and the drivers that feed them through the engine."""
import torch

import dorevik_oracle as oracle
from sovanex_cases import TraceReplay, error, feed, load_model, prompt, write_checkpoint
from fllm_b200.config import EngineConfig, ModelConfig
from fllm_b200.formats.dorevik_loader import dorevik_weights
from fllm_b200.runtime.engine import LLMEngine


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, shared=None):
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    return dict(out, shared=dict(ff=shared)) if shared else out


def heads(heads, kv_heads, dim, vdim, window, rot, base=1e4, scaling=None, sharp=2.0):
    r = dict(base=base, dims=rot)
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=sharp / dim ** 0.5, mask=dict(size=window), rot=r)


def diff(spec, lam=0.4, mlp=None):
    return dict(type="attention", mixer=dict(spec, diff=lam), mlp=mlp)


def parallel(left, decay, dim, vdim, mlp=None):
    return dict(type="parallel", mixer=dict(left=left, right=dict(heads=len(decay), dim=dim, vdim=vdim, decay=decay)), mlp=mlp)


def config(layers, vocab, width, cap=9.0, eps=1e-5):
    return dict(architecture="Dorevik", layers=layers, vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=cap)


CONFIGS = {
    # sizes that are not multiples of 8, a layer without a network, heads that forget within a token and heads that hardly forget
    "odd": config([diff(heads(6, 2, 20, 28, 19, 10, scaling=(4.0, 2000, 32.0, 1.0)), 0.3, moe(7, 3, 20, 36)),
                   parallel(heads(5, 5, 11, 9, 7, 6, 500.0), [0.004, 0.9, 0.9995], 13, 10, dense(50)), diff(heads(3, 1, 12, 7, 33, 12)),
                   parallel(heads(4, 2, 10, 12, 23, 4), [0.97], 24, 40, moe(5, 1, 12))], 203, 75),
    # widths of the tensor-core kernels and their paddings, groups of several heads, unequal key and value widths
    "tensor-cores": config([diff(heads(8, 2, 64, 128, 40, 64, scaling=(2.0, 30, 4.0, 0.5)), 0.6, dense(96)),
                            parallel(heads(8, 2, 128, 64, 50, 32, 1e6), [0.8, 0.99, 0.3, 0.999], 32, 64, moe(6, 2, 40, 24)),
                            diff(heads(12, 1, 128, 128, 21, 64), 0.2), parallel(heads(20, 2, 60, 100, 90, 60), [0.95, 0.5], 64, 128),
                            diff(heads(4, 4, 36, 56, 1000, 18, 300.0))], 264, 96),
    # wider than those kernels
    "wide": config([diff(heads(2, 1, 136, 72, 30, 100), 0.5, dense(40)), parallel(heads(3, 3, 72, 200, 18, 72), [0.99], 200, 72, dense(24)),
                    diff(heads(2, 2, 16, 140, 45, 8), 0.8, moe(3, 2, 24, 16))], 160, 64, cap=20.0, eps=1e-6),
    # sizes, windows and counts of one
    "ones": config([diff(heads(1, 1, 8, 24, 1, 2), 0.1, moe(1, 1, 16)), parallel(heads(1, 1, 8, 24, 1, 8), [0.5], 8, 24, dense(16)),
                    diff(heads(1, 1, 2, 16, 2, 2), 0.5), parallel(heads(2, 1, 8, 24, 3, 4), [0.5] * 12 + [1.0] * 12, 1, 1)], 48, 24, cap=1.0, eps=1e-3),
}


def tensors(cfg, seed=0, clear_calls=False):
    """Random tensors under checkpoint names: bf16 like a file would hold. ``clear_calls``: the routers see only the first columns
    of the residual, where the embedding holds well separated values and no layer adds anything, so that rounding elsewhere
    never changes a choice."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).bfloat16()
    mat = lambda name, rows, cols, gain=1.0: put(name, rows, cols, std=gain * cols ** -0.5)

    def network(p, ff):
        mat(p + "gate", ff, W)
        mat(p + "up", ff, W)
        mat(p + "down", W, ff)

    def attention(m, s, maps):
        rows = dict(q=s["heads"] * maps * s["dim"], k=s["kv_heads"] * maps * s["dim"], v=s["kv_heads"] * s["vdim"])
        for n, r in rows.items():
            mat(m + n, r, W)
            if maps == 2:
                put(m + n + ".b", r, std=0.3)
        for n in "qk":
            put(m + n + ".norm", s["dim"] if maps == 2 else rows[n], std=0.2, mean=1.0)
        mat(m + "o", W, s["heads"] * s["vdim"])
    put("embed", cfg["vocab"], W)
    put("final.norm", W, std=0.2, mean=1.0)
    mat("head", cfg["vocab"], W, gain=3.0)
    widest = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] or [1])
    for i, layer in enumerate(cfg["layers"]):
        p, m, s = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "attention":
            attention(m, s, 2)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(m + n, s["dim"], std=0.6 * s["dim"] ** -0.25)
        else:
            attention(m + "left.", s["left"], 1)
            r = s["right"]
            K, V = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            for n, rows in dict(q=K, k=K, v=V, g=V).items():
                mat(m + "right." + n, rows, W, gain=1.5)
            put(m + "right.norm", V, std=0.2, mean=1.0)
            mat(m + "right.o", W, V)
            put(m + "left.out", W, std=0.3, mean=1.0)
            put(m + "right.out", W, std=0.3, mean=0.7)
        put(p + "norm1", W, std=0.2, mean=0.8)
        mlp = layer["mlp"]
        if mlp:
            put(p + "norm2", W, std=0.2, mean=0.8)
        if mlp and mlp["kind"] == "dense":
            network(p + "mlp.", mlp["ff"])
        elif mlp:
            E = mlp["router"]["experts"]
            mat(p + "mlp.router", E, W, gain=1.5)
            if clear_calls:
                out[p + "mlp.router"] = torch.eye(W)[torch.randperm(widest, generator=g)[:E]].bfloat16()
            for e in range(E):
                network(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                network(p + "mlp.shared.", mlp["shared"]["ff"])
    if clear_calls:
        levels = torch.linspace(-2, 2, widest)
        out["embed"][:, :widest] = torch.stack([levels[torch.randperm(widest, generator=g)] for _ in range(cfg["vocab"])]).bfloat16()
        for n, t in out.items():
            if n.endswith("norm1") or n.endswith("norm2"):
                t[:widest] = 0
    return out


def load_tensors(cfg, w, device, dtype):
    """The loader's result without a file in between."""
    mc = ModelConfig.from_hf_config(cfg)
    return mc, dorevik_weights(mc, w.__getitem__, device, dtype)


def engine(cfg, w, device="cpu", f32=True, blocks=64, max_len=512, seqs=4, chunk=512, graphs=True, spare=0, ops=None, block_size=16):
    mc, weights = load_tensors(cfg, w, device, torch.float32 if f32 else torch.bfloat16)
    ec = EngineConfig(dtype="fp32" if f32 else "bf16", max_num_seqs=seqs, spare_state_rows=spare, num_kv_blocks=blocks, max_model_len=max_len,
                      max_num_batched_tokens=chunk, enable_prefix_caching=False, use_cuda_graphs=graphs, block_size=block_size)
    return LLMEngine(mc, ec, device=device, weights=weights, ops=ops)


_cache = {}


def expected(name, n, seed, clear_calls=False):
    """(config, tensors, prompt, oracle logits in fp64), computed once per session."""
    key = (name, n, seed, clear_calls)
    if key not in _cache:
        cfg = CONFIGS[name]
        w = tensors(cfg, 0, clear_calls)
        toks = prompt(cfg, n, seed)
        _cache[key] = (cfg, w, toks, oracle.forward(cfg, w, toks, torch.float64))
    return _cache[key]


__all__ = ["CONFIGS", "TraceReplay", "error", "feed", "load_model", "prompt", "write_checkpoint"]
