"""Small Milenex configurations and random weights for the tests, and the drivers that feed them through the engine."""
import torch

import milenex_oracle as oracle
from sovanex_cases import TraceReplay, error, feed, load_model, prompt, write_checkpoint
from fllm_b200.config import EngineConfig, ModelConfig
from fllm_b200.formats.milenex_loader import milenex_weights
from fllm_b200.runtime.engine import LLMEngine


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, limit=0.9, shared=None, groups=None):
    out = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if groups:
        out["router"]["groups"] = dict(zip(("count", "keep"), groups))
    if shared:
        out["shared"] = dict(zip(("ff", "limit"), shared))
    return out


def rotary(heads, kv_heads, dim, vdim, window, rot, conv=4, base=1e4, sharp=2.0, mlp=None):
    """Queries and keys have unit root mean square, so ``sharp`` sets the spread of the scores."""
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=sharp / dim ** 0.5, conv=conv,
                                                      mask=dict(size=window), rot=dict(base=base, dims=rot)))


def talking(heads, kv_heads, dim, vdim, window, sharp=2.0, mlp=None):
    return dict(type="attention_2", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=sharp / dim ** 0.5, mask=dict(size=window)))


def config(layers, vocab, width, loop=None, eps=1e-5):
    return dict(architecture="Milenex", layers=layers, vocab=vocab, width=width, norm=dict(eps=eps), loop=loop and dict(zip(("start", "stop", "times"), loop)))


CONFIGS = {
    # sizes that are not multiples of 8, a layer without a network, a loop in the middle
    "odd": config([rotary(6, 2, 20, 28, 19, 10, 3, 500.0, mlp=moe(6, 3, 20, 0.8, (36, 0.5), (3, 2))), talking(6, 3, 13, 9, 26, mlp=dense(50)),
                   rotary(3, 1, 12, 7, 33, 12, 5), talking(5, 1, 11, 10, 7, mlp=moe(7, 3, 12, 1.1))], 203, 75, (1, 3, 3)),
    # widths of the tensor-core kernels and their paddings, groups of several heads, unequal key and value widths, several value pieces
    "tensor-cores": config([talking(8, 2, 64, 40, 45, mlp=dense(96)), rotary(8, 2, 128, 64, 50, 32, 4, 1e6, mlp=moe(8, 3, 40, 1.0, (24, 2.0), (4, 2))),
                            talking(12, 4, 100, 64, 90, mlp=moe(10, 4, 24, 0.7, None, (5, 3))), rotary(10, 1, 60, 100, 130, 60, 2),
                            talking(3, 3, 36, 128, 1000)], 264, 96, (2, 4, 2)),
    # wider than those kernels, more query heads per key head than their table holds
    "wide": config([talking(4, 2, 136, 72, 30, mlp=dense(40)), rotary(3, 3, 200, 72, 45, 72, 7, mlp=moe(4, 2, 24, 1.5, (16, 1.0), (2, 2))),
                    talking(24, 1, 16, 140, 18), rotary(2, 1, 16, 140, 21, 0, 6)], 160, 64, (0, 4, 2), 1e-6),
    # sizes, windows and counts of one
    "ones": config([talking(1, 1, 8, 24, 1, mlp=moe(1, 1, 16, 1.0, (16, 1.0))), rotary(1, 1, 8, 24, 1, 2, 1, mlp=dense(16)), talking(2, 1, 1, 1, 2),
                    rotary(2, 2, 2, 16, 3, 2, 2)], 48, 24, (3, 4, 1), 1e-3),
    "no-loop": config([rotary(2, 1, 16, 24, 9, 8), talking(4, 2, 24, 8, 12, mlp=dense(24))], 71, 40),
}


def tensors(cfg, seed=0, clear_calls=False):
    """Random tensors under checkpoint names: bf16 like a file would hold. ``clear_calls``: the routers see only the first columns
    of the residual, where the embedding holds well separated values and no layer adds anything, so that rounding elsewhere
    hardly ever changes a choice."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).bfloat16()
    mat = lambda name, rows, cols, gain=1.0: put(name, rows, cols, std=gain * cols ** -0.5)

    def network(p, ff):
        mat(p + "gate", ff, W, gain=1.5)
        mat(p + "up", ff, W, gain=1.5)
        mat(p + "down", W, ff)
    put("embed", cfg["vocab"], W)
    put("final.norm", W, std=0.2)
    mat("head", cfg["vocab"], W, gain=3.0)
    widest = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"] or [1])
    for i, layer in enumerate(cfg["layers"]):
        p, m, s = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        H, G = s["heads"], s["kv_heads"]
        rows = dict(q=H * s["dim"], k=G * s["dim"], v=G * s["vdim"])
        for n, r in rows.items():
            mat(m + n, r, W)
        mat(m + "o", W, H * s["vdim"])
        put(m + "sink", H, std=1.0, mean=0.5)
        if layer["type"] == "attention":
            for n, r in rows.items():
                put(m + n + ".conv", r, s["conv"], std=s["conv"] ** -0.5)
        else:
            out[m + "r1"] = (0.2 + torch.rand(H, generator=g)).bfloat16()
            out[m + "r2"] = (0.1 + 1.5 * torch.rand(H, generator=g)).bfloat16()
            out[m + "talk"] = (torch.eye(H) + 0.6 * H ** -0.5 * torch.randn(H, H, generator=g)).bfloat16()
            mat(m + "g", H, W, gain=1.5)
        put(p + "norm1", W, std=0.2)
        out[p + "shift"] = (0.1 + 0.6 * torch.rand(W, generator=g)).bfloat16()
        mlp = layer["mlp"]
        if mlp:
            put(p + "norm2", W, std=0.2)
        if mlp and mlp["kind"] == "dense":
            mat(p + "mlp.up", mlp["ff"], W)
            mat(p + "mlp.down", W, mlp["ff"])
        elif mlp:
            E = mlp["router"]["experts"]
            mat(p + "mlp.router", E, W, gain=1.5)
            put(p + "mlp.correction", E, std=0.15, mean=-0.1)              # (choice scores of either sign)
            if clear_calls:
                out[p + "mlp.router"] = torch.eye(W)[torch.randperm(widest, generator=g)[:E]].bfloat16()
            for e in range(E):
                network(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                network(p + "mlp.shared.", mlp["shared"]["ff"])
                mat(p + "mlp.shared.sg", 1, W, gain=1.5)
    if clear_calls:
        levels = torch.linspace(-2, 2, widest)
        out["embed"][:, :widest] = torch.stack([levels[torch.randperm(widest, generator=g)] for _ in range(cfg["vocab"])]).bfloat16()
        for n, t in out.items():
            if n.endswith("norm2"):
                t[:widest] = 0
            elif n.endswith((".o", ".down")):
                t[:widest] = 0
    return out


def load_tensors(cfg, w, device, dtype):
    """The loader's result without a file in between."""
    mc = ModelConfig.from_hf_config(cfg)
    return mc, milenex_weights(mc, w.__getitem__, device, dtype)


def engine(cfg, w, device="cpu", f32=True, blocks=64, max_len=512, seqs=4, chunk=512, graphs=True, spare=0, ops=None, block_size=16, **more):
    mc, weights = load_tensors(cfg, w, device, torch.float32 if f32 else torch.bfloat16)
    more.setdefault("enable_prefix_caching", False)
    ec = EngineConfig(dtype="fp32" if f32 else "bf16", max_num_seqs=seqs, spare_state_rows=spare, num_kv_blocks=blocks, max_model_len=max_len,
                      max_num_batched_tokens=chunk, use_cuda_graphs=graphs, block_size=block_size, **more)
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
