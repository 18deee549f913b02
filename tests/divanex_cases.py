"""Small Divanex configurations and random weights for the tests, and the drivers that feed them through the engine."""
import torch

import divanex_oracle as oracle
from sovanex_cases import TraceReplay, error, feed, load_model, prompt, write_checkpoint
from fllm_b200.config import EngineConfig, ModelConfig
from fllm_b200.formats.divanex_loader import divanex_weights
from fllm_b200.runtime.engine import LLMEngine


def mamba(heads, vdim, state, groups=1, norm_groups=1, conv=4, ff=None, limit=7.0):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv),
                mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None)


def attn(heads, kv_heads, dim, ff=None, limit=7.0, cap=20.0, coef=0.3, every=10, sharp=2.0):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=sharp / dim ** 0.5, softcap=cap,
                                             q_temp=dict(coef=coef, every=every)),
                mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None)


def config(layers, vocab, width, side, alpha=1.7, scale=3.0, logit_scale=0.6, eps=1e-5):
    return dict(architecture="Divanex", layers=layers, vocab=vocab, width=width, token_side=dict(dim=side), postln_alpha=alpha,
                embedding=dict(scale=scale), logit_scale=logit_scale, norm=dict(eps=eps))


CONFIGS = {
    # sizes that are not multiples of 8; networks behind either mixer, with limits that bite
    "odd": config([attn(6, 2, 20, ff=50, limit=0.8), mamba(4, 9, 13, groups=2, norm_groups=3, conv=3, ff=36, limit=1.5), attn(5, 5, 11, cap=3.0),
                   mamba(3, 10, 24, conv=5)], 203, 75, 10),
    "mamba-only": config([mamba(6, 16, 64, groups=3, norm_groups=2), mamba(2, 40, 16, conv=2, ff=40), mamba(4, 24, 100, groups=4, norm_groups=4, conv=8)],
                         160, 64, 8, alpha=1.0),
    # attention only: tensor-core widths and others, unequal layers, a cap beyond the fixed-reference softmax, no cap at all
    "attention-only": config([attn(8, 2, 64, ff=96, every=16), attn(12, 1, 128, cap=80.0, coef=0.0), attn(3, 3, 24, ff=64), attn(4, 1, 48, cap=None),
                              attn(2, 1, 136)], 264, 96, 16, scale=1.0),
    # sizes of one
    "ones": config([mamba(1, 8, 8, conv=1, ff=8), attn(1, 1, 8, every=1, cap=1.0)], 48, 24, 1, alpha=0.5, logit_scale=1.0, eps=1e-3),
    # widths of large models on a narrow residual
    "wide-heads": config([mamba(4, 64, 128, groups=2, norm_groups=2), attn(16, 4, 128, ff=128), mamba(2, 64, 256), attn(20, 2, 64, every=100)], 512, 256, 40),
}


def tensors(cfg, seed=0):
    """Random tensors under checkpoint names: bf16 like a file would hold."""
    g = torch.Generator().manual_seed(seed)
    W, side = cfg["width"], cfg["token_side"]["dim"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).bfloat16()
    mat = lambda name, rows, cols, gain=1.0: put(name, rows, cols, std=gain * cols ** -0.5)
    put("embed", cfg["vocab"], W, std=0.5)
    put("side.embed", cfg["vocab"], side * len(cfg["layers"]))
    put("final.norm", W, std=0.2, mean=1.0)
    mat("head", cfg["vocab"], W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, s = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "mamba2":
            inner, bc, H = s["heads"] * s["vdim"], s["groups"] * s["state"], s["heads"]
            mat(m + "in", 2 * inner + 2 * bc + H, W)
            put(m + "conv", inner + 2 * bc, s["conv"], std=0.7)
            put(m + "conv.b", inner + 2 * bc, std=0.2)
            put(m + "dt_bias", H, std=0.5, mean=-2.5)
            put(m + "A_log", H, std=1.0, mean=-1.0)
            put(m + "D", H, std=0.3, mean=1.0)
            put(m + "norm", inner, std=0.2, mean=1.0)
            mat(m + "o", W, inner)
        else:
            mat(m + "q", s["heads"] * s["dim"], W)
            mat(m + "k", s["kv_heads"] * s["dim"], W)
            mat(m + "o", W, s["heads"] * s["dim"], gain=2.0)
        put(p + "norm1", W, std=0.2, mean=1.0)
        if layer["mlp"]:
            put(p + "norm2", W, std=0.2, mean=1.0)
            mat(p + "mlp.gate", layer["mlp"]["ff"], W)
            mat(p + "mlp.up", layer["mlp"]["ff"], W)
            mat(p + "mlp.down", W, layer["mlp"]["ff"])
        mat(p + "side.gate", side, W)
        mat(p + "side.proj", W, side)
        put(p + "side.norm", W, std=0.2, mean=0.5)
    return out


def load_tensors(cfg, w, device, dtype):
    """The loader's result without a file in between."""
    mc = ModelConfig.from_hf_config(cfg)
    return mc, divanex_weights(mc, w.__getitem__, device, dtype)


def engine(cfg, w, device="cpu", f32=True, blocks=64, max_len=512, seqs=4, chunk=512, graphs=True, spare=0, ops=None, block_size=16):
    mc, weights = load_tensors(cfg, w, device, torch.float32 if f32 else torch.bfloat16)
    ec = EngineConfig(dtype="fp32" if f32 else "bf16", max_num_seqs=seqs, spare_state_rows=spare, num_kv_blocks=blocks, max_model_len=max_len,
                      max_num_batched_tokens=chunk, enable_prefix_caching=False, use_cuda_graphs=graphs, block_size=block_size)
    return LLMEngine(mc, ec, device=device, weights=weights, ops=ops)


_cache = {}


def expected(name, n, seed, wseed=0):
    """(config, tensors, prompt, oracle logits in fp64), computed once per session."""
    key = (name, n, seed, wseed)
    if key not in _cache:
        cfg = CONFIGS[name]
        w = tensors(cfg, wseed)
        toks = prompt(cfg, n, seed)
        _cache[key] = (cfg, w, toks, oracle.forward(cfg, w, toks, torch.float64))
    return _cache[key]


__all__ = ["CONFIGS", "TraceReplay", "error", "feed", "load_model", "prompt", "write_checkpoint"]
