"""Small Sovanex configurations and random weights for the tests, and the drivers that feed them through the engine."""
import json
import math
import os

import torch

import sovanex_oracle as oracle
from fllm_b200.config import EngineConfig, ModelConfig
from fllm_b200.formats.loader import load_model
from fllm_b200.formats.safetensors_io import save_file
from fllm_b200.runtime.engine import LLMEngine
from fllm_b200.runtime.replay import TraceReplay


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
                mlp=dict(kind="dense", ff=ff) if ff else None)


def attn(heads, dim, rot_dim, vdim, kv_rank, ff=None, base=10000.0, kv_from=None, sharp=1.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim),
             scale=sharp / math.sqrt(dim + rot_dim))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None)


def config(layers, vocab, width, streams, residual_mult=0.7, eps=1e-5):
    return dict(architecture="Sovanex", layers=layers, vocab=vocab, width=width, streams=streams, residual_mult=residual_mult, norm=dict(eps=eps))


CONFIGS = {
    # sizes that are not multiples of 8, layers without a feed-forward network, two sharers of one layer's rows
    "odd": config([attn(3, 20, 6, 11, 37, ff=50, sharp=5.0), delta(4, 2, 20, 13, 3, ff=36), attn(5, 12, 6, 9, 37, kv_from=0, sharp=5.0),
                   delta(3, 3, 24, 10, 5), attn(2, 9, 6, 16, 37, ff=44, kv_from=0, sharp=5.0)], 203, 75, 3),
    # one plain stream, recurrent layers only
    "delta-only": config([delta(6, 2, 16, 24, 2, ff=72), delta(2, 2, 40, 32, 4, ff=40), delta(4, 1, 64, 40, 8)], 160, 64, 1, residual_mult=1.0),
    # attention only; rows of different widths in one model
    "attention-only": config([attn(4, 32, 16, 24, 144, ff=96, base=500.0, sharp=6.0), attn(9, 16, 32, 16, 80, ff=64, sharp=6.0),
                              attn(3, 24, 16, 8, 144, base=500.0, kv_from=0, sharp=6.0)], 264, 96, 2),
    # sizes of one
    "ones": config([delta(1, 1, 8, 8, 1, ff=8), attn(1, 8, 2, 8, 8, ff=16, sharp=4.0)], 48, 24, 1, residual_mult=0.5, eps=1e-3),
    # widths of large models on a narrow residual
    "wide-heads": config([delta(4, 4, 128, 128, 4, ff=256), attn(16, 128, 64, 128, 512, ff=128, base=1e6, sharp=6.0),
                          attn(20, 64, 64, 64, 512, base=1e6, kv_from=1, sharp=6.0), delta(2, 1, 256, 64, 4)], 512, 256, 4),
}


def tensors(cfg, seed=0):
    """Random tensors under checkpoint names: bf16 like a file would hold."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).bfloat16()
    mat = lambda name, rows, cols, gain=1.0: put(name, rows, cols, std=gain * cols ** -0.5)
    put("embed", cfg["vocab"], W)
    put("final.norm", W, std=0.2, mean=1.0)
    put("final.norm.b", W, std=0.2)
    for i, layer in enumerate(cfg["layers"]):
        p, m, s = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "delta":
            K, V, H = s["kv_heads"] * s["dim"], s["heads"] * s["vdim"], s["heads"]
            for n, r in (("q", K), ("k", K), ("v", V)):
                mat(m + n, r, W)
                put(m + n + ".conv", r, s["conv"], std=0.7)
            mat(m + "b", H, W)
            mat(m + "a", H, W)
            put(m + "A_log", H, std=0.5)
            put(m + "dt_bias", H, std=0.5, mean=-3.5)
            put(m + "norm", s["vdim"], std=0.2, mean=1.0)
            mat(m + "g", V, W)
            mat(m + "o", W, V)
        else:
            H, R = s["heads"], s["kv_rank"]
            mat(m + "q", H * (s["dim"] + s["rot_dim"]), W)
            if s.get("kv_from") is None:
                mat(m + "dkv", R + s["rot_dim"], W)
                put(m + "dkv.norm", R, std=0.2, mean=1.0)
            mat(m + "uk", H * s["dim"], R)
            mat(m + "uv", H * s["vdim"], R)
            mat(m + "g", H, W)
            mat(m + "o", W, H * s["vdim"])
        for q in (1, 2) if layer["mlp"] else (1,):
            put(f"{p}norm{q}", W, std=0.2, mean=1.0)
            put(f"{p}norm{q}.b", W, std=0.2)
            put(f"{p}hc{q}.in", S, std=0.3, mean=1.0 / S)
            put(f"{p}hc{q}.out", S, std=0.5, mean=1.0)
            out[f"{p}hc{q}.mix"] = (torch.eye(S) + 0.3 * torch.randn(S, S, generator=g)).bfloat16()
        if layer["mlp"]:
            mat(p + "mlp.up", layer["mlp"]["ff"], W)
            mat(p + "mlp.down", W, layer["mlp"]["ff"])
    return out


def write_checkpoint(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)


def load_tensors(cfg, w, device, dtype):
    """The loader's result without a file in between."""
    from fllm_b200.formats.sovanex_loader import sovanex_weights
    mc = ModelConfig.from_hf_config(cfg)

    def get(name, required=True):
        if name not in w and required:
            raise KeyError(name)
        return w.get(name)
    return mc, sovanex_weights(mc, get, device, dtype)


def engine(cfg, w, device="cpu", f32=True, blocks=64, max_len=512, seqs=4, chunk=512, graphs=True, spare=0, ops=None):
    mc, weights = load_tensors(cfg, w, device, torch.float32 if f32 else torch.bfloat16)
    ec = EngineConfig(dtype="fp32" if f32 else "bf16", max_num_seqs=seqs, spare_state_rows=spare, num_kv_blocks=blocks, max_model_len=max_len,
                      max_num_batched_tokens=chunk, enable_prefix_caching=False, use_cuda_graphs=graphs)
    return LLMEngine(mc, ec, device=device, weights=weights, ops=ops)


def prompt(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(replay, name, toks, cuts, end=True):
    """All logits of one request fed alone in portions that end at ``cuts``."""
    out, lo = [], 0
    for hi in list(cuts) + [len(toks)]:
        if hi > lo:
            out.append(replay.step([dict(id=name, tokens=toks[lo:hi], want=list(range(hi - lo)))], [name] if end and hi == len(toks) else []))
            lo = hi
    return torch.cat(out)


def error(got, want):
    """Largest difference of a position's logits (mean taken off) over the spread of the logits."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())


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


__all__ = ["CONFIGS", "TraceReplay", "load_model"]
