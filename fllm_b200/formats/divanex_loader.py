"""Divanex checkpoints (config.json with ``"architecture": "Divanex"`` and one safetensors file) into the decoder's weight
containers, and random tensors under the same names for benchmarks and tests.

Layer i's tensors are ``l<i>.*``: ``norm1`` / ``norm2``, ``mix.*`` (the mixer), ``mlp.gate`` / ``mlp.up`` / ``mlp.down`` (absent
without a feed-forward network), ``side.*`` (the per-layer token input, a slice of ``side.embed``). Row and column counts are
padded to multiples of 8 with zeros, which the kernels carry along as zeros.
"""
from __future__ import annotations

import hashlib
from typing import Callable, Dict

import torch

from ..config import ModelConfig
from ..models.recurrent import pack_mamba2, pad8, pad_cols, pad_rows
from ..models.tied import pack_tied
from ..models.weights import DecoderWeights, LayerWeights, SideInput


def tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    W, side = cfg.hidden_size, cfg.token_side_dim
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    if side:
        out["side.embed"] = (cfg.vocab_size, cfg.num_layers * side)
    for i in range(cfg.num_layers):
        p = f"l{i}."
        out[p + "norm1"] = (W,)
        if cfg.layer_kind(i) == "mamba2":
            s = cfg.ssm_of(i)
            inner, bc, H = s["d_inner"], s["n_groups"] * s["d_state"], s["n_heads"]
            C = inner + 2 * bc
            mix = {"in": (2 * inner + 2 * bc + H, W), "conv": (C, s["conv_taps"]), "conv.b": (C,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                   "norm": (inner,), "o": (W, inner)}
        else:
            c = cfg.attn_of(i)
            mix = {"q": (c["num_heads"] * c["head_dim"], W), "k": (c["num_kv_heads"] * c["head_dim"], W), "o": (W, c["num_heads"] * c["head_dim"])}
        out.update({p + "mix." + k: v for k, v in mix.items()})
        if cfg.ffn_kind(i) != "none":
            ff = cfg.ffn_of(i)["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
        if side:
            out.update({p + "side.gate": (side, W), p + "side.proj": (W, side), p + "side.norm": (W,)})
    return out


def divanex_weights(cfg: ModelConfig, get: Callable, device, dtype) -> DecoderWeights:
    """``get(name)`` returns a checkpoint tensor."""
    W, side = cfg.hidden_size, cfg.token_side_dim
    Wp, shapes = pad8(W), tensor_shapes(cfg)

    def tensor(name):
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the config says {shapes[name]}")
        return t

    put = lambda t: t.to(device=device, dtype=dtype).contiguous()
    vec = lambda name: put(pad_rows(tensor(name), Wp))
    proj_in = lambda name: pad_cols(tensor(name), Wp)              # reads the (padded) hidden state
    proj_out = lambda name: pad_rows(tensor(name), Wp)             # writes the (padded) hidden state

    layers = []
    for i in range(cfg.num_layers):
        p, m = f"l{i}.", f"l{i}.mix."
        if cfg.layer_kind(i) == "mamba2":
            s = cfg.ssm_of(i)
            conv = tensor(m + "conv")
            conv = torch.cat([torch.zeros(conv.shape[0], s["d_conv"] - s["conv_taps"], dtype=conv.dtype, device=conv.device), conv], 1)
            mixer = pack_mamba2(proj_in(m + "in"), conv, tensor(m + "conv.b"), tensor(m + "dt_bias"), tensor(m + "A_log"), tensor(m + "D"), tensor(m + "norm"),
                                proj_out(m + "o"), dtype, device, shapes=s)
        else:
            mixer = pack_tied(proj_in(m + "q"), proj_in(m + "k"), proj_out(m + "o"), dtype, device)
        lw = LayerWeights(attn_norm=vec(p + "norm1"), wqkv=None, wo=None, ffn_norm=None, mixer=mixer)
        if cfg.ffn_kind(i) != "none":
            f = cfg.ffn_of(i)
            rows = (f["ff"] + 15) // 16 * 16                       # gate and up rows of a feature side by side: 2 * rows in multiples of 32
            pair = torch.stack([pad_rows(proj_in(p + "mlp.gate"), rows), pad_rows(proj_in(p + "mlp.up"), rows)], 1)
            lw.ffn_norm, lw.act_limit = vec(p + "norm2"), f["limit"]
            lw.w_gate_up = put(pair.reshape(2 * rows, Wp))
            lw.w_down = put(pad_cols(proj_out(p + "mlp.down"), rows))
        if side:
            lw.side = SideInput(put(pad_rows(proj_in(p + "side.gate"), pad8(side))), put(pad_cols(proj_out(p + "side.proj"), pad8(side))), vec(p + "side.norm"))
        layers.append(lw)
    return DecoderWeights(embed=put(pad_cols(tensor("embed"), Wp)), layers=layers, final_norm=vec("final.norm"), lm_head=put(pad_cols(tensor("head"), Wp)),
                          vocab_start=0, vocab_local=cfg.vocab_size, side_embed=put(tensor("side.embed")) if side else None)


def random_tensors(cfg: ModelConfig, seed: int, device) -> Callable:
    """``get`` for :func:`divanex_weights` that draws tensors when asked: N(0, 1 / fan-in) matrices, norm weights around 1, decays
    and step sizes in the ranges trained models use."""
    shapes = tensor_shapes(cfg)

    def get(name):
        shape, leaf = shapes[name], name.split(".")[-1]
        g = torch.Generator(device=device)
        g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}/{name}".encode()).digest()[:6], "little"))
        t = torch.randn(shape, generator=g, device=device)
        if leaf in ("norm", "norm1", "norm2", "D"):
            return 1.0 + 0.1 * t
        if leaf == "A_log":
            return 0.5 * t
        if leaf == "dt_bias":
            return 0.5 * t - 3.0
        if leaf == "b":
            return 0.1 * t
        return t * (0.5 if leaf == "conv" else shape[-1] ** -0.5 if name not in ("embed", "side.embed") else 1.0)
    return get
