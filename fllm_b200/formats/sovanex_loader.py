"""Sovanex checkpoints (config.json with ``"architecture": "Sovanex"`` and one safetensors file) into the decoder's weight
containers, and random tensors under the same names for benchmarks and tests.

Layer i's tensors are ``l<i>.*``: ``norm1`` / ``norm2`` with ``.b`` biases, ``mix.*`` (the mixer), ``mlp.up`` / ``mlp.down``
(absent without a feed-forward network), ``hc1.*`` / ``hc2.*`` (the residual-stream coefficients ``in``, ``out``, ``mix``).
Row and column counts are padded to multiples of 8 with zeros, which the kernels carry along as zeros.
"""
from __future__ import annotations

import hashlib
from typing import Callable, Dict

import torch

from ..config import ModelConfig
from ..models.mla import pack_latent
from ..models.recurrent import pack_gated_delta, pad8, pad_cols, pad_rows
from ..models.weights import DecoderWeights, LayerWeights, StreamMix


def sovanex_weights(cfg: ModelConfig, get: Callable, device, dtype) -> DecoderWeights:
    """``get(name, required=True)`` returns a checkpoint tensor (or None)."""
    W, S = cfg.hidden_size, cfg.residual_streams
    Wp = pad8(W)

    def vec(name):
        return pad_rows(get(name), Wp).to(device=device, dtype=dtype)

    def shape(name, *want):
        t = get(name)
        if tuple(t.shape) != want:
            raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the config says {want}")
        return t

    def proj_in(name, rows):                   # reads the (padded) hidden state
        return pad_cols(shape(name, rows, W), Wp)

    def proj_out(name, cols):                  # writes the (padded) hidden state
        return pad_rows(shape(name, W, cols), Wp)

    def streams(p):
        if get(p + "in", False) is None:       # one plain residual
            if S != 1:
                raise KeyError(f"checkpoint has no tensor {p + 'in'!r}")
            one = torch.ones(1)
            return StreamMix(one.to(device), one.view(1, 1).to(device), (one * cfg.residual_mult).to(device))
        f32 = lambda t: t.float().to(device).contiguous()
        return StreamMix(f32(shape(p + "in", S)), f32(shape(p + "mix", S, S)), f32(shape(p + "out", S).float() * cfg.residual_mult))

    layers = []
    for i in range(cfg.num_layers):
        p, m = f"l{i}.", f"l{i}.mix."
        if cfg.layer_kind(i) == "gated_delta":
            s = cfg.ssm_of(i)
            Hk, Hv, Dk, Dv, taps = s["num_k_heads"], s["num_v_heads"], s["head_k_dim"], s["head_v_dim"], s["conv_taps"]
            conv = torch.cat([shape(m + f"{n}.conv", r, taps) for n, r in (("q", Hk * Dk), ("k", Hk * Dk), ("v", Hv * Dv))], 0)
            conv = torch.cat([torch.zeros(conv.shape[0], s["d_conv"] - taps, dtype=conv.dtype, device=conv.device), conv], 1)
            mixer = pack_gated_delta(proj_in(m + "q", Hk * Dk), proj_in(m + "k", Hk * Dk), proj_in(m + "v", Hv * Dv), proj_in(m + "g", Hv * Dv),
                                     proj_in(m + "b", Hv), proj_in(m + "a", Hv), conv, shape(m + "dt_bias", Hv), shape(m + "A_log", Hv),
                                     shape(m + "norm", Dv), proj_out(m + "o", Hv * Dv), dtype, device)
        else:
            c = cfg.mla_of(i)
            H, dn, dr, dv, R = c["num_heads"], c["qk_nope_head_dim"], c["qk_rope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
            own = c["kv_from"] is None
            mixer = pack_latent(proj_in(m + "q", H * (dn + dr)), proj_in(m + "dkv", R + dr) if own else None,
                                shape(m + "dkv.norm", R) if own else None, shape(m + "uk", H * dn, R), shape(m + "uv", H * dv, R),
                                proj_in(m + "g", H), proj_out(m + "o", H * dv), c, dtype, device)
        lw = LayerWeights(attn_norm=vec(p + "norm1"), attn_norm_b=vec(p + "norm1.b"), wqkv=None, wo=None, ffn_norm=None, mixer=mixer,
                          streams1=streams(p + "hc1."))
        if cfg.ffn_kind(i) != "none":
            up = get(p + "mlp.up")
            ff = up.shape[0]
            lw.ffn_norm, lw.ffn_norm_b, lw.streams2 = vec(p + "norm2"), vec(p + "norm2.b"), streams(p + "hc2.")
            lw.w_gate_up = pad_rows(proj_in(p + "mlp.up", ff), pad8(ff)).to(device=device, dtype=dtype)
            lw.w_down = pad_cols(proj_out(p + "mlp.down", ff), pad8(ff)).to(device=device, dtype=dtype)
        layers.append(lw)
    embed = pad_cols(shape("embed", cfg.vocab_size, W), Wp).to(device=device, dtype=dtype)
    return DecoderWeights(embed=embed, layers=layers, final_norm=vec("final.norm"), final_norm_b=vec("final.norm.b"), lm_head=embed,
                          vocab_start=0, vocab_local=cfg.vocab_size)


def random_tensors(cfg: ModelConfig, seed: int, device) -> Callable:
    """``get`` for :func:`sovanex_weights` that draws tensors when asked: N(0, 1 / fan-in) matrices, norm weights around 1,
    decays and step sizes in the ranges trained models use, stream mixes near the identity."""
    W, S, I = cfg.hidden_size, cfg.residual_streams, cfg.intermediate_size

    def draw(name, shape, std):
        g = torch.Generator(device=device)
        g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}/{name}".encode()).digest()[:6], "little"))
        return torch.randn(shape, generator=g, device=device) * std

    def shapes(i: int) -> Dict[str, tuple]:
        p = f"l{i}."
        out = {p + "norm1": (W,), p + "norm1.b": (W,)}
        if cfg.layer_kind(i) == "gated_delta":
            s = cfg.ssm_of(i)
            K, V, Hv, t = s["num_k_heads"] * s["head_k_dim"], s["num_v_heads"] * s["head_v_dim"], s["num_v_heads"], s["conv_taps"]
            out.update({p + "mix." + k: v for k, v in {
                "q": (K, W), "k": (K, W), "v": (V, W), "g": (V, W), "b": (Hv, W), "a": (Hv, W), "q.conv": (K, t), "k.conv": (K, t),
                "v.conv": (V, t), "dt_bias": (Hv,), "A_log": (Hv,), "norm": (s["head_v_dim"],), "o": (W, V)}.items()})
        else:
            c = cfg.mla_of(i)
            H, dn, dr, dv, R = c["num_heads"], c["qk_nope_head_dim"], c["qk_rope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
            out.update({p + "mix." + k: v for k, v in {
                "q": (H * (dn + dr), W), "uk": (H * dn, R), "uv": (H * dv, R), "g": (H, W), "o": (W, H * dv)}.items()})
            if c["kv_from"] is None:
                out.update({p + "mix.dkv": (R + dr, W), p + "mix.dkv.norm": (R,)})
        for q in (1, 2) if cfg.ffn_kind(i) != "none" else (1,):
            out.update({f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        if cfg.ffn_kind(i) != "none":
            out.update({p + "norm2": (W,), p + "norm2.b": (W,), p + "mlp.up": (I, W), p + "mlp.down": (W, I)})
        return out

    table: Dict[str, tuple] = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i in range(cfg.num_layers):
        table.update(shapes(i))

    def get(name, required=True):
        if name not in table:
            if required:
                raise KeyError(name)
            return None
        shape, leaf = table[name], name.split(".")[-1]
        if leaf == "b" and "norm" in name:
            return draw(name, shape, 0.1)
        if leaf in ("norm", "norm1", "norm2"):
            return 1.0 + draw(name, shape, 0.1)
        if leaf == "mix":
            return torch.eye(S, device=device) + draw(name, shape, 0.1)
        if leaf == "in":
            return 1.0 / S + draw(name, shape, 0.1)
        if leaf == "out":
            return 1.0 + draw(name, shape, 0.1)
        if leaf == "A_log":
            return draw(name, shape, 0.5)
        if leaf == "dt_bias":
            return draw(name, shape, 0.5) - 3.0
        return draw(name, shape, (shape[-1] if leaf != "conv" else 4) ** -0.5)
    return get
