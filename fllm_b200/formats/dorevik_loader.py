"""Dorevik checkpoints (config.json with ``"architecture": "Dorevik"`` and one safetensors file) into the decoder's weight
containers, and random tensors under the same names for benchmarks and tests.

Layer i's tensors are ``l<i>.*``: ``norm1`` / ``norm2`` (of the sublayers' outputs), ``mix.*`` (the mixer; two of them under
``mix.left`` and ``mix.right`` in a paired layer), ``mlp.*`` (``gate`` / ``up`` / ``down``, or ``router``, the experts
``e<j>.*`` and ``shared.*``). Row and column counts are padded to multiples of 8 (networks: 16) with zeros, which the kernels
carry along as zeros.
"""
from __future__ import annotations

import hashlib
from typing import Callable, Dict

import torch

from ..config import ModelConfig
from ..models.maps import pack_maps, pack_maps_lightning
from ..models.recurrent import pad8, pad_cols, pad_rows
from ..models.weights import DecoderWeights, LayerWeights


def _network(prefix: str, ff: int, W: int) -> Dict[str, tuple]:
    return {prefix + "gate": (ff, W), prefix + "up": (ff, W), prefix + "down": (W, ff)}


def tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    W = cfg.hidden_size
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    for i in range(cfg.num_layers):
        p, c = f"l{i}.", cfg.attn_of(i)
        out[p + "norm1"] = (W,)
        H, G, M, d, dv = c["num_heads"], c["num_kv_heads"], c["maps"], c["head_dim"], c["v_dim"]
        rows = {"q": H * M * d, "k": G * M * d, "v": G * dv}
        mix = {n: (r, W) for n, r in rows.items()}
        mix["o"] = (W, H * dv)
        if cfg.layer_kind(i) == "maps":
            mix.update({n + ".b": (r,) for n, r in rows.items()})
            mix.update({n: (d,) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
        else:
            mix.update({"q.norm": (H * d,), "k.norm": (G * d,)})
            K, V = c["lin_heads"] * c["lin_k_dim"], c["lin_heads"] * c["lin_v_dim"]
            mix = {"left." + n: s for n, s in mix.items()}
            mix.update({"right." + n: s for n, s in dict(q=(K, W), k=(K, W), v=(V, W), g=(V, W), norm=(V,), o=(W, V)).items()})
            mix.update({"left.out": (W,), "right.out": (W,)})
        out.update({p + "mix." + n: s for n, s in mix.items()})
        f = cfg.ffn_of(i)
        if cfg.ffn_kind(i) != "none":
            out[p + "norm2"] = (W,)
        if cfg.ffn_kind(i) == "glu":
            out.update(_network(p + "mlp.", f["ff"], W))
        elif cfg.ffn_kind(i) == "moe":
            out[p + "mlp.router"] = (f["experts"], W)
            for e in range(f["experts"]):
                out.update(_network(f"{p}mlp.e{e}.", f["ff"], W))
            if f["shared_ff"]:
                out.update(_network(p + "mlp.shared.", f["shared_ff"], W))
    return out


def dorevik_weights(cfg: ModelConfig, get: Callable, device, dtype) -> DecoderWeights:
    """``get(name)`` returns a checkpoint tensor."""
    Wp, shapes = pad8(cfg.hidden_size), tensor_shapes(cfg)

    def tensor(name):
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the config says {shapes[name]}")
        return t

    put = lambda t: t.to(device=device, dtype=dtype).contiguous()
    vec = lambda name: put(pad_rows(tensor(name), Wp))
    proj_in = lambda name: pad_cols(tensor(name), Wp)              # reads the (padded) hidden state
    proj_out = lambda name: pad_rows(tensor(name), Wp)             # writes the (padded) hidden state

    def network(p, ff):
        rows = (ff + 15) // 16 * 16
        return torch.cat([pad_rows(proj_in(p + "gate"), rows), pad_rows(proj_in(p + "up"), rows)], 0), pad_cols(proj_out(p + "down"), rows)

    layers = []
    for i in range(cfg.num_layers):
        p, m, c = f"l{i}.", f"l{i}.mix.", cfg.attn_of(i)
        if cfg.layer_kind(i) == "maps":
            mixer = pack_maps(proj_in(m + "q"), proj_in(m + "k"), proj_in(m + "v"), tensor(m + "q.norm"), tensor(m + "k.norm"), proj_out(m + "o"), dtype, device,
                              [tensor(m + n + ".b") for n in "qkv"], [tensor(m + n) for n in ("lq1", "lk1", "lq2", "lk2")], c["diff"])
        else:
            l, r = m + "left.", m + "right."
            left = pack_maps(proj_in(l + "q"), proj_in(l + "k"), proj_in(l + "v"), tensor(l + "q.norm"), tensor(l + "k.norm"), proj_out(l + "o"), dtype, device)
            mixer = pack_maps_lightning(left, *(proj_in(r + n) for n in "qkvg"), tensor(r + "norm"), proj_out(r + "o"), c["lin_decay"],
                                        pad_rows(tensor(l + "out"), Wp), pad_rows(tensor(r + "out"), Wp), dtype, device)
        lw = LayerWeights(attn_norm=vec(p + "norm1"), wqkv=None, wo=None, ffn_norm=None, mixer=mixer)
        f = cfg.ffn_of(i)
        if cfg.ffn_kind(i) != "none":
            lw.ffn_norm = vec(p + "norm2")
        if cfg.ffn_kind(i) == "glu":
            lw.w_gate_up, lw.w_down = (put(t) for t in network(p + "mlp.", f["ff"]))
        elif cfg.ffn_kind(i) == "moe":
            lw.moe = cfg.moe_of(i)
            lw.router_w = put(proj_in(p + "mlp.router"))
            rows = (f["ff"] + 15) // 16 * 16
            lw.exp_gate_up = torch.empty(f["experts"], 2 * rows, Wp, dtype=dtype, device=device)
            lw.exp_down = torch.empty(f["experts"], Wp, rows, dtype=dtype, device=device)
            for e in range(f["experts"]):
                gu, down = network(f"{p}mlp.e{e}.", f["ff"])
                lw.exp_gate_up[e].copy_(gu)
                lw.exp_down[e].copy_(down)
            if f["shared_ff"]:
                lw.shared_gate_up, lw.shared_down = (put(t) for t in network(p + "mlp.shared.", f["shared_ff"]))
        layers.append(lw)
    return DecoderWeights(embed=put(pad_cols(tensor("embed"), Wp)), layers=layers, final_norm=vec("final.norm"), lm_head=put(pad_cols(tensor("head"), Wp)),
                          vocab_start=0, vocab_local=cfg.vocab_size)


def random_tensors(cfg: ModelConfig, seed: int, device) -> Callable:
    """``get`` for :func:`dorevik_weights` that draws tensors when asked: N(0, 1 / fan-in) matrices, norm weights around 1, small
    biases and lambda vectors."""
    shapes = tensor_shapes(cfg)

    def get(name):
        shape, leaf = shapes[name], name.split(".")[-1]
        g = torch.Generator(device=device)
        g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}/{name}".encode()).digest()[:6], "little"))
        t = torch.randn(shape, generator=g, device=device)
        if leaf in ("norm", "norm1", "norm2", "out"):
            return 1.0 + 0.1 * t
        if len(shape) == 1:                                        # biases, lambda vectors
            return 0.1 * t
        return t if name == "embed" else t * shape[-1] ** -0.5
    return get
