"""Milenex checkpoints (config.json with ``"architecture": "Milenex"`` and one safetensors file) into the decoder's weight containers,
and random tensors under the same names for benchmarks and tests.

Layer i's tensors are ``l<i>.*``: ``norm1`` / ``norm2`` (weights around zero), ``shift`` (token shift), ``mix.*`` (the mixer) and ``mlp.*``
(``up`` / ``down``, or ``router``, ``correction``, the experts ``e<j>.*`` and ``shared.*``). A repeated layer appears once; all its runs
share one set of weights. Row and column counts are padded to multiples of 8 (networks: 16) with zeros, which the kernels carry along as
zeros.
"""
from __future__ import annotations

import hashlib
from typing import Callable, Dict

import torch

from ..config import ModelConfig
from ..models.maps import pack_maps
from ..models.recurrent import pad8, pad_cols, pad_rows
from ..models.weights import DecoderWeights, LayerWeights


def _checkpoint_layers(cfg: ModelConfig) -> Dict[int, int]:
    """Checkpoint layer -> its first place in the running order."""
    first: Dict[int, int] = {}
    for place, layer in enumerate(cfg.layer_source or range(cfg.num_layers)):
        first.setdefault(layer, place)
    return first


def _network(prefix: str, ff: int, W: int) -> Dict[str, tuple]:
    return {prefix + "gate": (ff, W), prefix + "up": (ff, W), prefix + "down": (W, ff)}


def tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    W = cfg.hidden_size
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    for layer, at in _checkpoint_layers(cfg).items():
        p, c, f, ffn = f"l{layer}.", cfg.attn_of(at), cfg.ffn_of(at), cfg.ffn_kind(at)
        H, G, d, dv = c["num_heads"], c["num_kv_heads"], c["head_dim"], c["v_dim"]
        out[p + "norm1"] = out[p + "shift"] = (W,)
        rows = {"q": H * d, "k": G * d, "v": G * dv}
        mix = {n: (r, W) for n, r in rows.items()}
        mix.update(o=(W, H * dv), sink=(H,))
        if c.get("talk"):
            mix.update(r1=(H,), r2=(H,), talk=(H, H), g=(H, W))
        else:
            mix.update({n + ".conv": (r, c["taps"]) for n, r in rows.items()})
        out.update({p + "mix." + n: s for n, s in mix.items()})
        if ffn != "none":
            out[p + "norm2"] = (W,)
        if ffn == "plain":
            out.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
        elif ffn == "moe":
            out.update({p + "mlp.router": (f["experts"], W), p + "mlp.correction": (f["experts"],)})
            for e in range(f["experts"]):
                out.update(_network(f"{p}mlp.e{e}.", f["ff"], W))
            if f["shared_ff"]:
                out.update(_network(p + "mlp.shared.", f["shared_ff"], W))
                out[p + "mlp.shared.sg"] = (1, W)
    return out


def milenex_weights(cfg: ModelConfig, get: Callable, device, dtype) -> DecoderWeights:
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
    up16 = lambda n: (n + 15) // 16 * 16

    def gated(p, ff):
        """Gate and up rows of a feature side by side, as the clamped activation reads them."""
        rows = up16(ff)
        pair = torch.stack([pad_rows(proj_in(p + "gate"), rows), pad_rows(proj_in(p + "up"), rows)], 1)
        return pair.reshape(2 * rows, Wp), pad_cols(proj_out(p + "down"), rows)

    def layer_weights(layer, at):
        p, m, c, f, ffn = f"l{layer}.", f"l{layer}.mix.", cfg.attn_of(at), cfg.ffn_of(at), cfg.ffn_kind(at)
        talk, convs = c.get("talk"), None
        if not talk:
            convs = [torch.nn.functional.pad(tensor(m + n + ".conv"), (c["conv"] - c["taps"], 0)) for n in "qkv"]
        mixer = pack_maps(proj_in(m + "q"), proj_in(m + "k"), proj_in(m + "v"), None, None, proj_out(m + "o"), dtype, device,
                          gate=proj_in(m + "g") if talk else None, convs=convs,
                          terms={n: tensor(m + n) for n in (("sink", "r1", "r2", "talk") if talk else ("sink",))})
        lw = LayerWeights(attn_norm=vec(p + "norm1"), wqkv=None, wo=None, ffn_norm=None, mixer=mixer, shift=vec(p + "shift"))
        if ffn != "none":
            lw.ffn_norm = vec(p + "norm2")
        if ffn == "plain":
            rows = up16(f["ff"])
            lw.plain_act = f["act"]
            lw.w_gate_up, lw.w_down = put(pad_rows(proj_in(p + "mlp.up"), rows)), put(pad_cols(proj_out(p + "mlp.down"), rows))
        elif ffn == "moe":
            rows = up16(f["ff"])
            lw.moe = cfg.moe_of(at)
            lw.router_w = put(proj_in(p + "mlp.router"))
            lw.router_select_b = tensor(p + "mlp.correction").to(device=device, dtype=torch.float32).contiguous()
            lw.exp_gate_up = torch.empty(f["experts"], 2 * rows, Wp, dtype=dtype, device=device)
            lw.exp_down = torch.empty(f["experts"], Wp, rows, dtype=dtype, device=device)
            for e in range(f["experts"]):
                gu, down = gated(f"{p}mlp.e{e}.", f["ff"])
                lw.exp_gate_up[e].copy_(gu)
                lw.exp_down[e].copy_(down)
            if f["shared_ff"]:
                lw.shared_gate_up, lw.shared_down = (put(t) for t in gated(p + "mlp.shared.", f["shared_ff"]))
                lw.shared_gate_w = put(proj_in(p + "mlp.shared.sg"))
        return lw

    own = {layer: layer_weights(layer, at) for layer, at in _checkpoint_layers(cfg).items()}
    return DecoderWeights(embed=put(pad_cols(tensor("embed"), Wp)), layers=[own[i] for i in cfg.layer_source or range(cfg.num_layers)],
                          final_norm=vec("final.norm"), lm_head=put(pad_cols(tensor("head"), Wp)), vocab_start=0, vocab_local=cfg.vocab_size)


def random_tensors(cfg: ModelConfig, seed: int, device) -> Callable:
    """``get`` for :func:`milenex_weights` that draws tensors when asked: N(0, 1 / fan-in) matrices, norm weights around 0, token shifts
    around a quarter, distance biases of positive numbers, nearly diagonal mixing of heads."""
    shapes = tensor_shapes(cfg)

    def get(name):
        shape, leaf = shapes[name], name.split(".")[-1]
        g = torch.Generator(device=device)
        g.manual_seed(int.from_bytes(hashlib.sha256(f"{seed}/{name}".encode()).digest()[:6], "little"))
        t = torch.randn(shape, generator=g, device=device)
        if leaf in ("norm", "norm1", "norm2", "correction"):
            return 0.1 * t
        if leaf == "shift":
            return 0.25 + 0.1 * t
        if leaf in ("r1", "r2"):
            return 0.5 * torch.exp(0.5 * t)
        if leaf == "talk":
            return torch.eye(shape[0], device=device) + 0.3 * shape[0] ** -0.5 * t
        if leaf == "sink" or name == "embed":
            return t
        return t * (0.5 if leaf == "conv" else shape[-1] ** -0.5)
    return get
