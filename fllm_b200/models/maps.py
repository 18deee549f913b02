"""Attention of one or two maps over shared values ("maps") and its pairing with lightning attention ("maps+lightning"), as layer
kinds of the decoder runner. One projection makes [queries | keys | values], followed in the paired kind by the
[queries | keys | values | gate] of the recurrent half; every segment starts on a multiple of 8 rows.

Two maps are differential attention: the difference of two softmax attentions, normalised per head. Lightning attention is a
linear attention whose state decays by a constant per head; its output is normalised over all heads and gated. One map may have a
short convolution over time on its projections, norms without weights, a sink, a distance bias, heads that mix their weights
(talking heads: the values of all key/value heads then share a cache row) and a gate per head (its logits are further columns of
the projection)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops.maps import Combine, ConvWindow, NormedPair, bias_range
from .recurrent import _batch_meta, pad8, pad_cols, pad_rows


def _attend(dec, li: int, m, proj, b) -> torch.Tensor:
    """The attention of a layer from its projection: [T, padded heads * v_dim]."""
    ops, c = dec.ops, dec.cfg.attn_of(li)
    H, G, M, dim, v_dim = c["num_heads"], c["num_kv_heads"], c["maps"], c["head_dim"], c["v_dim"]
    at, eps = dec.kv_index[li], dec.cfg.rms_eps
    keys, values = dec.kv.layer(at), dec.kv.values(at)
    inv_freq, factor = dec.layer_rope(c["rope"] or dict(dims=0, theta=1.0))
    nq, nk = pad8(H * M * dim), pad8(G * M * dim)
    talk, conv, gate = m.get("talk"), None, None
    if "conv" in m:
        qs, ss, pos = _batch_meta(b)
        if b.max_q_len == 1:                               # one token per sequence: inside the next kernel
            conv = ConvWindow(m["conv"], dec.rstate.conv[li], ss)
        else:
            proj = ops.causal_conv1d(proj[:, :m["conv"].shape[0]], m["conv"], None, dec.rstate.conv[li], qs, ss, pos, act=False, max_q_len=b.max_q_len)
    if c.get("gate"):
        gate = torch.empty(proj.shape[0], H, dtype=torch.float32, device=keys.device)
    q = ops.maps_prepare(proj, (0, nq, nq + nk), H * M, dim, v_dim if talk is None else G * v_dim, b.positions, b.slots, inv_freq, factor, m.get("q_norm"),
                         m.get("k_norm"), c["qk_norm"] == "full", -1.0 if c["qk_norm"] == "none" else eps, keys, values, m.get("in_bias"),
                         pairs=c.get("rope_style") == "pair", conv=conv, extra_out=gate, extra_offset=nq + nk + pad8(G * v_dim))
    terms = dict(sink=m.get("sink"), r1=m.get("r1"), r2=m.get("r2"), out_cols=m["wo"].shape[1])
    if talk is not None:
        return ops.attention_talk(q, keys, values, dim, v_dim, b, c["scale"], talk, c["window"], gate=gate, reach=m["bias_range"], **terms)
    combine = Combine(m["lam"], 1.0 - c["diff"], eps) if M == 2 else None
    return ops.attention_maps(q, keys, values, dim, v_dim, b, c["scale"], c["window"], combine, **terms)


def maps_mixer(dec, li: int, lw, h: torch.Tensor, b):
    m, ops = lw.mixer, dec.ops
    # (the convolution of longer portions reads finished rows)
    proj = ops.linear(h, m["in_proj"], defer=dec.defer_to_residual and not ("conv" in m and b.max_q_len > 1))
    return ops.linear(_attend(dec, li, m, proj, b), m["wo"], defer=dec.defer_to_residual)


def maps_lightning_mixer(dec, li: int, lw, h: torch.Tensor, b) -> NormedPair:
    m, ops, s = lw.mixer, dec.ops, dec.cfg.attn_of(li)
    qs, ss, pos = _batch_meta(b)
    H, K, V = s["lin_heads"], s["lin_k_dim"], s["lin_v_dim"]
    proj = ops.linear(h, m["in_proj"])
    ya = ops.linear(_attend(dec, li, m, proj, b), m["wo"])
    at, nk = m["lin_offset"], pad8(H * K)
    q, k, v = proj[:, at:at + H * K], proj[:, at + nk:at + nk + H * K], proj[:, at + 2 * nk:at + 2 * nk + H * V]
    gate = proj[:, at + 2 * nk + pad8(H * V):at + 2 * nk + pad8(H * V) + H * V]
    o = ops.decay_scan(q, k, v, m["lin_decay"], dec.rstate.scan[li], qs, ss, pos, H, K, V, 0, b.max_q_len, b.min_q_len)
    o = ops.gated_rmsnorm(o, gate, m["lin_norm"], s.get("norm_eps", dec.cfg.rms_eps), H * V, True, m["lin_wo"].shape[1], "sigmoid")
    return NormedPair(ya, ops.linear(o, m["lin_wo"], defer=dec.defer_to_residual), m["out_a"], m["out_b"])


MAPS_MIXERS = {"maps": maps_mixer, "maps+lightning": maps_lightning_mixer}


def pack_maps(q, k, v, q_norm, k_norm, o_proj, dtype, device, biases=None, lambdas=None, diff: float = 0.0, gate=None, convs=None,
              terms: Optional[Dict[str, torch.Tensor]] = None) -> Dict[str, object]:
    """q [H * maps * dim, in], k [G * maps * dim, in], v [G * v_dim, in], o_proj [out, H * v_dim]; ``biases``: those of q, k and v;
    ``lambdas``: the vectors lq1, lk1, lq2, lk2 of two maps; norm weights may be None; ``gate`` [H, in]; ``convs``: the taps [rows, taps]
    of q, k and v; ``terms``: fp32 numbers per head (sink, r1, r2) and the matrix over the heads (talk)."""
    put = lambda t: t.to(device=device, dtype=dtype).contiguous()
    p8 = lambda t: pad_rows(t, pad8(t.shape[0]))
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    m: Dict[str, object] = dict(in_proj=put(torch.cat([p8(t) for t in ((q, k, v) if gate is None else (q, k, v, gate))], 0)),
                                wo=put(pad_cols(o_proj, pad8(o_proj.shape[1]))))
    if q_norm is not None:
        m.update(q_norm=put(q_norm), k_norm=put(k_norm))
    if convs is not None:
        m["conv"] = f32(torch.cat([p8(t) for t in convs], 0))
    m.update({n: f32(t) for n, t in (terms or {}).items()})
    if "talk" in m:
        m["bias_range"] = bias_range(m.get("r1"), m.get("r2"))
    if biases is not None:
        m["in_bias"] = put(torch.cat([p8(t) for t in biases], 0))
    if lambdas is not None:
        a, b, c, d = (t.double() for t in lambdas)
        m["lam"] = float(torch.exp((a * b).sum()) - torch.exp((c * d).sum())) + diff
    return m


def pack_maps_lightning(attn: Dict[str, object], q, k, v, g, norm, o_proj, decay, out_a, out_b, dtype, device) -> Dict[str, object]:
    """``attn``: the attention half from :func:`pack_maps`; q, k [H * K, in], v, g [H * V, in], o_proj [out, H * V]."""
    put = lambda t: t.to(device=device, dtype=dtype).contiguous()
    p8 = lambda t: put(pad_rows(t, pad8(t.shape[0])))
    m = dict(attn)
    m["lin_offset"] = m["in_proj"].shape[0]
    m["in_proj"] = torch.cat([m["in_proj"]] + [p8(t) for t in (q, k, v, g)], 0)
    m.update(lin_decay=torch.tensor(decay, dtype=torch.float32, device=device), lin_norm=put(norm), lin_wo=put(pad_cols(o_proj, pad8(o_proj.shape[1]))),
             out_a=put(out_a), out_b=put(out_b))
    return m
