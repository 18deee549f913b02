"""Multi-head latent attention (DeepSeek-V2 / V3 family) as a layer kind of the decoder runner.

A token is cached as one row: the normalised KV latent (``kv_lora_rank`` values) followed by the rotated shared key
part (``qk_rope_head_dim`` values). The key up-projection is absorbed into the query and the value up-projection
is applied after the softmax, so attention itself is multi-query over those rows for prefill and decode alike
(the reference keeps an expanded prefill path in rust/engine/cuda/mla.cu next to the latent one in
rust/engine/cuda/mla_latent.cu / mla_decode.cu and rust/engine/src/rust_decoder/mla_latent.rs; here the latent form
is the only one).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config import ModelConfig


def mla_block(dec, li: int, lw, h: torch.Tensor, b) -> torch.Tensor:
    cfg, m, ops = dec.cfg, lw.mixer, dec.ops
    if "in_proj" in m:
        return latent_block(dec, li, lw, h, b)
    c = cfg.mla_of(li)
    H, dn, dr, dv, R = cfg.num_heads, c["qk_nope_head_dim"], c["qk_rope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
    T = h.shape[0]
    if "q_a" in m:
        q = ops.linear(ops.rmsnorm(ops.linear(h, m["q_a"]), None, m["q_a_norm"], cfg.rms_eps), m["q_b"])
    else:
        q = ops.linear(h, m["q_proj"])
    q = q.view(T, H, dn + dr)
    ckv = ops.linear(h, m["kv_a"])                                     # [T, pad8(R + dr)]
    cache = dec.kv.layer(dec.kv_index[li])
    q_pe = ops.mla_prepare(ckv, q, dn, b.positions, b.slots, dec.inv_freq, dec.attn_factor, m["kv_a_norm"], cfg.rms_eps, cache)
    q_abs = torch.bmm(q[:, :, :dn].transpose(0, 1), m["w_uk"])                                # [H, T, R]
    o_lat = ops.attention_mla(q_abs, q_pe, cache, b.block_tables, b.row_seq, b.positions, dec.scale, b.max_kv_len)     # [H, T, R]
    o = torch.bmm(o_lat, m["w_uv"]).transpose(0, 1).reshape(T, H * dv)
    return ops.linear(o, m["wo"], m.get("bo"))


def latent_block(dec, li: int, lw, h: torch.Tensor, b) -> torch.Tensor:
    """Latent attention of any size, with sizes, softmax scale and rotation of the layer's own, an optional sigmoid gate per
    head, and optionally another layer's cached rows (``kv_from``). One projection makes [q | latent, shared key part |
    head gates]; the absorbed query and its rotated part share one row, laid out like a cache row."""
    m, ops, c = lw.mixer, dec.ops, dec.cfg.mla_of(li)
    H, dn, dr, dv, R = c["num_heads"], c["qk_nope_head_dim"], c["qk_rope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
    T, pad8 = h.shape[0], lambda n: (n + 7) // 8 * 8
    cache = dec.kv.layer(dec.kv_index[dec.cfg.kv_source(li)])
    proj = ops.linear(h, m["in_proj"])
    nq, own = pad8(H * (dn + dr)), c.get("kv_from") is None
    q = proj[:, :H * (dn + dr)]
    ckv = proj[:, nq:nq + R + dr] if own else None
    ql = torch.empty(H, T, cache.shape[-1], dtype=h.dtype, device=h.device)
    q_nope = q.as_strided((H, T, dn), (dn + dr, proj.stride(0), 1))
    ops.bmm(q_nope, m["w_uk"], out=ql[:, :, :R])
    ops.latent_prepare(ckv, q, dn + dr, dn, b.positions, b.slots, dec.rope_table(dr, c["rope_theta"]), 1.0, m.get("kv_norm"),
                       dec.cfg.rms_eps, cache, ql, R, 0 if c.get("rope_style") == "neox" else 1)
    o = ops.bmm(ops.attention_latent(ql, cache, b, c["scale"], R), m["w_uv"])                     # [H, T, dv]
    og = nq + (pad8(R + dr) if own else 0)
    gate = proj[:, og:og + H] if c.get("head_gate") else None
    return ops.linear(ops.head_gate(o, gate, m["wo"].shape[1]), m["wo"], defer=getattr(dec, "defer_to_residual", False))


def pack_latent(q, dkv, kv_norm, uk, uv, gate, o_proj, c: Dict, dtype, device) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors of a layer ``latent_block`` runs: q [H * (dn + dr), in], dkv [R + dr, in] and its norm (None with
    shared rows), uk [H * dn, R], uv [H * dv, R], gate [H, in] or None, o_proj [out, H * dv]. Row counts are padded to
    multiples of 8."""
    from .recurrent import pad8, pad_cols, pad_rows
    H, dn, dv, R = c["num_heads"], c["qk_nope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
    bf = lambda t: t.to(device=device, dtype=dtype).contiguous()
    parts = [pad_rows(t, pad8(t.shape[0])) for t in (q, dkv, gate) if t is not None]
    m = dict(in_proj=bf(torch.cat(parts, 0)), w_uk=bf(uk.view(H, dn, R)), w_uv=bf(uv.view(H, dv, R).transpose(1, 2)),
             wo=bf(pad_cols(o_proj, pad8(H * dv))))
    if dkv is not None:
        m["kv_norm"] = bf(kv_norm)
    return m


def pack_mla(q_a, q_a_norm, q_b, q_proj, kv_a, kv_a_norm, kv_b, o_proj, cfg: ModelConfig, dtype, device) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors -> the runner's layout: kv_b [H * (dn + dv), R] is cut into the absorbed key matrix
    w_uk [H, dn, R] and the value matrix w_uv [H, R, dv]; kv_a is padded to a multiple of 8 rows."""
    c = cfg.mla
    H, dn, dv, R = cfg.num_heads, c["qk_nope_head_dim"], c["v_head_dim"], c["kv_lora_rank"]
    bf = lambda t: t.to(device=device, dtype=dtype).contiguous()
    kvb = kv_b.view(H, dn + dv, R)
    rows = (kv_a.shape[0] + 7) // 8 * 8
    kva = torch.zeros(rows, kv_a.shape[1], dtype=kv_a.dtype)
    kva[:kv_a.shape[0]] = kv_a
    m = dict(kv_a=bf(kva), kv_a_norm=bf(kv_a_norm), w_uk=bf(kvb[:, :dn, :]), w_uv=bf(kvb[:, dn:, :].transpose(1, 2)), wo=bf(o_proj))
    if q_proj is not None:
        m["q_proj"] = bf(q_proj)
    else:
        m.update(q_a=bf(q_a), q_a_norm=bf(q_a_norm), q_b=bf(q_b))
    return m


def init_random_mla(cfg: ModelConfig, full, li: int, dtype, device) -> Dict[str, torch.Tensor]:
    c = cfg.mla
    H, dn, dr, dv, R, Hd = cfg.num_heads, c["qk_nope_head_dim"], c["qk_rope_head_dim"], c["v_head_dim"], c["kv_lora_rank"], cfg.hidden_size
    ql = c.get("q_lora_rank")
    ones = lambda n: torch.ones(n, dtype=dtype)
    cpu = lambda t: t.cpu()
    if ql:
        q = dict(q_a=cpu(full((ql, Hd), li, 40)), q_a_norm=ones(ql), q_b=cpu(full((H * (dn + dr), ql), li, 41)), q_proj=None)
    else:
        q = dict(q_a=None, q_a_norm=None, q_b=None, q_proj=cpu(full((H * (dn + dr), Hd), li, 40)))
    return pack_mla(q["q_a"], q["q_a_norm"], q["q_b"], q["q_proj"], cpu(full((R + dr, Hd), li, 42)), ones(R),
                    cpu(full((H * (dn + dv), R), li, 43)), cpu(full((Hd, H * dv), li, 44)), cfg, dtype, device)
