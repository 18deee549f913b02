"""Attention whose values are the projected keys ("tied"), as a layer kind of the decoder runner: no value projection, queries
and keys over their root mean square per head, a query temperature that grows with the position, a soft cap on the scores, no
rotation. One projection makes [queries | keys]."""
from __future__ import annotations

from typing import Dict

import torch

from .recurrent import pad8, pad_cols, pad_rows


def tied_attention_mixer(dec, li: int, lw, h: torch.Tensor, b) -> torch.Tensor:
    m, ops, c = lw.mixer, dec.ops, dec.cfg.attn_of(li)
    H, dim, at = c["num_heads"], c["head_dim"], dec.kv_index[li]
    cache, factor = dec.kv.layer(at), dec.kv.factor(at)
    qk = ops.linear(h, m["in_proj"], defer=dec.defer_to_residual)
    q, qf = ops.tied_prepare(qk, pad8(H * dim), H, dim, b.positions, b.slots, c.get("norm_eps", dec.cfg.rms_eps), c["scale"], c.get("temp_coef", 0.0),
                             c.get("temp_every", 1.0), cache, factor)
    a = ops.attention_tied(q, qf, cache, factor, dim, b, c.get("softcap", 0.0), m["wo"].shape[1])
    return ops.linear(a, m["wo"], defer=dec.defer_to_residual)


def pack_tied(q, k, o_proj, dtype, device) -> Dict[str, torch.Tensor]:
    """q [H * dim, in], k [G * dim, in], o_proj [out, H * dim]; row counts are padded to multiples of 8."""
    put = lambda t: t.to(device=device, dtype=dtype).contiguous()
    return dict(in_proj=put(torch.cat([pad_rows(t, pad8(t.shape[0])) for t in (q, k)], 0)), wo=put(pad_cols(o_proj, pad8(o_proj.shape[1]))))
