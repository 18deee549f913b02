"""The residual with the norm in front of a sublayer, and the token shift: the fp32 PyTorch statement of the op (``PreNormRef``, mixed
into the reference ops) and the wrapper of the sm_100a kernel (``PreNormNative``).

The residual is fp32 [rows, width], zero beyond the model's width. ``prenorm_step`` adds what a sublayer made of it (and, on request,
the tokens' embeddings) and returns the normalised rows for the next sublayer, ``x / rms(x) (offset + w)`` in the activation type.
A token shift moves every normalised row towards that of the token before it, ``h_t + (h_(t-1) - h_t) mu``; the last row of every
sequence is kept in fp32 state rows.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F


@dataclass
class TokenShift:
    mu: torch.Tensor                 # [padded width]
    state: torch.Tensor              # fp32 [slots, padded width]
    batch: object                    # the step batch


class PreNormRef:
    def prenorm_step(self, x, y, norm_w, width, eps, offset=1.0, ids=None, table=None, shift: Optional[TokenShift] = None, rows=None):
        """``x`` None: the residual starts here. ``ids``, ``table``: rows of the table are added. ``rows``: only these rows, the residual is
        left as it is. Returns (the new residual, the normalised rows)."""
        from .recurrent import _seqs
        new = torch.zeros(ids.numel(), table.shape[1], device=table.device) if x is None else x
        new = new if y is None else new + y.float()
        if ids is not None:
            new = new + table[ids.long()].float()
        v = new if rows is None else new[rows.long()]
        h = v[:, :width] * torch.rsqrt(v[:, :width].pow(2).mean(-1, keepdim=True) + eps)
        h = F.pad(h, (0, v.shape[1] - width)) * (offset + norm_w.float())
        if shift is not None:
            before = torch.empty_like(h)
            for t0, t1, slot, fresh in _seqs(shift.batch.q_starts, shift.batch.seq_state, shift.batch.positions):
                before[t0] = 0 if fresh else shift.state[slot]
                before[t0 + 1:t1] = h[t0:t1 - 1]
                shift.state[slot] = h[t1 - 1]
            h = h + (before - h) * shift.mu.float()
        return new, h.to(norm_w.dtype)


class PreNormNative:
    """Kernel wrapper; ``y`` may be a deferred projection: its split-K partial sums are added by the kernel."""

    def prenorm_step(self, x, y, norm_w, width, eps, offset=1.0, ids=None, table=None, shift: Optional[TokenShift] = None, rows=None):
        n, ld, splits = (x.shape[0] if x is not None else ids.numel()), norm_w.numel(), getattr(y, "splits", 0)
        h = torch.empty(n if rows is None else rows.numel(), ld, dtype=norm_w.dtype, device=norm_w.device)
        # with a token shift rows are read again by other CTAs, so the new residual gets a buffer of its own
        new = x if x is not None and shift is None else torch.empty(n, ld, dtype=torch.float32, device=norm_w.device)
        seqs = (shift.mu, shift.state, shift.batch.q_starts, shift.batch.seq_state, shift.batch.row_seq, shift.batch.positions, shift.batch.max_q_len == 1) \
            if shift is not None else (None,) * 6 + (False,)
        self.k.prenorm(x, new if rows is None else None, ids, table, None if splits else y, self.workspace if splits else None, int(splits), norm_w, float(offset),
                       int(n), int(width), float(eps), rows, h, *seqs)
        self.launches += 1
        return new, h
