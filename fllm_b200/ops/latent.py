"""Hyper-connected residual streams and latent attention of any size: the fp32 PyTorch statement of each op
(``LatentRef``, mixed into the reference ops) and the wrappers of the sm_100a kernels (``LatentNative``).

Streams are one fp32 tensor [rows, streams, width]. A sublayer reads ``u = sum_s inp[s] x_s`` through a norm; its output y
goes back as ``x_t <- sum_s mix[s, t] x_s + out[t] y`` (any residual multiplier is part of ``out``). ``streams_step`` is
that update and the next sublayer's read and norm in one pass.

Latent attention caches one row per token, [latent | rotated shared key part | zeros], padded to a multiple of 16; a query
row has the same layout with the key up-projection absorbed into it.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F


def latent_width(rank: int, rot: int) -> int:
    """Padded length of a cache row."""
    return (rank + rot + 15) // 16 * 16


def _rotate(x, positions, inv_freq, factor, style):
    """x [T, ..., 2 * len(inv_freq)]; style 0: pairs (i, i + n / 2), 1: neighbours."""
    ang = positions[:x.shape[0]].float()[:, None] * inv_freq[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (inv_freq.numel(),)
    c, s = (torch.cos(ang) * factor).view(shape), (torch.sin(ang) * factor).view(shape)
    xf = x.float()
    if style == 0:
        a, b = xf.chunk(2, -1)
        return torch.cat([a * c - b * s, b * c + a * s], -1)
    a, b = xf[..., 0::2], xf[..., 1::2]
    return torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2)


class LatentRef:
    def _stream_norm(self, u, norm_w, norm_b, width, eps, rms, dtype):
        v = u[:, :width]
        if not rms:
            v = v - v.mean(-1, keepdim=True)
        v = v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)
        y = F.pad(v, (0, u.shape[1] - width)) * norm_w.float()
        return (y + norm_b.float() if norm_b is not None else y).to(dtype)

    def streams_begin(self, ids, table, streams, inp, norm_w, norm_b, width, eps, rms=False):
        """-> (streams, the first sublayer's input): every stream starts as the token's embedding row."""
        e = table[ids.long()].float()
        x = e[:, None, :].expand(-1, streams, -1).contiguous()
        return x, self._stream_norm(torch.einsum("s,tsd->td", inp, x), norm_w, norm_b, width, eps, rms, table.dtype)

    def streams_step(self, x, y, mix, out, inp, norm_w, norm_b, width, eps, rms=False, rows=None, write=True):
        """Update the streams behind a sublayer (in place unless ``write`` is off) and return the next one's normed input;
        ``inp`` of ones reads the sum of the streams. ``rows``: only these rows (nothing is written)."""
        xs, ys = (x, y) if rows is None else (x[rows.long()], y[rows.long()])
        new = torch.einsum("st,rsd->rtd", mix, xs) + out[None, :, None] * ys.float()[:, None, :]
        if write and rows is None:
            x.copy_(new)
        return self._stream_norm(torch.einsum("s,tsd->td", inp, new), norm_w, norm_b, width, eps, rms, norm_w.dtype)

    def bmm(self, a, m, out=None):
        y = torch.bmm(a.float(), m.float()).to(a.dtype)
        if out is not None:
            out.copy_(y)
            return out
        return y

    def latent_prepare(self, ckv, q, head, rope_offset, positions, slots, inv_freq, attn_factor, norm_w, eps, cache, q_out, rank, style):
        """Cache rows of the step's tokens (``ckv`` None: the layer reads another layer's rows) and the rotated part of
        every query into columns [rank, ...) of ``q_out`` [H, T, W]."""
        H, T, W = q_out.shape
        dr = 2 * inv_freq.numel()
        qh = q[:, :H * head].reshape(T, H, head)[..., rope_offset:rope_offset + dr]
        q_out[:, :, rank:] = 0
        q_out[:, :, rank:rank + dr] = _rotate(qh, positions, inv_freq, attn_factor, style).transpose(0, 1).to(q_out.dtype)
        if ckv is None:
            return
        lat = ckv[:, :rank].float()
        lat = lat * torch.rsqrt(lat.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
        row = torch.cat([lat, _rotate(ckv[:, rank:rank + dr], positions, inv_freq, attn_factor, style)], -1)
        keep = slots[:T] >= 0
        cache.view(-1, W)[slots[:T][keep].long()] = F.pad(row, (0, W - rank - dr)).to(cache.dtype)[keep]

    def attention_latent(self, q, cache, b, scale, rank, tensor_cores=True, splits=None):
        """q [H, T, W] against the cache rows every token may see -> [H, T, rank]. ``b``: the step batch."""
        H, T, W = q.shape
        bs = cache.shape[1]
        out = torch.empty(H, T, rank, dtype=q.dtype, device=q.device)
        for t in range(T):
            n = int(b.positions[t]) + 1
            blocks = b.block_tables[int(b.row_seq[t]), :(n + bs - 1) // bs].long()
            rows = cache[blocks].reshape(-1, W)[:n].float()
            p = torch.softmax(q[:, t].float() @ rows.T * scale, -1)
            out[:, t] = (p @ rows[:, :rank]).to(out.dtype)
        return out

    def head_gate(self, o, gate, cols):
        """o [H, T, dv] -> [T, cols]: heads side by side, each times the sigmoid of its gate logit; zeros behind."""
        H, T, dv = o.shape
        y = o.float().transpose(0, 1)
        if gate is not None:
            y = y * torch.sigmoid(gate[:, :H].float())[:, :, None]
        return F.pad(y.reshape(T, H * dv), (0, cols - H * dv)).to(o.dtype)


class LatentNative:
    """Kernel wrappers; ``self.k`` is the loaded extension and ``self.launches`` the launch counter of the ops object."""

    def streams_begin(self, ids, table, streams, inp, norm_w, norm_b, width, eps, rms=False):
        T, ld = ids.numel(), table.shape[1]
        x = torch.empty(T, streams, ld, dtype=torch.float32, device=table.device)
        h = torch.empty(T, ld, dtype=table.dtype, device=table.device)
        self.k.stream_mix_norm(x, ids, table, None, None, 0, None, None, inp, None, norm_w, norm_b, h, int(width), float(eps), bool(rms), True)
        self.launches += 1
        return x, h

    def streams_step(self, x, y, mix, out, inp, norm_w, norm_b, width, eps, rms=False, rows=None, write=True):
        """``y`` may be a deferred projection: its split-K partial sums are added here."""
        n = x.shape[0] if rows is None else rows.numel()
        h = torch.empty(n, x.shape[2], dtype=norm_w.dtype, device=x.device)
        splits = getattr(y, "splits", 0)
        self.k.stream_mix_norm(x, None, None, None if splits else y, self.workspace if splits else None, int(splits), mix, out, inp, rows,
                               norm_w, norm_b, h, int(width), float(eps), bool(rms), bool(write and rows is None))
        self.launches += 1
        return h

    def bmm(self, a, m, out=None):
        """Batched products of the absorbed projections: the vendor GEMM in bf16, the fp32 kernel in 32-bit."""
        if a.dtype != torch.float32:
            return torch.bmm(a, m) if out is None else torch.bmm(a, m, out=out)
        if out is None:
            out = torch.empty(a.shape[0], a.shape[1], m.shape[2], dtype=a.dtype, device=a.device)
        self.k.bmm_f32(a, m, out)
        self.launches += 1
        return out

    def latent_prepare(self, ckv, q, head, rope_offset, positions, slots, inv_freq, attn_factor, norm_w, eps, cache, q_out, rank, style):
        self.k.latent_prepare(ckv, q, int(head), int(rope_offset), positions, slots, inv_freq, float(attn_factor), norm_w, float(eps), cache,
                              q_out, int(rank), int(style))
        self.launches += 1

    def attention_latent(self, q, cache, b, scale, rank, tensor_cores=True, splits=None):
        H, T, _ = q.shape
        out = torch.empty(H, T, rank, dtype=q.dtype, device=q.device)
        if splits is None:
            splits = int(self.k.attention_latent_splits(b.num_seqs, T, b.max_q_len, H, b.max_kv_len)) if q.dtype == torch.bfloat16 else 1
        ws = None
        if splits > 1:
            need = int(self.k.attention_latent_workspace_bytes(T, H, rank, splits))
            held = self.__dict__.setdefault("_latent_ws", [])      # grow-only; captured graphs may still use the smaller ones
            if not held or held[-1].numel() < need:
                held.append(torch.empty(need, dtype=torch.uint8, device=q.device))
            ws = held[-1]
        self.launches += self.k.attention_latent(q, cache, b.block_tables, b.row_seq, b.positions, b.q_starts, out, b.num_seqs, b.max_q_len,
                                                 float(scale), int(splits), ws, bool(tensor_cores))
        return out

    def head_gate(self, o, gate, cols):
        out = torch.empty(o.shape[1], cols, dtype=o.dtype, device=o.device)
        self.k.head_gate(o, gate, out)
        self.launches += 1
        return out
