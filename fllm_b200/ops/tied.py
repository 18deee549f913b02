"""Attention whose values are the keys, and the residual with the norm after the sum: the fp32 PyTorch statement of each op
(``TiedRef``, mixed into the reference ops) and the wrappers of the sm_100a kernels (``TiedNative``).

A token caches one row per key/value head, the projected key, padded with zeros, and one fp32 factor (the reciprocal root mean
square of the key where keys are normalised). The factor multiplies the key where it meets a query, not where it is a value;
every query head has an fp32 factor of its own (norm, temperature by position, softmax scale). Normalised keys and queries
therefore exist only inside the fp32 scores.

The residual is fp32 [rows, width]. ``postnorm_step`` with ``add`` off is ``x <- rms(alpha x + y) w``, with ``add`` on
``x <- x + rms(y) w``; it returns the row in the activation type, or its final norm. Its ``y`` may be a pair of projections
with norms of their own (``ops.maps.NormedPair``).
"""
from __future__ import annotations

import torch
import torch.nn.functional as F


def tied_width(dim: int) -> int:
    """Padded length of a cache row: the widths of the tensor-core kernels, or a multiple of 16."""
    return 64 if dim <= 64 else (128 if dim <= 128 else (dim + 15) // 16 * 16)


def _rms(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


class TiedRef:
    def tied_prepare(self, x, k_offset, heads, dim, positions, slots, eps, scale, temp_coef, temp_every, cache, key_factor):
        """``x`` [T, >= k_offset + G dim]: query heads from column 0, key heads from ``k_offset``. Writes the tokens' cache rows
        and factors (slot < 0: none); returns (queries, query factors fp32 [T, heads]). ``eps`` < 0: no norms."""
        T, G, bs = x.shape[0], cache.shape[1], cache.shape[2]
        inv = lambda v: torch.rsqrt(v.pow(2).mean(-1) + eps) if eps >= 0 else torch.ones(v.shape[:-1], device=v.device)
        q = x[:, :heads * dim]
        k = x[:, k_offset:k_offset + G * dim].reshape(T, G, dim)
        temp = 1 + temp_coef * torch.log(torch.floor((positions[:T] + 1).float() / temp_every) + 1)
        qf = scale * temp[:, None] * inv(q.float().reshape(T, heads, dim))
        keep = slots[:T] >= 0
        s = slots[:T][keep].long()
        cache[s // bs, :, s % bs] = F.pad(k[keep], (0, cache.shape[3] - dim)).to(cache.dtype)
        key_factor[s // bs, :, s % bs] = inv(k[keep].float())
        return q, qf

    def attention_tied(self, q, q_factor, cache, key_factor, dim, b, softcap=0.0, out_cols=0, tensor_cores=True, splits=None):
        """q [T, H dim] against the rows every token may see -> [T, out_cols or H dim]. ``b``: the step batch."""
        T, H = q_factor.shape
        G, bs = cache.shape[1], cache.shape[2]
        out = torch.zeros(T, max(out_cols, H * dim), dtype=q.dtype, device=q.device)
        for t in range(T):
            n = int(b.positions[t]) + 1
            blocks = b.block_tables[int(b.row_seq[t]), :(n + bs - 1) // bs].long()
            k = cache[blocks].transpose(1, 2).reshape(-1, G, cache.shape[3])[:n, :, :dim].float()              # [n, G, dim]
            f = key_factor[blocks].transpose(1, 2).reshape(-1, G)[:n]
            qt = (q[t, :H * dim].float().view(G, H // G, dim))
            s = torch.einsum("ghd,ngd->ghn", qt, k) * f.t()[:, None] * q_factor[t].view(G, H // G)[:, :, None]
            if softcap > 0:
                s = softcap * torch.tanh(s / softcap)
            out[t, :H * dim] = torch.einsum("ghn,ngd->ghd", torch.softmax(s, -1), k).reshape(-1).to(out.dtype)
        return out

    def _row_out(self, x, final_w, final_scale, width, eps, rows, dtype):
        if rows is not None:
            x = x[rows.long()]
        if final_w is None:
            return x.to(dtype)
        return F.pad(_rms(x[:, :width], eps) * final_scale, (0, x.shape[1] - width)).mul(final_w.float()).to(dtype)

    def postnorm_begin(self, ids, table, scale):
        """-> (residual, first input)."""
        x = table[ids.long()].float() * scale
        return x, x.to(table.dtype)

    def postnorm_step(self, x, y, norm_w, width, eps, alpha=1.0, add=False, final_w=None, final_scale=1.0, rows=None):
        """``rows`` (with ``final_w``): only these rows, the residual is left as it is. ``y``: a tensor or a NormedPair."""
        if hasattr(y, "wa"):
            norm = lambda t, w: F.pad(_rms(t.float()[:, :width], eps), (0, x.shape[1] - width)) * w.float()
            y = 0.5 * (norm(y.a, y.wa) + norm(y.b, y.wb))
        y = y.float()
        v = y if add else alpha * x + y
        v = F.pad(_rms(v[:, :width], eps), (0, x.shape[1] - width)) * norm_w.float()
        new = x + v if add else v
        if rows is None:
            x.copy_(new)
        return self._row_out(new, final_w, final_scale, width, eps, rows, norm_w.dtype)

    def side_gate(self, gate, ids, table, offset, dim):
        """gelu_tanh(gate) * the layer's slice of the tokens' rows of ``table``; zeros behind ``dim``."""
        e = table[ids[:gate.shape[0]].long(), offset:offset + dim].float()
        return F.pad(F.gelu(gate[:, :dim].float(), approximate="tanh") * e, (0, gate.shape[1] - dim)).to(gate.dtype)


class TiedNative:
    """Kernel wrappers; ``self.k`` is the loaded extension and ``self.launches`` the launch counter of the ops object. ``x``, ``y``
    and ``gate`` may be deferred projections: their split-K partial sums are added by the kernel."""

    def tied_prepare(self, x, k_offset, heads, dim, positions, slots, eps, scale, temp_coef, temp_every, cache, key_factor):
        T, splits = x.shape[0], getattr(x, "splits", 0)
        qf = torch.empty(T, heads, dtype=torch.float32, device=cache.device)
        q = torch.empty(T, heads * dim, dtype=cache.dtype, device=cache.device) if splits else x[:, :heads * dim]
        self.k.tied_prepare(None if splits else x, self.workspace if splits else None, int(splits), int(x.shape[1]), q if splits else None, int(k_offset),
                            int(dim), positions, slots, float(eps), float(scale), float(temp_coef), float(temp_every), qf, cache, key_factor)
        self.launches += 1
        return q, qf

    def attention_tied(self, q, q_factor, cache, key_factor, dim, b, softcap=0.0, out_cols=0, tensor_cores=True, splits=None):
        T, H = q_factor.shape
        make = torch.zeros if out_cols > H * dim else torch.empty
        out = make(T, max(out_cols, H * dim), dtype=q.dtype, device=q.device)
        if splits is None:
            splits = int(self.k.attention_tied_splits(b.num_seqs, b.max_q_len, H, cache.shape[1], b.max_kv_len)) if q.dtype == torch.bfloat16 else 1
        ws = None
        if splits > 1:
            need = int(self.k.attention_tied_workspace_bytes(T, H, cache.shape[3], splits))
            held = self.__dict__.setdefault("_tied_ws", [])        # grow-only; captured graphs may still use the smaller ones
            if not held or held[-1].numel() < need:
                held.append(torch.empty(need, dtype=torch.uint8, device=q.device))
            ws = held[-1]
        self.launches += self.k.attention_tied(q, q_factor, cache, key_factor, int(dim), b.block_tables, b.row_seq, b.positions, b.q_starts, out,
                                               b.num_seqs, b.max_q_len, b.min_q_len, float(softcap), int(splits), ws, bool(tensor_cores), self.status)
        return out

    def postnorm_begin(self, ids, table, scale):
        T, ld = ids.numel(), table.shape[1]
        x = torch.empty(T, ld, dtype=torch.float32, device=table.device)
        h = torch.empty(T, ld, dtype=table.dtype, device=table.device)
        self.k.postnorm(x, ids, table, float(scale), None, None, 0, False, 0.0, None, None, 1.0, None, h, ld, 0.0, True, None, None, None)
        self.launches += 1
        return x, h

    def postnorm_step(self, x, y, norm_w, width, eps, alpha=1.0, add=False, final_w=None, final_scale=1.0, rows=None):
        h = torch.empty(x.shape[0] if rows is None else rows.numel(), x.shape[1], dtype=norm_w.dtype, device=x.device)
        first, wa, wb = (y.a, y.wa, y.wb) if hasattr(y, "wa") else (None, None, None)
        y = y.b if first is not None else y
        splits = getattr(y, "splits", 0)
        self.k.postnorm(x, None, None, 1.0, None if splits else y, self.workspace if splits else None, int(splits), bool(add), float(alpha), norm_w, final_w,
                        float(final_scale), rows, h, int(width), float(eps), rows is None, first, wa, wb)
        self.launches += 1
        return h

    def side_gate(self, gate, ids, table, offset, dim):
        splits = getattr(gate, "splits", 0)
        out = torch.empty(gate.shape[0], gate.shape[1], dtype=table.dtype, device=table.device)
        self.k.side_gate(None if splits else gate, self.workspace if splits else None, int(splits), ids, table, int(offset), int(dim), out)
        self.launches += 1
        return out
