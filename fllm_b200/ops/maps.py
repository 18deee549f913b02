"""Attention of one or two maps over shared values, and the recurrence of lightning attention: the fp32 PyTorch statement of each
op (``MapsRef``, mixed into the reference ops) and the wrappers of the sm_100a kernels (``MapsNative``).

A map is a softmax attention with queries and keys of its own. Every query head has ``maps`` of them over the values of its
key/value head; two maps are combined as ``rms(a1 - lam a2) * out_scale`` over the head's values. Map m of query head h is row
``h * maps + m`` of the query heads and reads key row ``g * maps + m``. Cache rows are padded with zeros to ``maps_width``; key
and value rows have widths of their own. A query at position i sees the keys j with 0 <= i - j < window (0: all up to i).

One map may have a sink per head (``exp(sink)`` joins the denominator) and a distance bias per head (``r1 ln(1 + r2 (i - j))`` is
taken off a score). Talking heads (``attention_talk``) mix the weights of all heads with a matrix before they meet the values; the
cache then holds one value row per token with the values of all key/value heads, so that every head can weigh all of them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .latent import _rotate
from .tied import tied_width


DECAY_CHUNK_TOKENS = 32          # sequences with at least this many tokens in a step run lightning attention in matrix form


def maps_width(dim: int) -> int:
    """Padded length of a key, value or query row."""
    return tied_width(dim)


def spread_width(dim: int) -> int:
    """Padded length of a row with the values of all heads."""
    return 64 if dim <= 64 else (dim + 127) // 128 * 128


MAX_BIAS_RANGE = 100.0           # (log2 units) a distance bias that changes more inside a tile of keys runs on the CUDA cores


def bias_range(r1, r2) -> float:
    """The most a distance bias can change between the tokens and the keys of one tile (within 320 of each other), in log2 units."""
    return 0.0 if r1 is None else float((r1.double().abs() * torch.log2(1 + r2.double() * 320)).nan_to_num(1e9).max())


@dataclass
class ConvWindow:
    """A causal convolution in front of the preparation of a step whose sequences have one token each: weights fp32 [columns, taps],
    state rows [slots, taps - 1, columns] that move on by the token, and the sequences' rows."""
    weight: torch.Tensor
    state: torch.Tensor
    seq_state: torch.Tensor


@dataclass
class Combine:
    """How the two maps of a head become its output."""
    lam: float
    out_scale: float
    eps: float


@dataclass
class NormedPair:
    """A sublayer output that is half the sum of two projections, each over its root mean square times a weight. ``b`` may be a
    deferred projection; ``postnorm_step`` takes the pair in place of a tensor."""
    a: torch.Tensor
    b: object
    wa: torch.Tensor
    wb: torch.Tensor


def _rms(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


class MapsRef:
    def maps_prepare(self, x, offsets, heads, dim, v_dim, positions, slots, inv_freq, rope_factor, q_norm, k_norm, full, eps, k_cache, v_cache, bias=None,
                     pairs=False, conv: Optional[ConvWindow] = None, extra_out=None, extra_offset=0):
        """``x`` [T, ...] (plus ``bias``): query maps at column offsets[0], key maps at offsets[1], values at offsets[2]. Norms (over a map, or with
        ``full`` over all maps at once; ``eps`` < 0: none; weights None: without weights), rotates the first 2 len(inv_freq) values of every
        map (values i and i + rot / 2, or with ``pairs`` 2 i and 2 i + 1), writes the tokens' cache rows (slot < 0: none) and returns the
        queries [T, heads, W], padded like the key rows. ``conv``: runs in front of it all (steps of single tokens). ``extra_out`` fp32
        [T, n] receives the columns from ``extra_offset`` on."""
        T, W, bs = x.shape[0], k_cache.shape[3], k_cache.shape[2]
        rot = 2 * inv_freq.numel()
        x = x.float() if bias is None else x.float() + bias.float()
        if extra_out is not None:
            extra_out.copy_(x[:, extra_offset:extra_offset + extra_out.shape[1]])
        if conv is not None:
            C, taps = conv.weight.shape
            rows = conv.seq_state[:T].long()
            seen = torch.where((positions[:T] == 0)[:, None, None], torch.zeros(1, device=x.device), conv.state[rows].float())
            seen = torch.cat([seen, x[:, None, :C]], 1)
            conv.state[rows] = seen[:, 1:].to(conv.state.dtype)
            x = (seen * conv.weight.t()).sum(1)

        def part(off, n, w):
            t = x[:, off:off + n * dim]
            t = t if full else t.reshape(T, n, dim)
            if eps >= 0:
                t = _rms(t, eps) if w is None else _rms(t, eps) * w.float()
            t = t.reshape(T, n, dim)
            turned = _rotate(t[..., :rot], positions, inv_freq, rope_factor, 1 if pairs else 0) if rot else t[..., :0]
            return F.pad(torch.cat([turned, t[..., rot:]], -1), (0, W - dim)).to(k_cache.dtype)
        q, k = part(offsets[0], heads, q_norm), part(offsets[1], k_cache.shape[1], k_norm)
        G = v_cache.shape[1]
        v = F.pad(x[:, offsets[2]:offsets[2] + G * v_dim].reshape(T, G, v_dim), (0, v_cache.shape[3] - v_dim)).to(v_cache.dtype)
        keep = slots[:T] >= 0
        s = slots[:T][keep].long()
        k_cache[s // bs, :, s % bs] = k[keep]
        v_cache[s // bs, :, s % bs] = v[keep]
        return q

    @staticmethod
    def _distance(s, n, lo, r1, r2):
        """Scores [G, heads of a group, ..., keys lo .. n - 1] of a query at position n - 1 without their distance bias."""
        if r1 is None:
            return s
        d = n - 1 - torch.arange(lo, n, device=s.device)
        return s - (r1.float()[:, None] * torch.log1p(r2.float()[:, None] * d)).view(s.shape)

    @staticmethod
    def _weights(s, sink):
        """Softmax over the last dimension with the heads' sinks in the denominator."""
        if sink is None:
            return torch.softmax(s, -1)
        return torch.softmax(torch.cat([s, sink.float().view(*s.shape[:-1], 1)], -1), -1)[..., :-1]

    def attention_maps(self, q, k_cache, v_cache, dim, v_dim, b, scale, window=0, combine: Optional[Combine] = None, out_cols=0, tensor_cores=True, splits=None,
                       sink=None, r1=None, r2=None):
        """q [T, heads * maps, W] against the rows every token may see -> [T, out_cols or heads * v_dim]. ``b``: the step batch.
        ``sink``, ``r1``, ``r2``: fp32, one per head of one map."""
        T, HM = q.shape[:2]
        G, bs = v_cache.shape[1], v_cache.shape[2]
        M = k_cache.shape[1] // G
        H = HM // M
        out = torch.zeros(T, max(out_cols, H * v_dim), dtype=q.dtype, device=q.device)
        for t in range(T):
            n = int(b.positions[t]) + 1
            lo = max(0, n - window) if window > 0 else 0
            blocks = b.block_tables[int(b.row_seq[t]), lo // bs:(n + bs - 1) // bs].long()
            cut = slice(lo - lo // bs * bs, n - lo // bs * bs)
            k = k_cache[blocks].transpose(1, 2).reshape(-1, G, M, k_cache.shape[3])[cut].float()
            v = v_cache[blocks].transpose(1, 2).reshape(-1, G, v_cache.shape[3])[cut, :, :v_dim].float()
            s = torch.einsum("ghmd,ngmd->ghmn", q[t].float().view(G, H // G, M, -1), k) * scale
            a = torch.einsum("ghmn,ngd->ghmd", self._weights(self._distance(s, n, lo, r1, r2), sink), v)
            y = _rms(a[:, :, 0] - combine.lam * a[:, :, 1], combine.eps) * combine.out_scale if M == 2 else a[:, :, 0]
            out[t, :H * v_dim] = y.reshape(-1).to(out.dtype)
        return out

    def attention_talk(self, q, k_cache, v_cache, dim, v_dim, b, scale, talk, window=0, sink=None, r1=None, r2=None, gate=None, out_cols=0, tensor_cores=True,
                       splits=None, reach=None):
        """Talking heads: head h weighs the values of its key/value head with sum_f talk[h, f] (weights of head f); its output is
        scaled by sigmoid(gate[:, h]). Value rows [.., 1, .., width] hold all heads' values (``v_dim`` each). ``reach``: the
        ``bias_range`` of r1 and r2 (None: it is computed, which waits for the device)."""
        T, H = q.shape[:2]
        G, bs = k_cache.shape[1], k_cache.shape[2]
        out = torch.zeros(T, max(out_cols, H * v_dim), dtype=q.dtype, device=q.device)
        for t in range(T):
            n = int(b.positions[t]) + 1
            lo = max(0, n - window) if window > 0 else 0
            blocks = b.block_tables[int(b.row_seq[t]), lo // bs:(n + bs - 1) // bs].long()
            cut = slice(lo - lo // bs * bs, n - lo // bs * bs)
            k = k_cache[blocks].transpose(1, 2).reshape(-1, G, k_cache.shape[3])[cut].float()
            v = v_cache[blocks].reshape(-1, v_cache.shape[3])[cut, :G * v_dim].float().view(-1, G, v_dim)
            s = torch.einsum("ghd,ngd->ghn", q[t].float().view(G, H // G, -1), k) * scale
            w = self._weights(self._distance(s, n, lo, r1, r2), sink).reshape(H, -1)
            y = torch.einsum("ghn,ngd->ghd", (talk.float() @ w).view(G, H // G, -1), v).reshape(H, v_dim)
            if gate is not None:
                y = y * torch.sigmoid(gate[t, :H].float())[:, None]
            out[t, :H * v_dim] = y.reshape(-1).to(out.dtype)
        return out

    def decay_scan(self, q, k, v, decay, state, q_starts, seq_state, positions, H, K, V, width=0, max_q_len=0, min_q_len=0, chunk_from=0):
        """Per head S <- decay S + silu(v) silu(k)^T, o = S silu(q), with S [V, K] in fp32: [T, width or H * V]."""
        from .recurrent import _seqs
        T = q.shape[0]
        out = torch.zeros(T, max(width, H * V), dtype=v.dtype, device=v.device)
        d = decay.float()[:, None, None]
        act = lambda x, n: F.silu(x.float()).reshape(-1, H, n)
        for t0, t1, slot, fresh in _seqs(q_starts, seq_state, positions):
            S = torch.zeros(H, V, K, dtype=torch.float32, device=v.device) if fresh else state[slot].clone()
            qf, kf, vf = act(q[t0:t1], K), act(k[t0:t1], K), act(v[t0:t1], V)
            for i in range(t1 - t0):
                S = d * S + vf[i][:, :, None] * kf[i][:, None, :]
                out[t0 + i, :H * V] = (S * qf[i][:, None, :]).sum(-1).reshape(-1).to(out.dtype)
            state[slot] = S
        return out


class MapsNative:
    """Kernel wrappers; ``self.k`` is the loaded extension and ``self.launches`` the launch counter of the ops object. The
    projection ``maps_prepare`` reads may be deferred: its split-K partial sums are added by the kernel."""

    def maps_prepare(self, x, offsets, heads, dim, v_dim, positions, slots, inv_freq, rope_factor, q_norm, k_norm, full, eps, k_cache, v_cache, bias=None,
                     pairs=False, conv: Optional[ConvWindow] = None, extra_out=None, extra_offset=0):
        T, splits = x.shape[0], getattr(x, "splits", 0)
        bias = bias if bias is not None or not splits else x.bias
        q = torch.empty(T, heads, k_cache.shape[3], dtype=k_cache.dtype, device=k_cache.device)
        self.k.maps_prepare(None if splits else x, self.workspace if splits else None, int(splits), int(x.shape[1]), bias,
                            int(offsets[0]), int(offsets[1]), int(offsets[2]), int(dim), int(v_dim), positions, slots, inv_freq, float(rope_factor), bool(pairs),
                            q_norm, k_norm, bool(full), float(eps), q, k_cache, v_cache, conv.weight if conv else None, conv.state if conv else None,
                            conv.seq_state if conv else None, extra_out, int(extra_offset))
        self.launches += 1
        return q

    def attention_maps(self, q, k_cache, v_cache, dim, v_dim, b, scale, window=0, combine: Optional[Combine] = None, out_cols=0, tensor_cores=True, splits=None,
                       sink=None, r1=None, r2=None):
        T, HM = q.shape[:2]
        M = k_cache.shape[1] // v_cache.shape[1]
        H = HM // M
        make = torch.zeros if out_cols > H * v_dim else torch.empty
        out = make(T, max(out_cols, H * v_dim), dtype=q.dtype, device=q.device)
        if splits is None:
            splits = int(self.k.attention_maps_splits(b.num_seqs, b.max_q_len, H, v_cache.shape[1], M, b.max_kv_len, int(window))) if q.dtype == torch.bfloat16 else 1
        ws = None
        if splits > 1:
            need = int(self.k.attention_maps_workspace_bytes(T, HM, v_cache.shape[3], splits))
            held = self.__dict__.setdefault("_maps_ws", [])        # grow-only; captured graphs may still use the smaller ones
            if not held or held[-1].numel() < need:
                held.append(torch.empty(need, dtype=torch.uint8, device=q.device))
            ws = held[-1]
        c = combine or Combine(0.0, 1.0, 0.0)
        self.launches += self.k.attention_maps(q, k_cache, v_cache, int(dim), int(v_dim), b.block_tables, b.row_seq, b.positions, b.q_starts, out, b.num_seqs,
                                               b.max_q_len, b.min_q_len, float(scale), int(window), float(c.lam), float(c.out_scale), float(c.eps),
                                               int(splits), ws, bool(tensor_cores), self.status, sink, r1, r2)
        return out

    def attention_talk(self, q, k_cache, v_cache, dim, v_dim, b, scale, talk, window=0, sink=None, r1=None, r2=None, gate=None, out_cols=0, tensor_cores=True,
                       splits=None, reach=None):
        T, H = q.shape[:2]
        G, wv = k_cache.shape[1], v_cache.shape[3]
        reach = bias_range(r1, r2) if reach is None else reach
        fast = tensor_cores and q.dtype == torch.bfloat16 and reach <= MAX_BIAS_RANGE and scale > 0 and self.k.attention_spread_tc_supported(H // G, k_cache.shape[3], wv, k_cache.shape[2])
        if not fast:
            splits = 1
        elif splits is None:
            splits = int(self.k.attention_spread_splits(b.num_seqs, b.max_q_len, H, G, wv, b.max_kv_len, int(window)))
        out = torch.empty(T, max(out_cols, H * v_dim), dtype=q.dtype, device=q.device)
        part_o = torch.empty(T, H, splits, wv, dtype=torch.float32, device=q.device)
        part_ml = torch.empty(T, H, splits, 2, dtype=torch.float32, device=q.device)
        self.launches += self.k.attention_talk(q, k_cache, v_cache, int(dim), int(v_dim), b.block_tables, b.row_seq, b.positions, b.q_starts, out, b.num_seqs,
                                               b.max_q_len, b.min_q_len, float(scale), int(window), sink, r1, r2, talk, gate, part_o, part_ml,
                                               bool(fast), float(reach), self.status)
        return out

    def decay_scan(self, q, k, v, decay, state, q_starts, seq_state, positions, H, K, V, width=0, max_q_len=0, min_q_len=0, chunk_from=DECAY_CHUNK_TOKENS):
        """``max_q_len`` / ``min_q_len``: host-side bounds on a sequence's tokens in the step (0: unknown). Sequences with at least
        ``chunk_from`` tokens run in matrix form on the tensor cores where it covers the sizes; q, k and v then hold their
        activations afterwards."""
        make = torch.zeros if width > H * V else torch.empty
        out = make(q.shape[0], max(width, H * V), dtype=v.dtype, device=v.device)
        args = (decay, state, q_starts, seq_state, positions, out, int(H), int(K), int(V))
        aligned = all(t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 for t in (q, k, v)) and out.stride(0) % 2 == 0
        chunks = chunk_from > 0 and max_q_len >= chunk_from and v.dtype == torch.bfloat16 and aligned and K % 8 == 0 and V % 8 == 0 and K <= 128
        if not chunks or min_q_len < chunk_from:
            self.k.decay_scan(q, k, v, *args, False, int(chunk_from) if chunks else 0, 0)
            self.launches += 1
        if chunks:
            ld, at = q.stride(0), q.data_ptr()
            if k.stride(0) == ld == v.stride(0) and k.data_ptr() == at + 2 * H * K and v.data_ptr() == at + 4 * H * K:     # one segment behind the other
                self.act_(q.as_strided((q.shape[0], 2 * H * K + H * V), (ld, 1)), "silu")
            else:
                for t in (q, k, v):
                    self.act_(t, "silu")
            self.k.decay_scan(q, k, v, *args, True, int(chunk_from), int(max_q_len))
            self.launches += 1
        return out
