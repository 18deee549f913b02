"""Paged pool of layers that keep rows of a layout of their own: latent attention (one row per token), attention whose values
are the keys (one row and one fp32 factor per token and key/value head) and attention of one or two maps (key rows of one
width, value rows of another, one or two keys per value). Every layer has its own shape."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..config import ModelConfig
from ..ops.latent import latent_width
from ..ops.maps import maps_width, spread_width
from ..ops.tied import tied_width


@dataclass(frozen=True)
class RowSpec:
    """Rows of ``width`` values per token; ``heads`` > 0: one per head, each with an fp32 factor, or (``value_heads`` > 0) beside
    ``value_heads`` rows of ``value_width`` values."""
    width: int
    heads: int = 0
    value_width: int = 0
    value_heads: int = 0

    def bytes_per_token(self, elem: int) -> int:
        if self.value_heads:
            return (self.heads * self.width + self.value_heads * self.value_width) * elem
        return self.heads * (self.width * elem + 4) if self.heads else self.width * elem


class RowCache:
    """Per layer that keeps rows: [blocks, block_size, width], or [blocks, heads, block_size, width] and factors
    [blocks, heads, block_size] or values [blocks, value_heads, block_size, value_width]."""

    def __init__(self, specs: List[RowSpec], num_blocks: int, block_size: int, device, dtype=torch.bfloat16):
        self.num_blocks, self.block_size = num_blocks, block_size
        shape = lambda s: (num_blocks, s.heads, block_size) if s.heads else (num_blocks, block_size)
        self.rows = [torch.zeros(*shape(s), s.width, device=device, dtype=dtype) for s in specs]
        self.factors: List[Optional[torch.Tensor]] = [torch.zeros(shape(s), device=device, dtype=torch.float32) if s.heads and not s.value_heads else None
                                                      for s in specs]
        self.value_rows: List[Optional[torch.Tensor]] = [torch.zeros(num_blocks, s.value_heads, block_size, s.value_width, device=device, dtype=dtype)
                                                         if s.value_heads else None for s in specs]

    def layer(self, i: int) -> torch.Tensor:
        return self.rows[i]

    def factor(self, i: int) -> torch.Tensor:
        return self.factors[i]

    def values(self, i: int) -> torch.Tensor:
        return self.value_rows[i]

    def copy_block(self, src: int, dst: int) -> None:
        for t in self.rows + [f for f in self.factors + self.value_rows if f is not None]:
            t[dst].copy_(t[src])

    @staticmethod
    def specs(cfg: ModelConfig, layer_range) -> List[RowSpec]:
        out = []
        for li in layer_range:
            if not cfg.has_kv(li):
                continue
            if cfg.layer_kind(li) == "mla":
                c = cfg.mla_of(li)
                R, dr = c["kv_lora_rank"], c["qk_rope_head_dim"]
                out.append(RowSpec(latent_width(R, dr) if cfg.layer_mixers else R + dr))
            elif cfg.layer_kind(li) == "tied":
                c = cfg.attn_of(li)
                out.append(RowSpec(tied_width(c["head_dim"]), c["num_kv_heads"]))
            elif cfg.layer_kind(li) in ("maps", "maps+lightning"):
                c = cfg.attn_of(li)
                one = c.get("talk")                # heads that mix their weights read the values of all heads as one row
                out.append(RowSpec(maps_width(c["head_dim"]), c["num_kv_heads"] * c["maps"], spread_width(c["num_kv_heads"] * c["v_dim"]) if one else
                                   maps_width(c["v_dim"]), 1 if one else c["num_kv_heads"]))
        return out

    @staticmethod
    def bytes_per_block(specs: List[RowSpec], block_size: int, elem: int = 2) -> int:
        return sum(s.bytes_per_token(elem) for s in specs) * block_size
