"""Paged pool of layers that keep rows of a layout of their own: latent attention (one row per token) and attention whose
values are the keys (one row and one fp32 factor per token and key/value head). Every layer has its own shape."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..config import ModelConfig
from ..ops.latent import latent_width
from ..ops.tied import tied_width


@dataclass(frozen=True)
class RowSpec:
    """Rows of ``width`` values per token; ``heads`` > 0: one per head, each with an fp32 factor."""
    width: int
    heads: int = 0

    def bytes_per_token(self, elem: int) -> int:
        return self.heads * (self.width * elem + 4) if self.heads else self.width * elem


class RowCache:
    """Per layer that keeps rows: [blocks, block_size, width], or [blocks, heads, block_size, width] and factors
    [blocks, heads, block_size]."""

    def __init__(self, specs: List[RowSpec], num_blocks: int, block_size: int, device, dtype=torch.bfloat16):
        self.num_blocks, self.block_size = num_blocks, block_size
        shape = lambda s: (num_blocks, s.heads, block_size) if s.heads else (num_blocks, block_size)
        self.rows = [torch.zeros(*shape(s), s.width, device=device, dtype=dtype) for s in specs]
        self.factors: List[Optional[torch.Tensor]] = [torch.zeros(shape(s), device=device, dtype=torch.float32) if s.heads else None for s in specs]

    def layer(self, i: int) -> torch.Tensor:
        return self.rows[i]

    def factor(self, i: int) -> torch.Tensor:
        return self.factors[i]

    def copy_block(self, src: int, dst: int) -> None:
        for t in self.rows + [f for f in self.factors if f is not None]:
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
        return out

    @staticmethod
    def bytes_per_block(specs: List[RowSpec], block_size: int, elem: int = 2) -> int:
        return sum(s.bytes_per_token(elem) for s in specs) * block_size
