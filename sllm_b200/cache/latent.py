"""Cache of models that mix latent-attention layers with recurrent layers, each layer with sizes of its own: a token's row
is [latent | rotated key part], one row for all heads; recurrent layers keep a 32-bit [heads, dim, dim] state per slot."""
from __future__ import annotations

from ..models.config import ModelConfig
from ..ops.latent import LatentPages
from .layered import LayeredCache


class LatentHybridCache(LayeredCache):
    def __init__(self, cfg: ModelConfig, num_pages: int, device, max_seqs: int, latent_widths: dict, state_shapes: dict):
        """latent_widths: layer -> row width; state_shapes: layer -> (heads, dim)."""
        super().__init__(cfg, num_pages, device, max_seqs, {l: [(1, w)] for l, w in latent_widths.items()},
                         {l: [(h, d, d)] for l, (h, d) in state_shapes.items()})

    def wrap(self, planes: list) -> LatentPages:
        pages = planes[0].squeeze(1)
        return LatentPages(pages, pages.shape[1])
