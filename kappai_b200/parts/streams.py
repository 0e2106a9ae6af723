"""A residual of several streams ("hyper-connections"): ``streams`` (category ``residual``).

Between the layers a row is ``streams`` float32 vectors that all start as the embedding output; what it stands for is their
sum.  The arrangement ``streams_residual`` (block.py) reads and writes the streams; this part makes them at the model's
entry and norms their sum, for picked rows, at its end (csrc/streams.cu).

Params: streams, hidden_size.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.schema import ConfigError
from ..ops import kernels as K
from .base import Part, register_part


def stream_norm(norm) -> bool:
    """Is ``norm`` centred?  (The kernels that read streams compute the layer norm without a shift and the RMS norm.)"""
    kind = type(norm).__name__
    if kind not in ("LayerNorm", "RMSNorm"):
        raise ConfigError(f"streams: a norm of the kind {kind} is not computed on streams")
    return kind == "LayerNorm"


class Streams(Part):
    category = "residual"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.S = int(self._p("streams"))
        self.d = int(self._p("hidden_size"))
        if not (1 <= self.S <= K.STREAMS_MAX):
            raise ConfigError(f"streams={self.S} outside 1..{K.STREAMS_MAX}")

    def enter(self, x: torch.Tensor) -> torch.Tensor:
        return K.streams_enter(x, torch.empty((x.shape[0], self.S, self.d), dtype=torch.float32, device=x.device))

    def rows(self, x: torch.Tensor) -> torch.Tensor:
        return x.sum(1)

    def normed(self, x: torch.Tensor, norm, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        h = torch.empty((x.shape[0] if rows is None else rows.numel(), self.d), dtype=self.env.dtype, device=x.device)
        K.streams_rows(x, norm_w=norm.weight, eps=norm.eps, centred=stream_norm(norm), h=h, rows=rows)
        return h


register_part("residual", "streams", Streams)
