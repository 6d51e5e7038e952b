"""Weight layout of layer-stack models: stacked bf16 matrices with rows padded to 16 bytes, heads padded to eight columns."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Sequence

import torch


def pad(n: int, to: int) -> int:
    return -(-n // to) * to


@dataclass
class Packed:
    """A stacked linear weight [z, n, ld] in bf16: rows padded to 16 bytes, ``k`` live columns."""

    w: torch.Tensor
    k: int

    @property
    def z(self) -> int:
        return self.w.shape[0]

    @property
    def n(self) -> int:
        return self.w.shape[1]

    @property
    def ld(self) -> int:
        return self.w.shape[2]

    @property
    def nbytes(self) -> int:
        return self.w.numel() * 2

    def rows(self, lo: int, n: int, z: int = 1) -> "Packed":
        """``z`` groups of ``n`` consecutive rows from row ``lo`` on (a view of a single matrix)."""
        return Packed(self.w[0, lo:lo + z * n].view(z, n, self.ld), self.k)


def pack(w: torch.Tensor, device) -> Packed:
    w = w.to(device=device, dtype=torch.bfloat16)
    w = w if w.dim() == 3 else w.unsqueeze(0)
    z, n, k = w.shape
    ld = pad(k, 8)
    if ld != k:
        full = torch.zeros(z, n, ld, dtype=torch.bfloat16, device=device)
        full[:, :, :k] = w
        w = full
    return Packed(w.contiguous(), k)


def vector(t: torch.Tensor, device) -> torch.Tensor:
    return t.to(device=device, dtype=torch.bfloat16).contiguous()


def head_rows(w: torch.Tensor, heads: int, dim: int, padded: int) -> torch.Tensor:
    """Rows laid out head by head, each head padded with zero rows."""
    if padded == dim:
        return w
    out = torch.zeros(heads, padded, w.shape[-1], dtype=w.dtype, device=w.device)
    out[:, :dim] = w.reshape(heads, dim, -1)
    return out.reshape(heads * padded, -1)


def head_columns(w: torch.Tensor, heads: int, dim: int, padded: int) -> torch.Tensor:
    """Columns laid out head by head, each head padded with zero columns."""
    if padded == dim:
        return w
    out = torch.zeros(w.shape[0], heads, padded, dtype=w.dtype, device=w.device)
    out[:, :, :dim] = w.reshape(w.shape[0], heads, dim)
    return out.reshape(w.shape[0], heads * padded)


def stacked_rows(parts: Sequence[torch.Tensor], stride: int) -> torch.Tensor:
    """Matrices one below the other, each but the last padded with zero rows to ``stride``."""
    out = []
    for i, p in enumerate(parts):
        out.append(p)
        if i + 1 < len(parts) and p.shape[0] < stride:
            out.append(torch.zeros(stride - p.shape[0], p.shape[1], dtype=p.dtype, device=p.device))
    return torch.cat(out)
