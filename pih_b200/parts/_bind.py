"""How parts bring loaded tensors onto the device for a compute path."""
from __future__ import annotations

import torch


def bind_matrix(t: torch.Tensor, rt) -> torch.Tensor:
    """Matrices take the compute dtype: bf16 widens exactly for the 32-bit
    path; a matrix stored in 32-bit is rounded to bf16 for the bf16 path,
    whose matrix products read bf16."""
    return t.to(device=rt.device, dtype=rt.dtype).contiguous()


def bind_vector(t: torch.Tensor, rt) -> torch.Tensor:
    """Vectors (norm weights) stay in 32-bit when stored so; bf16 vectors
    widen for the 32-bit path and stay bf16 for the bf16 path."""
    if t.dtype == torch.float32 or rt.dtype == torch.float32:
        return t.to(device=rt.device, dtype=torch.float32).contiguous()
    return t.to(device=rt.device, dtype=rt.dtype).contiguous()


def stack_rows(parts, align: int):
    """The rows of several matrices one below the other, every one beginning at a multiple of ``align`` (rows of zeros in
    between), the whole a multiple of 8 rows; returns ``(matrix, where each begins)``.  The columns of a product with it
    then begin where the kernels load 16 bytes at a time."""
    out, at, n = [], [], 0
    for i, p in enumerate(parts):
        at.append(n)
        out.append(p)
        n += p.shape[0]
        pad = -n % (align if i + 1 < len(parts) else 8)
        if pad:
            out.append(p.new_zeros((pad, p.shape[1])))
            n += pad
    return torch.cat(out, dim=0).contiguous(), at


def pad_columns(t: torch.Tensor, columns: int) -> torch.Tensor:
    """``t`` with columns of zeros behind its own, ``columns`` in all."""
    return torch.nn.functional.pad(t, (0, columns - t.shape[1]))
