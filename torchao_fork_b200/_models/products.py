"""Dense products of the sequence models: activations [n][K] (bf16 or fp32) with a weight matrix [M][K], fp32 result.  A few bf16
rows (decoded tokens) go through a matrix-vector kernel that reads the weights at memory speed, everything else through the
library GEMM."""
from typing import Optional

import torch

from .. import _lib

GEMV_ROWS = 8       # most rows the matrix-vector kernel takes
ACT_NONE, ACT_SQUARED_RELU = 0, 1


def gemv_takes(a: torch.Tensor, w: torch.Tensor) -> bool:
    return (a.dtype == torch.bfloat16 and a.shape[0] <= GEMV_ROWS and a.shape[1] % 8 == 0 and a.stride(0) % 8 == 0 and w.stride(0) % 8 == 0
            and a.stride(1) == 1 and w.stride(1) == 1 and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def gemv(L, a: torch.Tensor, w: torch.Tensor, act: int = ACT_NONE, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """act(a w^T) of a few rows: fp32, or bf16 behind an activation."""
    n, M = a.shape[0], w.shape[0]
    if out is None:
        out = torch.empty(n, M, dtype=torch.float32 if act == ACT_NONE else torch.bfloat16, device=a.device)
    st = torch.cuda.current_stream(a.device).cuda_stream
    _lib.lm_check(L.ao_lm_gemv_rows(a.data_ptr(), a.stride(0), w.data_ptr(), w.stride(0), n, M, a.shape[1], act, out.data_ptr(), out.stride(0), st),
                  "gemv_rows")
    return out


def mm_f32(L, a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """a @ w^T with an fp32 result (what fp32 kernels read next), into `out` when given."""
    if gemv_takes(a, w):
        return gemv(L, a, w, out=out)
    r = torch.mm(a, w.t(), out_dtype=torch.float32) if a.dtype == torch.bfloat16 else torch.mm(a, w.t())
    return r if out is None else out.copy_(r)
