"""Base of hybrid stacks: decoder stacks whose layers are listed one by one in the configuration (``ModelConfig.layer_specs``), keep
different things between steps (``cache_layout()``) and run as one stage on an fp32 residual.  Weight helpers and the small projection
helpers that the designs share."""
from __future__ import annotations

import torch

from ..ops import LinearWeight
from .base import StageModel


def pad_rows(w: torch.Tensor, mult: int = 8) -> torch.Tensor:
    n = w.shape[0]
    if n % mult == 0:
        return w.contiguous()
    return torch.cat([w, w.new_zeros((mult - n % mult, w.shape[1]))]).contiguous()


def pad_cols(w: torch.Tensor, mult: int = 8) -> torch.Tensor:
    """Zero columns behind a weight ``[out, in]`` whose input rows carry zero (or finite) padding up to a multiple of ``mult``."""
    n = w.shape[1]
    return w if n % mult == 0 else torch.cat([w, w.new_zeros((w.shape[0], mult - n % mult))], 1)


class HybridStage(StageModel):
    def __init__(self, cfg, spec=None, dtype=torch.bfloat16, device="cpu", backend=None):
        super().__init__(cfg, spec, dtype, device, backend)
        if not (self.spec.is_first and self.spec.is_last):
            raise NotImplementedError(f"{type(self).__name__} runs as a single stage (fp32 residual: the pipeline hand-off does not carry it)")
        self.specs = cfg.layer_specs

    def kv_geometry(self):
        raise NotImplementedError("hybrid stack: see cache_layout()")

    def sanitize(self, sd):
        return dict(sd)

    # ---- weights ----------------------------------------------------------------------------------------------------
    def _lw(self, w: torch.Tensor, bias: torch.Tensor = None) -> LinearWeight:
        """Linear weight ``[out, in]`` in the model dtype; output rows zero-padded to a multiple of 8 (GEMM tile rule), the real row
        count kept in ``n_real``."""
        lw = LinearWeight(weight=pad_rows(w.to(device=self.device, dtype=self.dtype)))
        if bias is not None:
            lw.bias = pad_rows(bias.to(device=self.device, dtype=self.dtype)[:, None])[:, 0].contiguous()
        lw.n_real = w.shape[0]
        return lw

    def _fused(self, parts):
        """One projection for several matrices that read the same input: ``parts`` = ``[(name, weight [rows, in], bias or None)]``.  Every
        segment starts at a multiple of 8 columns (a later product may read it in place).  Returns ``(LinearWeight, {name: (col0, rows)})``."""
        ws, bs, seg, col = [], [], {}, 0
        any_bias = any(b is not None for _, _, b in parts)
        for name, w, b in parts:
            n = w.shape[0]
            pad = (-n) % 8
            seg[name] = (col, n)
            ws.append(torch.cat([w, w.new_zeros(pad, w.shape[1])]) if pad else w)
            if any_bias:
                bb = b if b is not None else w.new_zeros(n)
                bs.append(torch.cat([bb, bb.new_zeros(pad)]) if pad else bb)
            col += n + pad
        return self._lw(torch.cat(ws), torch.cat(bs) if any_bias else None), seg

    def _f32(self, sd, key) -> torch.Tensor:
        return sd.pop(key).to(device=self.device, dtype=torch.float32).contiguous()

    # ---- forward ----------------------------------------------------------------------------------------------------
    def _mm(self, x, W: LinearWeight, f32: bool = False, act: str = "none"):
        y = self.ops.linear_any(x, W, torch.float32 if f32 else self.dtype, act)
        return y if y.shape[1] == W.n_real else y[:, :W.n_real]

    @staticmethod
    def _cols(u, seg, name):
        c0, n = seg[name]
        return u[:, c0:c0 + n]
