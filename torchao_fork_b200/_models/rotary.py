"""Rotary position constants shared by the model families: frequencies and the factor on cosine and sine, optionally with
YaRN scaling (slow pairs turn `factor` times slower, fast ones as before, a linear ramp between)."""
import math
from dataclasses import dataclass
from typing import Optional

import torch


@dataclass
class RotaryScaling:
    factor: float
    original: float             # context length the unscaled frequencies were made for
    fast: float                 # turns over the original context from which a pair keeps its frequency ...
    slow: float                 # ... and up to which it is slowed down by the whole factor


@dataclass
class RotaryArgs:
    dims: int = 0               # 0: no rotation
    base: float = 10000.0
    scaling: Optional[RotaryScaling] = None

    @classmethod
    def from_dict(cls, r: Optional[dict]) -> "RotaryArgs":
        if not r:
            return cls()
        s = r.get("scaling")
        return cls(int(r["dims"]), float(r["base"]),
                   RotaryScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None)

    def to_dict(self) -> Optional[dict]:
        if self.dims == 0:
            return None
        r = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            s = self.scaling
            r["scaling"] = {"factor": s.factor, "fast": s.fast, "original": s.original, "slow": s.slow}
        return r

    def inv_freq(self, device) -> Optional[torch.Tensor]:
        """Frequency of pair i < dims/2 (base^(-2i/dims), scaled), rounded once to fp32."""
        if self.dims == 0:
            return None
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / self.dims)
        s = self.scaling
        if s is not None:
            pair_of = [self.dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base)) for turns in (s.fast, s.slow)]
            lo, hi = max(math.floor(pair_of[0]), 0), min(math.ceil(pair_of[1]), self.dims - 1)
            slowed = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f * (slowed / s.factor + (1.0 - slowed))
        return f.to(torch.float32).to(device)

    @property
    def amplitude(self) -> float:
        """Factor on cosine and sine."""
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling.factor) + 1.0
