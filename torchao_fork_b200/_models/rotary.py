"""Rotary position constants shared by the model families: frequencies and the factor on cosine and sine, optionally scaled for
contexts longer than the original one: by YaRN (slow pairs turn `factor` times slower, fast ones as before, a linear ramp over
the pairs between) or in Llama 3.1's bands (the same by wavelength, a blend in the middle band)."""
import math
from dataclasses import dataclass
from typing import Optional, Union

import torch


@dataclass
class RotaryScaling:
    factor: float
    original: float             # context length the unscaled frequencies were made for
    fast: float                 # turns over the original context from which a pair keeps its frequency ...
    slow: float                 # ... and up to which it is slowed down by the whole factor
    keys = ("factor", "original", "fast", "slow")

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def scaled(self, f: torch.Tensor, dims: int, base: float) -> torch.Tensor:
        pair_of = [dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base)) for turns in (self.fast, self.slow)]
        lo, hi = max(math.floor(pair_of[0]), 0), min(math.ceil(pair_of[1]), dims - 1)
        slowed = torch.clamp((torch.arange(dims // 2, dtype=f.dtype) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return f * (slowed / self.factor + (1.0 - slowed))


@dataclass
class BandScaling:
    factor: float
    original: float             # context length the unscaled frequencies were made for
    low: float                  # below this many turns over the original context a pair is slowed down by the whole factor ...
    high: float                 # ... above this many it keeps its frequency
    keys = ("factor", "original", "low", "high")
    amplitude = 1.0

    def scaled(self, f: torch.Tensor, dims: int, base: float) -> torch.Tensor:
        turns = self.original * f / (2.0 * math.pi)
        keep = torch.clamp((turns - self.low) / max(self.high - self.low, 1e-12), 0.0, 1.0)      # 0: slowed, 1: kept
        return f * ((1.0 - keep) / self.factor + keep)


@dataclass
class RotaryArgs:
    dims: int = 0               # 0: no rotation
    base: float = 10000.0
    scaling: Optional[Union[RotaryScaling, BandScaling]] = None

    @classmethod
    def from_dict(cls, r: Optional[dict]) -> "RotaryArgs":
        if not r:
            return cls()
        s = r.get("scaling")
        if s:
            kind = BandScaling if "high" in s else RotaryScaling
            s = kind(*(float(s[k]) for k in kind.keys))
        return cls(int(r["dims"]), float(r["base"]), s or None)

    def to_dict(self) -> Optional[dict]:
        if self.dims == 0:
            return None
        r = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            r["scaling"] = {k: getattr(self.scaling, k) for k in self.scaling.keys}
        return r

    def inv_freq(self, device) -> Optional[torch.Tensor]:
        """Frequency of pair i < dims/2 (base^(-2i/dims), scaled), rounded once to fp32."""
        if self.dims == 0:
            return None
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / self.dims)
        if self.scaling is not None:
            f = self.scaling.scaled(f, self.dims, self.base)
        return f.to(torch.float32).to(device)

    @property
    def amplitude(self) -> float:
        """Factor on cosine and sine."""
        return 1.0 if self.scaling is None else self.scaling.amplitude
