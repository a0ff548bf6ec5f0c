"""Where model weights come from: a dictionary, seeded random tensors, or a checkpoint (`loader.CheckpointSource`)."""
from __future__ import annotations

import hashlib
from typing import Dict, Optional, Sequence, Tuple

import torch


RANDOM_EXTENT = 32           # of an extent that only a checkpoint could tell


def fits(shape: Sequence[int], want: Sequence[Optional[int]]) -> bool:
    """Whether a tensor's shape is the wanted one (None: any extent)."""
    return len(shape) == len(want) and all(w is None or s == w for s, w in zip(shape, want))


class WeightSource:
    """Hands out fp32 master tensors by checkpoint name.  An extent of None in a wanted shape is whatever the source has."""

    def get(self, name: str, shape: Tuple[int, ...], device) -> torch.Tensor:
        raise NotImplementedError


class DictSource(WeightSource):
    def __init__(self, tensors: Dict[str, torch.Tensor]):
        self.t = tensors

    def get(self, name, shape, device):
        t = self.t[name]
        assert fits(t.shape, shape), (name, t.shape, shape)
        return t.to(device)


class RandomSource(WeightSource):
    """Random-init weights: every tensor is a pure function of (seed, name), so replicated
    tensors agree across ranks without communication."""

    def __init__(self, seed: int = 0, std: float = 0.02):
        self.seed, self.std = seed, std

    def _gen(self, name: str, device) -> torch.Generator:
        h = int.from_bytes(hashlib.sha256(f"{self.seed}:{name}".encode()).digest()[:7], "little")
        g = torch.Generator(device=device)
        g.manual_seed(h)
        return g

    def get(self, name, shape, device):
        dev = torch.device(device)
        shape = tuple(RANDOM_EXTENT if n is None else n for n in shape)
        g = self._gen(name, dev)
        if name.endswith("tid2eid"):
            return torch.randint(0, 1 << 30, shape, generator=g, device=dev, dtype=torch.int64)
        if name.endswith(("norm.weight", "_scale", ".norm", ".norm1", ".norm2")):
            return torch.ones(shape, device=dev)
        if name.endswith(".f.b"):
            return 3.0 + 3.0 * torch.rand(shape, generator=g, device=dev)      # forget gates of a recurrence start near one
        if name.endswith(("_base", "attn_sink", ".sink", ".i.b", ".router.b")):
            return torch.zeros(shape, device=dev)
        if name.endswith("gate.bias"):
            return torch.rand(shape, generator=g, device=dev) * 0.2 - 0.1
        noise = torch.randn(shape, generator=g, device=dev) * self.std
        if name.endswith((".hc1.mix", ".hc2.mix")):
            return noise + torch.eye(shape[0], device=dev)                     # residual streams mostly stay themselves
        if ".hc" in name or name.endswith(".dt_bias"):
            return noise + (0.5 if ".hc" in name else -2.0)
        if name.endswith(".talk"):
            return noise + torch.eye(shape[0], device=dev)                     # heads mostly keep their own scores
        if name.endswith(".mix.right.w0"):
            return noise - 4.0                                                 # decays near one
        if name.endswith((".q.norm", ".k.norm", ".left.out", ".right.out")):
            return torch.ones(shape, device=dev)
        if name.endswith((".shift", ".mu.r", ".mu.k", ".mu.v", ".mu.g", ".mu.w")):
            return noise + 0.3
        return noise
