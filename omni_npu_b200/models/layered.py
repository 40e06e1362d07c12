"""What the models that list their layers share: padding of widths to whole 16-byte rows, a table of the
checkpoint's tensors (name -> shape and how it is placed), and the base of their mixers."""
from __future__ import annotations

from typing import Any, Callable, Dict, Iterable, List, Tuple

import torch
from torch import nn

from ..config import ModelConfig
from ..layers.linear import RowParallelLinear, SegmentedLinear
from ..parallel import state as pstate


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def fit(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` with zeros appended up to ``shape``."""
    if tuple(t.shape) == shape:
        return t
    out = t.new_zeros(shape)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


Want = Dict[str, Tuple[Tuple[int, ...], Callable[[torch.Tensor], Any]]]     # tensor -> (shape, how it is placed)


def place_tensors(weights: Iterable[Tuple[str, torch.Tensor]], want: Want, design: str,
                  idle: Callable[[str], bool] = lambda name: False) -> set:
    """Every tensor where ``want`` says.  Unknown names (but for idle ones), wrong shapes and missing tensors are
    errors."""
    loaded = set()
    for name, t in weights:
        if name not in want:
            if idle(name):
                continue
            raise ValueError(f"{design}: unknown tensor {name!r}")
        shape, place = want[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{design}: tensor {name!r} is {tuple(t.shape)}, expected {shape}")
        place(t)
        loaded.add(name)
    missing = sorted(set(want) - loaded)
    if missing:
        raise ValueError(f"{design}: {len(missing)} tensors missing, first {missing[:3]}")
    return loaded


class Mixer(nn.Module):
    """What the mixers share: this rank's part of heads and rows, and the output projection."""

    def __init__(self, cfg: ModelConfig) -> None:
        super().__init__()
        self.width, self.padded_width, self.eps = cfg.hidden_size, pad8(cfg.hidden_size), cfg.rms_norm_eps
        group = self.group = pstate.get_tp_group()
        self.tp, self.rank = group.world_size, group.rank_in_group
        self.out_scale = 1.0                     # of the mixer's result, for the residual kernel

    def share(self, n: int, what: str = "heads") -> int:
        if n % self.tp:
            raise ValueError(f"{type(self).__name__}: {n} {what} do not split over {self.tp} ranks")
        return n // self.tp

    def own(self, t: torch.Tensor, dim: int = 0) -> torch.Tensor:
        """This rank's part of a tensor that is split by heads."""
        n = t.shape[dim] // self.tp
        return t.narrow(dim, self.rank * n, n)

    def output_proj(self, cfg: ModelConfig, parts: List[int], device, prefix: str, bias: bool = False) -> None:
        """One product for the mixer's parts, each ``parts[i]`` columns of this rank at a whole 16-byte place."""
        self.parts, self.starts, at = parts, [], 0
        for n in parts:
            self.starts.append(at)
            at += pad8(n)
        self.o_proj = RowParallelLinear(at * self.tp, self.padded_width, bias=bias, dtype=cfg.dtype, device=device,
                                        prefix=f"{prefix}.o_proj")
        self.o_proj.weight.data.zero_()

    def expect_rows(self, want: Want, p: str, proj: SegmentedLinear) -> None:
        for name, n in proj.rows.items():
            rows = n * self.tp if proj.sharded[name] else n
            want[p + name] = (rows, self.width), lambda t, name=name: proj.weight_loader(proj.weight, t, name)
            if proj.bias is not None:
                want[f"{p}{name}.b"] = (rows,), lambda t, name=name: proj.weight_loader(proj.bias, t, name)

    def expect_output(self, want: Want, name: str, part: int) -> None:
        n, at = self.parts[part], self.starts[part]
        want[name] = (self.width, n * self.tp), lambda t: self.o_proj.weight.data[: self.width, at: at + n].copy_(
            self.own(t, 1))

    def expect_vector(self, want: Want, name: str, param: nn.Parameter, split: bool, shape=None) -> None:
        full = (param.shape[0] * (self.tp if split else 1), *param.shape[1:])
        want[name] = shape or full, lambda t: param.data.copy_((self.own(t) if split else t).view(param.shape))

    def expect_low(self, want: Want, name: str, low: SegmentedLinear, rank: int) -> None:
        want[name] = (low.rows["z"] * self.tp, rank), lambda t: low.weight_loader(
            low.weight, fit(t, t.shape[0], low.in_features), "z")

    @torch.no_grad()
    def clear(self, proj: SegmentedLinear, columns: int) -> None:
        """Zeros in the padding of a projection whose input has ``columns`` true columns."""
        w = proj.weight.data
        rows = proj.padding_rows().to(w.device)
        w[rows] = 0
        w[:, columns:] = 0
        if proj.bias is not None:
            proj.bias.data[rows] = 0

    @torch.no_grad()
    def clear_output(self) -> None:
        w = self.o_proj.weight.data
        w[self.width:] = 0
        for n, at in zip(self.parts, self.starts):
            w[:, at + n: at + pad8(n)] = 0
        if self.o_proj.bias is not None:
            self.o_proj.bias.data[self.width:] = 0

    def clear_padding(self) -> None:
        self.clear_output()
