"""Feed-forward blocks of designs that list their layers one by one.  A block reads the stream's normed copy ``h [T, ld]`` and
returns ``[T, ld]``, or ``(rows, places)`` whose rows the residual kernel sums (:func:`ops.experts_on_weighted_input`).

* :class:`GatedFeedForward`  ``W_down(act(W_gate h) * W_up h)``, the shared gated MLP with its fused activation
* :class:`PolyNormMLP`       ``W_down act(W_up h)``, act = normed powers of the row with learned coefficients
* :class:`WeightedInputMoE`  sigmoid router in fp32, the routing weight multiplies the expert's input, clamped gated experts

Widths are padded (rows to a multiple of 8 columns by the caller, inner widths here); padding is zero.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from ..config import round_up
from .dense import GatedMLP
from .layers import ReplicatedLinear, param
from .mixers import align, padded

MLP_TILE = 64       # inner widths: the fused gate / up epilogue and the grouped GEMM's k-blocks


class GatedFeedForward(GatedMLP):
    def __init__(self, ld: int, sizes: dict, act: str, eps: float, dtype, device):
        super().__init__(ld, round_up(int(sizes["ff"]), MLP_TILE), dtype, device, act=act)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        ff = int(sizes["ff"])
        return {"gate": (ff, width), "up": (ff, width), "down": (width, ff)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "down":
            dn = self.down_proj
            dn.load("weight", padded(w, dn.out_features, dn.in_features))
        else:
            gu = self.gate_up_proj
            gu.load("weight", padded(w, gu.output_sizes[0], gu.in_features), 0 if key == "gate" else 1)


class PolyNormMLP(nn.Module):
    def __init__(self, ld: int, sizes: dict, act: str, eps: float, dtype, device):
        super().__init__()
        self.ff, self.eps = int(sizes["ff"]), eps
        self.up = ReplicatedLinear(ld, align(self.ff), dtype=dtype, device=device)
        self.down = ReplicatedLinear(align(self.ff), ld, dtype=dtype, device=device)
        self.act = param(4, dtype=torch.float32, device=device)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        ff = int(sizes["ff"])
        return {"up": (ff, width), "down": (width, ff), "act": (4,)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "act":
            self.act.data.copy_(w)
        else:
            lin = self.up if key == "up" else self.down
            lin.weight.data.copy_(padded(w, *lin.weight.shape))

    def forward(self, h):
        return self.down(ops.poly_norm(self.up(h), self.act, self.ff, self.eps))


class WeightedInputMoE(nn.Module):
    """``sum over the chosen experts of expert(s h)``, ``s = sigmoid(W_router h)`` of the largest scores, not renormalised;
    ``expert(x) = W_down(g sigmoid(1.702 g) (u + 1))`` with ``g = min(W_gate x, limit)``, ``u = clamp(W_up x, +-limit)``."""

    def __init__(self, ld: int, sizes: dict, act: str, eps: float, dtype, device):
        super().__init__()
        ex, rt = sizes["expert"], sizes["router"]
        self.num_experts, self.top, self.limit = int(rt["experts"]), int(rt["top"]), float(ex["limit"])
        if not 0 < self.top <= min(self.num_experts, 16) or self.num_experts > 512:
            raise ValueError(f"{self.top} of {self.num_experts} experts: the router takes up to 16 of up to 512")
        self.ff = round_up(int(ex["ff"]), MLP_TILE)
        self.router = ReplicatedLinear(ld, self.num_experts, dtype=dtype, device=device)
        self.w13 = param(self.num_experts, 2 * self.ff, ld, dtype=dtype, device=device)       # gate rows, then up rows
        self.w2 = param(self.num_experts, ld, self.ff, dtype=dtype, device=device)
        for w in (self.w13, self.w2):
            w.data.zero_()

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        ff, E = int(sizes["expert"]["ff"]), int(sizes["router"]["experts"])
        out = {"router": (E, width)}
        for e in range(E):
            out.update({f"e{e}.gate": (ff, width), f"e{e}.up": (ff, width), f"e{e}.down": (width, ff)})
        return out

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "router":
            self.router.weight.data.copy_(padded(w, *self.router.weight.shape))
            return
        e, part = key[1:].split(".")
        if part == "down":
            self.w2.data[int(e), :w.shape[0], :w.shape[1]].copy_(w)
        else:
            off = self.ff * (part == "up")
            self.w13.data[int(e), off:off + w.shape[0], :w.shape[1]].copy_(w)

    def forward(self, h):
        w, ids = ops.router_and_route(h, self.router.weight, None, self.top, "sigmoid", False, fp32=True)
        return ops.experts_on_weighted_input(h, self.w13, self.w2, w, ids, "swiglu_limit", self.limit)


FEED_FORWARDS = {"dense": GatedFeedForward, "moe": WeightedInputMoE}
_BY_ACTIVATION = {("dense", "poly_norm"): PolyNormMLP}      # activations that come with a block of their own


def feed_forward_cls(sizes: dict, act: str):
    kind = sizes.get("kind", "dense")
    return _BY_ACTIVATION.get((kind, act), FEED_FORWARDS[kind])
