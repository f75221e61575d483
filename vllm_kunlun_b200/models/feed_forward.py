"""Feed-forward blocks of designs that list their layers one by one.  A block reads the stream's normed copy ``h [T, ld]`` and
returns ``[T, ld]``, or what the residual kernel sums: ``(rows, places)`` (:func:`ops.experts_on_weighted_input`) or a
:class:`ops.ChoicesSum`.

* :class:`GatedFeedForward`  ``W_down(act(W_gate h) * W_up h)``, the shared gated MLP with its fused activation
* :class:`PolyNormMLP`       ``W_down act(W_up h)``, act = normed powers of the row with learned coefficients
* :class:`WeightedInputMoE`  sigmoid router in fp32, the routing weight multiplies the expert's input, clamped gated experts
* :class:`CorrectedMoE`      softmax router with a choice correction and groups, identity experts, a shared expert, no gates

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


class CorrectedMoE(nn.Module):
    """``shared(h) + scale * sum over the chosen outputs of s expert(h)`` with ``s = softmax(W_router h)``, not renormalised, and
    ``expert(h) = W_down relu(W_up h)^2``.  The largest ``s + correction`` are chosen, inside the ``keep`` of ``count`` equal groups
    whose best member is largest.  The router's last ``identity`` outputs have no weights: they return h."""

    def __init__(self, ld: int, sizes: dict, act: str, eps: float, dtype, device):
        super().__init__()
        ex, rt, groups = sizes["expert"], sizes["router"], sizes["router"].get("groups") or {}
        self.act = act
        self.num_experts, self.top, self.scale = int(rt["experts"]), int(rt["top"]), float(rt.get("scale", 1.0))
        self.choices = self.num_experts + int(rt.get("identity") or 0)
        self.groups, self.keep = int(groups.get("count", 1)), int(groups.get("keep", 1))
        if self.choices > 512 or not 0 < self.top <= 16:
            raise ValueError(f"{self.top} of {self.choices} router outputs: the router takes up to 16 of up to 512")
        if self.choices % self.groups or self.groups > 32 or not 0 < self.keep <= self.groups:
            raise ValueError(f"{self.choices} router outputs in {self.groups} groups, {self.keep} of them kept")
        if self.top > self.keep * (self.choices // self.groups):
            raise ValueError(f"{self.top} choices from {self.keep} groups of {self.choices // self.groups}")
        self.router = ReplicatedLinear(ld, self.choices, dtype=dtype, device=device)
        self.correction = param(self.choices, dtype=torch.float32, device=device)
        ff = round_up(int(ex["ff"]), MLP_TILE)
        self.up = param(self.num_experts, ff, ld, dtype=dtype, device=device)
        self.down = param(self.num_experts, ld, ff, dtype=dtype, device=device)
        for w in (self.up, self.down):
            w.data.zero_()
        self.shared_up = self.shared_down = None
        if sizes.get("shared"):
            n = align(int(sizes["shared"]["ff"]))
            self.shared_up = ReplicatedLinear(ld, n, dtype=dtype, device=device)
            self.shared_down = ReplicatedLinear(n, ld, dtype=dtype, device=device)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        ff, rt = int(sizes["expert"]["ff"]), sizes["router"]
        E = int(rt["experts"])
        n = E + int(rt.get("identity") or 0)
        out = {"router": (n, width), "correction": (n,)}
        for e in range(E):
            out.update({f"e{e}.up": (ff, width), f"e{e}.down": (width, ff)})
        if sizes.get("shared"):
            ff = int(sizes["shared"]["ff"])
            out.update({"shared.up": (ff, width), "shared.down": (width, ff)})
        return out

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "correction":
            self.correction.data.copy_(w)
        elif key == "router" or key.startswith("shared."):
            lin = {"router": self.router, "shared.up": self.shared_up, "shared.down": self.shared_down}[key]
            lin.weight.data.copy_(padded(w, *lin.weight.shape))
        else:
            e, part = key[1:].split(".")
            (self.up if part == "up" else self.down).data[int(e), :w.shape[0], :w.shape[1]].copy_(w)

    def forward(self, h):
        w, ids = ops.router_and_route(h, self.router.weight, None, self.top, "softmax", False, self.correction, self.groups,
                                      self.keep, self.scale, fp32=True, group_top=1)
        rows, places = ops.expert_rows(h, self.up, self.down, ids, self.act, choices=self.choices)
        shared = None
        if self.shared_up is not None:
            shared = self.shared_down(ops.linear(h, self.shared_up.weight, act=self.act))
        return ops.ChoicesSum(shared, rows, places, w, h)


FEED_FORWARDS = {"dense": GatedFeedForward, "moe": WeightedInputMoE}
# activations that come with a block of their own
_BY_ACTIVATION = {("dense", "poly_norm"): PolyNormMLP, ("moe", "relu2"): CorrectedMoE}


def feed_forward_cls(sizes: dict, act: str):
    kind = sizes.get("kind", "dense")
    return _BY_ACTIVATION.get((kind, act), FEED_FORWARDS[kind])
