"""fp32 PyTorch forms of the output-normed stream with input convolutions and of the element-wise gated recurrence (CPU path of
``csrc/elementwise/postnorm.cu`` and ``csrc/linear_attn/blend.cu``)."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def layer_norm(y, weight, eps):
    n = weight.numel()
    out = torch.zeros_like(y)
    out[:, :n] = F.layer_norm(y[:, :n], (n,), weight.float(), None, eps)
    return out


def input_conv(x, h, conv, state, cu, slots, has_init):
    """``h = x + conv(x)``; ``state [slots, taps - 1, ld]`` holds and receives the last rows of every request."""
    n = conv.shape[0]
    for r in range(len(slots)):
        s, e, slot = int(cu[r]), int(cu[r + 1]), int(slots[r])
        if e == s:
            continue
        front = torch.zeros(n - 1, x.shape[1])
        if n > 1 and slot >= 0 and bool(has_init[r]):
            front = state[slot].clone()
        rows = torch.cat([front, x[s:e]])
        y = x[s:e].clone()
        for j in range(n):
            y += conv[j] * rows[j:j + e - s]
        h[s:e] = y.to(h.dtype)
        if n > 1 and slot >= 0:
            state[slot] = rows[len(rows) - (n - 1):]


def choices_sum(y, rows, places, weights, through):
    """``y`` (or zeros) plus, per token, the weighted rows of its choices; a place below zero stands for ``through``."""
    T, k = weights.shape
    p = places.reshape(T, k).long()
    picked = torch.where((p >= 0).unsqueeze(-1), rows.float()[p.clamp(min=0)], through.float().unsqueeze(1))
    out = (picked * weights.float().unsqueeze(-1)).sum(1)
    return out if y is None else out + y.float()


def gated_blend(out, z, x, g, z_bias, x_bias, state, cu, slots, has_init):
    a = torch.sigmoid(-(z.float() + z_bias))
    u = x.float() + x_bias
    b = torch.sigmoid(z.float() + z_bias) * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    gate = F.silu(g.float())
    n = z.shape[1]
    out[:, n:] = 0
    for r in range(len(slots)):
        s, e, slot = int(cu[r]), int(cu[r + 1]), int(slots[r])
        if e == s or slot < 0:
            continue
        S = state[slot].clone() if bool(has_init[r]) else torch.zeros(n)
        for t in range(s, e):
            S = a[t] * S + b[t]
            out[t, :n] = (S * gate[t]).to(out.dtype)
        state[slot] = S
