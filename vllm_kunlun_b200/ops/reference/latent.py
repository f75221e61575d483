"""fp32 PyTorch forms of the latent-attention steps and of the gated fp32 stream (CPU path of ``csrc/attention/latent.cu``
and ``csrc/elementwise/gated_stream.cu``)."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def rotary_table(positions, turns):
    a = positions.long().unsqueeze(1) * turns           # 64-bit fractions of a turn: the product wraps by itself
    angle = a.double() * (2 * math.pi * 2.0 ** -64)
    return torch.stack([angle.cos(), angle.sin()], -1).float()


def rotate(x, table):
    """``x [T, heads, n]`` (fp32): the first ``2 * pairs`` columns rotate, column i with i + pairs."""
    p = table.shape[1]
    c, s = table[:, None, :, 0], table[:, None, :, 1]
    u, v = x[..., :p], x[..., p:2 * p]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * p:]], -1)


def latent_prep(q_out, cache, q_down, kv_down, q_norm, kv_norm, table, slots, rot_off, eps):
    def rms(z, w):
        z = z.float()
        return z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w
    Q, C = q_down.shape[1], kv_norm.numel()
    q_out.zero_()
    q_out[:, :Q] = rms(q_down, q_norm).to(q_out.dtype)
    rows = torch.zeros(q_down.shape[0], cache.shape[2])
    rows[:, :C] = rms(kv_down[:, :C], kv_norm)
    R = kv_down.shape[1] - C
    rows[:, rot_off:rot_off + R] = rotate(kv_down[:, None, C:].float(), table)[:, 0]
    ok = slots >= 0
    bs = cache.shape[1]
    cache[slots[ok] // bs, slots[ok] % bs] = rows[ok].to(cache.dtype)


def absorb_query(q, w_uk, table, rot_off, row):
    T, H, D = q.shape[0], q.shape[1], w_uk.shape[1]
    C, R = w_uk.shape[2], q.shape[2] - D
    out = torch.zeros(T, H, row)
    out[:, :, :C] = torch.einsum("thd,hdc->thc", q[:, :, :D].float(), w_uk.float())
    out[:, :, rot_off:rot_off + R] = rotate(q[:, :, D:].float(), table)
    return out.to(q.dtype)


def expand_value(o, w_uv, gate, width):
    T, H, Dv = o.shape[0], w_uv.shape[0], w_uv.shape[1]
    y = torch.einsum("thc,hvc->thv", o.float(), w_uv.float())
    if gate is not None:
        y = y * torch.sigmoid(gate.float()).unsqueeze(-1)
    return F.pad(y.reshape(T, H * Dv), (0, width - H * Dv)).to(o.dtype)


def gather_window(cache, block_tables, seq_lens, lens):
    bs, rows = cache.shape[1], []
    for r, n in enumerate(lens.tolist()):
        pos = torch.arange(int(seq_lens[r]) - n, int(seq_lens[r]))
        rows.append(cache[block_tables[r, pos // bs].long(), pos % bs])
    return torch.cat(rows)


def bigram_rows(ids, state, cu, slots, has_init, mul_prev, mul_cur, buckets):
    out = torch.empty_like(ids)
    for r in range(len(slots)):
        s, e, slot = int(cu[r]), int(cu[r + 1]), int(slots[r])
        if e == s:
            continue
        cur = ids[s:e]
        out[s + 1:e] = (cur[:-1] * mul_prev + cur[1:] * mul_cur) % buckets
        before = int(state[slot]) if slot >= 0 and bool(has_init[r]) else -1
        out[s] = buckets if before < 0 else (before * mul_prev + int(cur[0]) * mul_cur) % buckets
        if slot >= 0:
            state[slot] = cur[-1]
    return out


def stream_layernorm(x, weight, eps, h, shift):
    """``h``: result in its dtype; returns the shifted rows or None.  ``shift``: ``(mix, state, cu, slots, has_init)``."""
    n = weight.numel()
    y = torch.zeros_like(x)
    y[:, :n] = F.layer_norm(x[:, :n], (n,), weight.float(), None, eps)
    h.copy_(y)
    if shift is None:
        return None
    mix, state, cu, slots, has_init = shift
    prev = torch.zeros_like(y)
    prev[1:] = y[:-1]
    for r in range(len(slots)):
        s, e, slot = int(cu[r]), int(cu[r + 1]), int(slots[r])
        if e == s:
            continue
        prev[s] = state[slot] if slot >= 0 and bool(has_init[r]) else 0.0
        if slot >= 0:
            state[slot] = y[e - 1]
    return (y + (prev - y) * mix).to(h.dtype)
