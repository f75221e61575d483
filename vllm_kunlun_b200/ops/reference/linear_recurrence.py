"""fp32 PyTorch forms of the fp32-stream norms and of the linear recurrences (CPU path of ``csrc/elementwise/layernorm.cu``
and ``csrc/linear_attn/recurrence.cu``)."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def _layer_norm(y, weight, eps):
    n = weight.numel()
    out = torch.zeros_like(y)
    out[:, :n] = F.layer_norm(y[:, :n], (n,), weight.float(), None, eps)
    return out


def embed_positions_layernorm(x, h, ids, positions, table, freq, weight, eps):
    n = weight.numel()
    turns = positions.long().unsqueeze(1) * freq           # 64-bit fractions of a turn: the product wraps by itself
    angle = (turns.double() * (2 * math.pi * 2.0 ** -64)).float()
    pe = torch.stack([angle.sin(), angle.cos()], -1).reshape(len(ids), -1)[:, :n]
    y = table[ids.long()].float()
    y[:, :n] += pe
    x.copy_(_layer_norm(y, weight, eps))
    if h is not x:
        h.copy_(x)


def layernorm_residual(x, h, y1, s1, y2, s2, weight, eps):
    if y1 is None:
        h.copy_(_layer_norm(x, weight, eps))
        return
    y = y1.float() * s1
    if y2 is not None:
        y = y + y2.float() * s2
    x += _layer_norm(y, weight, eps)
    if h is not x:
        h.copy_(x)


def gated_group_rmsnorm(out, o, gate, weight, eps):
    T, n = o.shape
    y = o.float().reshape(T, -1, weight.numel())
    y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps) * weight.float()
    y = y.reshape(T, n)
    out[:, :n] = (y if gate is None else y * torch.sigmoid(gate.float())).to(out.dtype)


def qk_unit_norm_cache(q, k, v, kv_cache, slot_mapping, num_heads, num_kv_heads, eps):
    T, bs, Dc = q.shape[0], kv_cache.shape[3], kv_cache.shape[4]

    def unit(z):
        z = z.float()
        return z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps)

    def pad(z):
        return F.pad(z, (0, Dc - z.shape[-1])).to(kv_cache.dtype)

    kh = pad(unit(k.reshape(T, num_kv_heads, -1)))
    vh = pad(v.reshape(T, num_kv_heads, -1))
    ok = slot_mapping >= 0
    slots = slot_mapping[ok].long()
    kv_cache[slots // bs, 0, :, slots % bs] = kh[ok]
    kv_cache[slots // bs, 1, :, slots % bs] = vh[ok]
    return pad(unit(q.reshape(T, num_heads, -1)))


def _segments(cu_seqlens, state_indices, has_initial_state):
    for r in range(len(state_indices)):
        s, e, slot = int(cu_seqlens[r]), int(cu_seqlens[r + 1]), int(state_indices[r])
        if e > s and slot >= 0:
            yield s, e, slot, bool(has_initial_state[r])


def channel_delta_rule(out, q, k, v, a, b, A_log, dt_bias, states, cu_seqlens, state_indices, has_initial_state, scale,
                       unit_eps):
    T, H, _ = v.shape
    Dk, rep = q.shape[2], H // q.shape[1]

    def unit(z):
        z = z.float()
        return (z * torch.rsqrt(z.pow(2).sum(-1, keepdim=True) + unit_eps)).repeat_interleave(rep, 1)

    qf, kf, vf = unit(q) * scale, unit(k), v.float()
    g = torch.exp(-torch.exp(A_log.float()).reshape(1, H, 1) * F.softplus(a.float() + dt_bias.float()).reshape(T, H, Dk))
    beta = torch.sigmoid(b.float())
    for s, e, slot, init in _segments(cu_seqlens, state_indices, has_initial_state):
        S = states[slot, :, :, :Dk].clone() if init else torch.zeros_like(states[slot, :, :, :Dk])    # [H, Dv, Dk]
        for t in range(s, e):
            S = S * g[t].unsqueeze(1)
            u = beta[t].unsqueeze(-1) * (vf[t] - torch.einsum("hvk,hk->hv", S, kf[t]))
            S = S + torch.einsum("hv,hk->hvk", u, kf[t])
            out[t] = torch.einsum("hvk,hk->hv", S, qf[t])
        states[slot].zero_()
        states[slot, :, :, :Dk] = S
    return out


def fixed_decay_attention(out, q, k, v, decay, states, cu_seqlens, state_indices, has_initial_state):
    D = q.shape[2]
    qf, kf, vf = F.silu(q.float()), F.silu(k.float()), F.silu(v.float())
    d = decay.float().reshape(-1, 1, 1)
    for s, e, slot, init in _segments(cu_seqlens, state_indices, has_initial_state):
        S = states[slot, :, :, :D].clone() if init else torch.zeros_like(states[slot, :, :, :D])
        for t in range(s, e):
            S = S * d + torch.einsum("hv,hk->hvk", vf[t], kf[t])
            out[t] = torch.einsum("hvk,hk->hv", S, qf[t])
        states[slot].zero_()
        states[slot, :, :, :D] = S
    return out


def gated_write_attention(out, q, v, f, f_bias, lower, states, cu_seqlens, state_indices, has_initial_state):
    T, H, D = q.shape
    z = f.float() + f_bias
    keep = (lower + (1 - lower) * torch.sigmoid(z)).reshape(T, H, D)
    write = ((1 - lower) * torch.sigmoid(-z)).reshape(T, H, D)
    qf, vf = F.silu(q.float()), v.float()
    for s, e, slot, init in _segments(cu_seqlens, state_indices, has_initial_state):
        S = states[slot, :, :, :D].clone() if init else torch.zeros_like(states[slot, :, :, :D])          # [H, Dv, D]
        for t in range(s, e):
            S = S * keep[t].unsqueeze(1) + torch.einsum("hv,hk->hvk", vf[t], write[t])
            out[t] = torch.einsum("hvk,hk->hv", S, qf[t])
        states[slot].zero_()
        states[slot, :, :, :D] = S
    return out
