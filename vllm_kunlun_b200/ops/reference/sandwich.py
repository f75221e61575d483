"""fp32 PyTorch forms of the sandwich norms, the polynomial activation, the attention split with value norms and the experts
on weighted inputs (CPU path of ``csrc/elementwise/sandwich.cu`` and of the routed experts)."""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import moe
from .latent import rotate


def _unit(x, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def _normed(x, weight, eps):
    out = torch.zeros_like(x)
    n = weight.numel()
    out[:, :n] = _unit(x[:, :n], eps) * weight
    return out


def embed_rmsnorm(x, h, ids, table, weight, eps):
    x.copy_(table[ids.long()])
    h.copy_(_normed(x, weight, eps))


def sandwich_rmsnorm(x, h, y, pos, w_post, w_pre, eps):
    y = y.float()
    if pos is not None:
        y = y[pos.long()].reshape(x.shape[0], -1, x.shape[1]).sum(1)
    x += _normed(y, w_post, eps)
    h.copy_(_normed(x, w_pre, eps))


def poly_norm(out, z, coeff, width, eps):
    x = z[:, :width].float()
    a, b, c, e = coeff.tolist()
    out.zero_()
    out[:, :width] = a * _unit(x, eps) + b * _unit(x ** 2, eps) + c * _unit(x ** 3, eps) + e


def attn_prep_cache(q_out, q, k, v, kv_cache, slot_mapping, positions, num_heads, num_kv_heads, coef, every, v_out, v_in, share,
                    eps, v_norm=True, q_norm=None, k_norm=None, table=None):
    T, bs, Dc = q.shape[0], kv_cache.shape[3], kv_cache.shape[4]

    def pad(z):
        return F.pad(z, (0, Dc - z.shape[-1])).to(kv_cache.dtype)

    def heads(z, n, weight):
        z = z.float().reshape(T, n, -1)
        if weight is not None:
            z = _unit(z, eps) * weight
        return z if table is None else rotate(z, table)

    vh = v.float().reshape(T, num_kv_heads, -1)
    if v_norm:
        vh = _unit(vh, eps)
    if v_out is not None:
        v_out.copy_(vh.reshape(T, -1))
    if v_in is not None:
        vh = (1 - share) * vh + share * v_in.float().reshape(vh.shape)
    ok = slot_mapping >= 0
    slots = slot_mapping[ok].long()
    kv_cache[slots // bs, 0, :, slots % bs] = pad(heads(k, num_kv_heads, k_norm))[ok]
    kv_cache[slots // bs, 1, :, slots % bs] = pad(vh)[ok]
    qf = heads(q, num_heads, q_norm)
    if every > 0:
        qf = qf * (1 + coef * torch.log(((positions + 1) // every + 1).float()))[:, None, None]
    q_out.copy_(pad(qf))


def swiglu_limit_and_mul(x, limit):
    g, u = x.float().chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).to(x.dtype)


def expert_rows(x, w_in, w_out, topk_ids, act, factors, choices):
    T, k = topk_ids.shape
    E = w_in.shape[0]
    pairs = x.unsqueeze(1).expand(T, k, -1)
    if factors is not None:
        pairs = (pairs.float() * factors.float().unsqueeze(-1)).to(x.dtype)
    xs, order, lod = moe.moe_permute(pairs.reshape(T * k, -1), topk_ids.reshape(T * k, 1), choices)
    y = moe.grouped_gemm(act(moe.grouped_gemm(xs, w_in, lod)), w_out, lod)      # rows behind the experts' stay zero
    pos = torch.empty(T * k, dtype=torch.int32)
    pos[order.long()] = torch.arange(T * k, dtype=torch.int32)
    return y, torch.where(topk_ids.reshape(-1) < E, pos, torch.full_like(pos, -1))
