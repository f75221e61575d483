"""Plain, slow implementation of the Seturax design, written from its equations: one function per mechanism, whole
sequences only (no cache, no batch, no absorbed products), every attention a full score matrix.

It shares no code with the package and is the ground truth of ``test_seturax``.  ``w`` maps tensor names to tensors,
``cfg`` is the dictionary of a ``config.json``; arithmetic runs in the dtype of the tensors handed in (float64 in the
tests).  Shapes: ``x [T, width]``; heads are laid out head by head.
"""
import math

import torch


def layer_norm(x, weight, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * weight, no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens, bigram):
    """Row of the bigram table per position; the first token of a sequence has the extra last row."""
    out = [bigram["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        out.append((prev * bigram["mul_prev"] + cur * bigram["mul_cur"]) % bigram["buckets"])
    return out


def embed_tokens(tokens, w, emb):
    return w["embed"][torch.as_tensor(tokens)] * emb["scale"] + w["bigram"][torch.as_tensor(bigram_rows(tokens, emb["bigram"]))]


def token_shift(h, mix):
    """h_t + (h_(t-1) - h_t) * mix per channel; zeros stand in front of the first token."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        prev = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out[t] = h[t] + (prev - h[t]) * mix
    return out


def rotate(x, base, start=0):
    """Rotate-half rotation of x [T, heads, n]: pair (i, i + n / 2) turns by position * base^(-2 i / n)."""
    T, _, n = x.shape
    out = x.clone()
    for i in range(n // 2):
        a = (start + torch.arange(T, dtype=torch.float64)) * base ** (-2.0 * i / n)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + n // 2]
        out[:, :, i] = u * c - v * s
        out[:, :, i + n // 2] = v * c + u * s
    return out


def sink_attention(q, k, v, scale, window, sink):
    """q, k [T, H, D], v [T, H, Dv]: position i sees j with 0 <= i - j < window; exp(sink[h]) joins the denominator."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    i = torch.arange(T)
    seen = (i[:, None] - i[None, :] >= 0) & (i[:, None] - i[None, :] < window)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = torch.maximum(m, sink[h])
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(sink[h] - m) if sink is not None else 0.0)
        out[:, h] = (e / den) @ v[:, h]
    return out


def latent_attention(h, w, p, m, eps):
    """``p`` is the tensor prefix ('l3.mix.'), ``m`` the mixer's sizes."""
    T = h.shape[0]
    H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :C], w[p + "dkv.norm"], eps)
    kr = rotate(down[:, None, C:], m["rot"]["base"])
    qr = rotate(q[:, :, D:], m["rot"]["base"])
    k = torch.cat([(c @ w[p + "uk"].T).reshape(T, H, D), kr.expand(T, H, R)], -1)
    q = torch.cat([q[:, :, :D], qr], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, Dv)
    o = sink_attention(q, k, v, m["scale"], m["mask"]["size"], w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention}


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer(x, w, p, spec, eps):
    """One norm; mixer (behind the token shift) and feed-forward side by side, each times its own gate."""
    h = layer_norm(x, w[p + "norm1"], eps)
    y = MIXERS[spec["type"]](token_shift(h, w[p + "shift"]), w, p + "mix.", spec["mixer"], eps)
    out = y * sigmoid(h @ w[p + "rg1"].T + w[p + "rg1.b"])
    if spec.get("mlp") is not None:
        out = out + feed_forward(h, w, p + "mlp.") * sigmoid(h @ w[p + "rg2"].T + w[p + "rg2.b"])
    return x + out


def forward(tokens, w, cfg):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    x = embed_tokens(tokens, w, cfg["embedding"])
    stream = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, f"l{i}.", spec, eps)
        stream.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"], torch.stack(stream)


# ------------------------------------------------------------------------------------------------ random models

def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W), "final.norm": (W,), "head": (V, W)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        H, D, R, Dv, C, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
        out.update({p + "norm1": (W,), p + "shift": (W,), p + "rg1": (W, W), p + "rg1.b": (W,)})
        out.update({p + "mix." + k: s for k, s in {
            "dq": (Q, W), "dq.norm": (Q,), "uq": (H * (D + R), Q), "dkv": (C + R, W), "dkv.norm": (C,), "uk": (H * D, C),
            "uv": (H * Dv, C), "sink": (H,), "g": (H, W), "o": (W, H * Dv)}.items()})
        if spec.get("mlp") is not None:
            f = spec["mlp"]["ff"]
            out.update({p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f), p + "rg2": (W, W),
                        p + "rg2.b": (W,)})
    return out


def random_weights(cfg, seed=0, dtype=torch.float64):
    """Seeded weights, already rounded to bfloat16 (what a checkpoint stores).  Queries are scaled up so that the
    attention is peaked: one key more or less then shows."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        z = torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith("norm1"):
            t = 1.0 + 0.1 * z
        elif name.endswith(".shift"):
            t = 0.5 + 0.4 * z
        elif name.endswith(".sink"):
            t = 1.0 + z
        elif name == "embed":
            t = z / cfg["embedding"]["scale"]
        elif name == "bigram":
            t = z * 0.7
        elif name.endswith(".b"):
            t = 0.5 * z
        elif name.endswith(".uq"):
            t = z * 2.5 / math.sqrt(shape[-1])
        else:
            t = z * 1.3 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out
