"""Plain, slow implementation of the Bolopel design, written from its equations: one function per mechanism, whole
sequences only (no cache, no batch), every recurrence a loop over tokens, every attention a full score matrix.

It shares no code with the package and is used as the ground truth of ``test_bolopel_*``.  ``w`` maps tensor names to
tensors, ``cfg`` is the dictionary of a ``config.json``; arithmetic runs in the dtype of the tensors handed in
(float64 in the tests).  Shapes: ``x [T, width]``; heads are laid out head by head.
"""
import math

import torch


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def position_vectors(n, width, start=0):
    """[n, width]: column pair i holds (sin, cos) of position / 10000^(2i / width)."""
    out = torch.zeros(n, width, dtype=torch.float64)
    for p in range(n):
        for j in range(width):
            angle = (start + p) * 10000.0 ** (-2.0 * (j // 2) / width)
            out[p, j] = math.sin(angle) if j % 2 == 0 else math.cos(angle)
    return out


def embed_tokens(tokens, w, width, eps):
    x = w["embed"][torch.as_tensor(tokens)]
    x = x + position_vectors(len(tokens), width).to(x.dtype)
    return layer_norm(x, w["embed.norm"], eps)


def causal_conv(x, taps):
    """x [T, C], taps [C, W]: y_t = sum_j taps[:, j] x_(t - W + 1 + j), zeros before the start."""
    T, C = x.shape
    W = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(W):
            s = t - (W - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def windowed_attention(q, k, v, scale, window, sink=True):
    """q [T, H, D], k [T, G, D], v [T, G, Dv]: position i sees j with 0 <= i - j < window; the denominator has one
    extra unit (a key of score 0 without a value)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    i = torch.arange(T)
    seen = (i[:, None] - i[None, :] >= 0) & (i[:, None] - i[None, :] < window)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)      # the sink's score is 0
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0.0)
        out[:, h] = (e / den) @ v[:, g]
    return out


def decayed_linear_attention(q, k, v, decay):
    """q, k [T, H, D], v [T, H, Dv], decay [H]: S <- decay S + k v^T, o = S^T q."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def channel_delta_rule(q, k, v, g, beta):
    """q, k [T, G, D], v [T, H, Dv], g [T, H, D], beta [T, H] (already activated / normalised)."""
    T, H, Dv = v.shape
    G, D = q.shape[1:]
    out = torch.zeros(T, H, Dv, dtype=q.dtype)
    for h in range(H):
        c = h // (H // G)
        S = torch.zeros(D, Dv, dtype=q.dtype)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, c])
            S = S + torch.outer(k[t, c], u)
            out[t, h] = S.T @ q[t, c]
    return out


def channel_delta_mixer(h, w, p, m, eps):
    """``p`` is the tensor prefix ('l3.mix.'), ``m`` the mixer's sizes."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, D)
    k = silu(causal_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, D)
    v = silu(causal_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, Dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = sigmoid(h @ w[p + "b"].T)
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(a).reshape(T, H, D))
    o = channel_delta_rule(q, k, v, g, beta)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, Dv)
    o = rms_unit(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def window_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit((h @ w[p + "q"].T).reshape(T, H, D), eps)
    k = rms_unit((h @ w[p + "k"].T).reshape(T, G, D), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, Dv)
    o = windowed_attention(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def lightning_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, D)
    k = silu(h @ w[p + "k"].T).reshape(T, H, D)
    v = silu(h @ w[p + "v"].T).reshape(T, H, Dv)
    o = decayed_linear_attention(q, k, v, m["decay"]).reshape(T, H * Dv)
    o = rms_unit(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    return (m["left_scale"] * window_mixer(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * lightning_mixer(h, w, p + "right.", m["right"], eps))


MIXERS = {"channel_delta": channel_delta_mixer, "parallel": parallel_mixer}


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(tokens, w, cfg):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    x = embed_tokens(tokens, w, cfg["width"], eps)
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + layer_norm(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + layer_norm(feed_forward(x, w, p + "mlp."), w[p + "norm2"], eps)
        stream.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)


# ------------------------------------------------------------------------------------------------ random models

def tensor_shapes(cfg, rank_a=None, rank_g=None):
    """Name -> shape of every tensor of a model with this configuration (low-rank widths are the caller's choice)."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            out.update({p + "left.q": (a["heads"] * a["dim"], W), p + "left.k": (a["kv_heads"] * a["dim"], W),
                        p + "left.v": (a["kv_heads"] * a["vdim"], W), p + "left.o": (W, a["heads"] * a["vdim"])})
            n = b["heads"] * b["vdim"]
            out.update({p + "right.q": (b["heads"] * b["dim"], W), p + "right.k": (b["heads"] * b["dim"], W),
                        p + "right.v": (n, W), p + "right.g": (n, W), p + "right.o": (W, n), p + "right.norm": (n,)})
        else:
            ck, cv = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, c in (("q", ck), ("k", ck), ("v", cv)):
                out[p + name], out[p + name + ".conv"] = (c, W), (c, m["conv"])
            ra, rg = rank_a or 8, rank_g or 8
            out.update({p + "b": (m["heads"], W), p + "A_log": (m["heads"],), p + "norm": (m["vdim"],),
                        p + "a1": (ra, W), p + "a2": (m["heads"] * m["dim"], ra), p + "dt_bias": (m["heads"] * m["dim"],),
                        p + "g1": (rg, W), p + "g2": (cv, rg), p + "o": (W, cv)})
        if layer.get("mlp") is not None:
            f = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.gate": (f, W), f"l{i}.mlp.up": (f, W), f"l{i}.mlp.down": (W, f)})
    return out


def random_weights(cfg, seed=0, rank_a=None, rank_g=None, dtype=torch.float64):
    """Seeded weights, already rounded to bfloat16 (what a checkpoint stores)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg, rank_a, rank_g).items()):
        z = torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            t = 1.0 + 0.1 * z
        elif name.endswith(".conv"):
            t = z / math.sqrt(shape[-1])
        elif name.endswith("A_log"):
            t = 0.5 * z - 1.0
        elif name.endswith("dt_bias"):
            t = z - 2.0
        elif name in ("embed",):
            t = z
        else:
            t = z * 1.3 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out
