"""Plain, slow implementation of the Kefesun design, written from its equations: one function per mechanism, whole sequences
only (no cache, no batch, no chunks), every attention a full score matrix, every recurrence a loop over tokens.

It shares no code with the package and is the ground truth of ``test_kefesun``.  ``w`` maps tensor names to tensors, ``cfg``
is the dictionary of a ``config.json``; arithmetic runs in the dtype of the tensors handed in (float64 in the tests).
Shapes: ``x [T, width]``; heads are laid out head by head.
"""
import math

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def input_conv(h, taps):
    """h plus its causal convolution over time, channel by channel; taps [width, n], the last one meets the token itself."""
    T, n = h.shape[0], taps.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * h[s]
    return out


def rotate(x, base, dims):
    """x [T, H, D]; column i turns with column i + dims / 2 by t * base^(-2 i / dims)."""
    half = dims // 2
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            a = t * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i], out[t, :, i + half] = u * c - v * s, v * c + u * s
    return out


def visible(T, size, keep_first):
    """[T, T]: query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def sigmoid_attention(q, k, v, scale, bias, seen):
    """q, k [T, H, D], v [T, H, Dv], bias [H]: every visible key counts with the sigmoid of its score."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[-1], dtype=q.dtype)
    for h in range(q.shape[1]):
        p = sigmoid((q[:, h] @ k[:, h].T) * scale + bias[h])
        out[:, h] = torch.where(seen, p, torch.zeros_like(p)) @ v[:, h]
    return out


def attention_mixer(h, w, pre, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(T, H, m["dim"])
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(T, G, m["dim"])
    v = (h @ w[pre + "v"].T + w[pre + "v.b"]).reshape(T, G, m["vdim"])
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = rotate(rms_norm(q, w[pre + "q.norm"], eps), base, dims)
    k = rotate(rms_norm(k, w[pre + "k.norm"], eps), base, dims)
    kv_of = [i // (H // G) for i in range(H)]
    o = sigmoid_attention(q, k[:, kv_of], v[:, kv_of], m["scale"], w[pre + "pb"],
                          visible(T, m["mask"]["size"], m["mask"]["keep_first"]))
    return o.reshape(T, -1) @ w[pre + "o"].T


def blend_recurrence(z, c):
    """z, c [T, n]: S <- (1 - z) S + z c from S = 0; all states."""
    S, out = torch.zeros_like(c[0]), torch.zeros_like(c)
    for t in range(c.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out


def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def mingru_mixer(h, w, pre):
    z = sigmoid(h @ w[pre + "z"].T + w[pre + "z.b"])
    c = candidate(h @ w[pre + "x"].T + w[pre + "x.b"])
    return (blend_recurrence(z, c) * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def expert(x, up, down):
    return torch.clamp(x @ up.T, min=0.0) ** 2 @ down.T


def route(h, router, correction, top, groups, keep, scale):
    """Chosen outputs [T, top] (best first) and their weights.  Outputs form ``groups`` runs; only the ``keep`` runs with the
    best member can be chosen from."""
    z = h @ router.T
    e = torch.exp(z - z.amax(-1, keepdim=True))
    s = e / e.sum(-1, keepdim=True)
    ids = []
    for t in range(h.shape[0]):
        choice = (s[t] + correction).tolist()
        n = len(choice) // groups
        best = sorted(range(groups), key=lambda g: -max(choice[g * n:(g + 1) * n]))[:keep]
        allowed = [e for e in range(len(choice)) if e // n in best]
        ids.append(sorted(allowed, key=lambda e: -choice[e])[:top])
    ids = torch.tensor(ids)
    return ids, torch.gather(s, 1, ids) * scale


def experts(h, w, pre, mlp):
    rt = mlp["router"]
    ids, weights = route(h, w[pre + "router"], w[pre + "correction"], rt["top"], rt["groups"]["count"], rt["groups"]["keep"],
                         rt["scale"])
    out = expert(h, w[pre + "shared.up"], w[pre + "shared.down"])
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), weights[t]):
            y = h[t] if e >= rt["experts"] else expert(h[t], w[f"{pre}e{e}.up"], w[f"{pre}e{e}.down"])
            out[t] = out[t] + c * y
    return out


def forward(tokens, w, cfg, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) collects the residual stream behind every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = input_conv(x, w[p + "canon1"])
        y = attention_mixer(h, w, p + "mix.", m, eps) if layer["type"] == "attention" else mingru_mixer(h, w, p + "mix.")
        x = x + layer_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = experts(input_conv(x, w[p + "canon2"]), w, p + "mlp.", layer["mlp"])
            x = x + layer_norm(y, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def tensor_shapes(cfg):
    W, V, n = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        out.update({p + "norm1": (W,), p + "canon1": (W, n)})
        if layer["type"] == "attention":
            H, G, D, Dv = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            mix = {"q": (H * D, W), "q.b": (H * D,), "k": (G * D, W), "k.b": (G * D,), "v": (G * Dv, W), "v.b": (G * Dv,),
                   "q.norm": (D,), "k.norm": (D,), "pb": (H,), "o": (W, H * Dv)}
        else:
            d = m["width"]
            mix = {"z": (d, W), "z.b": (d,), "x": (d, W), "x.b": (d,), "g": (d, W), "o": (W, d)}
        out.update({p + "mix." + k: s for k, s in mix.items()})
        if f is None:
            continue
        rt, ff = f["router"], f["expert"]["ff"]
        outputs = rt["experts"] + rt["identity"]
        out.update({p + "norm2": (W,), p + "canon2": (W, n), p + "mlp.router": (outputs, W), p + "mlp.correction": (outputs,),
                    p + "mlp.shared.up": (f["shared"]["ff"], W), p + "mlp.shared.down": (W, f["shared"]["ff"])})
        for e in range(rt["experts"]):
            out.update({f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def random_weights(cfg, seed=0, dtype=torch.float64):
    """Seeded weights, already rounded to bfloat16 (what a checkpoint stores).  Scores spread widely around a low bias, so that few
    keys count; half of the blend gates hardly move, so that early tokens still show late; corrections of both signs."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        z = torch.randn(shape, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith((".q.norm", ".k.norm")):
            t = 1.5 + 0.3 * z
        elif leaf.startswith("norm"):
            t = 1.0 + 0.15 * z
        elif leaf.startswith("canon"):
            t = 0.4 * z
        elif leaf == "pb":
            t = z - 2.5
        elif name.endswith(".z.b"):
            t = torch.where(torch.arange(shape[0]) % 2 == 0, z - 5.0, z)
        elif leaf == "b":
            t = 0.5 * z
        elif leaf == "correction":
            t = 0.3 * z - 0.2
        elif leaf == "embed":
            t = z / math.sqrt(shape[-1])
        elif leaf == "router":
            t = z * 2.0 / math.sqrt(shape[-1])
        else:
            t = z * 1.3 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out
