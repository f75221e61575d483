"""Plain, slow implementation of the Petipel design, written from its equations: one function per mechanism, whole sequences
only (no cache, no batch, no chunks), every attention a full score matrix, every recurrence a loop over tokens.

It shares no code with the package and is the ground truth of ``test_petipel``.  ``w`` maps tensor names to tensors, ``cfg``
is the dictionary of a ``config.json``; arithmetic runs in the dtype of the tensors handed in (float64 in the tests).
Shapes: ``x [T, width]``; heads are laid out head by head.
"""
import math

import torch


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def query_temperature(pos, coef, every):
    """Factor of a query at position pos."""
    return 1.0 + coef * math.log((pos + 1) // every + 1)


def distance_bucket(n, rows, far):
    """Row of a distance table with ``rows`` rows: one row per distance below rows / 2, then logarithmically wider ones that
    reach the end at ``far``; farther distances share the last row."""
    half = rows // 2
    if n < half:
        return n
    x = half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)
    return int(min(rows - 1, x))


def distance_bias(T, table, far):
    """[heads, T, T]: entry of query i and key j <= i."""
    rows, H = table.shape
    out = torch.zeros(H, T, T, dtype=table.dtype)
    near = torch.stack([table[distance_bucket(n, rows, far)] for n in range(T)])   # [distance, head]
    for i in range(T):
        out[:, i, :i + 1] = near[:i + 1].flip(0).T
    return out


def attention(q, k, v, scale, bias):
    """q, k [T, H, D], v [T, H, Dv], bias [H, T, T]; causal softmax."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale + bias[h]
        s = s.masked_fill(hidden, float("-inf"))
        e = torch.exp(s - s.amax(-1, keepdim=True))
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, h]
    return out


def mix_values(v, v_first, share):
    return (1.0 - share) * v + share * v_first


def attention_mixer(h, w, pre, m, eps, v_first):
    """Returns the output and the values [T, G, Dv] as they are attended."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[pre + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[pre + "k"].T).reshape(T, G, m["dim"])
    v = unit_rms((h @ w[pre + "v"].T).reshape(T, G, m["vdim"]), eps)
    t = m.get("q_temp")
    if t is not None:
        f = [query_temperature(p, t["coef"], t["every"]) for p in range(T)]
        q = q * torch.tensor(f, dtype=q.dtype)[:, None, None]
    if v_first is not None:
        v = mix_values(v, v_first, w[pre + "vmix"])
    kv_of = [i // (H // G) for i in range(H)]
    o = attention(q, k[:, kv_of], v[:, kv_of], m["scale"], distance_bias(T, w[pre + "rel"], m["bias_max"]))
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[pre + "o"].T, v


def hgrn2_recurrence(q, f, v):
    """q, f [T, H, D], v [T, H, Dv]: S <- f S + (1 - f) v^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def hgrn2_mixer(h, w, pre, m, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ w[pre + "q"].T).reshape(T, H, m["dim"])
    low = w[pre + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[pre + "f"].T + w[pre + "f.b"])).reshape(T, H, m["dim"])
    v = (h @ w[pre + "v"].T).reshape(T, H, m["vdim"])
    o = unit_rms(hgrn2_recurrence(q, f, v), eps) * w[pre + "norm"]
    return o.reshape(T, -1) @ w[pre + "o"].T


def poly_norm(z, coeffs, eps):
    a, b, c, e = coeffs
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def expert(x, gate, up, down, limit):
    g = torch.clamp(x @ gate.T, max=limit)
    u = torch.clamp(x @ up.T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, top):
    """[T, top] expert numbers, largest score first, and their scores."""
    s = sigmoid(h @ router.T)
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return order, torch.gather(s, 1, order)


def experts(h, w, pre, mlp):
    out = torch.zeros_like(h)
    ids, scores = route(h, w[pre + "router"], mlp["router"]["top"])
    for t in range(h.shape[0]):
        for e, s in zip(ids[t].tolist(), scores[t]):
            out[t] += expert(s * h[t], w[f"{pre}e{e}.gate"], w[f"{pre}e{e}.up"], w[f"{pre}e{e}.down"],
                             mlp["expert"]["limit"])
    return out


def feed_forward(h, w, pre, mlp, eps):
    if mlp["kind"] == "moe":
        return experts(h, w, pre, mlp)
    return poly_norm(h @ w[pre + "up"].T, w[pre + "act"], eps) @ w[pre + "down"].T


def forward(tokens, w, cfg, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) collects the residual stream behind every layer."""
    eps, scale = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, v = attention_mixer(h, w, p + "mix.", m, eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = v
        else:
            y = hgrn2_mixer(h, w, p + "mix.", m, eps)
        x = x + scale * norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], eps)
            x = x + scale * norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].T


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if layer["type"] == "attention":
            G = m["kv_heads"]
            mix = {"q": (H * D, W), "k": (G * D, W), "v": (G * Dv, W), "rel": (m["bias_rows"], H), "g": (H, W), "o": (W, H * Dv)}
            if m.get("v_mix"):
                mix["vmix"] = ()
        else:
            mix = {"q": (H * D, W), "f": (H * D, W), "f.b": (H * D,), "lower": (H * D,), "v": (H * Dv, W), "norm": (Dv,),
                   "o": (W, H * Dv)}
        out.update({p + "mix." + k: s for k, s in mix.items()})
        if f is None:
            continue
        out.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if f["kind"] == "dense":
            mlp = {"up": (f["ff"], W), "down": (W, f["ff"]), "act": (4,)}
        else:
            n, E = f["expert"]["ff"], f["router"]["experts"]
            mlp = {"router": (E, W)}
            for e in range(E):
                mlp.update({f"e{e}.gate": (n, W), f"e{e}.up": (n, W), f"e{e}.down": (W, n)})
        out.update({p + "mlp." + k: s for k, s in mlp.items()})
    return out


def random_weights(cfg, seed=0, dtype=torch.float64):
    """Seeded weights, already rounded to bfloat16 (what a checkpoint stores).  Queries are scaled up so that the attention
    is peaked; half of the forget gates hardly forget, so that early tokens still show late."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in sorted(tensor_shapes(cfg).items()):
        z = torch.randn(shape, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".mix.norm"):
            t = 1.0 + 0.1 * z
        elif leaf.startswith("norm"):
            t = 0.15 * z
        elif leaf == "rel":
            t = 1.5 * z
        elif leaf == "vmix":
            t = 0.2 + 0.5 * torch.sigmoid(z)
        elif leaf == "lower":
            t = torch.sigmoid(z) * (torch.arange(shape[0]) % 3 > 0)
        elif leaf == "b":
            t = torch.where(torch.arange(shape[0]) % 2 == 0, z + 6.0, z)
        elif leaf == "act":
            t = 0.5 + 0.3 * z
        elif leaf == "embed":
            t = z
        elif name.endswith(".mix.q"):
            t = z * 2.0 / math.sqrt(shape[-1])
        elif leaf == "router":
            t = z * 3.0 / math.sqrt(shape[-1])
        else:
            t = z * 1.3 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out
