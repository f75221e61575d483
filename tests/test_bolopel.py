"""Bolopel against the plain implementation in ``oracle_bolopel``: every mechanism alone, whole models through the
engine (whole prompts, portions, mixed batches, decoding, reused pages and slots), configuration and weight loading, the
replay program.  Each test runs on the CPU path and, on a GPU box, on the kernels (fp32 and bf16)."""
import copy

import json
import math
import os
import subprocess
import sys

import pytest
import torch

import oracle_bolopel as oracle
from vllm_kunlun_b200 import LLM, SamplingParams, ops
from vllm_kunlun_b200.config import ModelConfig, SchedulerConfig  # noqa: F401
from vllm_kunlun_b200.engine.replay import ScheduleReplay
from vllm_kunlun_b200.models.loader import save_safetensors

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
# kernels under test: fp32 on both devices, bf16 on the GPU
RUNS = [("cpu", "float32"), pytest.param("cuda", "float32", marks=pytest.mark.gpu),
        pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def parallel(heads=4, kv_heads=2, dim=12, vdim=20, size=7, scale=0.9, rheads=3, rdim=8, rvdim=16, decay=None, ls=0.8,
             rs=1.3):
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}},
            "right": {"heads": rheads, "dim": rdim, "vdim": rvdim,
                      "decay": decay or [0.5 + 0.49 * i / max(1, rheads - 1) for i in range(rheads)]},
            "left_scale": ls, "right_scale": rs}


def delta(heads=4, kv_heads=2, dim=12, vdim=8, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def layer(kind, mixer, ff=24):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=40, vocab=97, eps=1e-5):
    return {"architecture": "Bolopel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every branch, unequal sizes everywhere; a layer without feed-forward; widths that need padding
SMALL = config([layer("parallel", parallel()), layer("channel_delta", delta()), layer("parallel", parallel(
    heads=3, kv_heads=3, dim=16, vdim=6, size=1, rheads=1, rdim=5, rvdim=7, ls=-0.5, rs=0.7), ff=None),
    layer("channel_delta", delta(heads=3, kv_heads=1, dim=7, vdim=12, conv=2), ff=50)], width=36)
# head sizes of the tensor-core attention kernels, longer windows, decays close to 1
WIDE = config([layer("channel_delta", delta(heads=2, kv_heads=2, dim=32, vdim=40, conv=3), ff=72),
               layer("parallel", parallel(heads=6, kv_heads=2, dim=80, vdim=112, size=70, scale=0.12, rheads=2, rdim=64,
                                          rvdim=64, decay=[0.9, 0.998]), ff=136),
               layer("parallel", parallel(heads=8, kv_heads=1, dim=48, vdim=64, size=33, scale=0.2, rheads=4, rdim=36,
                                          rvdim=24, decay=[1.0, 0.0, 0.7, 0.99]), ff=64)], width=104, vocab=300, eps=1e-3)
CONFIGS = {"small": SMALL, "wide": WIDE}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Many tiny operations: one thread is several times faster than all of them."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    """name -> (directory, configuration, float64 weights)."""
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        w = oracle.random_weights(cfg, seed=3 + i, rank_a=5 + 6 * i, rank_g=3 + 13 * i)
        path = str(tmp_path_factory.mktemp(name))
        save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, path, cfg)
        out[name] = (path, cfg, w)
    return out


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, what=""):
    """fp32: rounding of 32-bit sums; bf16: a small fraction of the values' root mean square."""
    got, want = got.double().cpu(), want.double()
    scale = want.pow(2).mean().sqrt().clamp(min=1e-3)
    err = ((got - want).abs().max() / scale).item()
    limit = 2e-4 if dtype == "float32" else 0.12
    assert err < limit, f"{what}: error {err:.2e} of the root mean square (limit {limit})"


def close_rows(got, want, dtype, what=""):
    """Logits (or stream rows) of a whole model.  In bf16 single positions of a small random model amplify rounding, so
    rows are judged one by one: nearly all within 10 %, the median within 5 %, none far off."""
    if dtype == "float32":
        return close(got, want, dtype, what)
    d, want = got.double().cpu() - want.double(), want.double()
    rows = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    stats = (rows.median().item(), rows.max().item(), int((rows > 0.1).sum()))
    assert stats[0] < 0.05 and stats[1] < 0.4 and stats[2] <= max(2, 0.06 * len(rows)), f"{what}: {stats} of {len(rows)}"


def replay(path, dtype, device, max_tokens, **kw):
    return ScheduleReplay(path, dtype, max_tokens, device=device, **kw)


# ------------------------------------------------------------------------------------------------ mechanisms

@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width", [40, 37, 2048])
def test_embedding_positions_and_norms(device, dtype, width):
    g = torch.Generator().manual_seed(width)
    ld, V, T = -(-width // 8) * 8, 50, 9
    table = torch.zeros(V, ld)
    table[:, :width] = torch.randn(V, width, generator=g)
    table = table.to(torch.bfloat16)
    w = (1 + 0.2 * torch.randn(width, generator=g)).float()
    ids = torch.randint(0, V, (T,), generator=g)
    start = 70001                                   # positions far out: the angle must not lose bits
    pos = torch.arange(start, start + T)
    freq = ops.position_turns(width, 10000.0)
    x, h = ops.embed_positions_layernorm(ids.to(device), pos.to(device), table.to(DT[dtype]).to(device), freq.to(device),
                                         w.to(device), 1e-5)
    want = oracle.layer_norm(table[ids].double()[:, :width] + oracle.position_vectors(T, width, start), w.double(), 1e-5)
    close(x[:, :width], want, "float32", "stream")
    close(h[:, :width], want, dtype, "copy")
    assert x.dtype == torch.float32 and not x[:, width:].any() and not h[:, width:].any()
    # one and two summands, and the final norm
    y1, y2 = (torch.zeros(T, ld), torch.zeros(T, ld))
    y1[:, :width] = torch.randn(T, width, generator=g) * 3 + 5      # a mean that the norm has to remove
    y2[:, :width] = torch.randn(T, width, generator=g)
    y1, y2 = y1.to(DT[dtype]), y2.to(DT[dtype])
    for parts, total in (([(y1, 1.0)], y1.double()), ([(y1, 0.7), (y2, -1.9)], 0.7 * y1.double() - 1.9 * y2.double())):
        s = torch.zeros(T, ld)
        s[:, :width] = torch.randn(T, width, generator=g)
        xs = s.clone().to(device)
        hh = ops.layernorm_residual(xs, DT[dtype], [(y.to(device), c) for y, c in parts], w.to(device), 1e-2)
        want = s[:, :width].double() + oracle.layer_norm(total[:, :width], w.double(), 1e-2)
        close(xs[:, :width], want, "float32", "residual")
        close(hh[:, :width], want, dtype, "residual copy")
        before = xs.clone()
        fin = ops.layernorm_residual(xs, DT[dtype], [], w.to(device), 1e-5)
        close(fin[:, :width], oracle.layer_norm(want, w.double(), 1e-5), dtype, "final norm")
        assert torch.equal(before, xs)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("groups,D", [(3, 20), (1, 7), (1, 2048), (16, 128)])
def test_gated_group_norm(device, dtype, groups, D):
    g = torch.Generator().manual_seed(D)
    T, n = 5, groups * D
    o, wide = torch.randn(T, n, generator=g) * 3, torch.randn(T, n + 16, generator=g).to(DT[dtype])
    w = (1 + 0.2 * torch.randn(D, generator=g)).float()
    out = torch.zeros(T, -(-n // 8) * 8, dtype=DT[dtype], device=device)
    ops.gated_group_rmsnorm(o.to(device), wide.to(device)[:, 8:8 + n], w.to(device), 1e-3, out)
    want = oracle.rms_unit(o.double().reshape(T, groups, D), 1e-3) * w.double()
    want = want.reshape(T, n) * oracle.sigmoid(wide[:, 8:8 + n].double())
    close(out[:, :n], want, dtype)
    assert not out[:, n:].any()


def _paged(device, dtype, q, k, v, scale, window, sink, lens_before, bs=16, eps=1e-6, extra_blocks=3):
    """Run q / k / v [T, heads, size] of several requests (``lens_before``: list of (context, new tokens)) through the
    cache: the context is written first, then the new tokens attend."""
    from vllm_kunlun_b200.models.mixers import cache_head_dim
    H, G, dt = q.shape[1], k.shape[1], DT[dtype]
    Dc = cache_head_dim(q.shape[2], v.shape[2], dt)
    n_req = len(lens_before)
    nblk = [-(-(c + n) // bs) for c, n in lens_before]
    total = sum(nblk) + extra_blocks
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(1)).tolist()
    cache = torch.full((total, 2, G, bs, Dc), 7.0, dtype=dt, device=device)     # stale contents of earlier requests
    cache[..., max(q.shape[2], v.shape[2]):] = 0                                # padding dims are zero from the start
    cache[:, 0, :, :, q.shape[2]:] = 0
    cache[:, 1, :, :, v.shape[2]:] = 0
    bt = torch.zeros(n_req, max(nblk), dtype=torch.int32)
    flat = torch.cat([q.flatten(1), k.flatten(1), v.flatten(1)], 1)
    flat = torch.nn.functional.pad(flat, (0, -flat.shape[1] % 8)).to(dt).to(device)
    nq, nk = q[0].numel(), k[0].numel()
    off = at = 0
    new_rows, slots = [], torch.zeros(q.shape[0], dtype=torch.int64)
    for r, (c, n) in enumerate(lens_before):
        blocks = perm[at:at + nblk[r]]
        at += nblk[r]
        bt[r, :len(blocks)] = torch.tensor(blocks)
        p = torch.arange(c + n)
        slots[off:off + c + n] = torch.tensor(blocks)[p // bs] * bs + p % bs
        new_rows += list(range(off + c, off + c + n))
        off += c + n
    parts = flat[:, :nq], flat[:, nq:nq + nk], flat[:, nq + nk:nq + nk + v[0].numel()]
    qn = ops.qk_unit_norm_cache(*parts, cache, slots.to(device), H, G, eps)
    rows = torch.tensor(new_rows)
    lens = torch.tensor([c + n for c, n in lens_before], dtype=torch.int32)
    qsl = torch.tensor([0] + [n for _, n in lens_before]).cumsum(0).int()
    dec = 0
    while dec < n_req and lens_before[dec][1] == 1:
        dec += 1
    sinks = None if sink is None else torch.full((H,), sink, device=device)
    o = ops.paged_attention(qn[rows.to(device)].contiguous(), cache, bt.to(device), lens.to(device), qsl.to(device), scale,
                            max(n for _, n in lens_before), int(lens.max()), window, sinks, num_decodes=dec,
                            num_decode_tokens=dec)
    return o.reshape(len(rows), H, Dc)[:, :, :v.shape[2]], rows


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 12, 20), (3, 1, 64, 64), (6, 2, 96, 80), (4, 4, 128, 128), (2, 1, 200, 136)])
def test_windowed_attention_with_sink(device, dtype, H, G, D, Dv):
    """Unequal requests, decode rows beside prompt portions, windows from 1 to longer than everything; the first tokens
    (where the sink weighs most)."""
    g = torch.Generator().manual_seed(D)
    lens = [(37, 1), (64, 1), (0, 1), (0, 50), (30, 21), (63, 2)]
    T = sum(c + n for c, n in lens)
    q, k, v = (torch.randn(T, h, d, generator=g).to(DT[dtype]).float() for h, d in ((H, D), (G, D), (G, Dv)))
    for window in (1, 5, 16, 33, 500):
        got, rows = _paged(device, dtype, q, k, v, 2.0 / math.sqrt(D), window, 0.0, lens, bs=64 if window > 5 else 16)
        want, off = [], 0
        for c, n in lens:
            s = slice(off, off + c + n)
            off += c + n
            want.append(oracle.windowed_attention(oracle.rms_unit(q[s].double(), 1e-6), oracle.rms_unit(k[s].double(), 1e-6),
                                                  v[s].double(), 2.0 / math.sqrt(D), window)[c:])
        close(got, torch.cat(want), dtype, f"window {window}")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("window", [3, 16, 17, 64, 65])
def test_window_edge_and_page_borders(device, dtype, window):
    """One key per query stands out (same direction as the query, a value no other key has): it is seen at distance
    window - 1 and not at distance window, in a prompt and in decoding, across page borders."""
    H = G = 1
    D, Dv, L, scale = 32, 8, 150, 1.0
    for dist in (window - 1, window):
        for i in (window, 64, 79, 80, 127, 128, 149):
            if i < dist:
                continue
            q = torch.zeros(L, H, D)
            q[..., 1] = 1.0
            k = torch.zeros(L, G, D)
            k[..., 2] = 1.0                                     # orthogonal to every query: score 0
            k[i - dist, :, 2], k[i - dist, :, 1] = 0.0, 1.0     # score sqrt(D) * sqrt(D) * scale = 32
            v = torch.zeros(L, G, Dv)
            v[i - dist, :, 3] = 1.0
            for lens in ([(i, 1)], [(0, i + 1)], [(i - 1, 2)]):
                got, rows = _paged(device, dtype, q[:i + 1], k[:i + 1], v[:i + 1], scale, window, 0.0, lens)
                seen = float(got[-1, 0, 3])
                assert (seen > 0.99) == (dist < window) and (seen < 0.01) == (dist >= window), (dist, i, lens, seen)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_sink_of_the_first_token(device, dtype):
    q = torch.ones(1, 2, 16)
    k, v = torch.ones(1, 1, 16), torch.full((1, 1, 8), 3.0)
    got, _ = _paged(device, dtype, q, k, v, 0.1, 4, 0.0, [(0, 1)])
    s = 16 * 0.1
    close(got, torch.full((1, 2, 8), 3.0 * math.exp(s) / (1 + math.exp(s))), dtype)
    got, _ = _paged(device, dtype, q, k, v, 0.1, 4, None, [(0, 1)])
    close(got, torch.full((1, 2, 8), 3.0), dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("W", [1, 2, 3, 4, 8, 11])
def test_short_convolution(device, dtype, W):
    """Portions down to one and two tokens (shorter than the filter), a reused slot, a first portion of one token."""
    g = torch.Generator().manual_seed(W)
    C, T = 24, 29
    x = torch.randn(2, T, C, generator=g).to(DT[dtype])
    taps = torch.randn(C, W, generator=g).to(DT[dtype])
    want = [oracle.silu(oracle.causal_conv(x[r].double(), taps.double())) for r in range(2)]
    state = torch.full((3, W - 1, C), 9.0, dtype=DT[dtype], device=device)        # what earlier requests left
    at, cuts = [0, 0], [[1, 1, 2, 5, 1, 9, 2, 8], [4, 1, 1, 1, 7, 2, 13]]
    got = [[], []]
    for step in range(8):
        live = [r for r in range(2) if step < len(cuts[r])]
        n = [cuts[r][step] for r in live]
        xs = torch.cat([x[r, at[r]:at[r] + c] for r, c in zip(live, n)]).to(device)
        slots = torch.tensor([2 - r for r in live], dtype=torch.int32, device=device)
        init = torch.tensor([int(at[r] > 0) for r in live], dtype=torch.int32, device=device)
        cu = torch.tensor([0] + n).cumsum(0).int().to(device)
        if max(n) == 1:
            y = ops.causal_conv1d_update(xs, state, taps.to(device), None, slots, True, init)
        else:
            y = ops.causal_conv1d_fn(xs, taps.to(device), None, cu, state, slots, init, True)
        for j, r in enumerate(live):
            got[r].append(y[int(cu[j]):int(cu[j + 1])].cpu())
            at[r] += n[j]
    for r in range(2):
        close(torch.cat(got[r]), want[r], dtype, f"request {r}")
    assert bool((state[0] == 9.0).all())                       # a slot nobody used


def _recur(device, dtype, fn, T, cuts, make_args, state_shape):
    """Feed one request in the portions ``cuts`` next to a second request that always decodes; returns the outputs of
    both."""
    state = torch.full((4, *state_shape), 5.0, device=device)
    at, outs, outs2, i = 0, [], [], 0
    for n in cuts:
        rows = list(range(at, at + n))
        args = make_args([i] + rows)            # row 0: the decoding neighbour's i-th token
        cu = torch.tensor([0, 1, 1 + n], dtype=torch.int32, device=device)
        slots = torch.tensor([3, 1], dtype=torch.int32, device=device)
        init = torch.tensor([int(i > 0), int(at > 0)], dtype=torch.int32, device=device)
        o = fn(args, state, cu, slots, init)
        outs2.append(o[:1].cpu())
        outs.append(o[1:].cpu())
        at, i = at + n, i + 1
    assert at == T and bool((state[0] == 5.0).all()) and bool((state[2] == 5.0).all())
    return torch.cat(outs), torch.cat(outs2)


CUTS = [[150], [1] * 20 + [130], [2, 3, 1, 64, 16, 17, 2, 45], [70, 2, 1, 1, 1, 63, 12]]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,D,Dv", [(3, 8, 16), (2, 64, 48), (1, 5, 7), (2, 128, 128), (2, 96, 36), (1, 160, 24)])
def test_fixed_decay_attention(device, dtype, H, D, Dv):
    """Portions against the token-by-token rule, decays from 0 to 1, head sizes of every kernel instance."""
    g = torch.Generator().manual_seed(D)
    T = 150
    q, k, v = (torch.randn(T, H, d, generator=g).to(DT[dtype]) for d in (D, D, Dv))
    for decay in ([0.97, 0.0, 0.5], [1.0, 0.999, 1e-3]):
        dec = torch.tensor(decay[:H])
        s = [oracle.silu(z.double()) for z in (q, k, v)]
        want = oracle.decayed_linear_attention(*s, dec.double())
        pad = lambda z: torch.nn.functional.pad(z.reshape(T, -1), (0, -z[0].numel() % 8))  # noqa: E731
        flat = torch.cat([pad(z) for z in (q, k, v)], 1)
        offs = [0, pad(q).shape[1], 2 * pad(q).shape[1]]

        def args(rows):
            f = flat[rows].to(device)
            return [f.as_strided((len(rows), H, d), (f.stride(0), d, 1), o) for o, d in zip(offs, (D, D, Dv))]

        for cuts in CUTS:
            got, other = _recur(device, dtype, lambda a, st, cu, sl, ini: ops.fixed_decay_attention(
                *a, dec.to(device), st, cu, sl, ini, max(1, int((cu[1:] - cu[:-1]).max())), 1), T, cuts, args, (H, Dv, -(-D // 4) * 4))
            close(got, want, dtype, f"portions {cuts[:4]}")
            close(other, want[:len(cuts)], dtype, "neighbour")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 12, 8), (2, 2, 64, 40), (3, 1, 7, 20), (2, 1, 128, 128), (2, 2, 96, 36),
                                      (1, 1, 200, 12)])
def test_channel_delta_rule(device, dtype, H, G, D, Dv):
    """Strong and weak decays side by side (from nearly 1 to below the smallest fp32 number), portions, grouped heads."""
    g = torch.Generator().manual_seed(D)
    T = 150
    q, k, v = (torch.randn(T, h, d, generator=g).to(DT[dtype]) for h, d in ((G, D), (G, D), (H, Dv)))
    a = (torch.randn(T, H * D, generator=g) * 3).to(DT[dtype])
    b = (torch.randn(T, H, generator=g) * 2).to(DT[dtype])
    A_log = torch.linspace(-3.0, 2.0, H)
    dt = torch.randn(H * D, generator=g) * 3 - 3
    dt[::7] = 40.0                                             # these channels forget within a token
    dt[3::7] = -12.0                                           # these keep nearly everything
    unit = lambda z: z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)  # noqa: E731
    decay = torch.exp(-torch.exp(A_log.double())[None, :, None] * oracle.softplus(a.double() + dt.double()).reshape(T, H, D))
    want = oracle.channel_delta_rule(unit(q.double()) * D ** -0.5, unit(k.double()), v.double(), decay,
                                     oracle.sigmoid(b.double()))
    pad = lambda z: torch.nn.functional.pad(z.reshape(T, -1), (0, -z[0].numel() % 8))  # noqa: E731
    flat = torch.cat([pad(z) for z in (q, k, v)], 1)
    offs = [0, pad(q).shape[1], 2 * pad(q).shape[1]]

    def args(rows):
        f = flat[rows].to(device)
        return [f.as_strided((len(rows), h, d), (f.stride(0), d, 1), o) for o, (h, d) in zip(offs, ((G, D), (G, D), (H, Dv)))] + \
            [a[rows].to(device), b[rows].to(device)]

    for cuts in CUTS:
        got, other = _recur(device, dtype, lambda z, st, cu, sl, ini: ops.channel_delta_rule(
            *z, A_log.to(device), dt.to(device), st, cu, sl, ini, D ** -0.5, 1e-6, max(1, int((cu[1:] - cu[:-1]).max())), 1), T, cuts, args, (H, Dv, -(-D // 4) * 4))
        close(got, want, dtype, f"portions {cuts[:4]}")
        close(other, want[:len(cuts)], dtype, "neighbour")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,N,K", [(1, 3, 5), (7, 130, 33), (33, 64, 40), (200, 65, 129)])
def test_fp32_linear(device, T, N, K):
    g = torch.Generator().manual_seed(T)
    x, w, b = torch.randn(T, K, generator=g), torch.randn(N, K, generator=g), torch.randn(N, generator=g)
    y = ops.linear(x.to(device), w.to(device), b.to(device))
    torch.testing.assert_close(y.cpu().double(), x.double() @ w.double().T + b.double(), rtol=2e-6, atol=2e-5)
    assert ops.linear(x[:0].to(device), w.to(device)).shape == (0, N)


# ------------------------------------------------------------------------------------------------ whole models

@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_stream(checkpoints, device, dtype, name):
    path, cfg, w = checkpoints[name]
    toks = tokens(83, cfg["vocab"])
    want, stream = oracle.forward(toks, w, cfg)
    r = replay(path, dtype, device, 128)
    layers = []
    r.engine.runner.model.post_layer_hook = lambda i, h, x: layers.append(x.float().cpu().clone())
    got = r.step([{"id": "a", "tokens": toks, "want": list(range(len(toks)))}], ["a"])
    assert got.dtype == torch.float32
    close_rows(got, want, dtype, "logits")
    for i, (x, s) in enumerate(zip(layers, stream)):
        close_rows(x, s, dtype, f"stream after layer {i}")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_decoding(checkpoints, device, dtype, name):
    """Token by token from the start, portions of changing size down to two tokens, long decoding after a prompt: all
    give the logits of the whole prompt.  Every request runs in the pages and slots of the one before."""
    path, cfg, w = checkpoints[name]
    L = 150
    toks = tokens(L, cfg["vocab"], 1)
    want, _ = oracle.forward(toks, w, cfg)
    r = replay(path, dtype, device, 192)
    for cuts in ([1] * L, [64, 2, 1, 30, 3, 2, 48], [2] * 40 + [70], [33] + [1] * (L - 33)):
        if device == "cpu" and name == "wide" and cuts[0] == 1:
            continue
        at, got = 0, []
        for n in cuts:
            got.append(r.step([{"id": "a", "tokens": toks[at:at + n], "want": list(range(n))}]))
            at += n
        r.step([], ["a"])
        close_rows(torch.cat(got), want, dtype, f"portions {cuts[:4]}")


@pytest.mark.parametrize("device,dtype", RUNS)
def test_mixed_batches_and_reuse(checkpoints, device, dtype):
    """Up to four live requests, portions beside single tokens, requests that pause, pages and slots that go round: each
    request's logits are those it has alone."""
    path, cfg, w = checkpoints["small"]
    lens = {"a": 90, "b": 41, "c": 7, "d": 1, "e": 66, "f": 2, "g": 64}
    toks = {k: tokens(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: oracle.forward(t, w, cfg)[0] for k, t in toks.items()}
    r = replay(path, dtype, device, 320)
    pool = r.engine.pool
    gen = torch.Generator().manual_seed(5)
    at, got, waiting, live = {k: 0 for k in lens}, {k: [] for k in lens}, list(lens), []
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-lens[k] // 64) for k in live + waiting[:1]) <= 5:
            live.append(waiting.pop(0))
        entries, end = [], []
        for k in list(live):
            n = [0, 1, 1, 2, 17, 40][int(torch.randint(0, 6, (1,), generator=gen))]
            n = min(n, lens[k] - at[k])
            if n == 0:
                continue
            wants = [i for i in range(n) if (at[k] + i) % 3 != 1]          # not every place is asked for
            entries.append({"id": k, "tokens": toks[k][at[k]:at[k] + n], "want": wants})
            at[k] += n
            if at[k] == lens[k]:
                end.append(k)
                live.remove(k)
        if not entries:
            continue
        rows = r.step(entries, end)
        i = 0
        for e in entries:
            got[e["id"]].append(rows[i:i + len(e["want"])])
            i += len(e["want"])
    for k in lens:
        have, keep = torch.cat(got[k]), [i for i in range(lens[k]) if i % 3 != 1]
        close_rows(have, want[k][keep], dtype, f"request {k}")
    assert pool.num_free == pool.num_blocks and len(r.engine.scheduler.free_state_slots) == 4


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kind", ["parallel", "channel_delta"])
def test_models_of_one_kind(device, dtype, kind, tmp_path):
    """No paged cache at all, or no convolution state at all; grouped heads beyond one decode tile."""
    mix = parallel(heads=20, kv_heads=1, dim=24, vdim=8, size=50, rheads=2) if kind == "parallel" else delta(conv=1)
    cfg = config([layer(kind, mix, ff=40)] * 2, width=48)
    w = oracle.random_weights(cfg, seed=21)
    save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, str(tmp_path), cfg)
    t = tokens(90, cfg["vocab"], 3)
    want, _ = oracle.forward(t, w, cfg)
    r = replay(str(tmp_path), dtype, device, 128)
    got = [r.step([{"id": "a", "tokens": t[i:i + n], "want": list(range(n))}]) for i, n in
           [(0, 50), (50, 2), (52, 1), (53, 1), (54, 30)] + [(i, 1) for i in range(84, 90)]]
    close_rows(torch.cat(got), want, dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_one_token_prompt_in_a_used_slot(checkpoints, device, dtype):
    """A first portion of one token starts from zero state even when its slot still holds another request's."""
    path, cfg, w = checkpoints["small"]
    r = replay(path, dtype, device, 128)
    for i in range(3):
        t = tokens(20, cfg["vocab"], 40 + i)
        r.step([{"id": "x", "tokens": t, "want": []}], ["x"])
        want, _ = oracle.forward(t[:3], w, cfg)
        got = [r.step([{"id": "y", "tokens": [t[j]], "want": [0]}]) for j in range(3)]
        r.step([], ["y"])
        close_rows(torch.cat(got), want, dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_token_reaches_through_the_state(checkpoints, device, dtype):
    """Only the recurrent layers carry a token past every window: changing it changes the logits far behind it, by the
    same amount as in the plain implementation."""
    path, cfg, w = checkpoints["wide"]
    a = tokens(140, cfg["vocab"], 9)
    b = list(a)
    b[3] = (b[3] + 11) % cfg["vocab"]
    r = replay(path, dtype, device, 192)
    diff = []
    for t in (a, b):
        got = [r.step([{"id": "q", "tokens": t[:100], "want": [99]}])]
        got += [r.step([{"id": "q", "tokens": [x], "want": [0]}]) for x in t[100:]]
        r.step([], ["q"])
        diff.append(torch.cat(got))
    want = oracle.forward(b, w, cfg)[0][99:] - oracle.forward(a, w, cfg)[0][99:]
    assert want.abs().max() > 1e-3
    if dtype == "float32":
        close_rows(diff[1] - diff[0], want, dtype)


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation(checkpoints, device):
    """``LLM.generate`` through the scheduler: chunked prompts, a batch of unequal requests, more requests than slots."""
    path, cfg, w = checkpoints["small"]
    prompts = [tokens(n, cfg["vocab"], 60 + n) for n in (50, 1, 9, 33, 2)]
    llm = LLM(path, device=device, dtype="float32", block_size=16, max_model_len=96, max_num_seqs=3, num_gpu_blocks=14,
              max_num_batched_tokens=24)
    outs = llm.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for t in o.token_ids:
            logits = oracle.forward(seq, w, cfg)[0][-1]
            assert logits[t] > logits.max() - 1e-3          # the largest, up to rounding
            seq.append(t)
    assert len(llm.engine.scheduler.free_state_slots) == 3


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_decoding_equals_eager(checkpoints, dtype):
    """Capturing a decode step must not advance the recurrent state; padded batch sizes must not touch other slots."""
    path, cfg, w = checkpoints["wide"]
    prompts = [tokens(n, cfg["vocab"], 80 + n) for n in (40, 3, 17)]
    sp = SamplingParams(max_tokens=24, ignore_eos=True)
    kw = dict(device="cuda", dtype=dtype, block_size=64, max_model_len=128, max_num_seqs=4, num_gpu_blocks=16)
    a = [o.token_ids for o in LLM(path, enforce_eager=True, **kw).generate(prompts, sp)]
    llm = LLM(path, **kw)
    b = [o.token_ids for o in llm.generate(prompts, sp)]
    assert a == b and llm.engine.runner.graphs.hits > 0


def test_random_initialisation_serves(checkpoints):
    """A ModelConfig without a checkpoint: seeded weights through the same loading path."""
    cfg = ModelConfig.from_hf_config(copy.deepcopy(SMALL))
    kw = dict(device="cpu", dtype="float32", block_size=16, max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    a, b = (LLM(copy.deepcopy(cfg), **kw).generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].token_ids
            for _ in range(2))
    assert a == b and len(a) == 4


# ------------------------------------------------------------------------------------------------ configuration, loading

def test_configuration_is_read(checkpoints):
    path, cfg, _ = checkpoints["small"]
    m = ModelConfig.from_pretrained(path)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_layers, m.rms_norm_eps) == ("Bolopel", 36, 97, 4, 1e-5)
    assert m.has_recurrent_state and [s.type for s in m.layer_specs] == [x["type"] for x in cfg["layers"]]
    assert m.layer_specs[1].mixer["decay_rank"] == 5 and m.layer_specs[1].mixer["gate_rank"] == 3
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_config(bad)
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["kind"] = "routed"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        ModelConfig.from_hf_config(bad)


def test_incomplete_or_foreign_checkpoints_are_refused(checkpoints, tmp_path):
    path, cfg, w = checkpoints["small"]
    kw = dict(device="cpu", dtype="float32", block_size=16, max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    state = {k: v.to(torch.bfloat16) for k, v in w.items()}
    for change, match in ((lambda s: s.pop("l1.mix.a2"), "lacks"), (lambda s: s.update(extra=torch.zeros(2)), "unexpected"),
                          (lambda s: s.update(head=torch.zeros(3, 36)), "shape")):
        s = dict(state)
        change(s)
        d = str(tmp_path / match)
        save_safetensors(s, d, cfg)
        with pytest.raises(ValueError, match=match):
            LLM(d, **kw)


def test_replay_refuses_what_does_not_fit(checkpoints):
    path, cfg, _ = checkpoints["small"]
    r = replay(path, "float32", "cpu", 64)
    r.step([{"id": "a", "tokens": [1, 2], "want": [1]}])
    with pytest.raises(RuntimeError, match="blocks"):
        r.step([{"id": "b", "tokens": [1], "want": [0]}])
    with pytest.raises(ValueError, match="vocabulary"):
        r.step([{"id": "a", "tokens": [97], "want": [0]}])


@pytest.mark.parametrize("device,dtype", RUNS)
def test_replay_program(checkpoints, device, dtype, tmp_path):
    path, cfg, w = checkpoints["small"]
    t = tokens(30, cfg["vocab"], 7)
    want, _ = oracle.forward(t, w, cfg)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:20], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": t[:3], "want": [2]}, {"id": "a", "tokens": t[20:21], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": t[21:], "want": [8, 0]}], "end": ["a"]}]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "128", "--device", device], text=True, capture_output=True,
                       input="".join(json.dumps(s) + "\n" for s in steps), timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "0.f32").exists()
    V = cfg["vocab"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, V)  # noqa: E731
    close_rows(read(1), torch.stack([want[2], want[20]]), dtype)
    close_rows(read(2), torch.stack([want[29], want[21]]), dtype)


def test_command_line_knows_replay(capsys):
    from vllm_kunlun_b200.entrypoints.cli import main
    assert main(["--help"]) == 0 and "replay" in capsys.readouterr().out

