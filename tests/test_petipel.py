"""Petipel against the plain implementation in ``oracle_petipel``: every mechanism alone, whole models through the engine
(whole prompts, portions, mixed batches, decoding, reused pages and slots), configuration and weight loading, the replay
program.  Each test runs on the CPU path and, on a GPU box, on the kernels (fp32 and bf16)."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_petipel as oracle
from vllm_kunlun_b200 import LLM, SamplingParams, ops
from vllm_kunlun_b200.config import ModelConfig
from vllm_kunlun_b200.engine.replay import ScheduleReplay
from vllm_kunlun_b200.models.loader import save_safetensors
from vllm_kunlun_b200.models.mixers import cache_head_dim, distance_buckets

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
# kernels under test: fp32 on both devices, bf16 on the GPU
RUNS = [("cpu", "float32"), pytest.param("cuda", "float32", marks=pytest.mark.gpu),
        pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attn(mlp, heads=4, kv_heads=2, dim=10, vdim=6, scale=0.3, rows=6, far=20, v_mix=True, temp=(0.4, 8)):
    """``bias_rows`` is read from the checkpoint's table; it stands here for the oracle and for random weights."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_rows": rows, "bias_max": far,
         "v_mix": v_mix}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def hgrn(mlp, heads=3, dim=12, vdim=10):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def config(layers, width=36, vocab=97, eps=1e-5, mult=0.7):
    return {"architecture": "Petipel", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab,
            "width": width}


# every branch, unequal sizes everywhere, widths that need padding, layers that share values beside one that does not
SMALL = config([hgrn(dense(30)), attn(moe(5, 2, 20, 0.8)), attn(None, heads=3, kv_heads=3, dim=5, vdim=7, v_mix=False, temp=None),
                hgrn(moe(3, 3, 12, 5.0), heads=1, dim=20, vdim=3), hgrn(None, heads=2, dim=4, vdim=8),
                attn(dense(44), heads=6, kv_heads=2, dim=9, rows=10, far=70, temp=(1.1, 3))])
# head sizes of the tensor-core kernels, a bias beyond a key tile, many experts
WIDE = config([attn(dense(136), heads=6, kv_heads=3, dim=128, vdim=96, scale=0.09, rows=16, far=160, temp=(0.2, 64)),
               hgrn(moe(12, 4, 40, 1.5), heads=2, dim=128, vdim=72), hgrn(dense(64), heads=3, dim=64, vdim=64),
               attn(moe(4, 1, 128, 3.0), heads=54, kv_heads=3, dim=16, vdim=96, scale=0.2, rows=4, far=9)],
              width=104, vocab=300, eps=1e-3, mult=1.0)
# beyond the tensor-core kernels' sizes
LARGE = config([attn(dense(30), heads=3, kv_heads=1, dim=140, vdim=30, scale=0.08, rows=32, far=100),
                hgrn(moe(2, 1, 70, 2.0), heads=2, dim=136, vdim=140)], width=44, mult=0.25)
CONFIGS = {"small": SMALL, "wide": WIDE, "large": LARGE}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Many tiny operations: one thread is several times faster than all of them."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def plain_config(cfg):
    """What a checkpoint carries: the number of bias rows is in the table's shape only."""
    cfg = copy.deepcopy(cfg)
    for entry in cfg["layers"]:
        entry["mixer"].pop("bias_rows", None)
    return cfg


def checkpoint(path, cfg, seed, change=None):
    w = oracle.random_weights(cfg, seed=seed)
    if change is not None:
        change(w)
        w = {k: v.to(torch.bfloat16).double() for k, v in w.items()}
    save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, path, plain_config(cfg))
    return path, cfg, w


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    """name -> (directory, configuration, float64 weights)."""
    return {name: checkpoint(str(tmp_path_factory.mktemp(name)), cfg, 3 + i)
            for i, (name, cfg) in enumerate(CONFIGS.items())}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, what="", bf16=0.06):
    """fp32: rounding of 32-bit sums; bf16: a small fraction of the values' root mean square."""
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    scale = want.pow(2).mean().sqrt().clamp(min=1e-3)
    err = ((got - want).abs().max() / scale).item()
    limit = 1e-4 if dtype == "float32" else bf16
    assert err < limit, f"{what}: error {err:.2e} of the root mean square (limit {limit})"


def close_rows(got, want, dtype, what=""):
    """Logits (or stream rows) of a whole model: in bf16 rows are judged one by one (a router's close call moves a row)."""
    if dtype == "float32":
        return close(got, want, dtype, what)
    d, want = got.double().cpu() - want.double(), want.double()
    rows = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    stats = (rows.median().item(), int((rows > 0.15).sum()))
    assert stats[0] < 0.06 and stats[1] <= max(2, 0.15 * len(rows)), f"{what}: {stats} of {len(rows)}"


def replay(path, dtype, device, max_tokens, **kw):
    return ScheduleReplay(path, dtype, max_tokens, device=device, **kw)


def rounded(dtype, *xs):
    return [x.to(DT[dtype]).double() for x in xs]


# ------------------------------------------------------------------------------------------------ mechanisms

@pytest.mark.parametrize("rows,far", [(2, 5), (3, 9), (4, 6), (5, 40), (16, 128), (18, 90), (20, 320), (32, 128), (32, 33),
                                      (64, 8192), (9, 5)])
def test_distance_buckets(rows, far):
    """Boundaries that are powers of the step, as in (20, 320): 20, 40, 80, ... begin a row, whatever a logarithm says."""
    b = distance_buckets(rows, far)
    assert [b[min(n, len(b) - 1)] for n in range(far + 40)] == [oracle.distance_bucket(n, rows, far) for n in range(far + 40)]
    assert b[-1] == rows - 1 and len(b) <= far + 1 and (len(b) == 1 or b[-2] < rows - 1)
    if (rows, far) == (20, 320):
        assert [b.index(10 + 2 * k) for k in range(5)] == [10, 20, 40, 80, 160]


def test_distance_table_that_ends_too_early():
    with pytest.raises(ValueError, match="distance table"):
        distance_buckets(16, 8)


def attend(device, dtype, q, k, v, lens, scale, bias, gate=None, bs=64):
    """``lens``: (cached, new) tokens per request; q, k, v hold whole sequences.  Output rows of the new tokens."""
    dt, (H, D), (G, V) = DT[dtype], q.shape[1:], v.shape[1:]
    Dc = cache_head_dim(D, V, dt, (128,))
    nblk = [-(-(a + b) // bs) for a, b in lens]
    perm = torch.randperm(sum(nblk) + 3, generator=torch.Generator().manual_seed(1)).tolist()
    cache = torch.full((len(perm), 2, G, bs, Dc), 3.0)
    bt = torch.zeros(len(lens), max(nblk) + 1, dtype=torch.int32)
    off, new = 0, []
    for r, (a, b) in enumerate(lens):
        blocks = torch.tensor([perm.pop() for _ in range(nblk[r])])
        bt[r, :len(blocks)] = blocks
        p = torch.arange(a + b)
        for part, x in enumerate((k, v)):
            cells = torch.zeros(a + b, G, Dc)
            cells[..., :x.shape[-1]] = x[off:off + a + b]
            cache[blocks[p // bs], part, :, p % bs] = cells
        new += list(range(off + a, off + a + b))
        off += a + b
    qp = torch.zeros(len(new), H, Dc)
    qp[..., :D] = q[new]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32).to(device)  # noqa: E731
    nd = 0
    while nd < len(lens) and lens[nd][1] == 1:
        nd += 1
    wide = torch.zeros(len(new), H + 3, dtype=dt, device=device)      # gates are a column slice of a wider projection
    if gate is not None:
        wide[:, 2:2 + H] = gate.to(dt).to(device)
    sl, qsl = i32([a + b for a, b in lens]), i32([sum(b for _, b in lens[:i]) for i in range(len(lens) + 1)])
    o = ops.paged_attention(qp.to(dt).to(device), cache.to(dt).to(device), bt.to(device), sl, qsl, scale,
                            max(b for _, b in lens), max(a + b for a, b in lens), num_decodes=nd, num_decode_tokens=nd,
                            bias=bias.float().to(device), gate=None if gate is None else wide[:, 2:2 + H])
    return o[..., :V]


def plain_attention(q, k, v, lens, scale, table, far, gate=None):
    H, G = q.shape[1], k.shape[1]
    of = [i // (H // G) for i in range(H)]
    out, off = [], 0
    for a, b in lens:
        s = slice(off, off + a + b)
        out.append(oracle.attention(q[s].double(), k[s][:, of].double(), v[s][:, of].double(), scale,
                                    oracle.distance_bias(a + b, table.double(), far))[a:])
        off += a + b
    out = torch.cat(out)
    return out if gate is None else out * oracle.sigmoid(gate.double())[..., None]


def spread(table, far):
    """The table as the kernels read it: one column per distance."""
    return table[torch.tensor(distance_buckets(table.shape[0], far))].T.contiguous()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,V", [(6, 2, 64, 40), (3, 3, 10, 14), (8, 2, 128, 128), (20, 1, 24, 72), (2, 1, 140, 30)])
def test_attention_with_a_distance_bias(device, dtype, H, G, D, V):
    """Unequal requests, single tokens beside portions; tables that end inside a page, inside a tile and behind everything."""
    g = torch.Generator().manual_seed(D)
    for lens in ([(37, 1), (64, 1), (0, 1), (190, 1), (400, 1)], [(37, 1), (0, 130), (30, 41), (63, 2), (200, 3), (0, 1)]):
        T, n = sum(a + b for a, b in lens), sum(b for _, b in lens)
        q, k = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g)
        q, k, v, gate = rounded(dtype, q * 1.5, k, torch.randn(T, G, V, generator=g), torch.randn(n, H, generator=g) * 2)
        for rows, far in ((4, 6), (10, 70), (16, 150), (32, 2000)):
            table = torch.randn(rows, H, generator=g) * 2
            got = attend(device, dtype, q, k, v, lens, D ** -0.5, spread(table, far), gate)
            close(got, plain_attention(q, k, v, lens, D ** -0.5, table, far, gate), dtype, f"table {rows} {far}", 0.15)
        got = attend(device, dtype, q, k, v, lens, 0.02, spread(table, far))
        close(got, plain_attention(q, k, v, lens, 0.02, table, far), dtype, "no gate")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("far", [20, 64, 200])
def test_bias_at_its_borders(device, dtype, far):
    """Equal scores everywhere except one row of the table: exactly the keys whose distance falls into that row are attended,
    for single tokens and in portions, on both sides of page and tile borders and far behind the table's end."""
    H, D, V, L = 2, 8, 8, 330
    rows = 8
    row_of = [oracle.distance_bucket(n, rows, far) for n in range(L)]
    q, k = torch.zeros(L, H, D), torch.zeros(L, 1, D)
    pos = torch.arange(L, dtype=torch.float32)
    v = torch.zeros(L, 1, V)
    v[:, 0, 0], v[:, 0, 1] = pos // 64, pos % 64           # a key's position in numbers that bf16 holds
    for row in range(rows):
        table = torch.zeros(rows, H)
        table[row, 1] = 60.0
        for lens in ([(L - 1, 1)], [(0, L)], [(L - 70, 70)], [(L - 2, 2)]):
            o = attend(device, dtype, q, k, v, lens, 1.0, spread(table, far)).double().cpu()
            a, b = lens[0]
            for j in sorted({0, b // 2, b - 1}):
                i = a + j
                seen = [x for x in range(i + 1) if row_of[i - x] == row] or list(range(i + 1))
                for h, keys in ((0, list(range(i + 1))), (1, seen)):
                    want = torch.stack([v[keys, 0, c].double().mean() for c in (0, 1)])
                    assert (o[j, h, :2] - want).abs().max() < (2e-4 if dtype == "float32" else 0.3), (row, lens, i, h)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 8, 12), (3, 1, 10, 7), (2, 2, 128, 128)])
def test_split_norms_values_and_mixes_them(device, dtype, H, G, D, V):
    """Query temperature at and around its steps (far positions too), value norm, shared values, keys as they are, padding."""
    dt, T, bs = DT[dtype], 9, 64
    g = torch.Generator().manual_seed(V)
    off = [0, -(-H * D // 8) * 8, -(-H * D // 8) * 8 + -(-G * D // 8) * 8]
    y = torch.randn(T, off[2] + -(-G * V // 8) * 8, generator=g).to(dt)
    pos = torch.tensor([0, 1, 2, 3, 4, 5, 6, 2 ** 20 + 1, 10])
    slots = torch.tensor([5, 70, 200, -1, 33, 0, 1, 2, 3])
    first = torch.randn(T, G * V, generator=g).to(dt)
    Dc = cache_head_dim(D, V, dt, (128,))
    cache = torch.full((4, 2, G, bs, Dc), 7.0, dtype=dt).to(device)
    part = lambda t, i, n: t[:, off[i]:off[i] + n]  # noqa: E731
    yd = y.to(device)
    keep = torch.empty(T, G * V, dtype=dt, device=device)
    for temp, share in (((0.3, 3), 0.0), (None, 0.4)):
        v_in = first.to(device) if share else None
        q = ops.attn_prep_cache(part(yd, 0, H * D), part(yd, 1, G * D), part(yd, 2, G * V), cache, slots.to(device),
                                pos.to(device), H, G, 1e-2, temp, None if share else keep, v_in, share)
        f = torch.tensor([1.0 if temp is None else oracle.query_temperature(p, *temp) for p in pos.tolist()])
        close(q[..., :D], part(y, 0, H * D).double().reshape(T, H, D) * f.double()[:, None, None], dtype, "queries")
        assert not q[..., D:].any()
        k = part(y, 1, G * D).reshape(T, G, D)
        v = oracle.unit_rms(part(y, 2, G * V).double().reshape(T, G, V), 1e-2)
        close(keep.reshape(T, G, V), v, dtype, "values for later layers")
        if share:
            v = oracle.mix_values(v, first.double().reshape(T, G, V), share)
        for t, s in enumerate(slots.tolist()):
            if s >= 0:
                cell = cache[s // bs, :, :, s % bs].cpu()
                assert torch.equal(cell[0, :, :D], k[t]) and not cell[0, :, D:].any() and not cell[1, :, V:].any()
                close(cell[1, :, :V], v[t], dtype, "cached values")
        assert (cache[3, :, :, 9:].float() == 7.0).all()


def recur(device, dtype, q, v, f, bias, lower, states, lens, slots, init):
    i32 = lambda x: torch.tensor(x, dtype=torch.int32).to(device)  # noqa: E731
    nd = 0
    while nd < len(lens) and lens[nd] == 1:
        nd += 1
    n, H, D = q.shape
    V, ha, hv = v.shape[2], -(-H * D // 8) * 8, -(-H * v.shape[2] // 8) * 8
    y = torch.zeros(n, 2 * ha + hv, dtype=DT[dtype])
    y[:, :H * D], y[:, ha:ha + H * D], y[:, 2 * ha:2 * ha + H * V] = q.reshape(n, -1), f, v.reshape(n, -1)
    y = y.to(device)
    view = lambda o, d: y[:, o:o + H * d].as_strided((n, H, d), (y.stride(0), d, 1), y.storage_offset() + o)  # noqa: E731
    return ops.gated_write_attention(view(0, D), view(2 * ha, V), y[:, ha:ha + H * D], bias.float().to(device),
                                     lower.float().to(device), states, i32([sum(lens[:i]) for i in range(len(lens) + 1)]),
                                     i32(slots), i32(init), max(lens), nd)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,D,V", [(3, 16, 24), (2, 128, 128), (1, 12, 10), (2, 64, 136), (40, 128, 72), (1, 200, 33)])
def test_gated_write_recurrence(device, dtype, H, D, V):
    """Portions of every remainder modulo the chunk, single tokens, states that go on and slots that are used again; gates
    from almost closed to almost one, with and without a lower bound."""
    g = torch.Generator().manual_seed(D + V)
    lens = [1, 1, 16, 33, 2, 70, 15] if device == "cuda" and H < 40 else [1, 1, 17, 31]
    n = sum(lens)
    bias = torch.randn(H * D, generator=g) * 3
    bias[:D // 2] += 9.0
    lower = torch.rand(H * D, generator=g)
    lower[::3] = 0.0
    states = torch.full((len(lens) + 2, H, V, -(-D // 4) * 4), 9.0, device=device)     # what other requests left behind
    slots = torch.randperm(len(lens) + 2, generator=g).tolist()[:len(lens)]
    seqs = [[] for _ in lens]
    for step in range(3):
        q, v = torch.randn(n, H, D, generator=g), torch.randn(n, H, V, generator=g)
        q, v, f = rounded(dtype, q, v, torch.randn(n, H * D, generator=g) * 2)
        out = recur(device, dtype, q, v, f, bias, lower, states, lens, slots, [int(step > 0)] * len(lens))
        at = 0
        for r, L in enumerate(lens):
            seqs[r].append((q[at:at + L], f[at:at + L], v[at:at + L]))
            qs, fs, vs = (torch.cat(x) for x in zip(*seqs[r]))
            low = lower.double()
            gate = (low + (1 - low) * oracle.sigmoid(fs + bias.double())).reshape(-1, H, D)
            want = oracle.hgrn2_recurrence(oracle.silu(qs), gate, vs)[-L:]
            close(out[at:at + L], want, dtype, f"step {step} request {r}", 0.03)
            at += L
    assert (states[[s for s in range(len(lens) + 2) if s not in slots]] == 9.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_first_token_in_the_state(device, dtype):
    """Gates that never forget after the first token: what it wrote is there, unchanged, hundreds of tokens later."""
    H, D, V, L = 1, 16, 16, 300
    q, v, f = torch.zeros(L, H, D), torch.zeros(L, H, V), torch.full((L, H * D), 100.0)
    q[:, 0, 3] = 6.0
    v[0, 0, 5], v[1:, 0, 5] = 2.0, -50.0
    f[0] = -100.0                                      # writes everything once
    for lens in ([L], [100, 1, 199], [1] * 20 + [L - 20]):
        states = torch.full((1, H, V, D), 4.0, device=device)
        at, got = 0, []
        for i, n in enumerate(lens):
            s = slice(at, at + n)
            got.append(recur(device, dtype, q[s], v[s], f[s], torch.zeros(D), torch.zeros(D), states, [n], [0], [int(i > 0)]))
            at += n
        got = torch.cat(got).double().cpu()
        want = 2.0 * float(oracle.silu(torch.tensor(6.0).double()))
        assert (got[:, 0, 5] - want).abs().max() < (1e-4 if dtype == "float32" else 0.06)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,width,ld", [(3, 30, 32), (7, 64, 64), (2, 5000, 5000), (2, 17001, 17008)])
def test_poly_norm(device, dtype, T, width, ld):
    """Each power by itself, the constant, the epsilon of a row of almost nothing, values whose cubes are large."""
    g = torch.Generator().manual_seed(width)
    z = torch.randn(T, ld, generator=g)
    z[0] *= 1e-3
    z[1] *= 40.0
    z = z.to(DT[dtype])
    for coeff in ([1, 0, 0, 0], [0, 1, 0, 0], [0, 0, 1, 0], [0, 0, 0, 0.5], [0.6, -0.3, 0.8, -0.1]):
        c = torch.tensor(coeff, dtype=torch.float32)
        got = ops.poly_norm(z.to(device), c.to(device), width, 1e-5)
        want = oracle.poly_norm(z[:, :width].double(), c.double(), 1e-5)
        for t in range(T):
            close(got[t, :width], want[t], dtype, f"{coeff} row {t}")
        assert not got[:, width:].any()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,E,k,ff,width", [(5, 8, 1, 64, 40), (130, 5, 3, 64, 72), (700, 4, 2, 128, 64), (1, 3, 3, 64, 16)])
def test_experts_on_weighted_inputs(device, dtype, T, E, k, ff, width):
    """Scores as weights without renormalisation, on the experts' inputs; limits that cut both sides; uneven experts."""
    dt, limit = DT[dtype], 1.3
    g = torch.Generator().manual_seed(T)
    x = (torch.randn(T, width, generator=g) * 2).to(dt)
    r = (torch.randn(E, width, generator=g) / width ** 0.5).to(dt)          # scores well inside (0, 1): no ties
    w13 = (torch.randn(E, 2 * ff, width, generator=g) / width ** 0.5).to(dt)
    w2 = (torch.randn(E, width, ff, generator=g) / ff ** 0.5).to(dt)
    w, ids = ops.router_and_route(x.to(device), r.to(device), None, k, "sigmoid", False, fp32=True)
    order, scores = oracle.route(x.double(), r.double(), k)
    order_sorted = order.sort(-1)
    ids_sorted = ids.cpu().long().sort(-1)
    same = (order_sorted.values == ids_sorted.values).all(-1)
    assert same.float().mean() > 0.98
    got_w = w.double().cpu().gather(1, ids_sorted.indices)[same]
    assert (got_w - scores.gather(1, order_sorted.indices)[same]).abs().max() < 1e-5      # the logits are 32-bit sums
    rows, pos = ops.experts_on_weighted_input(x.to(device), w13.to(device), w2.to(device), w, ids, "swiglu_limit", limit)
    got = rows.double().cpu()[pos.cpu().long()].reshape(T, k, width).sum(1)
    want = torch.zeros(T, width, dtype=torch.float64)
    for t in range(T):
        for e, s in zip(order[t].tolist(), scores[t]):
            u = w13[e].double()
            want[t] += oracle.expert(s * x[t].double(), u[:ff], u[ff:], w2[e].double(), limit)
    close(got[same], want[same], dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width,ld", [(36, 40), (64, 64), (4100, 4104)])
def test_sandwich_norm(device, dtype, width, ld):
    """The sublayer's result is normed before it is added, the sum after it; rows of experts are summed; padding stays zero."""
    g = torch.Generator().manual_seed(width)
    T, k = 5, 3
    pad = lambda z: torch.nn.functional.pad(z, (0, ld - width))  # noqa: E731
    table = pad(torch.randn(9, width, generator=g)).to(DT[dtype])
    w_post, w_pre = torch.randn(width, generator=g), torch.randn(width, generator=g)
    ids = torch.tensor([3, 0, 8, 3, 1])
    x, h = ops.embed_rmsnorm(ids.to(device), table.to(device), w_pre.to(device), 1e-3)
    want_x = table[ids][:, :width].double()
    assert torch.equal(x[:, :width].double().cpu(), want_x)
    close(h[:, :width], oracle.unit_rms(want_x, 1e-3) * w_pre.double(), dtype)
    rows = pad(torch.randn(T * k + 2, width, generator=g)).to(DT[dtype])
    pos = torch.randperm(T * k + 2, generator=g)[:T * k].int()
    for y, plain in ((rows[:T], rows[:T].double()), ((rows, pos), rows.double()[pos.long()].reshape(T, k, ld).sum(1))):
        y = tuple(z.to(device) for z in y) if isinstance(y, tuple) else y.to(device)
        h = ops.sandwich_rmsnorm(x, y, w_post.to(device), w_pre.to(device), 1e-3)
        want_x = want_x + oracle.unit_rms(plain[:, :width], 1e-3) * w_post.double()
        close(x[:, :width], want_x, "float32", "stream")            # 32-bit also in 16-bit models
        close(h[:, :width], oracle.unit_rms(want_x, 1e-3) * w_pre.double(), dtype, "norm")
        assert not x[:, width:].any() and not h[:, width:].any() and h.dtype == DT[dtype]


# ------------------------------------------------------------------------------------------------ whole models

@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_stream(checkpoints, device, dtype, name):
    path, cfg, w = checkpoints[name]
    toks, stream = tokens(150, cfg["vocab"]), []
    want = oracle.forward(toks, w, cfg, stream)
    r = replay(path, dtype, device, 192)
    layers = []
    r.engine.runner.model.post_layer_hook = lambda i, h, x: layers.append(x.float().cpu().clone())
    got = r.step([{"id": "a", "tokens": toks, "want": list(range(len(toks)))}], ["a"])
    assert got.dtype == torch.float32 and len(layers) == len(stream)
    close_rows(got, want, dtype, "logits")
    for i, (x, s) in enumerate(zip(layers, stream)):
        close_rows(x, s, dtype, f"stream after layer {i}")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_decoding(checkpoints, device, dtype, name):
    """Token by token from the start, portions of changing size down to two tokens, long decoding after a prompt: all
    give the logits of the whole prompt.  Every request runs in the pages and slots of the one before."""
    path, cfg, w = checkpoints[name]
    L = 200
    toks = tokens(L, cfg["vocab"], 1)
    want = oracle.forward(toks, w, cfg)
    r = replay(path, dtype, device, 256)
    for cuts in ([1] * L, [64, 2, 1, 30, 3, 2, 98], [2] * 40 + [120], [33] + [1] * (L - 33)):
        if device == "cpu" and name != "small" and cuts[0] == 1:
            continue
        at, got = 0, []
        for n in cuts:
            got.append(r.step([{"id": "a", "tokens": toks[at:at + n], "want": list(range(n))}]))
            at += n
        r.step([], ["a"])
        close_rows(torch.cat(got), want, dtype, f"portions {cuts[:4]}")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", ["small", "wide"])
def test_mixed_batches_and_reuse(checkpoints, device, dtype, name):
    """Up to four live requests, portions beside single tokens, requests that pause, pages and slots that go round: each
    request's logits are those it has alone."""
    path, cfg, w = checkpoints[name]
    lens = {"a": 90, "b": 41, "c": 7, "d": 1, "e": 66, "f": 2, "g": 64}
    toks = {k: tokens(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: oracle.forward(t, w, cfg) for k, t in toks.items()}
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
def test_one_token_prompt_in_a_used_slot(checkpoints, device, dtype):
    """A first portion of one token starts from an empty state even when its slot still holds another request's."""
    path, cfg, w = checkpoints["small"]
    r = replay(path, dtype, device, 128)
    for i in range(3):
        t = tokens(20, cfg["vocab"], 40 + i)
        r.step([{"id": "x", "tokens": t, "want": []}], ["x"])
        want = oracle.forward(t[:3], w, cfg)
        got = [r.step([{"id": "y", "tokens": [t[j]], "want": [0]}]) for j in range(3)]
        r.step([], ["y"])
        close_rows(torch.cat(got), want, dtype)


def far_config(kind):
    if kind == "attention":
        return config([attn(None, heads=2, kv_heads=1, dim=16, vdim=16, scale=0.25, rows=8, far=40, v_mix=False, temp=None)],
                      width=48, mult=1.0)
    return config([hgrn(None, heads=1, dim=16, vdim=16)], width=48, mult=1.0)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kind", ["attention", "hgrn2"])
def test_far_token_reaches_every_place(device, dtype, kind, tmp_path):
    """One changed token far back - behind the end of the distance table, several pages away - moves the logits as in the
    plain implementation: in a prompt, across portions and decoded token by token."""
    def change(w):
        if kind == "attention":
            w["l0.mix.rel"].zero_()
            w["l0.mix.rel"][-1] = 6.0              # the last row stands out: the far keys count, the near ones hardly
            w["l0.mix.q"].mul_(0.1)
        else:
            w["l0.mix.f.b"].fill_(12.0)
            w["l0.mix.lower"].zero_()
    path, cfg, w = checkpoint(str(tmp_path), far_config(kind), 31, change)
    L, at = 300, 0 if kind == "hgrn2" else 3
    a = tokens(L, cfg["vocab"], 3)
    b = list(a)
    b[at] = (b[at] + 41) % cfg["vocab"]
    plain = [oracle.forward(t, w, cfg) for t in (a, b)]
    moved, size = plain[1] - plain[0], plain[0].pow(2).mean().sqrt()
    assert moved[-1].abs().max() > 1e-3 * size
    r = replay(path, dtype, device, 320)
    for cuts in ([L], [70, 2, 128, 100], [200] + [1] * 100):
        got = []
        for t in (a, b):
            p, rows = 0, []
            for n in cuts:
                rows.append(r.step([{"id": "q", "tokens": t[p:p + n], "want": list(range(n))}]))
                p += n
            r.step([], ["q"])
            got.append(torch.cat(rows))
        d = (got[1] - got[0]).double()
        if dtype == "float32":
            assert (d - moved).abs().max() < 3e-5 * size, cuts
        else:
            assert not torch.equal(got[0][-1], got[1][-1]), cuts


@pytest.mark.parametrize("device,dtype", RUNS)
def test_shared_values_are_the_same_tokens(device, dtype, tmp_path):
    """The second of two sharing layers attends (nearly) only the first one's values; a layer between them has its own."""
    def change(w):
        w["l2.mix.vmix"] = torch.tensor(0.98)
        w["l0.mix.vmix"] = torch.tensor(0.5)            # has no effect
    layers = [attn(None, rows=4, far=9), attn(None, v_mix=False, heads=2, kv_heads=1), attn(None, heads=2)]
    path, cfg, w = checkpoint(str(tmp_path), config(layers), 5, change)
    toks = tokens(90, cfg["vocab"], 2)
    want = oracle.forward(toks, w, cfg)
    other = dict(w)
    other["l2.mix.vmix"] = torch.tensor(0.0).double()
    assert (oracle.forward(toks, other, cfg) - want).abs().max() > 0.3 * want.pow(2).mean().sqrt()
    other = {**w, "l0.mix.vmix": torch.tensor(0.9).double()}
    assert torch.equal(oracle.forward(toks, other, cfg), want)
    r = replay(path, dtype, device, 128)
    got = [r.step([{"id": "a", "tokens": toks[:70], "want": list(range(70))}])]
    got += [r.step([{"id": "a", "tokens": [t], "want": [0]}]) for t in toks[70:]]
    close_rows(torch.cat(got), want, dtype)


def test_sharing_layers_of_different_widths_are_refused():
    cfg = ModelConfig.from_hf_config(config([attn(None, vdim=6), attn(None, vdim=8)]))
    with pytest.raises(ValueError, match="share values"):
        LLM(cfg, device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation(checkpoints, device):
    """``LLM.generate`` through the scheduler: chunked prompts, a batch of unequal requests, more requests than slots, a
    pool that runs dry (preemption and recomputation)."""
    path, cfg, w = checkpoints["small"]
    prompts = [tokens(n, cfg["vocab"], 60 + n) for n in (124, 126, 1, 9, 2)]
    llm = LLM(path, device=device, dtype="float32", max_model_len=256, max_num_seqs=3, num_gpu_blocks=5,
              max_num_batched_tokens=70)
    assert llm.engine.pool.block_size == 64
    outs = llm.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    assert llm.engine.stats["preemptions"] > 0
    for p, o in zip(prompts, outs):
        seq = list(p) + list(o.token_ids)
        logits = oracle.forward(seq, w, cfg)
        for j, t in enumerate(o.token_ids):
            row = logits[len(p) - 1 + j]
            assert row[t] > row.max() - 1e-3          # the largest, up to rounding
    assert len(llm.engine.scheduler.free_state_slots) == 3


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_decoding_equals_eager(checkpoints, dtype):
    """Capturing a decode step must not advance the per-request state; padded batch sizes must not touch other slots."""
    path, cfg, w = checkpoints["wide"]
    prompts = [tokens(n, cfg["vocab"], 80 + n) for n in (140, 3, 17)]
    sp = SamplingParams(max_tokens=24, ignore_eos=True)
    kw = dict(device="cuda", dtype=dtype, max_model_len=192, max_num_seqs=4, num_gpu_blocks=16)
    a = [o.token_ids for o in LLM(path, enforce_eager=True, **kw).generate(prompts, sp)]
    llm = LLM(path, **kw)
    b = [o.token_ids for o in llm.generate(prompts, sp)]
    assert a == b and llm.engine.runner.graphs.hits > 0


def test_random_initialisation_serves():
    """A ModelConfig without a checkpoint: seeded weights through the same loading path."""
    cfg = ModelConfig.from_hf_config(plain_config(SMALL))
    kw = dict(device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    for entry in cfg.layer_specs:           # no tensor tells the tables' rows: the default must fit
        if "bias_max" in entry.mixer:
            entry.mixer["bias_max"] = 50
    a, b = (LLM(copy.deepcopy(cfg), **kw).generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].token_ids
            for _ in range(2))
    assert a == b and len(a) == 4


# ------------------------------------------------------------------------------------------------ configuration, loading

def test_configuration_is_read(checkpoints):
    path, cfg, _ = checkpoints["small"]
    m = ModelConfig.from_pretrained(path)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_layers, m.rms_norm_eps) == ("Petipel", 36, 97, 6, 1e-5)
    assert (m.residual_multiplier, m.hidden_act, m.intermediate_size) == (0.7, "poly_norm", 44)
    assert m.has_recurrent_state and m.cache_block == 64
    assert [m.layer_specs[i].mixer["bias_rows"] for i in (1, 2, 5)] == [6, 6, 10]
    for change, match in ((lambda c: c["layers"][0].update(type="unknown"), "unknown mixer"),
                          (lambda c: c["layers"][0]["mlp"].update(kind="unknown"), "unknown feed-forward")):
        bad = copy.deepcopy(cfg)
        change(bad)
        with pytest.raises(ValueError, match=match):
            ModelConfig.from_hf_config(bad)
    only_attention = ModelConfig.from_hf_config(config([attn(dense(8))]))
    assert not only_attention.has_recurrent_state


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kind", ["attention", "hgrn2"])
def test_one_kind_of_layer(device, dtype, kind, tmp_path):
    """Models without any recurrent state, and models without any paged cache."""
    layers = [attn(dense(24), rows=5, far=33)] * 2 if kind == "attention" else [hgrn(moe(3, 1, 10, 1.0))] * 2
    path, cfg, w = checkpoint(str(tmp_path), config(layers, width=40, vocab=50), 8)
    toks = tokens(80, 50, 4)
    want = oracle.forward(toks, w, cfg)
    r = replay(path, dtype, device, 128)
    got = [r.step([{"id": "a", "tokens": toks[:67], "want": list(range(67))}])]
    got += [r.step([{"id": "a", "tokens": [t], "want": [0]}]) for t in toks[67:]]
    close_rows(torch.cat(got), want, dtype)


def test_incomplete_or_foreign_checkpoints_are_refused(checkpoints, tmp_path):
    path, cfg, w = checkpoints["small"]
    kw = dict(device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    state = {k: v.to(torch.bfloat16) for k, v in w.items()}
    for change, match in ((lambda s: s.pop("l1.mlp.e3.up"), "lacks"), (lambda s: s.update(extra=torch.zeros(2)), "unexpected"),
                          (lambda s: s.update({"l0.mix.lower": torch.zeros(35)}), "shape")):
        s = dict(state)
        change(s)
        d = str(tmp_path / match)
        save_safetensors(s, d, plain_config(cfg))
        with pytest.raises(ValueError, match=match):
            LLM(d, **kw)
    # tensors without effect: a share where no values are shared, norms of a feed-forward that is not there
    s = {**state, "l2.mix.vmix": torch.tensor(0.5), "l2.norm2": torch.ones(36), "l4.norm2b": torch.ones(36)}
    save_safetensors({k: v.to(torch.bfloat16) for k, v in s.items()}, str(tmp_path / "more"), plain_config(cfg))
    LLM(str(tmp_path / "more"), **kw)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_replay_program(checkpoints, device, dtype, tmp_path):
    path, cfg, w = checkpoints["small"]
    t = tokens(30, cfg["vocab"], 7)
    want = oracle.forward(t, w, cfg)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:20], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": t[:3], "want": [2]}, {"id": "a", "tokens": t[20:21], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": t[21:], "want": [8, 0]}], "end": ["a"]}]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "128", "--device", device], text=True, capture_output=True,
                       input="".join(json.dumps(s) + "\n" for s in steps), timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    V = cfg["vocab"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, V)  # noqa: E731
    close_rows(read(1), torch.stack([want[2], want[20]]), dtype)
    close_rows(read(2), torch.stack([want[29], want[21]]), dtype)
