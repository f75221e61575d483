"""Seturax against the plain implementation in ``oracle_seturax``: every mechanism alone, whole models through the engine
(whole prompts, portions, mixed batches, decoding, reused pages and slots), configuration and weight loading, the replay
program.  Each test runs on the CPU path and, on a GPU box, on the kernels (fp32 and bf16)."""
import copy
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import pytest
import torch

import oracle_seturax as oracle
from vllm_kunlun_b200 import LLM, SamplingParams, ops
from vllm_kunlun_b200.config import ModelConfig
from vllm_kunlun_b200.engine.replay import ScheduleReplay
from vllm_kunlun_b200.models.loader import save_safetensors
from vllm_kunlun_b200.models.mixers import LatentAttention

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
# kernels under test: fp32 on both devices, bf16 on the GPU
RUNS = [("cpu", "float32"), pytest.param("cuda", "float32", marks=pytest.mark.gpu),
        pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def latent(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=20, q_rank=12, size=7, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5}


def layer(mixer, ff=24):
    return {"type": "latent_attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=40, vocab=97, eps=1e-5, scale=3.0, buckets=53, mul_prev=7, mul_cur=3, logit_scale=0.4):
    return {"architecture": "Seturax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "logit_scale": logit_scale}


# every branch, unequal sizes everywhere, sizes and widths that need padding, a window of one token, no feed-forward
SMALL = config([layer(latent()), layer(latent(heads=4, dim=16, rot_dim=8, vdim=8, kv_rank=24, q_rank=40, size=1, base=77.0)),
                layer(latent(heads=1, dim=5, rot_dim=2, vdim=9, kv_rank=11, q_rank=9, size=40, scale=0.6), ff=None),
                layer(latent(heads=2, dim=12, rot_dim=12, vdim=12, kv_rank=12, q_rank=12, size=64, base=500.0), ff=50)],
               width=36, logit_scale=1.7)
# the kernels' own sizes and sizes in between, windows across pages, several groups of heads
WIDE = config([layer(latent(heads=6, dim=48, rot_dim=32, vdim=40, kv_rank=96, q_rank=72, size=70), ff=72),
               layer(latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96, size=129, base=1e6), ff=136),
               layer(latent(heads=36, dim=8, rot_dim=4, vdim=6, kv_rank=32, q_rank=32, size=33), ff=64)],
              width=104, vocab=300, eps=1e-3, scale=1.0, buckets=1, logit_scale=0.05)
# beyond the tensor-core kernels' sizes
LARGE = config([layer(latent(heads=3, dim=136, rot_dim=10, vdim=30, kv_rank=50, q_rank=20, size=66), ff=30),
                layer(latent(heads=2, dim=20, rot_dim=72, vdim=140, kv_rank=520, q_rank=44, size=20), ff=40)],
               width=44, buckets=1000, mul_prev=100003, mul_cur=99991)
CONFIGS = {"small": SMALL, "wide": WIDE, "large": LARGE}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Many tiny operations: one thread is several times faster than all of them."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def checkpoint(path, cfg, seed):
    w = oracle.random_weights(cfg, seed=seed)
    save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, path, cfg)
    return path, cfg, w


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    """name -> (directory, configuration, float64 weights)."""
    return {name: checkpoint(str(tmp_path_factory.mktemp(name)), cfg, 3 + i)
            for i, (name, cfg) in enumerate(CONFIGS.items())}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, what="", bf16=0.12):
    """fp32: rounding of 32-bit sums; bf16: a small fraction of the values' root mean square."""
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    scale = want.pow(2).mean().sqrt().clamp(min=1e-3)
    err = ((got - want).abs().max() / scale).item()
    limit = 2e-4 if dtype == "float32" else bf16
    assert err < limit, f"{what}: error {err:.2e} of the root mean square (limit {limit})"


def close_rows(got, want, dtype, what=""):
    """Logits (or stream rows) of a whole model: in bf16 rows are judged one by one."""
    if dtype == "float32":
        return close(got, want, dtype, what)
    d, want = got.double().cpu() - want.double(), want.double()
    rows = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    stats = (rows.median().item(), rows.max().item(), int((rows > 0.1).sum()))
    assert stats[0] < 0.05 and stats[1] < 0.4 and stats[2] <= max(2, 0.06 * len(rows)), f"{what}: {stats} of {len(rows)}"


def replay(path, dtype, device, max_tokens, **kw):
    return ScheduleReplay(path, dtype, max_tokens, device=device, **kw)


# ------------------------------------------------------------------------------------------------ mechanisms

def batch(device, lens, slots, init):
    """Metadata of a step: new tokens per request, their state slots, which of them continue."""
    dev = lambda x: torch.tensor(x, dtype=torch.int32).to(device)  # noqa: E731
    return SimpleNamespace(req_id_per_token=dev([r for r, n in enumerate(lens) for _ in range(n)]),
                           query_start_loc=dev([sum(lens[:i]) for i in range(len(lens) + 1)]), state_indices=dev(slots),
                           has_initial_state=dev([int(i) for i in init]))


CUTS = [[90], [1] * 90, [2, 3, 1, 64, 16, 2, 1, 1], [33, 2, 1, 1, 53]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", CUTS)
def test_bigram_rows(device, cuts):
    """Any portions; a neighbour that starts in every step, in a slot which another request has used; huge factors."""
    big = {"buckets": 1009, "mul_prev": 1 << 33, "mul_cur": 12345678901}
    t, u = tokens(sum(cuts), 5000, 1), tokens(3, 5000, 2)
    state = torch.tensor([77, 88, 99], dtype=torch.int64, device=device)
    at, got = 0, []
    for n in cuts:
        md = batch(device, [2, n], [2, 0], [False, at > 0])
        ids = torch.tensor(u[:2] + t[at:at + n], device=device)
        rows = ops.bigram_rows(ids, state, md.query_start_loc, md.state_indices, md.has_initial_state, big["mul_prev"],
                               big["mul_cur"], big["buckets"]).tolist()
        assert rows[:2] == oracle.bigram_rows(u[:2], big)
        got += rows[2:]
        at += n
        assert state.tolist() == [t[at - 1], 88, u[1]]
    assert got == oracle.bigram_rows(t, big)
    md = batch(device, [1], [-1], [True])           # no slot (a padded row): a first token, nothing is kept
    rows = ops.bigram_rows(torch.tensor([5], device=device), state, md.query_start_loc, md.state_indices,
                           md.has_initial_state, 1, 1, 1009)
    assert rows.tolist() == [1009] and state.tolist() == [t[-1], 88, u[1]]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width", [40, 37, 1030, 2056, 4200])
def test_embedding_norm_and_shift(device, dtype, width):
    """Start of the stream; the shift across portions and requests."""
    g = torch.Generator().manual_seed(width)
    ld, V, T = -(-width // 8) * 8, 30, 23

    def pad(x):
        out = torch.zeros(*x.shape[:-1], ld)
        out[..., :width] = x
        return out
    table, big = pad(torch.randn(V, width, generator=g) + 0.5).bfloat16(), pad(torch.randn(12, width, generator=g)).bfloat16()
    w, mix = 1 + 0.2 * torch.randn(width, generator=g), torch.rand(width, generator=g)
    ids, rows = torch.randint(0, V, (T,), generator=g), torch.randint(0, 12, (T,), generator=g)
    x0 = (table[ids].double() * 2.5 + big[rows].double())[:, :width]
    h0 = oracle.layer_norm(x0, w.double(), 1e-2)
    s0 = oracle.token_shift(h0, mix.double())
    for cuts in ([T], [1] * T, [2, 9, 1, 11]):
        state = torch.full((3, ld), 9.0, device=device)
        at, got = 0, []
        for n in cuts:
            md = batch(device, [1, n], [2, 1], [at > 0, at > 0])     # the neighbour repeats the request's first token
            pick = torch.tensor([0] + list(range(at, at + n)))
            x, h, s = ops.embed_stream_layernorm(ids[pick].to(device), table.to(DT[dtype]).to(device), 2.5,
                                                 (rows[pick].to(device), big.to(DT[dtype]).to(device)), w.to(device), 1e-2,
                                                 (pad(mix).to(device), state), md)
            assert not x[:, width:].any() and not h[:, width:].any() and not s[:, width:].any()
            close(s[0, :width], s0[0] if at == 0 else h0[0], dtype, "neighbour")     # same token again: h + 0 * mix
            got.append([z[1:, :width].cpu().double() for z in (x, h, s)])
            at += n
            close(state[1, :width], h0[at - 1], "float32", "state")
        for z, want, d in zip(zip(*got), (x0, h0, s0), ("float32", dtype, dtype)):
            close(torch.cat(z), want, d)
        assert bool((state[0] == 9.0).all())


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,width", [(5, 40), (70, 37), (1, 2048), (1500, 72), (1100, 2056), (1030, 4096), (9, 8200)])
def test_gated_sum_norm_and_shift(device, dtype, T, width):
    """One, two and no summands; runs of rows (long portions) and single rows; the final norm without a shift."""
    g = torch.Generator().manual_seed(T)
    ld = -(-width // 8) * 8

    def rows(scale=1.0, mean=0.0, n=1):
        out = torch.zeros(T, n * ld)
        for k in range(n):
            out[:, k * ld:k * ld + width] = torch.randn(T, width, generator=g) * scale + mean
        return out
    x, y1, y2, z = rows(2.0, 1.0), rows().to(DT[dtype]), rows(0.5, 3.0).to(DT[dtype]), rows(4.0, n=2).to(DT[dtype])
    w, mix = 1 + 0.2 * torch.randn(width, generator=g), torch.rand(ld, generator=g)
    mix[width:] = 0
    cuts = [1, 1, T - 2] if T > 2 else [T]
    md = batch(device, cuts, list(range(len(cuts))), [True, False, True][:len(cuts)])
    before = torch.randn(3, ld, generator=g)
    before[:, width:] = 0
    s1, s2 = oracle.sigmoid(z[:, :ld].double()), oracle.sigmoid(z[:, ld:].double())
    for parts, total in (([], 0.0), ([(y1, 0)], y1.double() * s1), ([(y1, 0), (y2, 1)], y1.double() * s1 + y2.double() * s2)):
        state = before.clone().to(device)
        p = [(y.to(device), z.to(device)[:, k * ld:(k + 1) * ld]) for y, k in parts]
        xs = x.to(device)
        new, h, sh = ops.gated_residual_layernorm(xs, p, w.to(device), 1e-3, DT[dtype], (mix.to(device), state), md)
        want = (x.double() + total)[:, :width]
        norm = oracle.layer_norm(want, w.double(), 1e-3)
        prev, at = torch.zeros_like(norm), 0
        for r, n in enumerate(cuts):
            prev[at] = before[r, :width].double() if [True, False, True][r] else 0.0
            prev[at + 1:at + n] = norm[at:at + n - 1]
            at += n
            close(state[r, :width], norm[at - 1], "float32", "state")
        close(new[:, :width], want, "float32", "stream")
        close(h[:, :width], norm, dtype, "norm")
        close(sh[:, :width], norm + (prev - norm) * mix[:width].double(), dtype, "shifted")
        assert torch.equal(xs.cpu(), x) and not h[:, width:].any() and not sh[:, width:].any()
        _, fin, none = ops.gated_residual_layernorm(xs, p, w.to(device), 1e-3, DT[dtype], keep_stream=False)
        close(fin[:, :width], norm, dtype, "final norm")
        assert none is None


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dims,base", [(2, 10.0), (6, 10000.0), (64, 5e5)])
def test_rotary_table(device, dims, base):
    """Positions far out keep their bits; the same numbers as the plain rotation."""
    pos = torch.tensor([0, 1, 2, 100, 4097, 1048577, 16777217])
    tab = ops.rotary_table(pos.to(device), ops.position_turns(dims, base).to(device)).cpu().double()
    for j, p in enumerate(pos.tolist()):
        x = torch.zeros(1, 1, dims, dtype=torch.float64)
        x[0, 0, :dims // 2] = 1.0
        r = oracle.rotate(x, base, start=p)[0, 0]
        torch.testing.assert_close(tab[j], torch.stack([r[:dims // 2], r[dims // 2:]], -1), rtol=0, atol=2e-6)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("Q,C,R,pairs", [(72, 48, 24, 12), (12, 20, 6, 3), (9, 11, 4, 1), (1536, 512, 64, 32), (40, 512, 24, 12)])
def test_latent_prep_and_rotation(device, dtype, Q, C, R, pairs):
    """Both norms, the rotated and the passing columns of the shared key part, the cache row with its zeros; rows without a
    slot are not stored; the same rotation on query heads.  Few tokens and many (the kernel's two shapes)."""
    g = torch.Generator().manual_seed(Q)
    off, bs = -(-C // 8) * 8 + 8, 4
    for T in (7, 300):
        _prep_and_rotate(device, dtype, Q, C, R, pairs, g, T, off, bs)


def _prep_and_rotate(device, dtype, Q, C, R, pairs, g, T, off, bs):
    row = off + -(-R // 8) * 8
    at = -(-Q // 8) * 8
    y = (torch.randn(T, at + C + R + 5, generator=g) * 3).to(DT[dtype])
    y = torch.nn.functional.pad(y, (0, -y.shape[1] % 8)).to(device)
    qn, kn = 1 + 0.3 * torch.randn(Q, generator=g), 1 + 0.3 * torch.randn(C, generator=g)
    pos = torch.randint(0, 5000, (T,), generator=g)
    tab = ops.rotary_table(pos.to(device), ops.position_turns(2 * pairs, 333.0).to(device))
    blocks = -(-(T + 5) // bs)
    cache = torch.full((blocks, bs, row), 5.0, dtype=DT[dtype], device=device)
    slots = torch.randperm(blocks * bs, generator=g)[:T]
    slots[T - 2] = -1
    q = ops.latent_prep(y[:, :Q], y[:, at:at + C + R], qn.to(device), kn.to(device), tab, cache, slots.to(device), off, at, 1e-2)
    z = y.cpu().double()
    close(q[:, :Q], oracle.rms_norm(z[:, :Q], qn.double(), 1e-2), dtype, "query latent", 0.03)
    assert not q[:, Q:].any()

    def turned(v, p):        # rotate-half over the first 2 * pairs columns
        return torch.cat([oracle.rotate(v[:, :, :2 * pairs], 333.0, start=p), v[:, :, 2 * pairs:]], -1)
    flat = cache.cpu().double().view(-1, row)
    for t, s in enumerate(slots.tolist()):
        if s < 0:
            continue
        want = torch.zeros(row, dtype=torch.float64)
        want[:C] = oracle.rms_norm(z[t, at:at + C], kn.double(), 1e-2)
        want[off:off + R] = turned(z[t:t + 1, None, at + C:at + C + R], int(pos[t]))[0, 0]
        close(flat[s], want, dtype, f"cache row {s}", 0.03)
    rest = sorted(set(range(blocks * bs)) - set(slots.tolist()))
    assert len(rest) >= 6 and bool((flat[rest] == 5.0).all())
    D = 6
    heads = torch.randn(T, 3, D + R, generator=g).to(DT[dtype])
    got = ops.rotate_heads(heads.clone().to(device), tab, D)
    want = torch.stack([torch.cat([heads[t:t + 1, :, :D].double(), turned(heads[t:t + 1, :, D:].double(), int(pos[t]))], -1)[0]
                        for t in range(T)])
    close(got, want, dtype, "query heads", 0.03)


def sizes_for(device, dtype, D, R, V, C):
    """Sizes as the kernels see them."""
    if device == "cuda" and dtype == "bfloat16":
        return LatentAttention.TENSOR_CORE
    return D, R, V, -(-C // 8) * 8


def attend(device, dtype, q, c, kr, w_uk, w_uv, lens, window, sink, scale, gate=None, form="absorbed", bs=64):
    """Windowed latent attention of several requests (``lens``: cached and new tokens of each) over a shuffled cache with
    stale contents: q [T, H, D + R] and kr [T, R] already rotated, c [T, C]; rows of all requests one after another, cached
    ones included.  Returns [new tokens, H, V]."""
    (T, H, _), C, R, dt = q.shape, c.shape[1], kr.shape[1], DT[dtype]
    D, V = w_uk.shape[1], w_uv.shape[1]
    Dp, Rp, Vp, Cp = sizes_for(device, dtype, D, R, V, C)
    up = torch.zeros(H, Dp + Vp, Cp)
    up[:, :D, :C], up[:, Dp:Dp + V, :C] = w_uk, w_uv
    up = up.to(dt).to(device)
    qp = torch.zeros(T, H, Dp + Rp)
    qp[..., :D], qp[..., Dp:Dp + R] = q[..., :D], q[..., D:]
    row = -(-(Cp + Rp) // 8) * 8
    nblk = [-(-(a + b) // bs) for a, b in lens]
    perm = torch.randperm(sum(nblk) + 3, generator=torch.Generator().manual_seed(1)).tolist()
    cache = torch.full((len(perm), bs, row), 3.0)
    bt = torch.zeros(len(lens), max(nblk) + 1, dtype=torch.int32)
    off, new = 0, []
    for r, (a, b) in enumerate(lens):
        blocks = torch.tensor([perm.pop() for _ in range(nblk[r])])
        bt[r, :len(blocks)] = blocks
        p = torch.arange(a + b)
        cells = torch.zeros(a + b, row)
        cells[:, :C], cells[:, Cp:Cp + R] = c[off:off + a + b], kr[off:off + a + b]
        cache[blocks[p // bs], p % bs] = cells
        new += list(range(off + a, off + a + b))
        off += a + b
    cache, bt = cache.to(dt).to(device), bt.to(device)
    qn = qp[new].to(dt).to(device).contiguous()
    i32 = lambda x: torch.tensor(x, dtype=torch.int32).to(device)  # noqa: E731
    sl, qsl = i32([a + b for a, b in lens]), i32([sum(b for _, b in lens[:i]) for i in range(len(lens) + 1)])
    mq, ms = max(b for _, b in lens), max(a + b for a, b in lens)
    sink = None if sink is None else sink.float().to(device)
    gate = None if gate is None else gate.to(dt).to(device)
    still = torch.zeros(len(new), Rp // 2, 2)
    still[..., 0] = 1.0                              # no rotation
    if form == "absorbed":
        qa = ops.absorb_query(qn, up[:, :Dp], still.to(device), Cp, row)
        o = ops.mla_attention(qa, cache, bt, sl, qsl, scale, Cp, mq, ms, window=window, sinks=sink)
        out = ops.expand_value(o, up[:, Dp:], gate).view(len(new), H, Vp)
    else:
        seen = [min(a + b, b + window - 1) for a, b in lens]
        starts = i32([sum(seen[:i]) for i in range(len(seen))])
        rows = ops.gather_window(cache, bt, sl, starts, i32(seen), sum(seen), max(seen))
        kv = ops.linear(rows[:, :Cp], up.view(H * (Dp + Vp), Cp))
        out = torch.zeros(len(new), H, Vp, dtype=dt, device=device)
        ops.mla_prefill_attention(qn, kv, rows[:, Cp:Cp + Rp], starts, i32(seen), qsl, True, scale, mq, out=out,
                                  window=window, sinks=sink, gate=gate)
    return out[..., :V]


def plain(q, c, kr, w_uk, w_uv, lens, window, sink, scale, gate=None):
    T, H, _ = q.shape
    c, kr, q = c.double(), kr.double(), q.double()
    k = torch.cat([torch.einsum("tc,hdc->thd", c, w_uk.double()), kr[:, None].expand(T, H, -1)], -1)
    v = torch.einsum("tc,hvc->thv", c, w_uv.double())
    out, off = [], 0
    for a, b in lens:
        s = slice(off, off + a + b)
        out.append(oracle.sink_attention(q[s], k[s], v[s], scale, window, None if sink is None else sink.double())[a:])
        off += a + b
    out = torch.cat(out)
    return out if gate is None else out * oracle.sigmoid(gate.double())[..., None]


# fp32 models attend in the absorbed form on the GPU
FORMS = [("cpu", "float32", "absorbed"), ("cpu", "float32", "up")] + [
    pytest.param("cuda", *x, marks=pytest.mark.gpu) for x in (("float32", "absorbed"), ("bfloat16", "absorbed"),
                                                              ("bfloat16", "up"))]


@pytest.mark.parametrize("device,dtype,form", FORMS)
@pytest.mark.parametrize("H,D,R,V,C", [(5, 40, 12, 24, 56), (3, 10, 6, 14, 20), (16, 128, 64, 128, 512), (37, 24, 8, 40, 72)])
def test_windowed_latent_attention(device, dtype, form, H, D, R, V, C):
    """Unequal requests, single tokens beside portions, windows from 1 to longer than everything, sinks, gates."""
    g = torch.Generator().manual_seed(D)
    few, many = [(37, 1), (64, 1), (0, 1), (190, 1), (130, 1)], [(37, 1), (0, 130), (30, 41), (63, 2), (200, 3), (0, 1)]
    for lens in (few, many):
        T = sum(a + b for a, b in lens)
        n = sum(b for _, b in lens)
        q, c, kr = torch.randn(T, H, D + R, generator=g) * 1.5, torch.randn(T, C, generator=g), torch.randn(T, R, generator=g)
        uk, uv = torch.randn(H, D, C, generator=g) / C ** 0.5, torch.randn(H, V, C, generator=g) / C ** 0.5
        q, c, kr, uk, uv = (z.to(DT[dtype]).float() for z in (q, c, kr, uk, uv))
        sink, gate = torch.randn(H, generator=g) * 2, torch.randn(n, H, generator=g).to(DT[dtype]).float()
        for window in (1, 5, 64, 65, 1000):
            if H > 16 and window not in (5, 65):
                continue
            a = (q, c, kr, uk, uv, lens, window, sink, (D + R) ** -0.5, gate)
            close(attend(device, dtype, *a, form=form), plain(*a), dtype, f"window {window}")
        a = (q, c, kr, uk, uv, lens, 70, None, 0.3 * (D + R) ** -0.5)
        close(attend(device, dtype, *a, form=form), plain(*a), dtype, "no sink, no gate")


@pytest.mark.parametrize("device,dtype,form", FORMS)
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 129])
def test_window_edge_and_page_borders(device, dtype, form, window):
    """One key stands out (through the latent, or through the shared rotated part) and has a value of its own: seen at
    distance window - 1, not at distance window; for single tokens, short and long portions, across page borders."""
    H, D, R, V, C = 2, 8, 4, 8, 16
    uk, uv = torch.zeros(H, D, C), torch.zeros(H, V, C)
    uk[:, 1, 1] = 1.0
    uv[:, 3, 2] = 1.0
    for through in ("latent", "rotated"):
        for dist in (window - 1, window):
            for i in sorted({window, 63, 64, 65, 127, 128, 200}):
                if i < dist:
                    continue
                q = torch.zeros(i + 1, H, D + R)
                q[..., 1 if through == "latent" else D + 2] = 8.0
                c, kr = torch.zeros(i + 1, C), torch.zeros(i + 1, R)
                c[i - dist, 2] = 1.0                                          # its value
                (c if through == "latent" else kr)[i - dist, 1 if through == "latent" else 2] = 4.0   # score 32
                for lens in ([(i, 1)], [(0, i + 1)], [(max(0, i - 1), min(2, i + 1))], [(max(0, i - 66), min(67, i + 1))]):
                    o = attend(device, dtype, q, c, kr, uk, uv, lens, window, torch.full((H,), -40.0), 1.0, form=form)
                    seen = float(o[-1, 0, 3])
                    assert (seen > 0.98) == (dist < window) and (seen < 0.02) == (dist >= window), (through, dist, i, lens, seen)


@pytest.mark.parametrize("device,dtype,form", FORMS)
def test_sink_per_head(device, dtype, form):
    """The sink is not scaled, counts once, and differs by head; far above and far below the scores."""
    H, C = 5, 16
    sink = torch.tensor([-90.0, 0.0, 1.5, 30.0, 100.0])
    for L in (1, 3, 200):
        q = torch.zeros(L, H, 12)
        q[..., 0] = 2.0
        uk, uv = torch.zeros(H, 8, C), torch.zeros(H, 4, C)
        uk[:, 0, 0] = 1.0
        uv[:, 1, 1] = 1.0
        c = torch.zeros(L, C)
        c[:, 0], c[:, 1] = 1.0, 3.0
        for lens in ([(L - 1, 1)], [(0, L)]):
            o = attend(device, dtype, q, c, torch.zeros(L, 4), uk, uv, lens, 500, sink, 0.5, form=form).double().cpu()
            for j, row in enumerate(o):
                n = lens[0][0] + j + 1                       # keys of score 2 * 1 * 0.5 = 1
                want = 3.0 * n * math.e / (n * math.e + torch.exp(sink.double()))
                torch.testing.assert_close(row[:, 1], want, rtol=1e-2 if dtype == "bfloat16" else 1e-5, atol=1e-6)


@pytest.mark.gpu
@pytest.mark.parametrize("window", [None, 100, 700])
@pytest.mark.parametrize("H", [16, 40])
def test_split_decoding_with_window_and_sink(H, window):
    """Splits merged in a cluster and through the workspace, one to four query tokens; splits that hold no visible page."""
    from vllm_kunlun_b200.ops import mla_cuda
    from vllm_kunlun_b200.ops.reference.attention import mla_decode
    g = torch.Generator().manual_seed(3)
    for q_len in (1, 2, 4):
        lens = [q_len, 65, 900, 1500]
        blocks = [-(-n // 64) for n in lens]
        bt = torch.zeros(len(lens), max(blocks), dtype=torch.int32)
        perm = torch.randperm(sum(blocks), generator=g).int()
        at = 0
        for r, n in enumerate(blocks):
            bt[r, :n] = perm[at:at + n]
            at += n
        cache = torch.randn(sum(blocks), 64, 576, generator=g).bfloat16()
        q = torch.randn(len(lens) * q_len, H, 576, generator=g).bfloat16()
        sl, qsl = torch.tensor(lens, dtype=torch.int32), torch.arange(0, len(lens) * q_len + 1, q_len, dtype=torch.int32)
        sink = torch.randn(H, generator=g) * 2 + 3
        want = mla_decode(q, cache, bt, sl, qsl, 0.05, 512, window=window, sinks=sink)
        dev = [t.cuda() for t in (q, cache, bt, sl, qsl)]
        for splits in (None, 1, 2, 3, 4, 8, 16):
            for force in (False, True):
                mla_cuda._FORCE_WORKSPACE[0] = force
                try:
                    got = mla_cuda.mla_decode_umma(*dev, 0.05, q_len, max(lens), splits, window=window, sinks=sink.cuda())
                finally:
                    mla_cuda._FORCE_WORKSPACE[0] = False
                close(got, want, "bfloat16", f"{splits} splits, {q_len} tokens", 0.05)


@pytest.mark.parametrize("device", DEVICES)
def test_gelu_in_fp32(device):
    """The activation of fp32 models keeps its bits, also where 1 + tanh cancels."""
    z = torch.linspace(-12, 12, 4096).reshape(2, -1)
    x = torch.cat([z, torch.ones_like(z)], -1)
    y = ops.act_and_mul(x.to(device), "gelu_tanh").cpu().double()
    torch.testing.assert_close(y, oracle.gelu_tanh(z.double()), rtol=1e-5, atol=1e-6)


# ------------------------------------------------------------------------------------------------ whole models

@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_stream(checkpoints, device, dtype, name):
    path, cfg, w = checkpoints[name]
    toks = tokens(150, cfg["vocab"])
    want, stream = oracle.forward(toks, w, cfg)
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
    want, _ = oracle.forward(toks, w, cfg)
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
def test_mixed_batches_and_reuse(checkpoints, device, dtype, name, monkeypatch):
    """Up to four live requests, portions beside single tokens, requests that pause, pages and slots that go round: each
    request's logits are those it has alone.  The bound on up-projected rows is so small that a step's portions need
    several attention calls."""
    path, cfg, w = checkpoints[name]
    monkeypatch.setattr(LatentAttention, "KV_BYTES", 60 * 4 * 512)
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
def test_one_token_prompt_in_a_used_slot(checkpoints, device, dtype):
    """A first portion of one token knows no previous token even when its slot still holds another request's."""
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
@pytest.mark.parametrize("dist", [6, 7, 8, 9])
def test_reach_of_one_layer(device, dtype, dist, tmp_path):
    """One layer with a window of 7: the shift reads one token further back than the window, the pair embedding one more;
    a change beyond that leaves the logits as they are - bit for bit - and one inside it shows, in a prompt and decoding."""
    cfg = config([layer(latent(size=7), ff=None)], width=48)
    path, cfg, w = checkpoint(str(tmp_path), cfg, 31)
    w["l0.shift"].fill_(0.75)
    w["l0.mix.uq"].mul_(0.25)                     # flat attention: every visible key counts
    save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, path, cfg)
    a = tokens(80, cfg["vocab"], 3)
    b = list(a)
    b[79 - dist] = (b[79 - dist] + 41) % cfg["vocab"]
    r = replay(path, dtype, device, 128)
    for cut in (80, 79, 78, 40):
        got = []
        for t in (a, b):
            if cut < 80:
                r.step([{"id": "q", "tokens": t[:cut], "want": []}])
            got.append(r.step([{"id": "q", "tokens": t[cut if cut < 80 else 0:], "want": [len(t) - 1 - (cut if cut < 80 else 0)]}], ["q"]))
        moved = (oracle.forward(a, w, cfg)[0][-1] - oracle.forward(b, w, cfg)[0][-1]).abs().max()
        assert (moved > 1e-3) == (dist <= 8)
        assert torch.equal(got[0], got[1]) == (dist > 8), (cut, dist)
        if dtype == "float32" and dist <= 8:
            close(got[0] - got[1], (oracle.forward(a, w, cfg)[0] - oracle.forward(b, w, cfg)[0])[-1:], dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_token_reaches_through_the_layers(device, dtype, tmp_path):
    """A token several windows back moves the logits through the stack of layers as in the plain implementation."""
    cfg = config([layer(latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, q_rank=24, size=50), ff=32)] * 4, width=64)
    path, cfg, w = checkpoint(str(tmp_path), cfg, 17)
    a = tokens(190, cfg["vocab"], 9)
    b = list(a)
    b[20] = (b[20] + 11) % cfg["vocab"]
    r = replay(path, dtype, device, 192)
    diff = []
    for t in (a, b):
        got = [r.step([{"id": "q", "tokens": t[:120], "want": [119]}])]
        got += [r.step([{"id": "q", "tokens": [x], "want": [0]}]) for x in t[120:]]
        r.step([], ["q"])
        diff.append(torch.cat(got))
    plain_a = oracle.forward(a, w, cfg)[0][119:]
    want, size = oracle.forward(b, w, cfg)[0][119:] - plain_a, plain_a.pow(2).mean().sqrt()
    assert want[50:].abs().max() > 2e-4 * size    # three windows away
    if dtype == "float32":
        assert ((diff[1] - diff[0]).double() - want).abs().max() < 2e-5 * size


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
        logits = oracle.forward(seq, w, cfg)[0]
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


def test_random_initialisation_serves(checkpoints):
    """A ModelConfig without a checkpoint: seeded weights through the same loading path."""
    cfg = ModelConfig.from_hf_config(copy.deepcopy(SMALL))
    kw = dict(device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    a, b = (LLM(copy.deepcopy(cfg), **kw).generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].token_ids
            for _ in range(2))
    assert a == b and len(a) == 4


# ------------------------------------------------------------------------------------------------ configuration, loading

def test_configuration_is_read(checkpoints):
    path, cfg, _ = checkpoints["small"]
    m = ModelConfig.from_pretrained(path)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_layers, m.rms_norm_eps) == ("Seturax", 36, 97, 4, 1e-5)
    assert (m.embedding_scale, m.logit_scale, m.hidden_act) == (3.0, 1.7, "gelu_tanh")
    assert m.bigram == {"buckets": 53, "mul_prev": 7, "mul_cur": 3}
    assert m.has_recurrent_state and m.cache_block == 64
    no_rank = copy.deepcopy(cfg)
    for entry in no_rank["layers"]:
        del entry["mixer"]["q_rank"]                       # the tensors' shapes tell it as well
    m = ModelConfig.from_hf_config(no_rank).complete_from_shapes({"l1.mix.dq": (40, 36)})
    assert m.layer_specs[1].mixer["q_rank"] == 40
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_config(bad)
    bad = copy.deepcopy(cfg)
    del bad["embedding"]["bigram"]
    with pytest.raises(ValueError, match="bigram"):
        LLM(ModelConfig.from_hf_config(bad), device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)


def test_incomplete_or_foreign_checkpoints_are_refused(checkpoints, tmp_path):
    path, cfg, w = checkpoints["small"]
    kw = dict(device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    state = {k: v.to(torch.bfloat16) for k, v in w.items()}
    for change, match in ((lambda s: s.pop("l1.mix.sink"), "lacks"), (lambda s: s.update(extra=torch.zeros(2)), "unexpected"),
                          (lambda s: s.update(bigram=torch.zeros(53, 36)), "shape")):
        s = dict(state)
        change(s)
        d = str(tmp_path / match)
        save_safetensors(s, d, cfg)
        with pytest.raises(ValueError, match=match):
            LLM(d, **kw)


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
    V = cfg["vocab"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, V)  # noqa: E731
    close_rows(read(1), torch.stack([want[2], want[20]]), dtype)
    close_rows(read(2), torch.stack([want[29], want[21]]), dtype)
