"""Kefesun against the plain implementation in ``oracle_kefesun``: every mechanism alone, whole models through the engine
(whole prompts, portions, mixed batches, decoding, reused pages and slots), configuration and weight loading, the replay
program.  Each test runs on the CPU path and, on a GPU box, on the kernels (fp32 and bf16)."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_kefesun as oracle
from vllm_kunlun_b200 import LLM, SamplingParams, ops
from vllm_kunlun_b200.attention.metadata import AttentionMetadata
from vllm_kunlun_b200.config import ModelConfig
from vllm_kunlun_b200.engine.replay import ScheduleReplay
from vllm_kunlun_b200.models.loader import save_safetensors
from vllm_kunlun_b200.models.mixers import cache_head_dim

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
# kernels under test: fp32 on both devices, bf16 on the GPU
RUNS = [("cpu", "float32"), pytest.param("cuda", "float32", marks=pytest.mark.gpu),
        pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def moe(experts=5, identity=1, top=2, ff=20, shared=28, count=2, keep=1, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "identity": identity, "top": top, "scale": scale,
                       "groups": {"count": count, "keep": keep}}}


def attn(mlp, heads=4, kv_heads=2, dim=10, vdim=6, scale=0.3, size=9, keep_first=2, base=100.0, dims=6):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "mask": {"size": size, "keep_first": keep_first}, "rot": {"base": base, "dims": dims}}}


def gru(mlp, width=22):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def config(layers, width=36, vocab=97, eps=1e-5, taps=3, scale=6.0):
    return {"architecture": "Kefesun", "layers": layers, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": scale}, "vocab": vocab, "width": width}


# every branch, unequal sizes everywhere, widths that need padding, layers without a feed-forward, one group, no identity expert
SMALL = config([gru(moe()), attn(moe(6, 3, 4, 12, 40, 3, 2)), attn(None, heads=3, kv_heads=3, dim=5, vdim=7, size=70, dims=4),
                gru(moe(3, 0, 3, 16, 8, 1, 1, 1.0), width=41), gru(None, width=7),
                attn(moe(4, 4, 1, 24, 24, 4, 1), heads=6, kv_heads=1, dim=8, size=1, keep_first=5, dims=8)])
# head sizes of the tensor-core kernels, windows and kept keys beyond a key tile, many experts, other taps
WIDE = config([attn(moe(14, 2, 5, 40, 100, 4, 2), heads=6, kv_heads=3, dim=128, vdim=96, scale=0.09, size=150, keep_first=3,
                    base=5e5, dims=64),
               gru(moe(12, 4, 6, 64, 64, 2, 1), width=300),
               attn(moe(4, 1, 1, 128, 72, 5, 3), heads=54, kv_heads=3, dim=16, vdim=72, scale=0.2, size=33, keep_first=130,
                    dims=12),
               attn(None, heads=8, kv_heads=4, dim=64, vdim=64, scale=0.125, size=64, keep_first=0, dims=64)],
              width=104, vocab=300, eps=1e-3, taps=4, scale=1.0)
# beyond the tensor-core kernels' sizes
LARGE = config([attn(moe(2, 1, 1, 70, 30, 3, 2), heads=3, kv_heads=1, dim=140, vdim=30, scale=0.08, size=40, keep_first=1,
                     dims=20),
                gru(moe(), width=515)], width=44, taps=2, scale=2.5)
CONFIGS = {"small": SMALL, "wide": WIDE, "large": LARGE}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Many tiny operations: one thread is several times faster than all of them."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def checkpoint(path, cfg, seed, change=None):
    w = oracle.random_weights(cfg, seed=seed)
    if change is not None:
        change(w)
        w = {k: v.to(torch.bfloat16).double() for k, v in w.items()}
    save_safetensors({k: v.to(torch.bfloat16) for k, v in w.items()}, path, cfg)
    return path, cfg, w


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    """name -> (directory, configuration, float64 weights)."""
    return {name: checkpoint(str(tmp_path_factory.mktemp(name)), cfg, 3 + i) for i, (name, cfg) in enumerate(CONFIGS.items())}


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got, want, dtype, what="", bf16=0.06):
    """fp32: rounding of 32-bit sums; bf16: a small fraction of the values' root mean square, and one unit in the last place of
    the value itself."""
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    scale = want.pow(2).mean().sqrt().clamp(min=1e-3)
    d = (got - want).abs() if dtype == "float32" else ((got - want).abs() - want.abs() / 128).clamp(min=0)
    err = (d.max() / scale).item()
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


def i32(x, device):
    return torch.tensor(x, dtype=torch.int32, device=device)


def starts(lens):
    return [sum(lens[:i]) for i in range(len(lens) + 1)]


# ------------------------------------------------------------------------------------------------ attention

def attend(device, dtype, q, k, v, lens, scale, pb, size, keep, bs=64, sigmoid=True):
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
    nd = 0
    while nd < len(lens) and lens[nd][1] == 1:
        nd += 1
    sl, qsl = i32([a + b for a, b in lens], device), i32(starts([b for _, b in lens]), device)
    o = ops.paged_attention(qp.to(dt).to(device), cache.to(dt).to(device), bt.to(device), sl, qsl, scale,
                            max(b for _, b in lens), max(a + b for a, b in lens), size, num_decodes=nd, num_decode_tokens=nd,
                            bias=None if pb is None else pb.float().reshape(H, 1).to(device), keep_first=keep, sigmoid=sigmoid)
    return o[..., :V]


def plain_attention(q, k, v, lens, scale, pb, size, keep):
    H, G = q.shape[1], k.shape[1]
    of = [i // (H // G) for i in range(H)]
    out, off = [], 0
    for a, b in lens:
        s = slice(off, off + a + b)
        out.append(oracle.sigmoid_attention(q[s][a:], k[s][:, of], v[s][:, of], scale, pb,
                                            oracle.visible(a + b, size if size else a + b, keep)[a:]))
        off += a + b
    return torch.cat(out)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,V", [(6, 2, 64, 40), (3, 3, 10, 14), (8, 2, 128, 128), (20, 1, 24, 72), (2, 1, 140, 30)])
def test_sigmoid_attention(device, dtype, H, G, D, V):
    """Unequal requests, single tokens beside portions; windows and kept keys of every relation to pages and tiles."""
    g = torch.Generator().manual_seed(D)
    for lens in ([(37, 1), (64, 1), (0, 1), (190, 1), (420, 1)], [(37, 1), (0, 130), (30, 41), (63, 2), (300, 3), (0, 1)],
                 [(2500, 1), (1700, 1)], [(1400, 140)]):
        T = sum(a + b for a, b in lens)
        q, k, v = rounded(dtype, torch.randn(T, H, D, generator=g) * 1.5, torch.randn(T, G, D, generator=g),
                          torch.randn(T, G, V, generator=g))
        pb = torch.randn(H, generator=g).double() - 2.0
        for size, keep in ((None, 0), (1, 0), (9, 3), (64, 0), (70, 4), (128, 64), (129, 140), (40, 5000), (1000, 2)):
            got = attend(device, dtype, q, k, v, lens, D ** -0.5, pb, size, keep)
            close(got, plain_attention(q, k, v, lens, D ** -0.5, pb, size, keep), dtype, f"window {size} {keep}", 0.05)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("D", [8, 160])
def test_one_loud_key_at_every_edge(device, dtype, D):
    """All scores are so low that their keys do not count, except one key's: it is seen by exactly the queries that the window
    and the kept keys allow, in prompts and by single tokens, on both sides of page, tile and window edges."""
    H, V, L = 2, 8, 400
    q = torch.zeros(L, H, D)
    q[:, :, 0] = 4.0
    v = torch.zeros(L, 1, V)
    v[:, 0, 1] = 1.0
    pb = torch.full((H,), -30.0).double()
    for size, keep in ((1, 1), (5, 0), (64, 4), (65, 63), (72, 64), (127, 65), (128, 1), (129, 128), (130, 129), (200, 260)):
        near = {L - size, L - size - 1, keep - 1, keep, 63, 64, 127, 128, L - 1, L - 2, 0, L - 70 - size, L - 70 - size + 1}
        for j in sorted(x for x in near if 0 <= x < L):
            k = torch.zeros(L, 1, D)
            k[j, 0, 0] = 10.0
            seen = oracle.visible(L, size, keep)[:, j].double()
            for lens in ([(L - 1, 1)], [(0, L)], [(L - 70, 70)], [(L - 2, 2)]):
                a = lens[0][0]
                o = attend(device, dtype, q, k, v, lens, 1.0, pb, size, keep)[:, :, 1].double().cpu()
                assert (o - seen[a:, None]).abs().max() < 1e-2, (size, keep, j, lens)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_extreme_scores(device, dtype):
    """Scores far out on both sides: weights of zero and one, nothing infinite."""
    H, D, V, L = 4, 16, 16, 200
    g = torch.Generator().manual_seed(1)
    q, k, v = rounded(dtype, torch.randn(L, H, D, generator=g) * 20, torch.randn(L, 2, D, generator=g) * 20,
                      torch.randn(L, 2, V, generator=g))
    pb = torch.tensor([0.0, 100.0, -100.0, 3.0]).double()
    for lens in ([(0, L)], [(L - 1, 1)], [(100, 100)]):
        got = attend(device, dtype, q, k, v, lens, 1.0, pb, 90, 3)
        close(got, plain_attention(q, k, v, lens, 1.0, pb, 90, 3), dtype, str(lens), 0.05)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_kept_keys_with_a_softmax(dtype):
    """The window that keeps first keys serves softmax attention as well."""
    H, G, D, L = 4, 2, 128, 420
    g = torch.Generator().manual_seed(2)
    q, k, v = rounded(dtype, torch.randn(L, H, D, generator=g), torch.randn(L, G, D, generator=g),
                      torch.randn(L, G, D, generator=g))
    of = [i // 2 for i in range(H)]
    for size, keep in ((70, 4), (129, 140), (16, 1)):
        s = torch.einsum("qhd,khd->hqk", q, k[:, of]) * 0.1
        want = torch.einsum("hqk,khd->qhd", torch.softmax(s.masked_fill(~oracle.visible(L, size, keep), float("-inf")), -1),
                            v[:, of])
        for lens in ([(0, L)], [(L - 1, 1)], [(L - 2, 2)], [(L - 90, 90)]):
            got = attend("cuda", dtype, q, k, v, lens, 0.1, None, size, keep, sigmoid=False)
            close(got, want[lens[0][0]:], dtype, f"{size} {keep} {lens}")


def test_sigmoid_weights_need_a_bias():
    if torch.cuda.is_available():
        with pytest.raises(ValueError, match="bias"):
            attend("cuda", "bfloat16", *(torch.zeros(4, 1, 8),) * 3, [(0, 4)], 1.0, None, 2, 0)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,V,dims", [(4, 2, 8, 12, 8), (3, 1, 10, 7, 6), (2, 2, 128, 72, 48), (2, 1, 64, 64, 64), (1, 1, 140, 9, 2)])
def test_split_norms_and_rotates(device, dtype, H, G, D, V, dims):
    """Norm weights per column, rotation of the first columns only (far positions too), values as they are, padding."""
    dt, T, bs, base, eps = DT[dtype], 8, 64, 1000.0, 1e-2
    g = torch.Generator().manual_seed(V)
    off = [0, -(-H * D // 8) * 8, -(-H * D // 8) * 8 + -(-G * D // 8) * 8]
    y = torch.randn(T, off[2] + -(-G * V // 8) * 8, generator=g).to(dt)
    pos = torch.tensor([0, 1, 2, 100, 4097, 5, 2 ** 20 + 1, 10])
    slots = torch.tensor([5, 70, 200, -1, 33, 0, 1, 2])
    qn, kn = torch.randn(D, generator=g), torch.randn(D, generator=g)
    Dc = cache_head_dim(D, V, dt, (128,))
    cache = torch.full((4, 2, G, bs, Dc), 7.0, dtype=dt).to(device)
    yd = y.to(device)
    parts = [(0, H * D), (off[1], G * D), (off[2], G * V)]
    table = ops.rotary_table(pos.to(device), ops.position_turns(dims, base).to(device))
    q = ops.attn_prep_cache(*(yd[:, o:o + n] for o, n in parts), cache, slots.to(device), pos.to(device), H, G, eps, v_norm=False,
                            qk_norm=(qn.to(device), kn.to(device)), table=table)
    plain = [y[:, o:o + n].double().reshape(T, -1, d) for (o, n), d in zip(parts, (D, D, V))]

    def turned(x, weight):
        x = oracle.rms_norm(x, weight.double(), eps)
        return torch.stack([oracle.rotate(x[t].expand(int(p) + 1, *x[t].shape), base, dims)[-1] if p < 200 else
                            far(x[t], int(p)) for t, p in enumerate(pos)])

    def far(x, p):
        out, half = x.clone(), dims // 2
        a = torch.tensor([p * base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
        out[:, :half], out[:, half:dims] = (x[:, :half] * a.cos() - x[:, half:dims] * a.sin(),
                                            x[:, half:dims] * a.cos() + x[:, :half] * a.sin())
        return out

    close(q[..., :D], turned(plain[0], qn), dtype, "queries")
    assert not q[..., D:].any()
    want_k = turned(plain[1], kn)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            cell = cache[s // bs, :, :, s % bs].cpu()
            close(cell[0, :, :D], want_k[t], dtype, "cached keys")
            assert torch.equal(cell[1, :, :V].double(), plain[2][t]) and not cell[0, :, D:].any() and not cell[1, :, V:].any()
    assert (cache[3, :, :, 9:].float() == 7.0).all()


# ------------------------------------------------------------------------------------------------ recurrence

def blend(device, dtype, z, x, gate, zb, xb, state, lens, slots, init):
    n, W = z.shape
    a = -(-W // 8) * 8
    y = torch.zeros(n, 3 * a, dtype=DT[dtype])
    y[:, :W], y[:, a:a + W], y[:, 2 * a:2 * a + W] = z, x, gate
    y = y.to(device)
    nd = 0
    while nd < len(lens) and lens[nd] == 1:
        nd += 1
    out = torch.full((n, a), 5.0, dtype=DT[dtype], device=device)
    out[:, W:] = 0
    ops.gated_blend(y[:, :W], y[:, a:a + W], y[:, 2 * a:2 * a + W], zb.float().to(device), xb.float().to(device), state,
                    i32(starts(lens), device), i32(slots, device), i32(init, device), out, max(lens), nd)
    assert not out[:, W:].any()
    return out[:, :W]


def plain_blend(z, x, gate, zb, xb):
    zz = oracle.sigmoid(z + zb.double())
    return oracle.blend_recurrence(zz, oracle.candidate(x + xb.double())) * oracle.silu(gate)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("W", [8, 33, 300])
def test_gated_blend(device, dtype, W):
    """Portions of every remainder modulo a run and a block of tokens, single tokens, states that go on and slots that are used
    again; gates from almost closed to almost open, candidates on both sides of zero."""
    g = torch.Generator().manual_seed(W)
    zb, xb = torch.randn(W, generator=g) * 3, torch.randn(W, generator=g)
    zb[::3] -= 8.0
    for lens in ([1, 1, 16, 33, 2, 130, 15, 128], [1, 1, 1], [3, 2, 9], [300]):
        n = sum(lens)
        state = torch.full((len(lens) + 2, W), 9.0, device=device)          # what other requests left behind
        slots = torch.randperm(len(lens) + 2, generator=g).tolist()[:len(lens)]
        seqs = [[] for _ in lens]
        for step in range(3):
            z, x, gate = rounded(dtype, *(torch.randn(n, W, generator=g) * 2 for _ in range(3)))
            out = blend(device, dtype, z, x, gate, zb, xb, state, lens, slots, [int(step > 0)] * len(lens))
            at = 0
            for r, m in enumerate(lens):
                seqs[r].append((z[at:at + m], x[at:at + m], gate[at:at + m]))
                want = plain_blend(*(torch.cat(p) for p in zip(*seqs[r])), zb, xb)[-m:]
                close(out[at:at + m], want, dtype, f"step {step} request {r}", 0.03)
                at += m
        assert (state[[s for s in range(len(lens) + 2) if s not in slots]] == 9.0).all()


@pytest.mark.parametrize("device,dtype", RUNS)
def test_first_token_stays_in_the_state(device, dtype):
    """Gates that open once and then stay shut: what the first token wrote is there, unchanged, hundreds of tokens later."""
    W, L = 16, 300
    z, x = torch.full((L, W), -100.0), torch.full((L, W), -50.0)
    z[0], x[0], gate = 100.0, 2.0, torch.full((L, W), 30.0)
    for lens in ([L], [100, 1, 199], [1] * 20 + [L - 20]):
        state = torch.full((1, W), 4.0, device=device)
        at, got = 0, []
        for i, n in enumerate(lens):
            s = slice(at, at + n)
            got.append(blend(device, dtype, z[s], x[s], gate[s], torch.zeros(W), torch.zeros(W), state, [n], [0], [int(i > 0)]))
            at += n
        assert (torch.cat(got).double().cpu() - 75.0).abs().max() < (1e-3 if dtype == "float32" else 0.5)


# ------------------------------------------------------------------------------------------------ stream

def metadata(lens, slots, init, device):
    z = torch.zeros(sum(lens), dtype=torch.int64, device=device)
    md = AttentionMetadata(num_tokens=sum(lens), num_reqs=len(lens), positions=z, slot_mapping=z,
                           block_tables=torch.zeros(len(lens), 1, dtype=torch.int32, device=device),
                           seq_lens=i32(lens, device), query_start_loc=i32(starts(lens), device), max_query_len=max(lens),
                           max_seq_len=max(lens))
    md.state_indices, md.has_initial_state = i32(slots, device), i32(init, device)
    return md


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("width,ld,taps", [(36, 40, 3), (64, 64, 1), (20, 24, 2), (520, 520, 4), (2100, 2104, 3), (4100, 4104, 7),
                                           (30, 32, 12)])
def test_stream_norm_and_convolution(device, dtype, width, ld, taps):
    """Embedding, sublayer results and experts' choices into the stream; the convolution over portions that are shorter and
    longer than its taps and over runs of rows, with states that go on in used slots; the last norm."""
    g = torch.Generator().manual_seed(width)
    pad = lambda z: torch.nn.functional.pad(z, (0, ld - width))  # noqa: E731
    dt, k, eps = DT[dtype], 3, 1e-3
    table = pad(torch.randn(9, width, generator=g)).to(dt)
    w, wf = torch.randn(width, generator=g), torch.randn(width, generator=g)
    c = torch.randn(width, taps, generator=g)
    conv_w = pad(c.T).contiguous().to(device)
    big = width > 2000
    for lens_by_step in (([1, 2, 70, 3, 1], [33, 1, 2, 1, 5]), ([1, 1, 2, 4], [1, 1, 1, 1], [3, 2, 1, 4])):
        if big and max(lens_by_step[0]) > 10 and device == "cpu":
            continue
        R = len(lens_by_step[0])
        slots = torch.randperm(R + 2, generator=g).tolist()[:R]
        state = None if taps == 1 else torch.full((R + 2, taps - 1, ld), 9.0, device=device)
        seqs = [torch.zeros(0, width, dtype=torch.float64) for _ in range(R)]
        for step, lens in enumerate(lens_by_step):
            T = sum(lens)
            md = metadata(lens, slots, [int(step > 0)] * R, device)
            ids = torch.randint(0, 9, (T,), generator=g)
            conv = (conv_w, state)

            def check(x, h, what):
                at = 0
                for r, n in enumerate(lens):
                    seqs[r] = torch.cat([seqs[r], x[at:at + n, :width].double().cpu()])
                    want = oracle.input_conv(seqs[r], c.double())[-n:]
                    close(h[at:at + n, :width], want, dtype, f"{what}: step {step} request {r}")
                    at += n
                assert not x[:, width:].any() and not h[:, width:].any() and h.dtype == dt

            if step == 0:
                x, h = ops.embed_input_conv(ids.to(device), table.to(device), 2.5, conv, md)
                want_x = table[ids][:, :width].double() * 2.5
                close(x[:, :width], want_x, "float32")
                check(x, h, "embedding")
                continue
            x = pad(torch.randn(T, width, generator=g)).to(device)
            start = x.clone().double().cpu()[:, :width]
            y = pad(torch.randn(T, width, generator=g) + 3.0).to(dt)
            if step == 1:
                h = ops.postnorm_input_conv(x, y.to(device), w.to(device), eps, dt, conv, md)
                s = y[:, :width].double()
            else:
                rows, through = (pad(torch.randn(n, width, generator=g)).to(dt) for n in (T * k + 2, T))
                places = torch.randperm(T * k + 2, generator=g)[:T * k].int()
                places[::4] = -1
                weights = torch.randn(T, k, generator=g)
                parts = ops.ChoicesSum(*(p.to(device) for p in (y, rows, places, weights, through)))
                h = ops.postnorm_input_conv(x, parts, w.to(device), eps, dt, conv, md)
                p = places.reshape(T, k).long()
                picked = torch.where((p >= 0)[..., None], rows.double()[p.clamp(min=0)], through.double()[:, None])
                s = (y.double() + (picked * weights.double()[..., None]).sum(1))[:, :width]
            close(x[:, :width], start + oracle.layer_norm(s, w.double(), eps), "float32", "stream")  # 32-bit in 16-bit models too
            check(x, h, "sublayer")
        if state is not None:
            assert (state[[s for s in range(R + 2) if s not in slots]] == 9.0).all()
    x = pad(torch.randn(5, width, generator=g)).to(device)
    y = pad(torch.randn(5, width, generator=g)).to(dt)
    want = x.double().cpu()[:, :width] + oracle.layer_norm(y[:, :width].double(), w.double(), eps)
    h = ops.postnorm_input_conv(x, y.to(device), w.to(device), eps, dt, final_weight=wf.to(device))
    close(h[:, :width], oracle.layer_norm(want, wf.double(), eps), dtype, "last norm")
    assert not h[:, width:].any()


# ------------------------------------------------------------------------------------------------ experts

@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,outputs,k,groups,keep,width", [(5, 14, 3, 2, 1, 40), (130, 12, 3, 4, 2, 72), (700, 9, 9, 1, 1, 64),
                                                           (3, 64, 8, 32, 8, 24), (65, 300, 16, 3, 3, 1200), (2, 40, 1, 20, 1, 16)])
def test_routing(device, dtype, T, outputs, k, groups, keep, width):
    """Choice by score plus correction inside the groups with the best member; weights without the correction.  Corrections
    below zero: a group that is left out must not be chosen from although its members' scores count as little as zero."""
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, width, generator=g).to(DT[dtype])
    r = (torch.randn(outputs, width, generator=g) * 3 / width ** 0.5).to(DT[dtype])
    for shift in (0.0, -2.0, 0.4):
        corr = torch.randn(outputs, generator=g) * 0.2 + shift
        w, ids = ops.router_and_route(x.to(device), r.to(device), None, k, "softmax", False, corr.to(device), groups, keep, 2.2,
                                      fp32=True, group_top=1)
        order, weights = oracle.route(x.double(), r.double(), corr.double(), k, groups, keep, 2.2)
        a, b = ids.cpu().long().sort(-1), order.sort(-1)
        same = (a.values == b.values).all(-1)
        assert same.float().mean() > 0.98
        got = w.double().cpu().gather(1, a.indices)[same]
        assert (got - weights.gather(1, b.indices)[same]).abs().max() < 1e-5       # the logits are 32-bit sums


def test_routing_keeps_its_defaults():
    """Softmax scores know no groups unless asked; sigmoid scores rank groups by their two best members."""
    z = torch.tensor([[4.0, -8.0, -9.0, 3.9, 3.8, 3.7]])
    assert ops.moe_route(z, 2, "softmax", n_group=2, topk_group=1)[1].tolist() == [[0, 3]]
    assert ops.moe_route(z, 2, "sigmoid", n_group=2, topk_group=1)[1].tolist() == [[3, 4]]
    assert ops.moe_route(z, 2, "softmax", n_group=2, topk_group=1, group_top=1)[1].tolist() == [[0, 1]]
    assert ops.moe_route(z, 2, "softmax", n_group=2, topk_group=1, group_top=2)[1].tolist() == [[3, 4]]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,E,outputs,k,ff,width", [(5, 7, 9, 4, 64, 40), (130, 5, 5, 3, 64, 72), (700, 4, 6, 2, 128, 64),
                                                    (1, 3, 6, 3, 64, 16), (3, 2, 9, 1, 64, 24)])
def test_expert_rows(device, dtype, T, E, outputs, k, ff, width):
    """Ungated experts in any order, choices without an expert, uneven experts; no expert at all for some batches."""
    dt = DT[dtype]
    g = torch.Generator().manual_seed(T)
    x = (torch.randn(T, width, generator=g)).to(dt)
    up = (torch.randn(E, ff, width, generator=g) / width ** 0.5).to(dt)
    down = (torch.randn(E, width, ff, generator=g) / ff ** 0.5).to(dt)
    every = torch.stack([torch.randperm(outputs, generator=g)[:k] for _ in range(T)])
    for ids in (every, torch.arange(outputs - k, outputs).expand(T, k)):
        rows, places = ops.expert_rows(x.to(device), up.to(device), down.to(device), ids.int().to(device), "relu2", choices=outputs)
        places = places.cpu().reshape(T, k)
        assert torch.equal(places < 0, ids >= E)
        got = rows.double().cpu()[places.clamp(min=0).long()]
        want = torch.stack([torch.stack([oracle.expert(x[t].double(), up[min(e, E - 1)].double(), down[min(e, E - 1)].double())
                                         for e in ids[t].tolist()]) for t in range(T)])
        if (ids < E).any():
            close(got[ids < E], want[ids < E], dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("T,N,K", [(1, 40, 64), (16, 200, 1032), (33, 136, 264), (64, 128, 8192), (300, 1000, 512)])
def test_projection_with_squared_relu(device, dtype, T, N, K):
    """In the epilogue of every product kernel: few rows, split sums, whole tiles; with and without a bias."""
    g = torch.Generator().manual_seed(T)
    x, w, b = rounded(dtype, torch.randn(T, K, generator=g), torch.randn(N, K, generator=g) / K ** 0.5, torch.randn(N, generator=g))
    on = lambda t: t.to(DT[dtype]).to(device)  # noqa: E731
    for bias in (None, b):
        want = torch.clamp(x @ w.T + (0.0 if bias is None else bias), min=0.0) ** 2
        close(ops.linear(on(x), on(w), None if bias is None else on(bias), act="relu2"), want, dtype)


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
def test_short_prompts_in_a_used_slot(checkpoints, device, dtype):
    """A first portion shorter than the convolution's taps starts from an empty state even when its slot still holds another
    request's; the rows in front of a second such portion come from both."""
    path, cfg, w = checkpoints["wide"]
    r = replay(path, dtype, device, 128)
    want, got = [], []
    for i, cuts in enumerate(([1, 1, 1, 1, 1], [2, 1, 2], [1, 2, 2], [5], [3, 2], [1, 3, 1], [4, 1], [1, 4])):
        t = tokens(20, cfg["vocab"], 40 + i)
        r.step([{"id": "x", "tokens": t, "want": []}], ["x"])
        want.append(oracle.forward(t[:5], w, cfg))
        at = 0
        for n in cuts:
            got.append(r.step([{"id": "y", "tokens": t[at:at + n], "want": list(range(n))}]))
            at += n
        r.step([], ["y"])
    close_rows(torch.cat(got), torch.cat(want), dtype)


def moved_rows(path, cfg, w, device, dtype, at, L, cuts_list, seed=3):
    """The two runs (with and without another token at ``at``) of the framework per way of cutting, and the plain ones."""
    a = tokens(L, cfg["vocab"], seed)
    b = list(a)
    b[at] = (b[at] + 41) % cfg["vocab"]
    plain = [oracle.forward(t, w, cfg) for t in (a, b)]
    r = replay(path, dtype, device, -(-L // 64) * 64)
    out = []
    for cuts in cuts_list:
        got = []
        for t in (a, b):
            p, rows = 0, []
            for n in cuts:
                rows.append(r.step([{"id": "q", "tokens": t[p:p + n], "want": list(range(n))}]))
                p += n
            r.step([], ["q"])
            got.append(torch.cat(rows))
        out.append(got)
    return plain, out


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("size,keep", [(70, 0), (64, 5), (20, 129)])
def test_a_token_reaches_as_far_as_the_window(device, dtype, size, keep, tmp_path):
    """One changed token in a model of one attention layer moves the logits of exactly the places that see it: up to the window's
    edge, or everywhere behind it if it is among the kept ones (the convolution carries it two rows further)."""
    def change(w):
        w["l0.mix.q"].mul_(0.1)
        w["l0.mix.pb"].fill_(1.0)
        w["l0.canon1"].zero_()
    layers = [attn(None, heads=2, kv_heads=1, dim=16, vdim=16, scale=0.25, size=size, keep_first=keep, dims=8)]
    path, cfg, w = checkpoint(str(tmp_path), config(layers, width=48), 31, change)
    L = 260
    for at in sorted({0, max(keep - 1, 0), keep, 100, 131}):
        plain, runs = moved_rows(path, cfg, w, device, dtype, at, L, ([L], [70, 2, 100, 88], [200] + [1] * 60))
        moved, scale = plain[1] - plain[0], plain[0].pow(2).mean().sqrt()
        seen = moved.abs().amax(-1) > 0
        assert torch.equal(seen, oracle.visible(L, size, keep)[:, at])
        for a, b in runs:
            d = (b - a).double()
            assert not d[~seen].any()                                # not a bit outside
            if dtype == "float32":
                assert (d - moved).abs().max() < 3e-5 * scale
            else:
                assert d[seen].abs().amax(-1).gt(0).float().mean() > 0.9


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_token_through_the_recurrence(device, dtype, tmp_path):
    """One changed token hundreds of places back still moves the logits as in the plain implementation."""
    def change(w):
        w["l0.mix.z.b"].fill_(-6.0)
        w["l0.mix.z"].mul_(0.3)
    path, cfg, w = checkpoint(str(tmp_path), config([gru(None, width=24)], width=48), 31, change)
    L = 300
    plain, runs = moved_rows(path, cfg, w, device, dtype, 0, L, ([L], [70, 2, 128, 100], [200] + [1] * 100))
    moved, size = plain[1] - plain[0], plain[0].pow(2).mean().sqrt()
    assert moved[-1].abs().max() > 1e-3 * size
    for a, b in runs:
        if dtype == "float32":
            assert ((b - a).double() - moved).abs().max() < 3e-5 * size
        else:
            assert not torch.equal(a[-1], b[-1])


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
    kw = dict(device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)
    a, b = (LLM(ModelConfig.from_hf_config(SMALL), **kw).generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0]
            .token_ids for _ in range(2))
    assert a == b and len(a) == 4


# ------------------------------------------------------------------------------------------------ configuration, loading

def test_configuration_is_read(checkpoints):
    path, cfg, _ = checkpoints["small"]
    m = ModelConfig.from_pretrained(path)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_layers, m.rms_norm_eps) == ("Kefesun", 36, 97, 6, 1e-5)
    assert (m.embedding_scale, m.input_conv_taps, m.hidden_act, m.tie_word_embeddings) == (6.0, 3, "relu2", True)
    assert m.has_recurrent_state and m.cache_block == 64
    assert [s.type for s in m.layer_specs] == ["mingru", "sigmoid_attention", "sigmoid_attention", "mingru", "mingru",
                                               "sigmoid_attention"]
    for change, match in ((lambda c: c["layers"][0].update(type="unknown"), "unknown mixer"),
                          (lambda c: c["layers"][0]["mlp"].update(kind="unknown"), "unknown feed-forward")):
        bad = copy.deepcopy(cfg)
        change(bad)
        with pytest.raises(ValueError, match=match):
            ModelConfig.from_hf_config(bad)


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), "choices from"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12), "rotated columns"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "do not divide"),
    (lambda c: c["canon"].update(taps=17), "taps"), (lambda c: c.pop("canon"), "taps")])
def test_configurations_that_cannot_be_served(change, match):
    bad = copy.deepcopy(SMALL)
    change(bad)
    with pytest.raises(ValueError, match=match):
        LLM(ModelConfig.from_hf_config(bad), device="cpu", dtype="float32", max_model_len=64, max_num_seqs=2, num_gpu_blocks=8)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("kind", ["attention", "mingru", "no convolution state"])
def test_one_kind_of_layer(device, dtype, kind, tmp_path):
    """Models without any recurrence, without any paged cache, and without any state at all."""
    layers = [gru(moe(), width=10)] * 2 if kind == "mingru" else [attn(moe(), size=30)] * 2
    path, cfg, w = checkpoint(str(tmp_path), config(layers, width=40, vocab=50, taps=1 if "state" in kind else 5), 8)
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
    for change, match in ((lambda s: s.pop("l1.mlp.e3.up"), "lacks"), (lambda s: s.update(head=torch.zeros(97, 36)), "unexpected"),
                          (lambda s: s.update({"l0.canon1": torch.zeros(36, 4)}), "shape")):
        s = dict(state)
        change(s)
        d = str(tmp_path / match)
        save_safetensors(s, d, cfg)
        with pytest.raises(ValueError, match=match):
            LLM(d, **kw)
    # tensors without effect: norm and convolution of a feed-forward that is not there
    s = {**state, "l2.norm2": torch.ones(36), "l4.canon2": torch.ones(36, 3)}
    save_safetensors({k: v.to(torch.bfloat16) for k, v in s.items()}, str(tmp_path / "more"), cfg)
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
