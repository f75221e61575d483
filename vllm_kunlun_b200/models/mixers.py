"""Sequence mixers of designs that list their layers one by one, with every size and constant a parameter.

A mixer reads the residual stream's 16-bit (or fp32) copy ``h [T, ld]`` and returns the summands of its output as
``[(y, scale), ...]`` for :func:`ops.layernorm_residual`.  It declares what it keeps between steps - paged tensors
(``kv_cache_spec``) and per-request state (``state_spec``) - and finds both in the forward context:
``kv_caches[layer] = (paged ..., state ...)``.

* :class:`WindowAttention`   softmax attention, unit-RMS q / k heads, optional sliding window, optional constant sink
* :class:`LightningAttention` linear attention with a fixed decay per head, jointly normed and gated output
* :class:`ParallelMixer`     both of them on the same input, one input projection, scaled sum
* :class:`ChannelDelta`      short convolutions + delta rule with one decay per head and key channel
* :class:`DistanceBiasAttention` softmax attention with a learned score bias by distance, a query temperature, unit-RMS values
  that layers may share, output gate per head
* :class:`SigmoidAttention` sigmoid weights without normalisation, rotated and normed q / k, window with kept first tokens
* :class:`MinGRU`            element-wise recurrence whose gates read only the current token
* :class:`GatedWriteAttention` linear attention whose forget gate decides what is written (HGRN2)
* :class:`LatentAttention`   windowed attention over a shared latent row per token, learned sink, output gate per head

Checkpoint rows are padded so that every column slice of a fused projection starts on a 16-byte boundary; padding rows
and columns are zero.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..attention.metadata import get_forward_context
from ..config import round_up
from .layers import ReplicatedLinear, param

ALIGN = 8                       # elements: 16 bytes of a 16-bit row
_TENSOR_CORE_HEADS = (64, 128, 256)
UNIT_NORM_EPS = 1e-6            # inside the root of the delta rule's unit vectors


def align(n: int) -> int:
    return round_up(n, ALIGN)


def cache_head_dim(dim: int, vdim: int, dtype: torch.dtype, served=_TENSOR_CORE_HEADS) -> int:
    """Head size of the paged cache: keys and values share it, zero-padded to one the attention kernels serve."""
    n = max(dim, vdim)
    if dtype == torch.float32:
        return round_up(n, 4)
    return next((d for d in served if d >= n), align(n))


def padded(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    if tuple(w.shape) == (rows, cols):
        return w
    out = w.new_zeros(rows, cols)
    out[:w.shape[0], :w.shape[1]] = w
    return out


class FusedProjection(ReplicatedLinear):
    """Several projections of the same input in one GEMM; part ``i`` is a column slice starting at a multiple of 8."""

    def __init__(self, in_features: int, sizes: dict, dtype, device, bias: bool = False):
        self.parts, off = {}, 0
        for name, n in sizes.items():
            self.parts[name] = (off, n)
            off += align(n)
        super().__init__(in_features, off, bias, dtype=dtype, device=device)
        self.weight.data.zero_()
        if bias:
            self.bias.data.zero_()

    def load_part(self, name: str, w: torch.Tensor):
        off, n = self.parts[name]
        if w.shape[0] != n or w.shape[1] > self.in_features:
            raise ValueError(f"projection {name}: checkpoint shape {tuple(w.shape)}, expected [{n}, <= {self.in_features}]")
        self.weight.data[off:off + n, :w.shape[1]].copy_(w)

    def load_bias(self, name: str, b: torch.Tensor):
        off, n = self.parts[name]
        self.bias.data[off:off + n].copy_(b)

    def slice(self, y: torch.Tensor, name: str) -> torch.Tensor:
        off, n = self.parts[name]
        return y[:, off:off + n]


def output_projection(in_features: int, width: int, dtype, device) -> ReplicatedLinear:
    lin = ReplicatedLinear(in_features, width, dtype=dtype, device=device)
    lin.weight.data.zero_()
    return lin


def _rows(T: int, n: int, dtype, device) -> torch.Tensor:
    """Buffer ``[T, align(n)]`` whose padding columns are zero (they meet zero weight columns)."""
    return torch.empty(T, n, dtype=dtype, device=device) if align(n) == n else \
        torch.zeros(T, align(n), dtype=dtype, device=device)


class WindowAttention(nn.Module):
    """Causal softmax attention over the paged cache; no rotation.  Every q / k head is divided by its root mean
    square.  ``window``: position i sees the last ``window`` positions up to itself (None = all of them).  ``sink``: a
    constant score without a value that joins the softmax denominator (None = no sink)."""

    served_heads = _TENSOR_CORE_HEADS       # cache head sizes of the tensor-core kernels that this attention can use

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: Optional[int],
                 sink: Optional[float], eps: float, dtype, device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads do not divide over {kv_heads} key / value heads")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.window, self.eps = float(scale), window, eps
        self.cache_dim = cache_head_dim(dim, vdim, dtype, self.served_heads)
        self.sinks = None if sink is None else param(heads, dtype=torch.float32, device=device)
        if sink is not None:
            self.sinks.data.fill_(sink)
        self.o = output_projection(heads * self.cache_dim, width, dtype, device)

    def proj_sizes(self) -> dict:
        return {"q": self.heads * self.dim, "k": self.kv_heads * self.dim, "v": self.kv_heads * self.vdim}

    def kv_cache_spec(self, block_size: int, dtype):
        return ((2, self.kv_heads, block_size, self.cache_dim), dtype)

    def load_o(self, w: torch.Tensor):
        """Columns are spread to the cache's head size (the padded value dims are zero)."""
        g = self.o.weight.data.view(self.o.out_features, self.heads, self.cache_dim)
        g[:w.shape[0], :, :self.vdim].copy_(w.reshape(w.shape[0], self.heads, self.vdim))

    def forward(self, q, k, v, kv_cache, md):
        T = q.shape[0]
        qn = ops.qk_unit_norm_cache(q, k, v, kv_cache, md.slot_mapping, self.heads, self.kv_heads, self.eps)
        span = md.max_seq_len if self.window is None else min(md.max_seq_len, self.window + 127)
        o = ops.paged_attention(
            qn, kv_cache, md.block_tables, md.seq_lens, md.query_start_loc, self.scale, md.max_query_len, span,
            self.window, self.sinks, md.seq_lens_cpu, md.query_start_loc_cpu, workspace=md.workspace,
            num_decodes=md.num_decodes, decode_query_len=1 + md.num_spec_tokens,
            num_decode_tokens=md.num_decode_tokens, stable_metadata=True)
        return self.o(o.reshape(T, self.heads * self.cache_dim))


def distance_buckets(rows: int, far: int) -> list:
    """Row of a distance table per distance 0, 1, ... up to the first one from which on all share the last row.  The first
    half of the rows serve one distance each; row ``h + m`` (``h = rows // 2``) starts at ``h (far / h)^(m / (rows - h))``,
    decided in integers, so that no rounding moves a boundary."""
    h, n_log = rows // 2, rows - rows // 2
    if not 0 < h < far:
        raise ValueError(f"a distance table of {rows} rows that ends at {far}")

    def start(m: int) -> int:       # first distance of row h + m
        want, unit = far ** m * h ** n_log, h ** m
        lo, hi = h, far             # the last row starts at or before ``far``
        while lo < hi:
            mid = (lo + hi) // 2
            lo, hi = (lo, mid) if mid ** n_log * unit >= want else (mid + 1, hi)
        return lo

    starts = [start(m) for m in range(n_log)]
    out = list(range(h))
    for m in range(n_log - 1):
        out += [h + m] * (starts[m + 1] - starts[m])
    return out + [rows - 1]


class DistanceBiasAttention(WindowAttention):
    """Causal softmax attention without rotation: positions enter through a learned bias per head and distance (added to the
    scaled scores) and through a temperature ``1 + coef ln(floor((p + 1) / every) + 1)`` of the query at position p.  Every
    value head is divided by its root mean square; layers that share values (``v_mix``) blend them with those of the first
    such layer (same token), and the cache holds the blend.  Every head's output is multiplied by ``sigmoid`` of its gate."""

    has_state = False
    cache_block = 64                        # tokens per cache block that the tensor-core kernels take
    served_heads = (128,)
    VALUES = "first_values"                 # where the first sharing layer leaves its values for the step's later layers

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        if "rel" in shapes:
            sizes["bias_rows"] = int(shapes["rel"][0])

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        m = sizes
        super().__init__(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], None, None, eps, dtype, device)
        self.layer_idx = layer_idx
        temp = m.get("q_temp")
        self.temperature = None if temp is None else (float(temp["coef"]), int(temp["every"]))
        self.shares_values, self.first_of_sharing, self.value_share = bool(m.get("v_mix")), False, 0.0
        self.buckets = torch.tensor(distance_buckets(self._bias_rows(m), int(m["bias_max"])), device=device)
        self.bias = param(self.heads, self.buckets.numel(), dtype=torch.float32, device=device)
        self.in_proj = FusedProjection(width, {**self.proj_sizes(), "g": self.heads}, dtype, device)

    @staticmethod
    def _bias_rows(sizes: dict) -> int:
        return int(sizes.get("bias_rows", 32))

    @classmethod
    def tensor_shapes(cls, sizes: dict, width: int) -> dict:
        H, G, D, V = (sizes[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        out = {"q": (H * D, width), "k": (G * D, width), "v": (G * V, width), "rel": (cls._bias_rows(sizes), H),
               "g": (H, width), "o": (width, H * V)}
        return {**out, "vmix": ()} if sizes.get("v_mix") else out

    @staticmethod
    def unused_tensors(sizes: dict) -> tuple:
        return () if sizes.get("v_mix") else ("vmix",)

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "o":
            self.load_o(w)
        elif key == "rel":
            self.bias.data.copy_(w.to(self.bias.device).float()[self.buckets].T)
        elif key == "vmix":
            self.value_share = float(w)
        else:
            self.in_proj.load_part(key, w)

    def state_spec(self, dtype):
        return []

    def workspace_size(self) -> tuple:
        return self.heads, self.cache_dim

    def forward(self, h):
        ctx = get_forward_context()
        md, p, T = ctx.attn, self.in_proj, h.shape[0]
        kv_cache = ctx.kv_caches[self.layer_idx]
        y = p(h)
        v_out = v_in = None
        if self.shares_values:
            if self.first_of_sharing:
                v_out = md.extras[self.VALUES] = torch.empty(T, self.kv_heads * self.vdim, dtype=h.dtype, device=h.device)
            else:
                v_in = md.extras[self.VALUES]
        q = ops.attn_prep_cache(p.slice(y, "q"), p.slice(y, "k"), p.slice(y, "v"), kv_cache, md.slot_mapping, md.positions,
                                self.heads, self.kv_heads, self.eps, self.temperature, v_out, v_in, self.value_share)
        o = ops.paged_attention(
            q, kv_cache, md.block_tables, md.seq_lens, md.query_start_loc, self.scale, md.max_query_len, md.max_seq_len,
            None, None, md.seq_lens_cpu, md.query_start_loc_cpu, workspace=md.workspace, num_decodes=md.num_decodes,
            decode_query_len=1 + md.num_spec_tokens, num_decode_tokens=md.num_decode_tokens, stable_metadata=True,
            bias=self.bias, gate=p.slice(y, "g"))
        return [(self.o(o.reshape(T, self.heads * self.cache_dim)), 1.0)]


class SigmoidAttention(WindowAttention):
    """Causal attention without a softmax: a visible key counts with ``sigmoid(score + b)`` (a learned ``b`` per head), not
    normalised over the keys.  q, k and v have biases; q and k heads are RMS-normed with a weight that the heads share, then
    rotated on their first columns.  ``mask``: a position sees the last ``size`` ones up to itself and the first ``keep_first``."""

    has_state = False
    cache_block = 64                        # tokens per cache block that the tensor-core kernels take
    served_heads = (128,)

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        pass

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        m, mask, rot = sizes, sizes.get("mask") or {}, sizes.get("rot")
        window = mask.get("size")
        super().__init__(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"],
                         None if window is None else int(window), None, eps, dtype, device)
        self.layer_idx, self.keep_first = layer_idx, int(mask.get("keep_first") or 0)
        self.in_proj = FusedProjection(width, self.proj_sizes(), dtype, device, bias=True)
        self.q_norm, self.k_norm = (param(self.dim, dtype=torch.float32, device=device) for _ in range(2))
        self.bias = param(self.heads, 1, dtype=torch.float32, device=device)
        self.rotary_key = None
        if rot is not None:
            self.rotary_key = (int(rot.get("dims", self.dim)), float(rot["base"]))
            if self.rotary_key[0] > self.dim or self.rotary_key[0] % 2:
                raise ValueError(f"{self.rotary_key[0]} rotated columns in heads of {self.dim}")
            self.register_buffer("turns", ops.position_turns(*self.rotary_key).to(device))

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        H, G, D, V = (sizes[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        return {"q": (H * D, width), "q.b": (H * D,), "k": (G * D, width), "k.b": (G * D,), "v": (G * V, width), "v.b": (G * V,),
                "q.norm": (D,), "k.norm": (D,), "pb": (H,), "o": (width, H * V)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "o":
            self.load_o(w)
        elif key == "pb":
            self.bias.data[:, 0].copy_(w)
        elif key.endswith(".norm"):
            (self.q_norm if key == "q.norm" else self.k_norm).data.copy_(w)
        elif key.endswith(".b"):
            self.in_proj.load_bias(key.removesuffix(".b"), w)
        else:
            self.in_proj.load_part(key, w)

    def state_spec(self, dtype):
        return []

    def workspace_size(self) -> tuple:
        return self.heads, self.cache_dim

    def forward(self, h):
        ctx = get_forward_context()
        md, p, T = ctx.attn, self.in_proj, h.shape[0]
        kv_cache = ctx.kv_caches[self.layer_idx]
        kv_cache = kv_cache[0] if isinstance(kv_cache, tuple) else kv_cache
        table = None if self.rotary_key is None else md.extras["rotary"][self.rotary_key]
        y = p(h)
        q = ops.attn_prep_cache(p.slice(y, "q"), p.slice(y, "k"), p.slice(y, "v"), kv_cache, md.slot_mapping, md.positions,
                                self.heads, self.kv_heads, self.eps, v_norm=False, qk_norm=(self.q_norm, self.k_norm),
                                table=table)
        span = md.max_seq_len if self.window is None else min(md.max_seq_len, self.window + self.keep_first + 127)
        o = ops.paged_attention(
            q, kv_cache, md.block_tables, md.seq_lens, md.query_start_loc, self.scale, md.max_query_len, span, self.window,
            None, md.seq_lens_cpu, md.query_start_loc_cpu, workspace=md.workspace, num_decodes=md.num_decodes,
            decode_query_len=1 + md.num_spec_tokens, num_decode_tokens=md.num_decode_tokens, stable_metadata=True,
            bias=self.bias, keep_first=self.keep_first, sigmoid=True)
        return [(self.o(o.reshape(T, self.heads * self.cache_dim)), 1.0)]


def link_shared_values(mixers) -> None:
    """The first of the layers that share values is their source; the others need values of the same shape."""
    sharing = [m for m in mixers if getattr(m, "shares_values", False)]
    for i, m in enumerate(sharing):
        m.first_of_sharing = i == 0
        if (m.kv_heads, m.vdim) != (sharing[0].kv_heads, sharing[0].vdim):
            raise ValueError("layers that share values have different numbers or sizes of value heads")


class LightningAttention(nn.Module):
    """``S <- decay_h S + k v^T``, ``o = S^T q`` with SiLU on q, k and v; the concatenated heads are RMS-normed together,
    multiplied by ``sigmoid`` of the gate projection and projected."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay, eps: float, dtype, device):
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decay constants for {heads} heads")
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.register_buffer("decay", torch.tensor([float(d) for d in decay], dtype=torch.float32, device=device))
        self.norm = nn.Module()
        self.norm.weight = param(heads * vdim, dtype=torch.float32, device=device)
        self.o = output_projection(align(heads * vdim), width, dtype, device)

    def proj_sizes(self) -> dict:
        n = self.heads * self.vdim
        return {"q": self.heads * self.dim, "k": self.heads * self.dim, "v": n, "g": n}

    def state_spec(self):
        return [((self.heads, self.vdim, round_up(self.dim, 4)), torch.float32)]

    def load_o(self, w: torch.Tensor):
        self.o.weight.data[:w.shape[0], :w.shape[1]].copy_(w)

    def forward(self, q, k, v, g, state, md):
        T, H = q.shape[0], self.heads
        o = ops.fixed_decay_attention(_heads(q, H, self.dim), _heads(k, H, self.dim), _heads(v, H, self.vdim), self.decay,
                                      state, md.query_start_loc, md.state_indices, md.has_initial_state, md.max_query_len,
                                      md.num_decodes)
        n = H * self.vdim
        y = ops.gated_group_rmsnorm(o.reshape(T, n), g, self.norm.weight, self.eps, _rows(T, n, q.dtype, q.device))
        return self.o(y)


def _heads(x: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """``[T, heads * dim]`` column slice -> ``[T, heads, dim]`` view."""
    return x.as_strided((x.shape[0], heads, dim), (x.stride(0), dim, 1))


class ParallelMixer(nn.Module):
    """Windowed softmax attention and lightning attention on the same input, added with constant scales."""

    has_state = True
    cache_block = None          # any cache block size
    sink_score = 0.0            # one unit in the softmax denominator

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        pass

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        super().__init__()
        a, b = sizes["left"], sizes["right"]
        self.layer_idx = layer_idx
        mask = a.get("mask") or {}
        window = mask.get("size")
        self.left = WindowAttention(width, a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"],
                                    None if window is None else int(window), self.sink_score, eps, dtype, device)
        self.right = LightningAttention(width, b["heads"], b["dim"], b["vdim"], b["decay"], eps, dtype, device)
        self.scales = (float(sizes["left_scale"]), float(sizes["right_scale"]))
        self.in_proj = FusedProjection(width, {**{f"left.{k}": n for k, n in self.left.proj_sizes().items()},
                                               **{f"right.{k}": n for k, n in self.right.proj_sizes().items()}}, dtype, device)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        a, b = sizes["left"], sizes["right"]
        n = b["heads"] * b["vdim"]
        return {"left.q": (a["heads"] * a["dim"], width), "left.k": (a["kv_heads"] * a["dim"], width),
                "left.v": (a["kv_heads"] * a["vdim"], width), "left.o": (width, a["heads"] * a["vdim"]),
                "right.q": (b["heads"] * b["dim"], width), "right.k": (b["heads"] * b["dim"], width), "right.v": (n, width),
                "right.g": (n, width), "right.o": (width, n), "right.norm": (n,)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "left.o":
            self.left.load_o(w)
        elif key == "right.o":
            self.right.load_o(w)
        elif key == "right.norm":
            self.right.norm.weight.data.copy_(w)
        else:
            self.in_proj.load_part(key, w)

    def kv_cache_spec(self, block_size: int, dtype):
        return self.left.kv_cache_spec(block_size, dtype)

    def state_spec(self, dtype):
        return self.right.state_spec()

    def workspace_size(self) -> tuple:
        return self.left.heads, self.left.cache_dim

    def forward(self, h):
        ctx = get_forward_context()
        md = ctx.attn
        kv_cache, state = ctx.kv_caches[self.layer_idx]
        p = self.in_proj
        y = p(h)
        yl = self.left(p.slice(y, "left.q"), p.slice(y, "left.k"), p.slice(y, "left.v"), kv_cache, md)
        yr = self.right(p.slice(y, "right.q"), p.slice(y, "right.k"), p.slice(y, "right.v"), p.slice(y, "right.g"), state, md)
        return [(yl, self.scales[0]), (yr, self.scales[1])]


class ChannelDelta(nn.Module):
    """Gated delta rule with one decay per head and key channel.  ``q | k | v`` pass one short causal convolution and
    SiLU; q and k become unit vectors inside the recurrence kernel; decay and output gate come from low-rank pairs
    whose second factors run as one block-diagonal GEMM."""

    has_state = True
    cache_block = None

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
            if name in shapes:
                sizes[key] = int(shapes[name][0])

    @staticmethod
    def _ranks(sizes: dict) -> tuple:
        return int(sizes.get("decay_rank", sizes["dim"])), int(sizes.get("gate_rank", sizes["vdim"]))

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        super().__init__()
        self.layer_idx, self.eps = layer_idx, eps
        self.heads, self.kv_heads, self.dim, self.vdim = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} value heads do not divide over {self.kv_heads} key heads")
        self.taps = int(sizes["conv"])
        ra, rg = self._ranks(sizes)
        H, nk, nv = self.heads, self.kv_heads * self.dim, self.heads * self.vdim
        self.in_proj = FusedProjection(width, {"q": nk, "k": nk, "v": nv, "a1": ra, "g1": rg, "b": H}, dtype, device)
        self.conv_dim = self.in_proj.parts["v"][0] + align(nv)          # q | k | v with their padding
        self.conv_weight = param(self.conv_dim, self.taps, dtype=dtype, device=device)
        self.conv_weight.data.zero_()
        self.low = (self.in_proj.parts["a1"][0], align(ra) + align(rg))  # columns of a1 | g1
        self.rank_a, self.n_decay = align(ra), align(H * self.dim)
        self.up = ReplicatedLinear(self.low[1], self.n_decay + align(nv), dtype=dtype, device=device)
        self.up.weight.data.zero_()
        self.A_log = param(H, dtype=torch.float32, device=device)
        self.dt_bias = param(H * self.dim, dtype=torch.float32, device=device)
        self.norm = nn.Module()
        self.norm.weight = param(self.vdim, dtype=torch.float32, device=device)
        self.o = output_projection(align(nv), width, dtype, device)

    @classmethod
    def tensor_shapes(cls, sizes: dict, width: int) -> dict:
        H, nk, nv = sizes["heads"], sizes["kv_heads"] * sizes["dim"], sizes["heads"] * sizes["vdim"]
        ra, rg = cls._ranks(sizes)
        W = sizes["conv"]
        return {"q": (nk, width), "q.conv": (nk, W), "k": (nk, width), "k.conv": (nk, W), "v": (nv, width),
                "v.conv": (nv, W), "b": (H, width), "A_log": (H,), "norm": (sizes["vdim"],), "a1": (ra, width),
                "a2": (H * sizes["dim"], ra), "dt_bias": (H * sizes["dim"],), "g1": (rg, width), "g2": (nv, rg),
                "o": (width, nv)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key.endswith(".conv"):
            off, n = self.in_proj.parts[key.removesuffix(".conv")]
            self.conv_weight.data[off:off + n].copy_(w)
        elif key == "a2":
            self.up.weight.data[:w.shape[0], :w.shape[1]].copy_(w)
        elif key == "g2":
            self.up.weight.data[self.n_decay:self.n_decay + w.shape[0], self.rank_a:self.rank_a + w.shape[1]].copy_(w)
        elif key in ("A_log", "dt_bias"):
            getattr(self, key).data.copy_(w)
        elif key == "norm":
            self.norm.weight.data.copy_(w)
        elif key == "o":
            self.o.weight.data[:w.shape[0], :w.shape[1]].copy_(w)
        else:
            self.in_proj.load_part(key, w)

    def kv_cache_spec(self, block_size: int, dtype):
        return None

    def state_spec(self, dtype):
        return [((self.taps - 1, self.conv_dim), dtype),
                ((self.heads, self.vdim, round_up(self.dim, 4)), torch.float32)]

    def workspace_size(self) -> tuple:
        return 0, 0

    def forward(self, h):
        ctx = get_forward_context()
        md = ctx.attn
        conv_state, state = ctx.kv_caches[self.layer_idx]
        T, H, p = h.shape[0], self.heads, self.in_proj
        y = p(h)
        if md.max_query_len == 1:
            x = ops.causal_conv1d_update(y[:, :self.conv_dim], conv_state, self.conv_weight, None, md.state_indices, True,
                                         md.has_initial_state)
        else:
            x = ops.causal_conv1d_fn(y[:, :self.conv_dim], self.conv_weight, None, md.query_start_loc, conv_state,
                                     md.state_indices, md.has_initial_state, True)
        up = self.up(y[:, self.low[0]:self.low[0] + self.low[1]])
        q, k, v = (_heads(p.slice(x, n), m, d) for n, m, d in
                   (("q", self.kv_heads, self.dim), ("k", self.kv_heads, self.dim), ("v", H, self.vdim)))
        o = ops.channel_delta_rule(q, k, v, up[:, :H * self.dim], p.slice(y, "b"), self.A_log, self.dt_bias, state,
                                   md.query_start_loc, md.state_indices, md.has_initial_state, self.dim ** -0.5,
                                   UNIT_NORM_EPS, md.max_query_len, md.num_decodes)
        n = H * self.vdim
        z = ops.gated_group_rmsnorm(o.reshape(T, n), up[:, self.n_decay:self.n_decay + n], self.norm.weight, self.eps,
                                    _rows(T, n, h.dtype, h.device))
        return [(self.o(z), 1.0)]


class GatedWriteAttention(nn.Module):
    """HGRN2: ``S <- diag(f) S + (1 - f) v^T``, ``o = S^T silu(q)``; the forget gate ``f = l + (1 - l) sigmoid(W_f h + b)`` per
    head and channel has a lower bound l.  Every head's output is RMS-normed with a weight that the heads share."""

    has_state = True
    cache_block = None

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        pass

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        super().__init__()
        self.layer_idx, self.eps = layer_idx, eps
        self.heads, self.dim, self.vdim = sizes["heads"], sizes["dim"], sizes["vdim"]
        n, nv = self.heads * self.dim, self.heads * self.vdim
        self.in_proj = FusedProjection(width, {"q": n, "f": n, "v": nv}, dtype, device)
        self.f_bias, self.lower = (param(n, dtype=torch.float32, device=device) for _ in range(2))
        self.norm = nn.Module()
        self.norm.weight = param(self.vdim, dtype=torch.float32, device=device)
        self.o = output_projection(align(nv), width, dtype, device)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        n, nv = sizes["heads"] * sizes["dim"], sizes["heads"] * sizes["vdim"]
        return {"q": (n, width), "f": (n, width), "f.b": (n,), "lower": (n,), "v": (nv, width), "norm": (sizes["vdim"],),
                "o": (width, nv)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "o":
            self.o.weight.data[:w.shape[0], :w.shape[1]].copy_(w)
        elif key in ("f.b", "lower", "norm"):
            {"f.b": self.f_bias, "lower": self.lower, "norm": self.norm.weight}[key].data.copy_(w)
        else:
            self.in_proj.load_part(key, w)

    def kv_cache_spec(self, block_size: int, dtype):
        return None

    def state_spec(self, dtype):
        return [((self.heads, self.vdim, round_up(self.dim, 4)), torch.float32)]

    def workspace_size(self) -> tuple:
        return 0, 0

    def forward(self, h):
        ctx = get_forward_context()
        md, p, T, H = ctx.attn, self.in_proj, h.shape[0], self.heads
        state, = ctx.kv_caches[self.layer_idx]
        y = p(h)
        o = ops.gated_write_attention(_heads(p.slice(y, "q"), H, self.dim), _heads(p.slice(y, "v"), H, self.vdim),
                                      p.slice(y, "f"), self.f_bias, self.lower, state, md.query_start_loc, md.state_indices,
                                      md.has_initial_state, md.max_query_len, md.num_decodes)
        n = H * self.vdim
        z = ops.gated_group_rmsnorm(o.reshape(T, n), None, self.norm.weight, self.eps, _rows(T, n, h.dtype, h.device))
        return [(self.o(z), 1.0)]


class MinGRU(nn.Module):
    """``S <- (1 - z) S + z c`` element by element with ``z = sigmoid(W_z h + b_z)`` and, for ``u = W_x h + b_x``, the candidate
    ``c = u + 1/2`` where ``u >= 0`` and ``sigmoid(u)`` elsewhere; output ``W_o (S * silu(W_g h))``."""

    has_state = True
    cache_block = None

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        pass

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        super().__init__()
        self.layer_idx, self.size = layer_idx, int(sizes["width"])
        self.in_proj = FusedProjection(width, {"z": self.size, "x": self.size, "g": self.size}, dtype, device)
        self.z_bias, self.x_bias = (param(self.size, dtype=torch.float32, device=device) for _ in range(2))
        self.o = output_projection(align(self.size), width, dtype, device)

    @staticmethod
    def tensor_shapes(sizes: dict, width: int) -> dict:
        n = int(sizes["width"])
        return {"z": (n, width), "z.b": (n,), "x": (n, width), "x.b": (n,), "g": (n, width), "o": (width, n)}

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "o":
            self.o.weight.data[:w.shape[0], :w.shape[1]].copy_(w)
        elif key in ("z.b", "x.b"):
            (self.z_bias if key == "z.b" else self.x_bias).data.copy_(w)
        else:
            self.in_proj.load_part(key, w)

    def kv_cache_spec(self, block_size: int, dtype):
        return None

    def state_spec(self, dtype):
        return [((self.size,), torch.float32)]

    def workspace_size(self) -> tuple:
        return 0, 0

    def forward(self, h):
        ctx = get_forward_context()
        md, p = ctx.attn, self.in_proj
        y = p(h)
        out = ops.gated_blend(p.slice(y, "z"), p.slice(y, "x"), p.slice(y, "g"), self.z_bias, self.x_bias,
                              ctx.kv_caches[self.layer_idx][0], md.query_start_loc, md.state_indices, md.has_initial_state,
                              _rows(h.shape[0], self.size, h.dtype, h.device), md.max_query_len, md.num_decodes)
        return [(self.o(out), 1.0)]


class LatentAttention(nn.Module):
    """Multi-head attention over one latent row per token.  Queries come through their own latent; keys and values are
    per-head products of the cached latent, plus one rotated key part that all heads share.  Optional sliding ``window``,
    a learned sink per head, the output of every head times ``sigmoid`` of its gate.

    Single tokens attend in the absorbed form (the query moves into the latent space, ``W_uk`` never meets the cache);
    prompt portions in the up-projected form: the cached rows that the portion can see and its own ones are gathered
    contiguously, up-projected by one GEMM and attended by the prefill kernel.  16-bit models up to the kernels' head sizes
    run both on the tensor cores, with every part zero-padded to them; other sizes and fp32 take the absorbed form on the
    CUDA cores throughout."""

    has_state = False
    cache_block = 64                       # tokens per cache block that the decode kernel takes
    TENSOR_CORE = (128, 64, 128, 512)      # unrotated and rotated query / key dims, value dims, latent
    KV_BYTES = 512 << 20                   # bound of the up-projected keys and values of one attention call

    @staticmethod
    def complete_sizes(sizes: dict, shapes: dict) -> None:
        if "dq" in shapes:
            sizes["q_rank"] = int(shapes["dq"][0])

    @staticmethod
    def _sizes(m: dict) -> tuple:
        return m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]

    def __init__(self, width: int, sizes: dict, layer_idx: int, eps: float, dtype, device):
        super().__init__()
        H, D, R, V, C, Q = self._sizes(sizes)
        self.layer_idx, self.eps, self.scale = layer_idx, eps, float(sizes["scale"])
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank, self.q_rank = H, D, R, V, C, Q
        rot = sizes["rot"]
        self.rotary_key = (int(rot.get("dims", R)), float(rot["base"]))
        if self.rotary_key[0] > R or self.rotary_key[0] % 2:
            raise ValueError(f"{self.rotary_key[0]} rotated columns in a rotated part of {R}")
        window = (sizes.get("mask") or {}).get("size")
        self.window = None if window is None else int(window)
        self.tensor_cores = (torch.device(device).type == "cuda" and dtype in (torch.bfloat16, torch.float16)
                             and all(n <= m for n, m in zip((D, R, V, C), self.TENSOR_CORE)))
        # sizes as the kernels see them, and the place of the rotated key part in a cache row
        self.D, self.R, self.V, self.C = self.TENSOR_CORE if self.tensor_cores else (D, R, V, align(C))
        self.row = align(self.C + self.R)
        self.in_proj = FusedProjection(width, {"dq": Q, "dkv": C + R, "g": H}, dtype, device)
        self.uq = ReplicatedLinear(align(Q), align(H * (self.D + self.R)), dtype=dtype, device=device)
        self.up = ReplicatedLinear(self.C, H * (self.D + self.V), dtype=dtype, device=device)      # per head keys | values
        for lin in (self.uq, self.up):
            lin.weight.data.zero_()
        self.o = output_projection(align(H * self.V), width, dtype, device)
        self.q_norm, self.kv_norm, self.sinks = (param(n, dtype=torch.float32, device=device) for n in (Q, C, H))
        self.register_buffer("turns", ops.position_turns(*self.rotary_key).to(device))

    @classmethod
    def tensor_shapes(cls, sizes: dict, width: int) -> dict:
        H, D, R, V, C, Q = cls._sizes(sizes)
        return {"dq": (Q, width), "dq.norm": (Q,), "uq": (H * (D + R), Q), "dkv": (C + R, width), "dkv.norm": (C,),
                "uk": (H * D, C), "uv": (H * V, C), "sink": (H,), "g": (H, width), "o": (width, H * V)}

    def _up(self) -> tuple:
        """``w_uk [H, D, C]`` and ``w_uv [H, V, C]``, views of the up-projection's weight."""
        w = self.up.weight.view(self.heads, self.D + self.V, self.C)
        return w[:, :self.D], w[:, self.D:]

    def load_tensor(self, key: str, w: torch.Tensor):
        H = self.heads
        if key in ("dq", "dkv", "g"):
            self.in_proj.load_part(key, w)
        elif key == "uq":
            q, g = w.reshape(H, self.dim + self.rot_dim, -1), self.uq.weight.data[:H * (self.D + self.R)].view(H, self.D + self.R, -1)
            g[:, :self.dim, :self.q_rank].copy_(q[:, :self.dim])
            g[:, self.D:self.D + self.rot_dim, :self.q_rank].copy_(q[:, self.dim:])
        elif key in ("uk", "uv"):
            n = self.dim if key == "uk" else self.vdim
            self._up()[key == "uv"].data[:, :n, :self.rank].copy_(w.reshape(H, n, -1))
        elif key == "o":
            g = self.o.weight.data[:, :H * self.V].view(self.o.out_features, H, self.V)
            g[:w.shape[0], :, :self.vdim].copy_(w.reshape(w.shape[0], H, self.vdim))
        else:
            {"dq.norm": self.q_norm, "dkv.norm": self.kv_norm, "sink": self.sinks}[key].data.copy_(w)

    def kv_cache_spec(self, block_size: int, dtype):
        return ((block_size, self.row), dtype)

    def state_spec(self, dtype):
        return []

    def workspace_size(self) -> tuple:
        return 0, 0

    def _portions(self, md, first: int) -> list:
        """Attention calls of the prompt portions (requests ``first ..``): runs of requests whose visible rows, cached and
        new, fit the bound on up-projected keys and values.  The same for every layer with this window and row size."""
        key = ("latent_portions", self.window, self.heads)
        if key not in md.extras:
            lens = md.seq_lens_cpu.tolist()
            qsl = md.query_start_loc_cpu.tolist()
            limit = max(1, self.KV_BYTES // (self.heads * (self.D + self.V) * 2))
            calls, lo, rows = [], first, []
            for b in range(first, md.num_reqs + 1):
                n = 0
                if b < md.num_reqs:
                    q = qsl[b + 1] - qsl[b]
                    n = lens[b] if self.window is None else min(lens[b], q + self.window - 1)
                if rows and (b == md.num_reqs or sum(rows) + n > limit):
                    starts = [sum(rows[:i]) for i in range(len(rows))]
                    both = torch.tensor([starts, rows], dtype=torch.int32).to(md.seq_lens.device, non_blocking=True)
                    calls.append((lo, b, both[0], both[1], sum(rows), max(rows),
                                  max(qsl[i + 1] - qsl[i] for i in range(lo, b))))
                    lo, rows = b, []
                rows.append(n)
            md.extras[key] = calls
        return md.extras[key]

    def forward(self, h):
        ctx = get_forward_context()
        md = ctx.attn
        cache = ctx.kv_caches[self.layer_idx]
        cache = cache[0] if isinstance(cache, tuple) else cache
        T, H, p = h.shape[0], self.heads, self.in_proj
        table = md.extras["rotary"][self.rotary_key]
        y = p(h)
        g = p.slice(y, "g")
        cq = ops.latent_prep(p.slice(y, "dq"), p.slice(y, "dkv"), self.q_norm, self.kv_norm, table, cache, md.slot_mapping,
                             self.C, self.uq.in_features, self.eps)
        q = self.uq(cq)[:, :H * (self.D + self.R)].contiguous().view(T, H, self.D + self.R)
        out = _rows(T, H * self.V, h.dtype, h.device)
        nd = md.num_decodes if self.tensor_cores else md.num_reqs
        nt = md.num_decode_tokens if self.tensor_cores else T
        if nd:
            w_uk, w_uv = self._up()
            qa = ops.absorb_query(q[:nt], w_uk, table[:nt], self.C, self.row)
            cpu = (md.seq_lens_cpu[:nd], md.query_start_loc_cpu[:nd + 1]) if md.seq_lens_cpu is not None else (None, None)
            o = ops.mla_attention(qa, cache, md.block_tables[:nd], md.seq_lens[:nd], md.query_start_loc[:nd + 1], self.scale,
                                  self.C, 1 + md.num_spec_tokens if self.tensor_cores else md.max_query_len, md.max_seq_len,
                                  *cpu, stable_metadata=True, window=self.window, sinks=self.sinks)
            ops.expand_value(o, w_uv, g[:nt], out[:nt])
        if nd < md.num_reqs:
            ops.rotate_heads(q[nt:], table[nt:], self.D)
            heads = out.view(T, H, self.V)
            for lo, hi, starts, lens, total, longest, max_q in self._portions(md, nd):
                rows = ops.gather_window(cache, md.block_tables[lo:hi], md.seq_lens[lo:hi], starts, lens, total, longest)
                ops.mla_prefill_attention(q, self.up(rows[:, :self.C]), rows[:, self.C:], starts, lens,
                                          md.query_start_loc[lo:hi + 1], True, self.scale, max_q, out=heads,
                                          window=self.window, sinks=self.sinks, gate=g, want_lse=False)
        return [(self.o(out), 1.0)]


def rotary_tables(mixers, md) -> None:
    """cos / sin of the step's positions for every rotation among ``mixers``: made once per step, before the layers."""
    md.extras["rotary"] = {}
    for m in mixers:
        key = getattr(m, "rotary_key", None)
        if key is not None and key not in md.extras["rotary"]:
            md.extras["rotary"][key] = ops.rotary_table(md.positions, m.turns)


MIXERS = {"attention": DistanceBiasAttention, "channel_delta": ChannelDelta, "hgrn2": GatedWriteAttention,
          "latent_attention": LatentAttention, "mingru": MinGRU, "parallel": ParallelMixer, "sigmoid_attention": SigmoidAttention}
