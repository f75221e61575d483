"""Seturax: decoder-only model with windowed latent attention beside the feed-forward in every layer, each result gated, and
an embedding of token pairs.

    x = scale * embed[token] + bigram[row(previous token, token)]
    per layer:  h = LayerNorm(x);  s = h + (h of the previous token - h) * shift
                x += sigmoid(RG1 h + b1) * mixer(s) + sigmoid(RG2 h + b2) * W_down(gelu(W_gate h) * W_up h)
    logits = logit_scale * head . LayerNorm(x)

The stream, the norms, the gates' sigmoid and the shift are fp32.  A layer's sum, the next layer's norm and its shift are
one kernel (``ops.gated_residual_layernorm``); both gates are one GEMM; the logit scale is folded into the final norm's
weight.  Per request the model keeps the last token and, per layer, the last token's h.

Checkpoint names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.shift``, ``l<i>.mix.*``, ``l<i>.mlp.{gate,up,down}``,
``l<i>.rg1``, ``l<i>.rg1.b`` (mixer), ``l<i>.rg2``, ``l<i>.rg2.b`` (feed-forward), ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..attention.metadata import get_forward_context
from ..config import LayerSpec, ModelConfig
from .layer_list import LayerListForCausalLM, ListedLayer, NormWeight
from .layers import ReplicatedLinear, param
from .mixers import padded, rotary_tables

EMBEDDING = "embedding"         # key of the embedding's per-request state among the layers' caches


class SeturaxDecoderLayer(ListedLayer):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__(cfg, layer_idx, dtype, device)
        self.layer_idx = layer_idx
        self.input_norm = NormWeight(cfg.hidden_size, device)
        self.shift = param(self.ld, dtype=torch.float32, device=device)
        self.shift.data.zero_()
        self.num_gates = 1 if self.mlp is None else 2
        self.gates = ReplicatedLinear(self.ld, self.num_gates * self.ld, bias=True, dtype=dtype, device=device)
        self.gates.weight.data.zero_()
        self.gates.bias.data.zero_()

    @classmethod
    def tensor_shapes(cls, spec: LayerSpec, width: int, act: str) -> dict:
        out = {"norm1": (width,), "shift": (width,), **super().tensor_shapes(spec, width, act)}
        for k in range(1 if spec.mlp is None else 2):
            out.update({f"rg{k + 1}": (width, width), f"rg{k + 1}.b": (width,)})
        return out

    @classmethod
    def unused_tensors(cls, spec: LayerSpec) -> tuple:
        return ("rg2", "rg2.b") if spec.mlp is None else ()       # the gate of a feed-forward that is not there

    def state_spec(self, dtype) -> list:
        return super().state_spec(dtype) + [((self.ld,), torch.float32)]

    def shift_args(self):
        """``(mix, state)`` of the token shift for the norm kernels; the state is the layer's last cache tensor."""
        return self.shift, get_forward_context().kv_caches[self.layer_idx][-1]

    def forward(self, h, shifted):
        """Summands of the layer with their raw gates."""
        g = self.gates(h)
        (y, c), *more = self.mixer(shifted)
        if more or c != 1.0:
            y = sum((y2.float() * c2 for y2, c2 in more), y.float() * c).to(y.dtype)
        parts = [(y, g[:, :self.ld])]
        if self.mlp is not None:
            parts.append((self.mlp(h), g[:, self.ld:]))
        return parts

    def load_tensor(self, key: str, w: torch.Tensor):
        if key == "norm1":
            self.input_norm.weight.data.copy_(w)
        elif key == "shift":
            self.shift.data[:w.shape[0]].copy_(w)
        elif key in ("rg1", "rg2"):
            off = self.ld * (key == "rg2")
            self.gates.weight.data[off:off + w.shape[0], :w.shape[1]].copy_(w)
        elif key in ("rg1.b", "rg2.b"):
            off = self.ld * (key == "rg2.b")
            self.gates.bias.data[off:off + w.shape[0]].copy_(w)
        else:
            super().load_tensor(key, w)


class SeturaxForCausalLM(LayerListForCausalLM):
    layer_cls = SeturaxDecoderLayer

    def __init__(self, cfg: ModelConfig, device="cpu", dtype: Optional[torch.dtype] = None):
        super().__init__(cfg, device, dtype)
        if not cfg.bigram:
            raise ValueError(f"{cfg.architecture}: the configuration lacks embedding.bigram")
        self.bigram = param(cfg.bigram["buckets"] + 1, self.ld, dtype=self.dtype, device=device)

    def forward(self, input_ids, hidden=None, residual=None):
        ctx = get_forward_context()
        md, b, layers = ctx.attn, self.cfg.bigram, [self.layers[str(i)] for i in range(self.last_layer)]
        rotary_tables([layer.mixer for layer in layers], md)
        rows = ops.bigram_rows(input_ids, ctx.kv_caches[EMBEDDING][0], md.query_start_loc, md.state_indices,
                               md.has_initial_state, b["mul_prev"], b["mul_cur"], b["buckets"])
        after = layers[1:] + [None]
        x, h, s = ops.embed_stream_layernorm(
            input_ids, self.embed_tokens.weight, self.cfg.embedding_scale, (rows, self.bigram),
            layers[0].input_norm.weight if layers else self.norm.weight, self.eps,
            layers[0].shift_args() if layers else None, md)
        for i, (layer, nxt) in enumerate(zip(layers, after)):
            parts = layer(h, s)
            x, h, s = ops.gated_residual_layernorm(
                x, parts, self.norm.weight if nxt is None else nxt.input_norm.weight, self.eps, self.dtype,
                None if nxt is None else nxt.shift_args(), md,
                keep_stream=nxt is not None or self.post_layer_hook is not None)
            if self.post_layer_hook is not None:
                self.post_layer_hook(i, h, x[:, :self.width])
        return h, None

    def state_cache_spec(self):
        return {**super().state_cache_spec(), EMBEDDING: [((1,), torch.int64)]}

    def outer_tensor_shapes(self) -> dict:
        return {**super().outer_tensor_shapes(), "bigram": (self.cfg.bigram["buckets"] + 1, self.width)}

    def load_outer_tensor(self, name: str, w: torch.Tensor):
        if name == "bigram":
            self.bigram.data.copy_(padded(w, w.shape[0], self.ld))
        elif name == "final.norm":
            self.norm.weight.data.copy_(w.float() * self.cfg.logit_scale)
        else:
            super().load_outer_tensor(name, w)
