"""Bolopel: decoder-only model whose layers are listed one by one in its configuration (``models/layer_list.py``), with an
fp32 residual stream normalised on the sublayers' outputs.

    stream = LayerNorm(embed[token] + sinusoid(position))
    per layer:  stream += LayerNorm(mixer(stream));  stream += LayerNorm(W_down(silu(W_gate s) * W_up s))
    logits = head . LayerNorm(stream)

The norm kernels write the stream's copy for the GEMMs beside it.

Checkpoint names: ``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.mlp.{gate,up,down}``,
``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..attention.metadata import get_forward_context
from ..config import LayerSpec, ModelConfig
from .layer_list import LayerListForCausalLM, ListedLayer, NormWeight

POSITION_BASE = 10000.0


class BolopelDecoderLayer(ListedLayer):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__(cfg, layer_idx, dtype, device)
        self.mixer_norm = NormWeight(cfg.hidden_size, device)
        self.mlp_norm = None if self.mlp is None else NormWeight(cfg.hidden_size, device)

    @classmethod
    def tensor_shapes(cls, spec: LayerSpec, width: int, act: str) -> dict:
        norms = ("norm1",) if spec.mlp is None else ("norm1", "norm2")
        return {**{n: (width,) for n in norms}, **super().tensor_shapes(spec, width, act)}

    def forward(self, x, h):
        h = ops.layernorm_residual(x, self.dtype, self.mixer(h), self.mixer_norm.weight, self.eps)
        if self.mlp is not None:
            h = ops.layernorm_residual(x, self.dtype, [(self.mlp(h), 1.0)], self.mlp_norm.weight, self.eps)
        return h

    def load_tensor(self, key: str, w: torch.Tensor):
        if key in ("norm1", "norm2"):
            (self.mixer_norm if key == "norm1" else self.mlp_norm).weight.data.copy_(w)
        else:
            super().load_tensor(key, w)


class BolopelForCausalLM(LayerListForCausalLM):
    layer_cls = BolopelDecoderLayer

    def __init__(self, cfg: ModelConfig, device="cpu", dtype: Optional[torch.dtype] = None):
        super().__init__(cfg, device, dtype)
        self.embed_norm = NormWeight(self.width, device)
        self.register_buffer("turns", ops.position_turns(self.width, POSITION_BASE).to(device))

    def forward(self, input_ids, hidden=None, residual=None):
        md = get_forward_context().attn
        x, h = ops.embed_positions_layernorm(input_ids, md.positions, self.embed_tokens.weight, self.turns,
                                             self.embed_norm.weight, self.eps)
        for i in range(self.last_layer):
            h = self.layers[str(i)](x, h)
            if self.post_layer_hook is not None:
                self.post_layer_hook(i, h, x[:, :self.width])
        return ops.layernorm_residual(x, self.dtype, [], self.norm.weight, self.eps), None

    def outer_tensor_shapes(self) -> dict:
        return {**super().outer_tensor_shapes(), "embed.norm": (self.width,)}

    def load_outer_tensor(self, name: str, w: torch.Tensor):
        if name == "embed.norm":
            self.embed_norm.weight.data.copy_(w)
        else:
            super().load_outer_tensor(name, w)
