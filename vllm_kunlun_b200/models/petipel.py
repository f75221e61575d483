"""Petipel: decoder-only model whose layers are listed one by one (``models/layer_list.py``): softmax attention with a bias by
distance and values shared between layers, or HGRN2; dense polynomial or routed feed-forwards; a norm before and after every
sublayer around an fp32 residual stream.

    x = embed[token]
    per layer:  x += m * Norm(mixer(Norm(x)));  x += m * Norm(feed_forward(Norm(x)))      Norm(z) = z / rms(z) * (1 + w)
    logits = head . Norm(x)

A sublayer's end and the next one's start are one kernel (``ops.sandwich_rmsnorm``), which also sums the experts' rows.  The
weights are kept ready to multiply in fp32: ``1 + w``, and ``m (1 + w)`` behind the sublayers.

Checkpoint names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mlp.*``,
``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config import LayerSpec, ModelConfig
from .layer_list import LayerListForCausalLM, ListedLayer, NormWeight
from .mixers import link_shared_values


class PetipelDecoderLayer(ListedLayer):
    NORMS = {"norm1": "mixer_norm", "norm1b": "mixer_post_norm", "norm2": "mlp_norm", "norm2b": "mlp_post_norm"}

    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__(cfg, layer_idx, dtype, device)
        self.multiplier = cfg.residual_multiplier
        for key, name in self.NORMS.items():
            if self.mlp is not None or key.startswith("norm1"):
                setattr(self, name, NormWeight(cfg.hidden_size, device))

    @classmethod
    def tensor_shapes(cls, spec: LayerSpec, width: int, act: str) -> dict:
        norms = [k for k in cls.NORMS if spec.mlp is not None or k.startswith("norm1")]
        return {**{k: (width,) for k in norms}, **super().tensor_shapes(spec, width, act)}

    @classmethod
    def unused_tensors(cls, spec: LayerSpec) -> tuple:
        return super().unused_tensors(spec) + (("norm2", "norm2b") if spec.mlp is None else ())

    def forward(self, x, h, next_norm):
        """``x``: the stream, updated in place; ``h``: its norm for the mixer.  Returns the stream under ``next_norm``."""
        (y, _), = self.mixer(h)
        if self.mlp is None:
            return ops.sandwich_rmsnorm(x, y, self.mixer_post_norm.weight, next_norm.weight, self.eps)
        h = ops.sandwich_rmsnorm(x, y, self.mixer_post_norm.weight, self.mlp_norm.weight, self.eps)
        return ops.sandwich_rmsnorm(x, self.mlp(h), self.mlp_post_norm.weight, next_norm.weight, self.eps)

    def load_tensor(self, key: str, w: torch.Tensor):
        if key in self.NORMS:
            scale = self.multiplier if key.endswith("b") else 1.0
            getattr(self, self.NORMS[key]).weight.data.copy_((1.0 + w.float()) * scale)
        else:
            super().load_tensor(key, w)


class PetipelForCausalLM(LayerListForCausalLM):
    layer_cls = PetipelDecoderLayer
    unit_norm_init = 0.0

    def __init__(self, cfg: ModelConfig, device="cpu", dtype: Optional[torch.dtype] = None):
        super().__init__(cfg, device, dtype)
        link_shared_values([self.layers[str(i)].mixer for i in range(self.last_layer)])

    def forward(self, input_ids, hidden=None, residual=None):
        layers = [self.layers[str(i)] for i in range(self.last_layer)]
        norms = [layer.mixer_norm for layer in layers] + [self.norm]
        x, h = ops.embed_rmsnorm(input_ids, self.embed_tokens.weight, norms[0].weight, self.eps)
        for i, layer in enumerate(layers):
            h = layer(x, h, norms[i + 1])
            if self.post_layer_hook is not None:
                self.post_layer_hook(i, h, x[:, :self.width])
        return h, None

    def load_outer_tensor(self, name: str, w: torch.Tensor):
        if name == "final.norm":
            self.norm.weight.data.copy_(1.0 + w.float())
        else:
            super().load_outer_tensor(name, w)
