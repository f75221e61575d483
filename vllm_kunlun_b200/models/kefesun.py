"""Kefesun: decoder-only model whose layers are listed one by one (``models/layer_list.py``): windowed sigmoid attention or
minGRU, then routed experts (or nothing), each sublayer reading the stream through a short causal convolution and normed on its
output; the output head is the embedding table.

    x = scale * embed[token]
    per layer:  x += Norm1(mixer(x + conv1(x)));  x += Norm2(experts(x + conv2(x)))        Norm = LayerNorm without a bias
    logits = embed . Norm(x)

The stream is fp32.  A sublayer's end - the experts' weighted sum, its norm, the residual sum - and the next one's convolution are
one kernel for single tokens, two for prompt portions (``ops.postnorm_input_conv``).  Per request and sublayer the model keeps the
last ``taps - 1`` rows of the stream (fp32).

Checkpoint names: ``embed``, ``l<i>.canon1``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.canon2``, ``l<i>.norm2``, ``l<i>.mlp.*``,
``final.norm``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..attention.metadata import get_forward_context
from ..config import LayerSpec, ModelConfig
from .layer_list import LayerListForCausalLM, ListedLayer, NormWeight
from .layers import param
from .mixers import rotary_tables

MAX_TAPS = 16           # of the convolution kernels


class KefesunDecoderLayer(ListedLayer):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__(cfg, layer_idx, dtype, device)
        self.layer_idx, self.taps = layer_idx, cfg.input_conv_taps
        self.sublayers = 1 if self.mlp is None else 2
        for k in range(1, self.sublayers + 1):
            conv = param(self.taps, self.ld, dtype=torch.float32, device=device)
            conv.data.zero_()
            self.register_parameter(f"conv{k}", conv)
            setattr(self, f"norm{k}", NormWeight(cfg.hidden_size, device))

    def outer_shapes(self, width: int) -> dict:
        """Name -> shape of the layer's tensors outside its sublayers."""
        return {n: s for k in range(1, self.sublayers + 1) for n, s in ((f"norm{k}", (width,)), (f"canon{k}", (width, self.taps)))}

    @classmethod
    def unused_tensors(cls, spec: LayerSpec) -> tuple:
        return super().unused_tensors(spec) + (("norm2", "canon2") if spec.mlp is None else ())

    def state_spec(self, dtype) -> list:
        rows = [((self.taps - 1, self.ld), torch.float32)] * self.sublayers if self.taps > 1 else []
        return super().state_spec(dtype) + rows

    def conv(self, k: int) -> tuple:
        """``(taps, state)`` of sublayer k's convolution; the states are the layer's last cache tensors."""
        state = None if self.taps < 2 else get_forward_context().kv_caches[self.layer_idx][k - 1 - self.sublayers]
        return getattr(self, f"conv{k}"), state

    def mix(self, h):
        (y, _), = self.mixer(h)
        return y

    def steps(self) -> list:
        """``(sublayer, its convolution, its norm weight)`` in order."""
        out = [(self.mix, self.conv(1), self.norm1.weight)]
        return out if self.mlp is None else out + [(self.mlp, self.conv(2), self.norm2.weight)]

    def load_tensor(self, key: str, w: torch.Tensor):
        if key in ("norm1", "norm2"):
            getattr(self, key).weight.data.copy_(w)
        elif key in ("canon1", "canon2"):
            getattr(self, f"conv{key[-1]}").data[:, :w.shape[0]].copy_(w.T)
        else:
            super().load_tensor(key, w)


class KefesunForCausalLM(LayerListForCausalLM):
    layer_cls = KefesunDecoderLayer

    def __init__(self, cfg: ModelConfig, device="cpu", dtype: Optional[torch.dtype] = None):
        if not 1 <= cfg.input_conv_taps <= MAX_TAPS:
            raise ValueError(f"{cfg.architecture}: convolutions of {cfg.input_conv_taps} taps; 1 to {MAX_TAPS} are served")
        super().__init__(cfg, device, dtype)

    def tensor_shapes(self) -> dict:
        out = super().tensor_shapes()
        for i in range(self.last_layer):
            out.update({f"l{i}.{n}": s for n, s in self.layers[str(i)].outer_shapes(self.width).items()})
        return out

    def forward(self, input_ids, hidden=None, residual=None):
        md = get_forward_context().attn
        layers = [self.layers[str(i)] for i in range(self.last_layer)]
        rotary_tables([layer.mixer for layer in layers], md)
        steps = [(i, *s) for i, layer in enumerate(layers) for s in layer.steps()]
        x, h = ops.embed_input_conv(input_ids, self.embed_tokens.weight, self.cfg.embedding_scale, steps[0][2], md)
        for (i, sublayer, _, weight), after in zip(steps, steps[1:] + [None]):
            y = sublayer(h)
            if after is None:
                h = ops.postnorm_input_conv(x, y, weight, self.eps, self.dtype, final_weight=self.norm.weight)
            else:
                h = ops.postnorm_input_conv(x, y, weight, self.eps, self.dtype, after[2], md)
            if self.post_layer_hook is not None and (after is None or after[0] != i):
                self.post_layer_hook(i, h, x[:, :self.width])
        return h, None
