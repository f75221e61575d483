"""Bolopel: decoder-only model whose layers are listed one by one in its configuration (``models/mixers.py``), with an
fp32 residual stream normalised on the sublayers' outputs.

    stream = LayerNorm(embed[token] + sinusoid(position))
    per layer:  stream += LayerNorm(mixer(stream));  stream += LayerNorm(W_down(silu(W_gate s) * W_up s))
    logits = head . LayerNorm(stream)

The stream and every norm are fp32; the GEMMs read the stream's copy in the model's dtype, which the norm kernels write
beside it.  Rows are padded to a multiple of 8 columns (zeros) and the feed-forward width to a multiple of 64 (the fused
gate / up epilogue), so any width runs through the tensor-core GEMMs.

Checkpoint names: ``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.mlp.{gate,up,down}``,
``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from .. import ops
from ..attention.metadata import get_forward_context
from ..config import ModelConfig, round_up
from ..parallel.state import get_state
from .dense import DenseForCausalLM, GatedMLP
from .layers import DTYPES, ParallelLMHead, VocabParallelEmbedding, param
from .mixers import MIXERS, ParallelMixer, align, padded

MLP_TILE = 64
POSITION_BASE = 10000.0


class LayerNormWeight(nn.Module):
    def __init__(self, width: int, device):
        super().__init__()
        self.weight = param(width, dtype=torch.float32, device=device)


class BolopelDecoderLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec = cfg.layer_specs[layer_idx]
        ld = align(cfg.hidden_size)
        self.eps, self.dtype = cfg.rms_norm_eps, dtype
        self.mixer = MIXERS[spec.type](ld, spec.mixer, layer_idx, cfg.rms_norm_eps, dtype, device)
        self.mixer_norm = LayerNormWeight(cfg.hidden_size, device)
        self.mlp = None
        if spec.mlp is not None:
            self.ff = int(spec.mlp["ff"])
            self.mlp = GatedMLP(ld, round_up(self.ff, MLP_TILE), dtype, device)
            self.mlp_norm = LayerNormWeight(cfg.hidden_size, device)

    def forward(self, x, h):
        h = ops.layernorm_residual(x, self.dtype, self.mixer(h), self.mixer_norm.weight, self.eps)
        if self.mlp is not None:
            h = ops.layernorm_residual(x, self.dtype, [(self.mlp(h), 1.0)], self.mlp_norm.weight, self.eps)
        return h

    def load_tensor(self, key: str, w: torch.Tensor):
        if key in ("norm1", "norm2"):
            (self.mixer_norm if key == "norm1" else self.mlp_norm).weight.data.copy_(w)
        elif key in ("mlp.gate", "mlp.up"):
            gu = self.mlp.gate_up_proj
            gu.load("weight", padded(w, gu.output_sizes[0], gu.in_features), 0 if key == "mlp.gate" else 1)
        elif key == "mlp.down":
            dn = self.mlp.down_proj
            dn.load("weight", padded(w, dn.out_features, dn.in_features))
        elif key.startswith("mix."):
            self.mixer.load_tensor(key.removeprefix("mix."), w)
        else:
            raise KeyError(key)


class BolopelForCausalLM(DenseForCausalLM):
    layer_cls = BolopelDecoderLayer

    def __init__(self, cfg: ModelConfig, device="cpu", dtype: Optional[torch.dtype] = None):
        nn.Module.__init__(self)
        st = get_state()
        if st.tp_size > 1 or st.pp_size > 1:
            raise ValueError(f"{cfg.architecture} runs on one GPU (no tensor or pipeline parallelism)")
        if cfg.quantization:
            raise ValueError(f"{cfg.architecture}: quantised checkpoints are not supported")
        self.cfg = cfg
        self.dtype = dtype or DTYPES[cfg.dtype]
        self.device = torch.device(device)
        self.first_layer, self.last_layer = 0, cfg.num_layers
        self.width, self.ld, self.eps = cfg.hidden_size, align(cfg.hidden_size), cfg.rms_norm_eps
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, self.ld, self.dtype, device)
        self.embed_norm = LayerNormWeight(self.width, device)
        self.layers = nn.ModuleDict({str(i): self.layer_cls(cfg, i, self.dtype, device) for i in range(cfg.num_layers)})
        self.norm = LayerNormWeight(self.width, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, self.ld, self.dtype, device)
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

    # ---- caches
    def kv_cache_spec(self, block_size: int):
        specs = {i: self.layers[str(i)].mixer.kv_cache_spec(block_size, self.dtype) for i in range(self.last_layer)}
        return {i: s for i, s in specs.items() if s is not None}

    def state_cache_spec(self):
        return {i: self.layers[str(i)].mixer.state_spec(self.dtype) for i in range(self.last_layer)
                if self.layers[str(i)].mixer.has_state}

    @property
    def uses_state_cache(self) -> bool:
        return self.cfg.has_recurrent_state

    def attn_workspace_size(self) -> tuple:
        """(heads, head size) that cover every layer's split-KV partials (heads x size) and log-sum-exps (heads)."""
        left = [m.left for m in (self.layers[str(i)].mixer for i in range(self.last_layer)) if isinstance(m, ParallelMixer)]
        return max([1] + [a.heads for a in left]), max([1] + [a.cache_dim for a in left])

    # ---- weights
    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor of a checkpoint with this configuration."""
        W, V = self.width, self.cfg.vocab_size
        out = {"embed": (V, W), "embed.norm": (W,)}
        for i, spec in enumerate(self.cfg.layer_specs):
            out[f"l{i}.norm1"] = (W,)
            out.update({f"l{i}.mix.{k}": s for k, s in MIXERS[spec.type].tensor_shapes(spec.mixer, W).items()})
            if spec.mlp is not None:
                ff = int(spec.mlp["ff"])
                out.update({f"l{i}.norm2": (W,), f"l{i}.mlp.gate": (ff, W), f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff)})
        out.update({"final.norm": (W,), "head": (V, W)})
        return out

    def init_random(self, seed: int = 0, std: float = 0.02):
        """Seeded weights through the checkpoint path: ``N(0, std)`` matrices, norm weights 1, decay parameters in the
        range of a trained model."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def tensors():
            for name, shape in self.tensor_shapes().items():
                t = torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
                leaf = name.rsplit(".", 1)[-1]
                if "norm" in leaf:
                    t = torch.ones_like(t)
                elif leaf == "A_log":
                    t = t.clamp(-1.0, 1.0)
                elif leaf == "dt_bias":
                    t = t.clamp(-1.0, 1.0) - 3.0
                elif leaf == "conv":
                    t = t * (10.0 * std)
                else:
                    t = t * std
                yield name, t.to(self.dtype)
        self.load_weights(tensors())

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]):
        want = self.tensor_shapes()
        loaded = set()
        for m in self.modules():
            if isinstance(m, GatedMLP):
                m.set_act_fused(False)  # checkpoints carry the plain [gate | up] order
        for name, w in weights:
            if name not in want:
                raise ValueError(f"unexpected tensor {name!r} in the checkpoint")
            if tuple(w.shape) != tuple(want[name]):
                raise ValueError(f"tensor {name!r}: shape {tuple(w.shape)}, expected {tuple(want[name])}")
            if name == "embed":
                self.embed_tokens.load("weight", padded(w, w.shape[0], self.ld))
            elif name == "head":
                self.lm_head.load("weight", padded(w, w.shape[0], self.ld))
            elif name == "embed.norm":
                self.embed_norm.weight.data.copy_(w)
            elif name == "final.norm":
                self.norm.weight.data.copy_(w)
            else:
                layer, key = name.split(".", 1)
                self.layers[layer[1:]].load_tensor(key, w)
            loaded.add(name)
        missing = sorted(set(want) - loaded)
        if missing:
            raise ValueError(f"the checkpoint lacks {len(missing)} tensors, e.g. {missing[:3]}")
        self.finish_loading()
        return loaded
