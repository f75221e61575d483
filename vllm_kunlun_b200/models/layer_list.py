"""Shared frame of decoders whose configuration lists the layers one by one (``models/mixers.py``): checks, caches and
per-request state, strict checkpoint loading, random initialisation.  A design adds its layer class, its forward pass and
the tensors outside the layers.

The residual stream and every norm are fp32; the GEMMs read copies in the model's dtype.  Rows are padded to a multiple of 8
columns (zeros), so any width runs through the tensor-core GEMMs.  Checkpoint tensors of layer i are named ``l<i>.*``, its
mixer's ``l<i>.mix.*``, its feed-forward's (``models/feed_forward.py``) ``l<i>.mlp.*``.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from ..config import LayerSpec, ModelConfig
from ..parallel.state import get_state
from .dense import DenseForCausalLM, GatedMLP
from .feed_forward import feed_forward_cls
from .layers import DTYPES, ParallelLMHead, VocabParallelEmbedding, param
from .mixers import MIXERS, align, padded


class NormWeight(nn.Module):
    def __init__(self, width: int, device):
        super().__init__()
        self.weight = param(width, dtype=torch.float32, device=device)


class ListedLayer(nn.Module):
    """Mixer and feed-forward of one listed layer; subclasses arrange them."""

    def __init__(self, cfg: ModelConfig, layer_idx: int, dtype, device):
        super().__init__()
        spec = cfg.layer_specs[layer_idx]
        self.ld, self.eps, self.dtype = align(cfg.hidden_size), cfg.rms_norm_eps, dtype
        self.mixer = MIXERS[spec.type](self.ld, spec.mixer, layer_idx, cfg.rms_norm_eps, dtype, device)
        self.mlp = None
        if spec.mlp is not None:
            self.mlp = feed_forward_cls(spec.mlp, cfg.hidden_act)(self.ld, spec.mlp, cfg.hidden_act, cfg.rms_norm_eps, dtype,
                                                                  device)

    @classmethod
    def tensor_shapes(cls, spec: LayerSpec, width: int, act: str) -> dict:
        """Name (behind ``l<i>.``) -> shape of the mixer's and the feed-forward's tensors."""
        out = {f"mix.{k}": s for k, s in MIXERS[spec.type].tensor_shapes(spec.mixer, width).items()}
        if spec.mlp is not None:
            shapes = feed_forward_cls(spec.mlp, act).tensor_shapes(spec.mlp, width)
            out.update({f"mlp.{k}": s for k, s in shapes.items()})
        return out

    @classmethod
    def unused_tensors(cls, spec: LayerSpec) -> tuple:
        """Names that a checkpoint may carry without effect."""
        unused = getattr(MIXERS[spec.type], "unused_tensors", None)
        return () if unused is None else tuple(f"mix.{k}" for k in unused(spec.mixer))

    def state_spec(self, dtype) -> list:
        """``(shape per request, dtype)`` of everything the layer keeps per request, the mixer's first."""
        return self.mixer.state_spec(dtype) if self.mixer.has_state else []

    def load_tensor(self, key: str, w: torch.Tensor):
        if key.startswith("mlp."):
            self.mlp.load_tensor(key.removeprefix("mlp."), w)
        elif key.startswith("mix."):
            self.mixer.load_tensor(key.removeprefix("mix."), w)
        else:
            raise KeyError(key)


class LayerListForCausalLM(DenseForCausalLM):
    layer_cls = ListedLayer
    unit_norm_init = 1.0        # what a norm weight of a freshly initialised model is stored as

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
        self.layers = nn.ModuleDict({str(i): self.layer_cls(cfg, i, self.dtype, device) for i in range(cfg.num_layers)})
        self.norm = NormWeight(self.width, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, self.ld, self.dtype, device)
        if cfg.tie_word_embeddings:
            self.lm_head.weight = self.embed_tokens.weight

    # ---- caches
    def kv_cache_spec(self, block_size: int):
        specs = {i: self.layers[str(i)].mixer.kv_cache_spec(block_size, self.dtype) for i in range(self.last_layer)}
        return {i: s for i, s in specs.items() if s is not None}

    def state_cache_spec(self):
        specs = {i: self.layers[str(i)].state_spec(self.dtype) for i in range(self.last_layer)}
        return {i: s for i, s in specs.items() if s}

    @property
    def uses_state_cache(self) -> bool:
        return self.cfg.has_recurrent_state

    def attn_workspace_size(self) -> tuple:
        """(heads, head size) that cover every layer's split-KV partials (heads x size) and log-sum-exps (heads)."""
        sizes = [self.layers[str(i)].mixer.workspace_size() for i in range(self.last_layer)]
        return tuple(max([1] + [s[k] for s in sizes]) for k in (0, 1))

    # ---- weights
    def outer_tensor_shapes(self) -> dict:
        """Name -> shape of the tensors outside the layers."""
        W, V = self.width, self.cfg.vocab_size
        out = {"embed": (V, W), "final.norm": (W,)}
        return out if self.cfg.tie_word_embeddings else {**out, "head": (V, W)}

    def load_outer_tensor(self, name: str, w: torch.Tensor):
        if name == "embed":
            self.embed_tokens.load("weight", padded(w, w.shape[0], self.ld))
        elif name == "head":
            self.lm_head.load("weight", padded(w, w.shape[0], self.ld))
        elif name == "final.norm":
            self.norm.weight.data.copy_(w)
        else:
            raise KeyError(name)

    def tensor_shapes(self) -> dict:
        """Name -> shape of every tensor of a checkpoint with this configuration."""
        out = dict(self.outer_tensor_shapes())
        for i, spec in enumerate(self.cfg.layer_specs):
            out.update({f"l{i}.{k}": s for k, s in self.layer_cls.tensor_shapes(spec, self.width, self.cfg.hidden_act).items()})
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
                    # norms inside a mixer have plain weights
                    t = torch.full_like(t, 1.0 if ".mix." in name else self.unit_norm_init)
                elif leaf == "A_log":
                    t = t.clamp(-1.0, 1.0)
                elif leaf == "dt_bias":
                    t = t.clamp(-1.0, 1.0) - 3.0
                elif leaf == "conv" or leaf.startswith("canon"):
                    t = t * (10.0 * std)
                elif leaf in ("shift", "lower", "vmix"):
                    t = torch.sigmoid(t)
                elif leaf in ("rel", "act"):
                    t = t.clamp(-1.0, 1.0)
                else:
                    t = t * std
                yield name, t.to(self.dtype)
        self.load_weights(tensors())

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]):
        want, outer = self.tensor_shapes(), self.outer_tensor_shapes()
        unused = {f"l{i}.{k}" for i, spec in enumerate(self.cfg.layer_specs) for k in self.layer_cls.unused_tensors(spec)}
        loaded = set()
        for m in self.modules():
            if isinstance(m, GatedMLP):
                m.set_act_fused(False)  # checkpoints carry the plain [gate | up] order
        for name, w in weights:
            if name in unused:
                continue
            if name not in want:
                raise ValueError(f"unexpected tensor {name!r} in the checkpoint")
            if tuple(w.shape) != tuple(want[name]):
                raise ValueError(f"tensor {name!r}: shape {tuple(w.shape)}, expected {tuple(want[name])}")
            if name in outer:
                self.load_outer_tensor(name, w)
            else:
                layer, key = name.split(".", 1)
                self.layers[layer[1:]].load_tensor(key, w)
            loaded.add(name)
        missing = sorted(set(want) - loaded)
        if missing:
            raise ValueError(f"the checkpoint lacks {len(missing)} tensors, e.g. {missing[:3]}")
        self.finish_loading()
        return loaded
