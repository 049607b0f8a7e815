"""Base of the layer-list decoders: weights by file name, a cache per layer run, one packed step.

A design gives ``layers[i]`` as a list of sublayers whose ``body`` is a module of ``mixers.py``, the order in which the layers run,
``tensor_shapes`` of its configuration, and the step itself (``_step``). The model has one forward: ``step(cache, batch)`` runs the
packed new tokens of any number of sequences against a ``StepCache`` and returns the logits asked for. Generation, batching, scoring
and trace replay all go through it."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..inference.state_cache import StepBatch, StepCache
from ..ops.gemm import full_fp32_matmul
from .mixers import MIXERS, GatedMLP


def check_layers(layers: List[dict]):
    for i, layer in enumerate(layers):
        if layer["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        MIXERS[layer["type"]].check(layer["mixer"], i)
        if layer.get("mlp") is not None and layer["mlp"].get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {layer['mlp']!r}")


class SteppedDecoder(nn.Module):
    config_class: type
    HOST_SOURCES = ("importers.cpp",)

    def __init__(self, cfg, dtype):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"{dtype}: bfloat16 or float32")
        self.cfg, self.dtype = cfg, dtype

    def set_runs(self, order: List[int]):
        """Layer and cache index of every run; each kind of cache counts its own runs."""
        self.runs, counts = [], {}
        for i in order:
            kind = self.layers[i][0].body.cache_kind
            self.runs.append((i, counts.setdefault(kind, 0)))
            counts[kind] += 1

    # ------------------------------------------------------------------ weights
    @classmethod
    def fit_config(cls, cfg, shapes: Dict[str, tuple]):
        """Take into ``cfg`` the sizes that only the tensors give."""

    def complete(self, tensors: Dict[str, torch.Tensor], shapes: Dict[str, tuple]) -> Dict[str, torch.Tensor]:
        """Add tensors that a file may leave out."""
        return tensors

    @classmethod
    def from_tensors(cls, config: dict, tensors: Dict[str, torch.Tensor], dtype=torch.bfloat16, device=None) -> "SteppedDecoder":
        cfg = cls.config_class.from_dict(config)
        cls.fit_config(cfg, {n: tuple(t.shape) for n, t in tensors.items()})
        model = cls(cfg, dtype=dtype)
        model.load_tensors(tensors)
        return model.to(device) if device is not None else model

    @torch.no_grad()
    def load_tensors(self, tensors: Dict[str, torch.Tensor]):
        shapes = self.cfg.tensor_shapes()
        tensors = self.complete(tensors, shapes)
        missing = [n for n in shapes if n not in tensors]
        if missing:
            raise KeyError(f"model file lacks {len(missing)} tensors: {', '.join(missing[:8])}")
        t = {}
        for n, shp in shapes.items():
            if tensors[n].numel() != torch.Size(shp).numel():
                raise ValueError(f"{n}: shape {tuple(tensors[n].shape)}, expected {shp}")
            t[n] = tensors[n].view(shp)
        self.put_tensors(t)

    def num_params(self) -> int:
        return sum(torch.Size(s).numel() for s in self.cfg.tensor_shapes().values())

    # ------------------------------------------------------------------ cache and step
    def make_cache(self, max_batch: int, max_seq: int, device=None, num_pages: Optional[int] = None) -> StepCache:
        specs: Dict[str, list] = {}
        for i, _ in self.runs:
            body = self.layers[i][0].body
            specs.setdefault(body.cache_kind, []).append(body.cache_spec)
        return StepCache(max_batch, max_seq, device or self.embed.weight.device, self.dtype, num_pages, **specs)

    @torch.no_grad()
    def step(self, cache: StepCache, batch: StepBatch, hidden: bool = False, residuals: Optional[list] = None):
        """Run the batch's new tokens; returns fp32 logits [wanted, vocab] (or the final normed states with ``hidden``), None when
        nothing is wanted. ``residuals`` collects the residual (the sum of its streams) after every layer run."""
        with full_fp32_matmul(self.dtype):
            return self._step(cache, batch, hidden, residuals)

    # ------------------------------------------------------------------ whole-sequence forms (scoring, embedding, beam search)
    def _whole(self, ids: torch.Tensor, hidden: bool):
        B, S = ids.shape
        cache = self.make_cache(B, S, self.embed.weight.device)
        for b in range(B):
            cache.reserve(b, S)
        batch = StepBatch(cache, ids.tolist(), [0] * B, list(range(B)), want=range(B * S), vocab=self.cfg.vocab_size)
        return self.step(cache, batch, hidden=hidden).view(B, S, -1)

    def hidden_states(self, ids: torch.Tensor) -> torch.Tensor:
        return self._whole(ids, True)

    def forward(self, ids: torch.Tensor) -> torch.Tensor:
        """[B, S] token ids -> logits [B, S, vocab]."""
        return self._whole(ids, False)


def mlp_shapes(width: int, mlp: dict, p: str) -> Dict[str, tuple]:
    return {p + "gate": (mlp["ff"], width), p + "up": (mlp["ff"], width), p + "down": (width, mlp["ff"])}


def layer_bodies(width: int, layer: dict, eps: float, dtype, shapes=None) -> List[nn.Module]:
    """The mixer of a layer and, if it has one, its feed-forward."""
    bodies = [MIXERS[layer["type"]](width, layer["mixer"], eps, dtype, shapes)]
    if layer.get("mlp") is not None:
        bodies.append(GatedMLP(width, layer["mlp"]["ff"], dtype))
    return bodies
