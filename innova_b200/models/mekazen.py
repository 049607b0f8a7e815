"""Mekazen: a decoder given as a list of layers, each with gated attention in chunks and an optional gated MLP.

The residual is one fp32 row with an RMS norm in front of every sublayer and another behind it (weights stored around zero;
``ops/sandwich.py``). The attention (``mixers.GatedAttention``) normalises whole query and key rows, rotates pairs of the first
dimensions with scaled frequencies, uses the projected keys as values, sees the earlier tokens of its own chunk, and has an output
gate. Logits come from a head of their own and pass a soft limit."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..ops.sandwich import sandwich_step
from .mixers import MIXERS, Proj, StepContext, frozen, put
from .registry import register
from .stepped import SteppedDecoder, check_layers, layer_bodies, mlp_shapes

NORM_OFFSET = 1.0      # the stored weight of a residual norm is its distance from one


@dataclass
class MekazenConfig:
    """The contents of ``config.json`` plus the run-time limit ``max_seq_len`` (cache size; the model itself has none)."""
    vocab_size: int
    width: int
    layers: List[dict]
    norm_eps: float = 1e-5
    logit_softcap: Optional[float] = None
    max_seq_len: int = 4096

    @staticmethod
    def from_dict(d: dict) -> "MekazenConfig":
        check_layers(d["layers"])
        return MekazenConfig(vocab_size=d["vocab"], width=d["width"], layers=d["layers"], norm_eps=d["norm"]["eps"],
                             logit_softcap=d.get("logit_softcap"), max_seq_len=d.get("max_seq_len", 4096))

    def to_dict(self) -> dict:
        return {"architecture": "Mekazen", "vocab": self.vocab_size, "width": self.width, "layers": self.layers, "norm": {"eps": self.norm_eps},
                "logit_softcap": self.logit_softcap, "max_seq_len": self.max_seq_len}

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Every tensor of a model file."""
        V, E = self.vocab_size, self.width
        out = {"embed": (V, E), "final.norm": (E,), "head": (V, E)}
        for i, layer in enumerate(self.layers):
            l = f"l{i}."
            out.update(MIXERS[layer["type"]].shapes(E, layer["mixer"], l + "mix.", None))
            out[l + "norm1"] = out[l + "norm1b"] = (E,)
            if layer.get("mlp") is not None:
                out.update(mlp_shapes(E, layer["mlp"], l + "mlp."))
                out[l + "norm2"] = out[l + "norm2b"] = (E,)
        return out


class Sublayer(nn.Module):
    """A mixer or MLP between its two norms."""

    def __init__(self, body: nn.Module, width: int):
        super().__init__()
        self.body = body
        self.norm, self.post = frozen(width, dtype=torch.float32), frozen(width, dtype=torch.float32)


@register("Mekazen")
class MekazenModel(SteppedDecoder):
    # what a fresh checkout compiles to run this model
    CUDA_SOURCES = ("sandwich.cu", "kv_attn.cu", "hyper.cu", "skinny_gemm.cu", "flash_attn_fwd.cu", "gemm_tcgen05.cu", "gemm_tcgen05_2cta.cu",
                    "elementwise.cu", "sampler.cu")
    config_class = MekazenConfig

    def __init__(self, cfg: MekazenConfig, dtype=torch.bfloat16, device=None, seed: Optional[int] = None):
        super().__init__(cfg, dtype)
        E = cfg.width
        self.embed, self.head = Proj(cfg.vocab_size, E, dtype), Proj(cfg.vocab_size, E, dtype)
        self.final = frozen(E, dtype=torch.float32)
        self.layers = nn.ModuleList(nn.ModuleList(Sublayer(body, E) for body in layer_bodies(E, layer, cfg.norm_eps, dtype)) for layer in cfg.layers)
        self.set_runs(list(range(len(cfg.layers))))
        if seed is not None:
            self.reset_parameters(seed)
        if device is not None:
            self.to(device)

    def put_tensors(self, t: Dict[str, torch.Tensor]):
        put(self.embed, t["embed"])
        put(self.head, t["head"])
        self.final.copy_(t["final.norm"])
        for i, subs in enumerate(self.layers):
            for q, sub in enumerate(subs, 1):
                sub.body.load(t, f"l{i}." + ("mix." if q == 1 else "mlp."))
                sub.norm.copy_(t[f"l{i}.norm{q}"])
                sub.post.copy_(t[f"l{i}.norm{q}b"])

    def state_dict_reference(self) -> Dict[str, torch.Tensor]:
        """fp32 tensors under their file names (``formats.export.save_model``)."""
        V, E = self.cfg.vocab_size, self.cfg.width
        out = {"embed": self.embed.weight[:V, :E], "head": self.head.weight[:V, :E], "final.norm": self.final}
        for i, subs in enumerate(self.layers):
            for q, sub in enumerate(subs, 1):
                out.update(sub.body.export(f"l{i}." + ("mix." if q == 1 else "mlp.")))
                out.update({f"l{i}.norm{q}": sub.norm, f"l{i}.norm{q}b": sub.post})
        return {k: v.detach().float().cpu().contiguous() for k, v in out.items()}

    def reset_parameters(self, seed: int = 0):
        """Random weights of the usual scales (benchmarks and tests; the design is served, not trained, here)."""
        g = torch.Generator().manual_seed(seed)
        t = {}
        for n, shp in self.cfg.tensor_shapes().items():
            if len(shp) == 1:
                t[n] = torch.ones(shp) if n.endswith((".q.norm", ".k.norm")) else torch.zeros(shp)
            else:
                t[n] = torch.randn(shp, generator=g) * (1.0 if n == "embed" else shp[-1] ** -0.5)
        self.load_tensors(t)

    def _step(self, cache, batch, hidden, residuals):
        cfg, eps = self.cfg, self.cfg.norm_eps
        ctx = StepContext(self, cache, batch)
        x = torch.empty(batch.T, cfg.width, dtype=torch.float32, device=cache.device)
        todo = dict(ids=batch.ids, table=self.embed.weight)       # what the residual takes in at the next step between sublayers
        for i, index in self.runs:
            for q, sub in enumerate(self.layers[i]):
                h = sandwich_step(x, self.dtype, eps, NORM_OFFSET, norm_w=sub.norm, **todo)
                if residuals is not None and q == 0 and i > 0:
                    residuals.append(x.clone())
                todo = dict(y=sub.body.run(ctx, h, index), post_w=sub.post)
        if residuals is not None:
            sandwich_step(x, self.dtype, eps, NORM_OFFSET, **todo)
            residuals.append(x.clone())
            todo = {}
        if batch.n_want == 0:
            return None
        rows = None if batch.want_all else batch.want
        h = sandwich_step(x, self.dtype, eps, NORM_OFFSET, norm_w=self.final, rows=rows, **todo)
        if hidden:
            return h
        return ctx.logits(h, self.head, cfg.vocab_size, cfg.logit_softcap)
