"""Vebesun: a decoder given as a list of layers, each with its own kind of mixer and an optional gated MLP.

The residual is a bundle of streams joined by hyper-connections (``ops/hyper.py``), norms are LayerNorm in front of every
sublayer, a stretch of layers can be run several times with the same weights (each pass with a cache of its own), positions
enter through the mixers only, and the output head is the embedding table. Mixers: windowed latent attention and the
channel-wise gated delta rule (``models/mixers.py``); weights, cache and step are those of ``models/stepped.py``."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops.hyper import HyperIn, HyperOut, hyper_step
from .mixers import MIXERS, Proj, StepContext, frozen, put
from .registry import register
from .stepped import SteppedDecoder, check_layers, layer_bodies, mlp_shapes


@dataclass
class VebesunConfig:
    """The contents of ``config.json`` plus the run-time limit ``max_seq_len`` (cache size; the model itself has none)."""
    vocab_size: int
    width: int
    layers: List[dict]
    streams: int = 1
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    loop: Optional[dict] = None
    max_seq_len: int = 4096
    ranks: Dict[str, Tuple[int, int]] = field(default_factory=dict)   # layer -> inner sizes of its low-rank products (tensor shapes)

    @staticmethod
    def from_dict(d: dict) -> "VebesunConfig":
        c = VebesunConfig(vocab_size=d["vocab"], width=d["width"], layers=d["layers"], streams=d.get("streams") or 1, norm_eps=d["norm"]["eps"],
                          embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), loop=d.get("loop"),
                          max_seq_len=d.get("max_seq_len", 4096), ranks={k: tuple(v) for k, v in d.get("ranks", {}).items()})
        c.order()
        return c

    def to_dict(self) -> dict:
        return {"architecture": "Vebesun", "vocab": self.vocab_size, "width": self.width, "layers": self.layers, "streams": self.streams,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "loop": self.loop, "max_seq_len": self.max_seq_len,
                "ranks": self.ranks}

    def order(self) -> List[int]:
        """Layer index of every run."""
        n = len(self.layers)
        check_layers(self.layers)
        if not self.loop:
            return list(range(n))
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        if not (0 <= a <= b <= n and times >= 0):
            raise ValueError(f"bad loop {self.loop}")
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Every tensor of a model file, with the low-rank sizes of ``ranks``."""
        E, S = self.width, self.streams
        out = {"embed": (self.vocab_size, E), "final.norm": (E,), "final.norm.b": (E,)}
        for i, layer in enumerate(self.layers):
            l = f"l{i}."
            out.update(MIXERS[layer["type"]].shapes(E, layer["mixer"], l + "mix.", self.ranks.get(str(i))))
            if layer.get("mlp") is not None:
                out.update(mlp_shapes(E, layer["mlp"], l + "mlp."))
            for q in ((1, 2) if layer.get("mlp") is not None else (1,)):
                out[f"{l}norm{q}"] = out[f"{l}norm{q}.b"] = (E,)
                out[f"{l}hc{q}.in"] = out[f"{l}hc{q}.out"] = (S,)
                out[f"{l}hc{q}.mix"] = (S, S)
        return out


class Sublayer(nn.Module):
    """A mixer or MLP with its norm and its place in the streams."""

    def __init__(self, body: nn.Module, width: int, streams: int):
        super().__init__()
        self.body = body
        self.norm_w, self.norm_b = frozen(width, dtype=torch.float32), frozen(width, dtype=torch.float32)
        self.inw, self.outw, self.mix = (frozen(streams, dtype=torch.float32), frozen(streams, dtype=torch.float32),
                                         frozen(streams, streams, dtype=torch.float32))


@register("Vebesun")
class VebesunModel(SteppedDecoder):
    # what a fresh checkout compiles to run this model
    CUDA_SOURCES = ("hyper.cu", "delta_rule.cu", "latent_attn.cu", "skinny_gemm.cu", "flash_attn_fwd.cu", "gemm_tcgen05.cu", "gemm_tcgen05_2cta.cu", "elementwise.cu",
                    "sampler.cu")
    config_class = VebesunConfig

    def __init__(self, cfg: VebesunConfig, dtype=torch.bfloat16, device=None, seed: Optional[int] = None):
        super().__init__(cfg, dtype)
        E, S = cfg.width, cfg.streams
        self.embed = Proj(cfg.vocab_size, E, dtype)
        self.final_w, self.final_b = frozen(E, dtype=torch.float32), frozen(E, dtype=torch.float32)
        self.ones = frozen(S, dtype=torch.float32)
        layers = []
        for i, layer in enumerate(cfg.layers):
            sh = {"a1": (cfg.ranks[str(i)][0],), "g1": (cfg.ranks[str(i)][1],)} if str(i) in cfg.ranks else None
            layers.append(nn.ModuleList(Sublayer(body, E, S) for body in layer_bodies(E, layer, cfg.norm_eps, dtype, sh)))
        self.layers = nn.ModuleList(layers)
        self.set_runs(cfg.order())
        if seed is not None:
            self.reset_parameters(seed)
        if device is not None:
            self.to(device)

    # ------------------------------------------------------------------ weights
    @staticmethod
    def ranks_from(shapes: Dict[str, tuple], cfg: VebesunConfig) -> Dict[str, Tuple[int, int]]:
        """Low-rank sizes are given by the tensors, not by ``config.json``."""
        return {str(i): (shapes[f"l{i}.mix.a1"][0], shapes[f"l{i}.mix.g1"][0]) for i in range(len(cfg.layers)) if f"l{i}.mix.a1" in shapes}

    @classmethod
    def fit_config(cls, cfg: VebesunConfig, shapes: Dict[str, tuple]):
        cfg.ranks = cls.ranks_from(shapes, cfg) or cfg.ranks

    def complete(self, tensors, shapes):
        if self.cfg.streams == 1:      # a model with a plain residual has no stream weights: they are ones
            tensors = dict(tensors)
            for n in shapes:
                if ".hc" in n and n not in tensors:
                    tensors[n] = torch.ones(shapes[n])
        return tensors

    def put_tensors(self, t: Dict[str, torch.Tensor]):
        put(self.embed, t["embed"])
        self.final_w.copy_(t["final.norm"])
        self.final_b.copy_(t["final.norm.b"])
        self.ones.fill_(1.0)
        for i, subs in enumerate(self.layers):
            for q, sub in enumerate(subs, 1):
                l = f"l{i}."
                sub.body.load(t, l + ("mix." if q == 1 else "mlp."))
                sub.norm_w.copy_(t[f"{l}norm{q}"])
                sub.norm_b.copy_(t[f"{l}norm{q}.b"])
                sub.inw.copy_(t[f"{l}hc{q}.in"])
                sub.outw.copy_(t[f"{l}hc{q}.out"])
                sub.mix.copy_(t[f"{l}hc{q}.mix"])

    def state_dict_reference(self) -> Dict[str, torch.Tensor]:
        """fp32 tensors under their file names (``formats.export.save_model``)."""
        out = {"embed": self.embed.weight[: self.cfg.vocab_size, : self.cfg.width], "final.norm": self.final_w, "final.norm.b": self.final_b}
        for i, subs in enumerate(self.layers):
            for q, sub in enumerate(subs, 1):
                l = f"l{i}."
                out.update(sub.body.export(l + ("mix." if q == 1 else "mlp.")))
                out.update({f"{l}norm{q}": sub.norm_w, f"{l}norm{q}.b": sub.norm_b, f"{l}hc{q}.in": sub.inw, f"{l}hc{q}.out": sub.outw,
                            f"{l}hc{q}.mix": sub.mix})
        return {k: v.detach().float().cpu().contiguous() for k, v in out.items()}

    def reset_parameters(self, seed: int = 0):
        """Random weights of the usual scales (benchmarks and tests; the design is served, not trained, here)."""
        g = torch.Generator().manual_seed(seed)
        t = {}
        for n, shp in self.cfg.tensor_shapes().items():
            if n.endswith(".b") and not n.endswith("mix.b"):
                t[n] = torch.zeros(shp)
            elif "norm" in n:
                t[n] = torch.ones(shp)
            elif ".hc" in n:
                t[n] = torch.eye(shp[0]) if len(shp) == 2 else torch.full(shp, 1.0 / shp[0] if n.endswith(".in") else 1.0)
            elif n.endswith("A_log"):
                t[n] = torch.rand(shp, generator=g) * 2 - 1
            elif n.endswith("dt_bias"):
                t[n] = torch.randn(shp, generator=g) - 4
            else:
                t[n] = torch.randn(shp, generator=g) * shp[-1] ** -0.5
        self.load_tensors(t)

    def _step(self, cache, batch, hidden, residuals):
        cfg = self.cfg
        ctx = StepContext(self, cache, batch)
        x = torch.empty(batch.T, cfg.streams, cfg.width, dtype=torch.float32, device=cache.device)
        prev, table = None, self.embed.weight
        for run, (i, index) in enumerate(self.runs):
            for q, sub in enumerate(self.layers[i]):
                nxt = HyperIn(sub.inw, sub.norm_w, sub.norm_b, cfg.norm_eps)
                first = prev is None
                h = hyper_step(x, self.dtype, prev, nxt, batch.ids if first else None, table if first else None, cfg.embedding_scale)
                if residuals is not None and q == 0 and run > 0:
                    residuals.append(x.sum(1))
                prev = HyperOut(sub.body.run(ctx, h, index), sub.mix, sub.outw)
        if prev is None:               # no layers at all
            hyper_step(x, self.dtype, None, None, batch.ids, table, cfg.embedding_scale)
        head = HyperIn(self.ones, self.final_w, self.final_b, cfg.norm_eps)
        if batch.n_want == batch.T and batch.want_all:
            h = hyper_step(x, self.dtype, prev, head)
        else:
            hyper_step(x, self.dtype, prev)
            if batch.n_want == 0:
                return None
            h = hyper_step(x, self.dtype, None, head, rows=batch.want)
        if residuals is not None:
            residuals.append(x.sum(1))
        if hidden:
            return h
        return ctx.logits(h, self.embed, cfg.vocab_size)
