"""Nomivik `Model`: the per-model surface of the package (`language_model`, `get_input_embeddings`, `sanitize`,
`load_weights`, `engine`, `config`) for a text-only decoder of plain pre-norm layers (decoder_blocks.PreNormLayer): an
attention beside a matrix memory with exponential gates, or a gated linear recurrence; silu-gated units; an input that the
token brings to every layer.  The embedding adds a second table addressed by the token and the one before it.  A span of
layers may run several times with the same weights; every run has its own cache rows and state, and before every pass after
the first the embedding output is added to the stream.  All weights are packed into ONE device arena, the embedding table is
the head; the arithmetic is csrc/layer_ops.cu, mixer_ops.cu and recurrent_ops.cu driven by `LayerEngine`."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import numpy as np
import torch

from ...layer_engine import LayerEngine
from ..base import InputEmbeddingsFeatures
from ..decoder_blocks import PreNormLayer, StepCtx, whole_vectors
from ..qwen2_vl.qwen2_vl import WeightArena
from .config import ModelConfig
from .language import LanguageModel

TOKEN_STATE = whole_vectors(1)      # numbers of a slot's state in front of the layers': the last token


@dataclass
class Run:
    layer: int
    opens_pass: bool              # the embedding output is added to the stream before this run
    kv_base: int                  # the pool's caching layer of this run's attention
    state_base: int               # offset of this run's state in a slot


class Model:
    norm_offset = 0.0             # the norms' weights are stored plainly

    def __init__(self, config: ModelConfig, device=None, dtype: str = "bfloat16"):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype: 'bfloat16' (serving) or 'float32' (everything in true 32-bit)")
        self.config = config
        self.exact = dtype == "float32"
        self._device = torch.device(device) if device is not None else torch.device("cuda", 0)
        self._eng: Optional[LayerEngine] = None
        self.width, self.vocab = config.width, config.vocab
        self.eps, self.embed_scale, self.logit_softcap = config.norm_eps, 1.0, None
        self.layers = [PreNormLayer(i, c, config.width, side_dim=config.side_dim) for i, c in enumerate(config.layers)]
        self.runs, kv, st = [], 0, TOKEN_STATE
        for i, opens in config.layer_runs():
            self.runs.append(Run(i, opens, kv, st))
            kv += 1 if self.layers[i].kv_dim else 0
            st += self.layers[i].state_floats
        self.n_cache_layers, self.state_floats = kv, st
        self.row_dim = (max([L.kv_dim for L in self.layers] + [0]) + 7) // 8 * 8      # rows of whole 16-byte vectors
        self.embed = self.bigram = self.final_norm = self.head = None
        self.arena: Optional[WeightArena] = None
        self.language_model = LanguageModel(config, self, self._engine)

    # ------------------------------------------------------------------ engine
    def _engine(self) -> LayerEngine:
        if self._eng is None:
            self._eng = LayerEngine(self._device, exact=self.exact)
            self._eng.bind_model(self)
        return self._eng

    @property
    def engine(self) -> LayerEngine:
        return self._engine()

    def embed_rows(self, ctx, tokens: torch.Tensor) -> torch.Tensor:
        """the embedding output of a step (T, width) fp32; a second copy for the passes that add it again, and the first layer's
        norm, are left in ctx"""
        ops = ctx.ops
        again = any(r.opens_pass for r in self.runs)
        if self.config.bigram is None:
            x = ops.embed(tokens, self.embed, self.embed_scale)
            ctx.carry["embedding"] = ops.embed(tokens, self.embed, self.embed_scale) if again else None
            ctx.carry["normed"] = None
            return x
        b = self.config.bigram
        x, kept, ctx.carry["normed"], ctx.x_operand = ops.embed_bigram(
            tokens, self.embed, self.embed_scale, self.bigram, b["mul_prev"], b["mul_cur"], ctx.pool.state, ctx, keep=again,
            norm=self.layers[self.runs[0].layer].w["norm1"] if self.runs else None, eps=self.eps)
        ctx.carry["embedding"] = kept
        return x

    def run_layers(self, ctx, x: torch.Tensor, embed_again) -> torch.Tensor:
        """the layer runs of one step over the residual rows x (T, width) fp32, updated in place"""
        normed = ctx.carry["normed"]
        for k, run in enumerate(self.runs):
            nxt = self.runs[k + 1] if k + 1 < len(self.runs) else None
            ctx.kv_base, ctx.state_base = run.kv_base, run.state_base
            normed = self.layers[run.layer].forward(
                ctx, x, normed, next_norm=self.layers[nxt.layer].w["norm1"] if nxt is not None else None,
                extra=ctx.carry["embedding"] if nxt is not None and nxt.opens_pass else None)
        return x

    # ------------------------------------------------------------------ weights
    def _globals(self):
        W, V, c = self.width, self.vocab, self.config
        out = [("embed", (V, W)), ("final.norm", (W,))]
        if c.bigram is not None:
            out.append(("bigram", (c.bigram["buckets"] + 1, W)))
        if c.side_dim:
            out.append(("side.embed", (V, len(self.layers) * c.side_dim)))
        return out

    def manifest(self):
        out = self._globals()
        for i, L in enumerate(self.layers):
            out += L.manifest(f"l{i}.")
        return out

    def checkpoint_tensors(self) -> Dict[str, tuple]:
        """checkpoint name -> shape of every tensor this configuration reads"""
        out = dict(self._globals())
        for i, L in enumerate(self.layers):
            out.update(L.checkpoint_tensors(f"l{i}."))
        return out

    def expected_tensors(self):
        return list(self.checkpoint_tensors())

    @staticmethod
    def sanitize(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
        return {k[len("model."):] if k.startswith("model.") else k: v for k, v in weights.items()}

    def _bind(self, view):
        for i, L in enumerate(self.layers):
            L.bind(f"l{i}.", view)
            if L.side is not None:
                L.side.table = view("side.embed")[:, i * L.side.dim:(i + 1) * L.side.dim]
        self.embed, self.final_norm = view("embed"), view("final.norm")
        self.bigram = view("bigram") if self.config.bigram is not None else None
        self.head = self.embed        # the logits are products with the embedding rows

    def load_weights(self, weights: Dict[str, torch.Tensor], strict: bool = True):
        need = self.checkpoint_tensors()
        missing = [n for n in need if n not in weights]
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors, e.g. {missing[:4]}")
        wrong = [n for n, shape in need.items() if tuple(weights[n].shape) != tuple(shape)]
        if wrong:
            n = wrong[0]
            raise ValueError(f"checkpoint tensor {n} has shape {tuple(weights[n].shape)}, the configuration says {need[n]}")
        extra = sorted(set(weights) - set(need))
        if strict and extra:
            raise ValueError(f"checkpoint has {len(extra)} tensors this configuration does not use, e.g. {extra[:4]}")
        eng = self._engine()
        with torch.cuda.stream(eng.stream):
            self.arena = WeightArena(self.manifest(), eng.device)
            ck = {n: weights[n].to(device=eng.device, dtype=torch.bfloat16) for n in need}
            view = self.arena.view
            for n, _ in self._globals():
                view(n).copy_(ck[n])
            for i, L in enumerate(self.layers):
                L.pack(f"l{i}.", ck, view)
            self._bind(view)
        eng.stream.synchronize()
        return self

    def init_random(self, seed: int = 0):
        """seeded random weights of this configuration, generated on the device straight into the arena (benchmarks,
        no checkpoint): matrices N(0, 1/fan-in), norm weights around one, slow decays, the other vectors small"""
        eng = self._engine()
        g = torch.Generator(device=eng.device).manual_seed(seed)
        with torch.cuda.stream(eng.stream):
            self.arena = WeightArena(self.manifest(), eng.device)
            view = self.arena.view
            for name, shape in self.manifest():
                v = view(name)
                if len(shape) == 1:
                    last = name.rsplit(".", 1)[-1]
                    mean = {"lam": -4.0}.get(last, 1.0 if last.startswith("norm") or last == "out" else 0.0)
                    v.copy_(mean + 0.05 * torch.randn(shape, generator=g, device=eng.device))
                else:
                    s = 1.0 if name in ("embed", "bigram", "side.embed") else 1.0 / float(shape[-1]) ** 0.5
                    for part in (v.unbind(0) if v.numel() > (1 << 28) else (v,)):     # bounded fp32 staging
                        part.copy_(torch.randn(part.shape, generator=g, device=eng.device) * s)
            self._bind(view)
        eng.stream.synchronize()
        return self

    # ------------------------------------------------------------------ inputs
    def get_input_embeddings(self, input_ids=None, pixel_values=None, **kwargs) -> InputEmbeddingsFeatures:
        """text only: the embedding rows (1, T, width) fp32 of a sequence from its first token on"""
        if pixel_values is not None:
            raise ValueError("Nomivik is a text-only decoder")
        eng = self._engine()
        ids = np.asarray(input_ids.cpu() if isinstance(input_ids, torch.Tensor) else input_ids).reshape(-1)
        tok, T = eng.ops.to_device(ids), ids.shape[0]
        if self.config.bigram is None:
            return InputEmbeddingsFeatures(inputs_embeds=eng.ops.embed(tok, self.embed, self.embed_scale).unsqueeze(0))
        ctx = StepCtx(eng.ops, eng.ops.to_device(np.zeros(T)), eng.ops.to_device(np.arange(T)), None, self.eps, [(0, T, 0, 0)])
        b = self.config.bigram
        x = eng.ops.embed_bigram(tok, self.embed, self.embed_scale, self.bigram, b["mul_prev"], b["mul_cur"],
                                 eng.ops.empty((1, TOKEN_STATE)), ctx)[0]
        return InputEmbeddingsFeatures(inputs_embeds=x.unsqueeze(0))
