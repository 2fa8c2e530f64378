"""Futidra `Model`: the per-model surface of the package (`language_model`, `get_input_embeddings`, `sanitize`,
`load_weights`, `engine`, `config`) for a text-only decoder of layers that norm the sum of the scaled stream and a
branch (decoder_blocks.NormedSumLayer), with the embedding table as head.  Mixers: grouped attention whose values are the
projected keys (norms per head, paired rotary with frequencies scaled by wavelength, a sliding window, one in the
softmax's denominator); latent attention without positions (a window, a gate per head, its own or an earlier layer's
latent); a delta rule with a decay per head and key channel.  Feed-forward: a relu-gated unit.  All weights are packed
into ONE device arena; the arithmetic is csrc/layer_ops.cu + csrc/mixer_ops.cu driven by `LayerEngine`."""
from __future__ import annotations

from typing import Dict, Optional

import numpy as np
import torch

from ...layer_engine import LayerEngine
from ..base import InputEmbeddingsFeatures
from ..decoder_blocks import ChannelDeltaRule, NormedSumLayer, assign_cache_layers
from ..qwen2_vl.qwen2_vl import WeightArena
from .config import ModelConfig
from .language import LanguageModel

DEFAULT_RANK = 64


class Model:
    norm_offset = 0.0             # the norms' weights are stored plainly
    norm_center = True            # the model's norm takes the mean off, like the layers'

    def __init__(self, config: ModelConfig, device=None, dtype: str = "bfloat16"):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype: 'bfloat16' (serving) or 'float32' (everything in true 32-bit)")
        self.config = config
        self.exact = dtype == "float32"
        self._device = torch.device(device) if device is not None else torch.device("cuda", 0)
        self._eng: Optional[LayerEngine] = None
        self.width, self.vocab = config.width, config.vocab
        self.eps, self.embed_scale, self.logit_softcap = config.norm_eps, 1.0, None
        self.layers = [NormedSumLayer(i, c, config.width, alpha=config.postln_alpha) for i, c in enumerate(config.layers)]
        self.n_cache_layers = assign_cache_layers(self.layers)
        st = 0
        for L in self.layers:     # every recurrent layer gets its span of the slot's state
            L.mixer.state_off, st = st, st + L.state_floats
            if isinstance(L.mixer, ChannelDeltaRule):
                for s in ChannelDeltaRule.LOW_RANK:
                    L.mixer.set_rank(s, L.mixer.rank[s] or DEFAULT_RANK)
        self.state_floats = st
        self.row_dim = (max([L.kv_dim for L in self.layers] + [0]) + 7) // 8 * 8      # rows of whole 16-byte vectors
        self.embed = self.final_norm = self.final_norm_bias = self.head = None
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

    # ------------------------------------------------------------------ weights
    def _globals(self):
        return [("embed", (self.vocab, self.width)), ("final.norm", (self.width,)), ("final.norm.b", (self.width,))]

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
        self.embed, self.final_norm, self.final_norm_bias = view("embed"), view("final.norm"), view("final.norm.b")
        self.head = self.embed        # the logits are products with the embedding rows

    def _ranks_from(self, weights: Dict[str, torch.Tensor]):
        """sizes that only the checkpoint gives: the ranks of the low-rank projections"""
        for i, L in enumerate(self.layers):
            if isinstance(L.mixer, ChannelDeltaRule):
                for s in ChannelDeltaRule.LOW_RANK:
                    t = weights.get(f"l{i}.mix.{s}1")
                    if t is not None and f"{s}_rank" not in self.config.layers[i]["mixer"]:
                        L.mixer.set_rank(s, t.shape[0])

    def load_weights(self, weights: Dict[str, torch.Tensor], strict: bool = True):
        self._ranks_from(weights)
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
        no checkpoint): matrices N(0, 1/fan-in), norm weights around one, decay biases negative, the other vectors small"""
        eng = self._engine()
        g = torch.Generator(device=eng.device).manual_seed(seed)
        with torch.cuda.stream(eng.stream):
            self.arena = WeightArena(self.manifest(), eng.device)
            view = self.arena.view
            for name, shape in self.manifest():
                v = view(name)
                if len(shape) == 1:
                    last = name.rsplit(".", 1)[-1]
                    mean = {"dt_bias": -3.0}.get(last, 1.0 if last.startswith("norm") else 0.0)
                    v.copy_(mean + 0.05 * torch.randn(shape, generator=g, device=eng.device))
                else:
                    s = 1.0 if name == "embed" else 1.0 / float(shape[-1]) ** 0.5
                    for part in (v.unbind(0) if v.numel() > (1 << 28) else (v,)):     # bounded fp32 staging
                        part.copy_(torch.randn(part.shape, generator=g, device=eng.device) * s)
            self._bind(view)
        eng.stream.synchronize()
        return self

    # ------------------------------------------------------------------ inputs
    def get_input_embeddings(self, input_ids=None, pixel_values=None, **kwargs) -> InputEmbeddingsFeatures:
        """text only: the embedding rows (1, T, width) fp32"""
        if pixel_values is not None:
            raise ValueError("Futidra is a text-only decoder")
        eng = self._engine()
        ids = np.asarray(input_ids.cpu() if isinstance(input_ids, torch.Tensor) else input_ids).reshape(-1)
        x = eng.ops.embed(eng.ops.to_device(ids), self.embed, self.embed_scale)
        return InputEmbeddingsFeatures(inputs_embeds=x.unsqueeze(0))
