"""The Dilavik decoder on the B200 kernels: window attention and matrix-memory layers over a 32-bit residual stream whose
input to every layer is a weighted sum of all earlier layers' results."""
from typing import Dict, List

import torch

from . import _lib, mixers
from .configuration_dilavik import DilavikConfig
from .modeling_stream import StreamDecoder, StreamLayer


class DecoderLayer(StreamLayer):
    """A layer and the depth-average coefficients of what goes on after it."""

    def __init__(self, cfg, index: int, model_cfg: DilavikConfig, rotary: mixers.RotaryTables, scratch: mixers.Scratch):
        H, c = model_cfg.hidden_size, cfg.mixer
        if cfg.type == "attention":
            visible = mixers.Visibility(_lib.MASK_WINDOW, c.window, c.keep_first)
            mixer = mixers.GroupedAttention(c, H, rotary, visible, gated=True)
        else:
            mixer = mixers.MatrixMemory(c, H, model_cfg.norm_eps, scratch)
        super().__init__(H, mixer, mixers.DenseFeedForward(H, cfg.ff) if cfg.ff is not None else None)
        self.dwa = mixers.weight(index + 2)

    def load(self, take) -> None:
        super().load(take)
        self.dwa.copy_(take("dwa"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {**super().tensors(), "dwa": self.dwa.detach()}


class DilavikForCausalLM(StreamDecoder):
    config_class = DilavikConfig

    @property
    def norm_groups(self) -> int:
        return self.config.norm_groups

    def _make_layers(self) -> List[DecoderLayer]:
        return [DecoderLayer(c, i, self.config, self.rotary, self.scratch) for i, c in enumerate(self.config.layers)]

    def _init_parameter(self, leaf, prm, normal, std) -> None:
        """Gate biases that remember, and a depth average that is mostly the layer's own result."""
        if leaf == "dwa":
            normal(prm, 0.1)
            prm[-1] += 1.0
        elif leaf == "bias_f":
            normal(prm, 1.0)
            prm += 4.0
        elif leaf in ("bias_i", "act"):
            normal(prm, 0.5)
        else:
            super()._init_parameter(leaf, prm, normal, std)

    def _invalidate(self) -> None:
        super()._invalidate()
        self._dwa: List[torch.Tensor] = []

    def _prepare(self) -> None:
        if not self._ready:
            self._dwa = [l.dwa.detach().float().contiguous() for l in self.layers]
        super()._prepare()

    def _extra_buffers(self, rows: int) -> Dict[str, torch.Tensor]:
        # the embedding output and every layer's result, which the depth averages read
        return {"hist": torch.empty(self.n_layers + 1, rows, self.config.hidden_size, dtype=torch.float32, device=self.device)}

    def _run_layers(self, ctx, cache, tok_ids, layer_outputs) -> None:
        ws = ctx.ws
        hist, x, mid, xn = ws["hist"], ws["x"], ws["mid"], ws["xn"]
        self._norm(ctx, self.layers[0].norm1, xn, x_out=hist[0], ids=tok_ids, scale=self.config.embedding_scale)
        residual = hist[0]
        for i, l in enumerate(self.layers):
            result = hist[i + 1]
            l.mixer.run(ctx, cache.layers[i], xn, residual, result if l.mlp is None else mid)
            if l.mlp is not None:
                self._norm(ctx, l.norm2, xn, src=mid)
                l.mlp.run(ctx, xn, mid, result)
            last = i + 1 == self.n_layers
            keep = not last or layer_outputs is not None
            self._norm(ctx, self.final_norm if last else self.layers[i + 1].norm1, ws["hidden"] if last else xn, src=hist,
                       x_out=x if keep else None, coeff=self._dwa[i], n_hist=i + 2, hist_stride=hist.stride(0))
            residual = x
            if layer_outputs is not None:
                layer_outputs.append(x[: ctx.m_max].clone())
