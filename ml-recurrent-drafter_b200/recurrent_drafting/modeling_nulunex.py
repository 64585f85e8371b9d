"""The Nulunex decoder on the B200 kernels: chunked grouped attention whose values are the keys and latent attention over a
sliding window, clamped gated feed-forwards, a plain 32-bit residual stream; layers may share their weights."""
from typing import List, Optional

import torch

from . import _lib, mixers
from .configuration_nulunex import GLU_ALPHA, LayerConfig, NulunexConfig
from .modeling_stream import StreamDecoder, StreamLayer


class NulunexForCausalLM(StreamDecoder):
    config_class = NulunexConfig

    def _make_layers(self) -> List[StreamLayer]:
        owners = [self.config.owner(i) for i in range(self.n_layers)]
        made = {i: self._make_layer(self.config.layers[i]) for i in sorted(set(owners))}
        return [made[i] for i in owners]

    def _make_layer(self, cfg: LayerConfig) -> StreamLayer:
        H, eps, c = self.config.hidden_size, self.config.norm_eps, cfg.mixer
        mixer: torch.nn.Module
        if cfg.type == "attention":
            mixer = mixers.GroupedAttention(c, H, self.rotary, mixers.Visibility(_lib.MASK_CHUNK, c.chunk), values_are_keys=True,
                                            unit_norm_eps=eps, zero_sink=True)
        else:
            mixer = mixers.LatentAttention(c, H, eps, self.rotary, self.scratch, mixers.Visibility(_lib.MASK_WINDOW, c.window))
        mlp: Optional[torch.nn.Module] = None
        if cfg.mlp is not None:
            mlp = mixers.ClampedGatedFeedForward(H, cfg.mlp.ff, cfg.mlp.limit, GLU_ALPHA)
        return StreamLayer(H, mixer, mlp)

    def _owners(self):
        return [(i, self.layers[i]) for i in sorted({self.config.owner(i) for i in range(self.n_layers)})]

    def _run_layers(self, ctx, cache, tok_ids, layer_outputs) -> None:
        ws = ctx.ws
        x, xn = ws["x"], ws["xn"]
        self._norm(ctx, self.layers[0].norm1, xn, x_out=x, ids=tok_ids)
        for i, l in enumerate(self.layers):
            l.mixer.run(ctx, cache.layers[i], xn, x, x)
            if l.mlp is not None:
                self._norm(ctx, l.norm2, xn, src=x)
                l.mlp.run(ctx, xn, x, x)
            if layer_outputs is not None:
                layer_outputs.append(x[: ctx.m_max].clone())
            last = i + 1 == self.n_layers
            self._norm(ctx, self.final_norm if last else self.layers[i + 1].norm1, ws["hidden"] if last else xn, src=x)
