"""The Dilavik decoder on the B200 kernels: window attention and matrix-memory layers over a 32-bit residual stream whose
input to every layer is a weighted sum of all earlier layers' results.

The model offers the interface the decode loops use (backbone, heads, new_cache, commit_draft, workspace), so prefill,
autoregressive decoding, speculative decoding and the trace runner serve it as they serve LlamaForCausalLM."""
from typing import Dict, List, Optional, Tuple

import torch
from torch import nn

from . import _lib, checkpoint, kv_cache, mixers
from .configuration_dilavik import DilavikConfig
from .modeling_common import Linear, LMHead


class DecoderLayer(nn.Module):
    """norm1 + mixer, optionally norm2 + feed-forward, and the depth-average coefficients of what goes on."""

    def __init__(self, cfg, index: int, model_cfg: DilavikConfig, rotary: mixers.RotaryTables, scratch: mixers.Scratch):
        super().__init__()
        H = model_cfg.hidden_size
        if cfg.type == "attention":
            self.mixer = mixers.WindowAttention(cfg.mixer, H, rotary)
        else:
            self.mixer = mixers.MatrixMemory(cfg.mixer, H, model_cfg.norm_eps, scratch)
        self.mlp = mixers.DenseFeedForward(H, cfg.ff) if cfg.ff is not None else None
        self.norm1 = mixers.weight(H)
        self.norm2 = mixers.weight(H) if cfg.ff is not None else None
        self.dwa = mixers.weight(index + 2)


class DilavikForCausalLM(LMHead, nn.Module):
    config_class = DilavikConfig
    positions_are_columns = False  # positions count from each sequence's first real token

    def __init__(self, config: DilavikConfig):
        super().__init__()
        self.config = config
        H = config.hidden_size
        self.n_layers = config.num_hidden_layers
        self.embed_tokens = nn.Embedding(config.vocab_size, H)
        self.embed_tokens.weight.requires_grad_(False)
        self.rotary, self.scratch = mixers.RotaryTables(), mixers.Scratch()
        self.layers = nn.ModuleList([DecoderLayer(c, i, config, self.rotary, self.scratch) for i, c in enumerate(config.layers)])
        self.final_norm = mixers.weight(H)
        self.lm_head = nn.Linear(H, config.vocab_size, bias=False)
        self.lm_head.weight.requires_grad_(False)
        self.gemm_status: Optional[torch.Tensor] = None
        self._invalidate()

    # ----------------------------------------------------------------- surface shared with the other base models
    @property
    def base_model(self):
        return self

    @property
    def dtype(self) -> torch.dtype:
        return self.lm_head.weight.dtype

    @property
    def device(self) -> torch.device:
        return self.lm_head.weight.device

    def get_input_embeddings(self):
        return self.embed_tokens

    def get_output_embeddings(self):
        return self.lm_head

    @property
    def graph_capturable(self) -> bool:
        return True  # no kernel of a step is sized by the live sequence length

    def new_cache(self, batch_size: int, max_length: int, draft_tokens: int = 0, device=None) -> kv_cache.HybridCache:
        return kv_cache.HybridCache([l.mixer.cache_spec() for l in self.layers], batch_size, max_length, self.dtype,
                                    self.device if device is None else device, draft_tokens=draft_tokens)

    # ----------------------------------------------------------------- weights
    def init_random(self, std: float = 0.02, seed: int = 0) -> "DilavikForCausalLM":
        """Random weights in place: matrices normal(0, std), norms 1, gate biases that remember, and a depth average that
        is mostly the layer's own result."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def normal(prm: torch.Tensor, s: float) -> None:
            prm.copy_(torch.randn(prm.shape, generator=g, device=prm.device, dtype=torch.float32).mul_(s))

        for name, prm in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf == "dwa":
                normal(prm, 0.1)
                prm[-1] += 1.0
            elif leaf == "bias_f":
                normal(prm, 1.0)
                prm += 4.0
            elif leaf in ("bias_i", "act"):
                normal(prm, 0.5)
            elif prm.ndim == 1:
                prm.fill_(1.0)
            else:
                normal(prm, std)
        self._invalidate()
        return self

    def load_state_dict(self, state_dict, strict: bool = True, assign: bool = False):
        """Accepts the checkpoint's names ('l<i>.mix.q', ...) and packs them into the kernel layouts."""
        sd = state_dict if isinstance(state_dict, checkpoint.LazyCheckpoint) else dict(state_dict)
        if "lm_head.weight" in sd:  # this module's own layout
            out = super().load_state_dict(sd, strict=strict)
            self._invalidate()
            return out

        def take(name: str) -> torch.Tensor:
            return sd.pop(name).to(device=self.device, dtype=self.dtype)

        with torch.no_grad():
            self.embed_tokens.weight.copy_(take("embed"))
            for i, l in enumerate(self.layers):
                pre = f"l{i}."
                l.norm1.copy_(take(pre + "norm1"))
                l.mixer.load(lambda n: take(pre + "mix." + n))
                if l.mlp is not None:
                    l.norm2.copy_(take(pre + "norm2"))
                    l.mlp.load(lambda n: take(pre + "mlp." + n))
                l.dwa.copy_(take(pre + "dwa"))
            self.final_norm.copy_(take("final.norm"))
            self.lm_head.weight.copy_(take("head"))
        leftover = list(sd.keys())
        if strict and leftover:
            raise KeyError(f"unexpected keys in state dict: {leftover[:5]}")
        self._invalidate()
        return leftover

    def checkpoint_state_dict(self) -> Dict[str, torch.Tensor]:
        """The weights under the checkpoint's names."""
        sd = {"embed": self.embed_tokens.weight.detach()}
        for i, l in enumerate(self.layers):
            pre = f"l{i}."
            sd[pre + "norm1"] = l.norm1.detach()
            sd.update({pre + "mix." + n: v for n, v in l.mixer.tensors().items()})
            if l.mlp is not None:
                sd[pre + "norm2"] = l.norm2.detach()
                sd.update({pre + "mlp." + n: v for n, v in l.mlp.tensors().items()})
            sd[pre + "dwa"] = l.dwa.detach()
        sd["final.norm"] = self.final_norm.detach()
        sd["head"] = self.lm_head.weight.detach()
        return {k: v.clone() for k, v in sd.items()}

    @classmethod
    def from_pretrained(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16, device="cuda") -> "DilavikForCausalLM":
        with torch.device(device):
            model = cls(DilavikConfig.from_pretrained(path)).to(torch_dtype)
        model.load_state_dict(checkpoint.LazyCheckpoint(path))
        return model

    def save_pretrained(self, path: str) -> None:
        checkpoint.save_directory(path, self.config, self.checkpoint_state_dict())

    # ----------------------------------------------------------------- derived state
    def _apply(self, fn, *args, **kwargs):
        out = super()._apply(fn, *args, **kwargs)
        self._invalidate()
        return out

    def _invalidate(self) -> None:
        self._ready = False
        self._head: Optional[Linear] = None
        self._dwa: List[torch.Tensor] = []
        self._ws: Dict[Tuple[int, int], Dict[str, torch.Tensor]] = {}
        self._ws_full: Dict[str, torch.Tensor] = {}
        self._ws_cap: Tuple[int, int] = (0, 0)
        self._head_ws: Optional[torch.Tensor] = None

    def _prepare(self) -> None:
        if self._ready:
            return
        for l in self.layers:
            l.mixer.prepare()
            if l.mlp is not None:
                l.mlp.prepare()
        self._dwa = [l.dwa.detach().float().contiguous() for l in self.layers]
        self._head = Linear(self.lm_head.weight)
        self._ready = True

    def _lin(self) -> Dict[str, Linear]:
        self._prepare()
        return {"head": self._head}

    def _drop_plans(self) -> None:
        if self._ready:
            for l in self.layers:
                if isinstance(l.mixer, mixers.WindowAttention):
                    l.mixer.drop_plans()
                for lin in l.mixer.linears() + (l.mlp.linears() if l.mlp is not None else []):
                    lin.drop_plans()
            self._head.drop_plans()

    def workspace(self, m_max: int, logit_rows: int) -> Dict[str, torch.Tensor]:
        """Activation buffers for m_max packed tokens and fp32 logits for logit_rows rows: one grow-only set, smaller
        requests get its leading part."""
        key = (m_max, logit_rows)
        ws = self._ws.get(key)
        if ws is not None:
            return ws
        H, dt, dev = self.config.hidden_size, self.dtype, self.device
        cap_m, cap_l = self._ws_cap
        full = dict(self._ws_full)
        if m_max > cap_m:
            cap_m = m_max
            mix = [l.mixer for l in self.layers]
            gates = max([2 * m.cfg.heads for m in mix if isinstance(m, mixers.MatrixMemory)] or [1])
            for name, width, t in (("x", H, torch.float32), ("mid", H, torch.float32), ("xn", H, dt), ("hidden", H, dt),
                                   ("proj", max(mixers.row_stride(m.proj_width()) for m in mix), dt), ("gates", gates, torch.float32),
                                   ("head_gate", mixers.row_stride(max([m.cfg.heads for m in mix if isinstance(m, mixers.WindowAttention)] or [1])), dt),
                                   ("mixed", max(m.out_width() for m in mix), dt),
                                   ("act", mixers.row_stride(max([l.mlp.ff for l in self.layers if l.mlp is not None] or [1])), dt)):
                full[name] = torch.empty(cap_m, width, dtype=t, device=dev)
            # the embedding output and every layer's result, which the depth averages read
            full["hist"] = torch.empty(self.n_layers + 1, cap_m, H, dtype=torch.float32, device=dev)
        if logit_rows > cap_l:
            cap_l = logit_rows
            full["logits"] = torch.empty(cap_l, self.config.vocab_size, dtype=torch.float32, device=dev)
        if (cap_m, cap_l) != self._ws_cap:
            self._ws_full, self._ws_cap = full, (cap_m, cap_l)
            self._ws = {}
            self._drop_plans()
        ws = {k: (v[:logit_rows] if k == "logits" else v if k == "hist" else v[:m_max]) for k, v in full.items()}
        if len(self._ws) >= 16:
            self._ws.pop(next(iter(self._ws)))
        self._ws[key] = ws
        return ws

    # ----------------------------------------------------------------- forward
    def backbone(self, ws, cache: kv_cache.HybridCache, m_max: int, m_dev, tok_ids, tok_row, tok_pos, tok_slot, row_start, kv_begin,
                 base_len, batch: int, max_new: int, max_kv: int, mode: int, tree_mask=None, mask_words: int = 0,
                 n_pos: int = 4096, layer_outputs: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Embedding, all layers and the final norm over m_max (or *m_dev) packed tokens; keys, values and recurrent states
        of their rows are extended.  Returns the post-norm hidden states.  In mode ATTN_TREE (verification of a packed
        draft) the recurrent states stay as they are until commit_draft().  layer_outputs, a list, receives a copy of the
        residual stream after every layer."""
        self._prepare()
        code, st = _lib.dtype_code(self.dtype), _lib.stream()
        H, groups, eps = self.config.hidden_size, self.config.norm_groups, self.config.norm_eps
        ctx = mixers.StepContext(m_max, m_dev, tok_row, tok_pos, tok_slot, row_start, kv_begin, base_len, batch, max_new, max_kv,
                                 mode, tree_mask, mask_words, n_pos, self.gemm_status, ws)
        md = _lib.ptr(m_dev)
        hist, x, mid, xn = ws["hist"], ws["x"], ws["mid"], ws["xn"]
        stride = hist.stride(0)

        def norm(src, coeff, n_hist, x_out, weight, y):
            _lib.call("rd_stream_norm", code, None, None, 0.0, _lib.ptr(src), stride, _lib.ptr(coeff), n_hist, _lib.ptr(x_out),
                      _lib.ptr(weight), _lib.ptr(y), m_max, md, H, groups, eps, st)

        _lib.call("rd_stream_norm", code, _lib.ptr(self.embed_tokens.weight), _lib.ptr(tok_ids), self.config.embedding_scale, None, 0,
                  None, 0, _lib.ptr(hist[0]), _lib.ptr(self.layers[0].norm1), _lib.ptr(xn), m_max, md, H, groups, eps, st)
        residual = hist[0]
        for i, l in enumerate(self.layers):
            result = hist[i + 1]
            l.mixer.run(ctx, cache.layers[i], xn, residual, result if l.mlp is None else mid)
            if l.mlp is not None:
                norm(mid, None, 1, None, l.norm2, xn)
                l.mlp.run(ctx, xn, mid, result)
            last = i + 1 == self.n_layers
            keep = not last or layer_outputs is not None
            norm(hist, self._dwa[i], i + 2, x if keep else None, self.final_norm if last else self.layers[i + 1].norm1,
                 ws["hidden"] if last else xn)
            residual = x
            if layer_outputs is not None:
                layer_outputs.append(x[:m_max].clone())
        return ws["hidden"]

    def commit_draft(self, cache: kv_cache.HybridCache, fp, n_accepted, seq_in_beam, beam_shape, kv_begin=None) -> None:
        """After acceptance: keys and values of the accepted path move to the tail of their row, recurrent states take its
        tokens in."""
        for l, state in zip(self.layers, cache.layers):
            l.mixer.commit_draft(state, kv_begin, fp, n_accepted, seq_in_beam, beam_shape)
