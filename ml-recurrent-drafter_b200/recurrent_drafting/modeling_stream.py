"""What the decoders with a 32-bit residual stream share: layers of norm1 + mixer and norm2 + feed-forward built from the
blocks of mixers.py, checkpoint names, workspace, and the interface the decode loops use (backbone, heads, new_cache,
commit_draft, workspace), so that prefill, autoregressive decoding, speculative decoding and the trace runner serve them as
they serve LlamaForCausalLM."""
from typing import Callable, Dict, List, Optional, Tuple

import torch
from torch import nn

from . import _lib, checkpoint, kv_cache, mixers
from .modeling_common import Linear, LMHead


class StreamLayer(nn.Module):
    """norm1 + mixer, optionally norm2 + feed-forward."""

    def __init__(self, width: int, mixer: nn.Module, mlp: Optional[nn.Module]):
        super().__init__()
        self.mixer, self.mlp = mixer, mlp
        self.norm1 = mixers.weight(width)
        self.norm2 = mixers.weight(width) if mlp is not None else None

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        """take(name): the layer's tensor of that name in the checkpoint."""
        self.norm1.copy_(take("norm1"))
        self.mixer.load(lambda n: take("mix." + n))
        if self.mlp is not None:
            self.norm2.copy_(take("norm2"))
            self.mlp.load(lambda n: take("mlp." + n))

    def tensors(self) -> Dict[str, torch.Tensor]:
        out = {"norm1": self.norm1.detach(), **{"mix." + n: v for n, v in self.mixer.tensors().items()}}
        if self.mlp is not None:
            out["norm2"] = self.norm2.detach()
            out.update({"mlp." + n: v for n, v in self.mlp.tensors().items()})
        return out

    def linears(self) -> List[Linear]:
        return self.mixer.linears() + (self.mlp.linears() if self.mlp is not None else [])


class StreamDecoder(LMHead, nn.Module):
    """A subclass names its configuration class, makes its layers and runs them (_run_layers).  Several places of the
    stack may hold the same layer object: they share its weights and have a cache or state each."""

    config_class = None
    norm_groups = 1
    positions_are_columns = False  # positions count from each sequence's first real token

    def __init__(self, config):
        super().__init__()
        self.config = config
        H = config.hidden_size
        self.n_layers = config.num_hidden_layers
        self.embed_tokens = nn.Embedding(config.vocab_size, H)
        self.embed_tokens.weight.requires_grad_(False)
        self.rotary, self.scratch = mixers.RotaryTables(), mixers.Scratch()
        self.layers = nn.ModuleList(self._make_layers())
        self.final_norm = mixers.weight(H)
        self.lm_head = nn.Linear(H, config.vocab_size, bias=False)
        self.lm_head.weight.requires_grad_(False)
        self.gemm_status: Optional[torch.Tensor] = None
        self._invalidate()

    # ----------------------------------------------------------------- what a subclass provides
    def _make_layers(self) -> List[StreamLayer]:
        raise NotImplementedError

    def _run_layers(self, ctx: mixers.StepContext, cache: kv_cache.HybridCache, tok_ids: torch.Tensor,
                    layer_outputs: Optional[List[torch.Tensor]]) -> None:
        """From token ids to the post-norm hidden states in ctx.ws["hidden"]."""
        raise NotImplementedError

    def _own_buffers(self) -> mixers.Buffers:
        H, f32 = self.config.hidden_size, torch.float32
        return {"x": (H, f32), "mid": (H, f32), "xn": (H, self.dtype), "hidden": (H, self.dtype)}

    def _extra_buffers(self, rows: int) -> Dict[str, torch.Tensor]:
        """Buffers that are not [rows, width]."""
        return {}

    def _init_parameter(self, leaf: str, prm: torch.Tensor, normal: Callable[[torch.Tensor, float], None], std: float) -> None:
        if prm.ndim == 1:
            prm.fill_(1.0)
        else:
            normal(prm, std)

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

    def held_buffers(self) -> List[Optional[torch.Tensor]]:
        """Device memory besides the workspace that captured launches address."""
        return [self.scratch.held()] + self.rotary.held()

    def new_cache(self, batch_size: int, max_length: int, draft_tokens: int = 0, device=None) -> kv_cache.HybridCache:
        return kv_cache.HybridCache([l.mixer.cache_spec() for l in self.layers], batch_size, max_length, self.dtype,
                                    self.device if device is None else device, draft_tokens=draft_tokens)

    def commit_draft(self, cache: kv_cache.HybridCache, fp, n_accepted, seq_in_beam, beam_shape, kv_begin=None) -> None:
        """After acceptance: what the cache holds of the accepted path moves to the tail of its row, recurrent states take
        its tokens in."""
        for l, state in zip(self.layers, cache.layers):
            l.mixer.commit_draft(state, kv_begin, fp, n_accepted, seq_in_beam, beam_shape)

    # ----------------------------------------------------------------- weights
    def _owners(self) -> List[Tuple[int, StreamLayer]]:
        """(index under which the checkpoint names its tensors, layer) of every layer with weights of its own."""
        return [(i, l) for i, l in enumerate(self.layers) if not any(l is e for e in list(self.layers)[:i])]

    def init_random(self, std: float = 0.02, seed: int = 0) -> "StreamDecoder":
        """Random weights in place: matrices normal(0, std), norms 1, the rest as the subclass says."""
        g = torch.Generator(device=self.device).manual_seed(seed)

        def normal(prm: torch.Tensor, s: float) -> None:
            prm.copy_(torch.randn(prm.shape, generator=g, device=prm.device, dtype=torch.float32).mul_(s))

        for name, prm in self.named_parameters():
            self._init_parameter(name.rsplit(".", 1)[-1], prm, normal, std)
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
            for i, l in self._owners():
                l.load(lambda n: take(f"l{i}.{n}"))
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
        for i, l in self._owners():
            sd.update({f"l{i}.{n}": v for n, v in l.tensors().items()})
        sd["final.norm"] = self.final_norm.detach()
        sd["head"] = self.lm_head.weight.detach()
        return {k: v.clone() for k, v in sd.items()}

    @classmethod
    def from_pretrained(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16, device="cuda") -> "StreamDecoder":
        with torch.device(device):
            model = cls(cls.config_class.from_pretrained(path)).to(torch_dtype)
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
        self._ws: Dict[Tuple[int, int], Dict[str, torch.Tensor]] = {}
        self._ws_full: Dict[str, torch.Tensor] = {}
        self._ws_cap: Tuple[int, int] = (0, 0)
        self._head_ws: Optional[torch.Tensor] = None

    def _prepare(self) -> None:
        if self._ready:
            return
        for _, l in self._owners():
            l.mixer.prepare()
            if l.mlp is not None:
                l.mlp.prepare()
        self._head = Linear(self.lm_head.weight)
        self._ready = True

    def _lin(self) -> Dict[str, Linear]:
        self._prepare()
        return {"head": self._head}

    def _drop_plans(self) -> None:
        if self._ready:
            for _, l in self._owners():
                l.mixer.drop_plans()
                for lin in l.linears():
                    lin.drop_plans()
            self._head.drop_plans()

    def workspace(self, m_max: int, logit_rows: int) -> Dict[str, torch.Tensor]:
        """Activation buffers for m_max packed tokens and fp32 logits for logit_rows rows: one grow-only set, smaller
        requests get its leading part."""
        key = (m_max, logit_rows)
        ws = self._ws.get(key)
        if ws is not None:
            return ws
        dev = self.device
        cap_m, cap_l = self._ws_cap
        full = dict(self._ws_full)
        extra = self._extra_buffers(0)
        if m_max > cap_m:
            cap_m = m_max
            needs = [self._own_buffers()] + [b.buffers(self.dtype) for _, l in self._owners() for b in (l.mixer, l.mlp) if b is not None]
            for name, (width, t) in mixers.widest(needs).items():
                full[name] = torch.empty(cap_m, width, dtype=t, device=dev)
            full.update(self._extra_buffers(cap_m))
        if logit_rows > cap_l:
            cap_l = logit_rows
            full["logits"] = torch.empty(cap_l, self.config.vocab_size, dtype=torch.float32, device=dev)
        if (cap_m, cap_l) != self._ws_cap:
            self._ws_full, self._ws_cap = full, (cap_m, cap_l)
            self._ws = {}
            self._drop_plans()
        ws = {k: (v[:logit_rows] if k == "logits" else v if k in extra else v[:m_max]) for k, v in full.items()}
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
        ctx = mixers.StepContext(m_max, m_dev, tok_row, tok_pos, tok_slot, row_start, kv_begin, base_len, batch, max_new, max_kv,
                                 mode, tree_mask, mask_words, n_pos, self.gemm_status, ws)
        self._run_layers(ctx, cache, tok_ids, layer_outputs)
        return ws["hidden"]

    def _norm(self, ctx: mixers.StepContext, weight: torch.Tensor, y: torch.Tensor, src: Optional[torch.Tensor] = None, x_out=None,
              coeff: Optional[torch.Tensor] = None, n_hist: int = 1, hist_stride: int = 0, ids=None, scale: float = 1.0) -> None:
        """y = norm(x) * weight in the model's dtype, with x a row of src, a weighted sum of n_hist rows hist_stride apart, or
        (ids given) a scaled embedding; x_out, when given, receives x."""
        _lib.call("rd_stream_norm", _lib.dtype_code(self.dtype), _lib.ptr(self.embed_tokens.weight) if ids is not None else None,
                  _lib.ptr(ids), scale, _lib.ptr(src), hist_stride, _lib.ptr(coeff), n_hist, _lib.ptr(x_out), _lib.ptr(weight), _lib.ptr(y),
                  ctx.m_max, _lib.ptr(ctx.m_dev), self.config.hidden_size, self.norm_groups, self.config.norm_eps, _lib.stream())
