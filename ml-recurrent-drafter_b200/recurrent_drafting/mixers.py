"""Building blocks of decoders with a 32-bit residual stream: grouped attention over a window or a chunk, latent attention,
the matrix-memory recurrence, dense feed-forwards.  A block owns its weights in the layouts the kernels consume and runs
packed tokens (see StepContext); every constant is a parameter of the block."""
import ctypes
import math
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Tuple

import torch
from torch import nn

from . import _lib, kv_cache
from .modeling_common import Linear


@dataclass
class StepContext:
    """The packed tokens of one step.  Row b of the batch owns tokens [row_start[b], row_start[b+1]); it already holds
    base_len[b] tokens, from slot kv_begin[b] of the cache on."""

    m_max: int
    m_dev: Optional[torch.Tensor]
    tok_row: torch.Tensor
    tok_pos: torch.Tensor
    tok_slot: torch.Tensor
    row_start: torch.Tensor
    kv_begin: torch.Tensor
    base_len: torch.Tensor
    batch: int
    max_new: int
    max_kv: int  # bounds base_len + new tokens of every row; decides nothing but launch shapes
    mode: int
    tree_mask: Optional[torch.Tensor]
    mask_words: int
    n_pos: int
    status: Optional[torch.Tensor]
    ws: Dict[str, torch.Tensor]


@dataclass(frozen=True)
class Visibility:
    """Which earlier positions a query at position p sees: the `size` last ones, its own included (MASK_WINDOW), or those of
    its own chunk of `size` positions (MASK_CHUNK); the sequence's keep_first first ones in any case."""

    kind: int
    size: int
    keep_first: int = 0


def weight(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.empty(*shape), requires_grad=False)


def row_stride(width: int) -> int:
    """Row length of an activation buffer: 16-byte rows in bf16."""
    return (width + 7) // 8 * 8


def rows_of(buffer: torch.Tensor, width: int) -> torch.Tensor:
    """The leading part of a workspace buffer as rows of `width` elements."""
    return buffer.view(-1)[: buffer.shape[0] * width].view(-1, width)


class Scratch:
    """Grow-only device memory that the layers of a model share within a launch."""

    def __init__(self):
        self._buf: Optional[torch.Tensor] = None

    def get(self, nbytes: int, device) -> torch.Tensor:
        if self._buf is None or self._buf.numel() < nbytes or self._buf.device != device:
            self._buf = torch.empty((nbytes + 255) // 256 * 256, dtype=torch.uint8, device=device)
        return self._buf

    def held(self) -> Optional[torch.Tensor]:
        return self._buf


class RotaryTables:
    """cos/sin tables in fp32, formed in fp64 on the host; one pair per (dims, base, head), grown on demand."""

    def __init__(self):
        self._tables: Dict[Tuple[int, float, int], Tuple[torch.Tensor, torch.Tensor]] = {}

    def get(self, dims: int, base: float, n_pos: int, device, head: int = 0) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
        """[n_pos, dims/2], one column per rotated pair; with head given [n_pos, head], one column per feature of the head
        (cos 1, sin 0 past dims)."""
        if dims == 0 and head == 0:
            return None, None
        key = (dims, base, head)
        have = self._tables.get(key)
        if have is None or have[0].shape[0] < n_pos or have[0].device != torch.device(device):
            n = max(n_pos, 2048)
            freq = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
            a = torch.arange(n, dtype=torch.float64)[:, None] * freq[None, :]
            cos, sin = a.cos(), a.sin()
            if head:
                rest = torch.zeros(n, head - dims, dtype=torch.float64)
                cos, sin = torch.cat([cos, cos, rest + 1.0], dim=1), torch.cat([sin, sin, rest], dim=1)
            have = (cos.float().contiguous().to(device), sin.float().contiguous().to(device))
            self._tables[key] = have
        return have

    def held(self) -> List[torch.Tensor]:
        return [t for pair in self._tables.values() for t in pair]


Buffers = Dict[str, Tuple[int, torch.dtype]]  # workspace buffers a block needs: name -> (elements per token, type)


def widest(needs: List[Buffers]) -> Buffers:
    """One set of buffers that serves all blocks."""
    out: Buffers = {}
    for need in needs:
        for name, (width, dtype) in need.items():
            if name in out and out[name][1] != dtype:
                raise ValueError(f"buffer {name} is wanted in two types")
            out[name] = (max(width, out[name][0]) if name in out else width, dtype)
    return out


class _Mixer(nn.Module):
    """What the blocks that mix tokens share."""

    def linears(self) -> List[Linear]:
        return list(self.lin or ())

    def drop_plans(self) -> None:
        """Forgets TMA descriptors of buffers that are about to be replaced."""

    def _commit_planes(self, planes, kv_begin, fp, n_accepted, seq_in_beam, beam_shape) -> None:
        for plane in planes:
            B, heads, max_len, dim = plane.shape
            _lib.call("rd_cache_commit", _lib.dtype_code(plane.dtype), _lib.ptr(plane), B, heads, max_len, dim, _lib.ptr(kv_begin),
                      _lib.ptr(fp.base_len), _lib.ptr(fp.unpacker), beam_shape.width, beam_shape.length, _lib.ptr(n_accepted),
                      _lib.ptr(seq_in_beam), _lib.stream())


class AttentionPlans:
    """TMA descriptors of the tcgen05 attention, by the buffers they address."""

    MAX_PLANS = 8

    def __init__(self, destroy: str = "rd_attention_plan_destroy"):
        self._destroy = destroy
        self._plans: Dict[Tuple, int] = {}

    def get(self, key: Tuple, entry: str, *args) -> int:
        plan = self._plans.get(key)
        if plan is None:
            plan = getattr(_lib.load(), entry)(*args)
            if not plan:
                raise _lib.RedrafterError(f"{entry} failed (TMA descriptor could not be encoded)")
            if len(self._plans) >= self.MAX_PLANS:
                self.drop()
            self._plans[key] = plan
        return plan

    def drop(self) -> None:
        plans, self._plans = self._plans, {}
        if plans:
            destroy = getattr(_lib.load(), self._destroy)
            for p in plans.values():
                destroy(p)

    def __del__(self):
        try:
            self.drop()
        except Exception:
            pass


def attention_desc(ctx: StepContext, visible: Visibility, scale: float, dtype: torch.dtype, **fields) -> _lib.AttentionDesc:
    """A descriptor of the step's tokens; tensors among the fields become pointers."""
    d = _lib.AttentionDesc(dtype=_lib.dtype_code(dtype), B=ctx.batch, max_new=ctx.max_new, max_kv=ctx.max_kv, mode=ctx.mode,
                           mask_words=ctx.mask_words, mask_kind=visible.kind, window=visible.size, keep_first=visible.keep_first,
                           scale=scale)
    tensors = dict(row_start=ctx.row_start, kv_begin=ctx.kv_begin, base_len=ctx.base_len, tok_pos=ctx.tok_pos, tree_mask=ctx.tree_mask)
    for name, v in {**tensors, **fields}.items():
        setattr(d, name, _lib.ptr(v) if v is None or isinstance(v, torch.Tensor) else v)
    return d


def cache_strides(plane: torch.Tensor, name: str) -> Dict[str, int]:
    return {f"{name}_batch": plane.stride(0), f"{name}_head": plane.stride(1), f"{name}_row": plane.stride(2)}


class GroupedAttention(_Mixer):
    """Grouped-query attention with rotary embedding on a part of each head, keys and values of different sizes.  Options:
    one output gate per head (gated), values that are the keys as projected (values_are_keys), queries and keys over
    their root mean square after the rotation (unit_norm_eps), a sink of score 0 in the softmax (zero_sink)."""

    def __init__(self, cfg, width: int, rotary: RotaryTables, visible: Visibility, gated: bool = False, values_are_keys: bool = False,
                 unit_norm_eps: Optional[float] = None, zero_sink: bool = False):
        super().__init__()
        self.cfg, self.rotary, self.visible = cfg, rotary, visible
        self.gated, self.values_are_keys, self.unit_norm_eps, self.zero_sink = gated, values_are_keys, unit_norm_eps, zero_sink
        c = cfg
        if values_are_keys and c.vdim != c.dim:
            raise ValueError(f"values that are the keys have their size: {c.vdim} != {c.dim}")
        parts = {"q": c.heads * c.dim, "k": c.kv_heads * c.dim, "v": 0 if values_are_keys else c.kv_heads * c.vdim,
                 "g": c.heads if gated else 0}
        self.parts = {n: size for n, size in parts.items() if size}  # checkpoint name -> rows of w_in
        self.w_in = weight(sum(self.parts.values()), width)
        self.w_out = weight(width, c.heads * c.vdim)
        self.lin: Optional[Tuple[Linear, Linear]] = None
        self.sink: Optional[torch.Tensor] = None
        self._plans = AttentionPlans()

    def drop_plans(self) -> None:
        self._plans.drop()

    def cache_spec(self) -> kv_cache.LayerSpec:
        return kv_cache.KeyValueSpec(self.cfg.kv_heads, self.cfg.dim, self.cfg.vdim)

    def buffers(self, dtype: torch.dtype) -> Buffers:
        c = self.cfg
        need = {"proj": (row_stride(self.w_in.shape[0]), dtype), "mixed": (c.heads * c.vdim, dtype)}
        if self.gated:
            need["head_gate"] = (row_stride(c.heads), dtype)
        return need

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.w_in.copy_(torch.cat([take(n) for n in self.parts], dim=0))
        self.w_out.copy_(take("o"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        split = torch.split(self.w_in.detach(), list(self.parts.values()), dim=0)
        return {**dict(zip(self.parts, split)), "o": self.w_out.detach()}

    def prepare(self) -> None:
        self.lin = (Linear(self.w_in), Linear(self.w_out))
        self.sink = torch.zeros(self.cfg.heads, dtype=torch.float32, device=self.w_in.device) if self.zero_sink else None

    def run(self, ctx: StepContext, state: kv_cache.LayerKeyValues, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        """out = residual + mixer(xn); residual and out are fp32 rows, xn the normed rows in the model's dtype."""
        mixed = rows_of(ctx.ws["mixed"], self.cfg.heads * self.cfg.vdim)
        if self._heads_of_128() and os.environ.get("RD_FUSED_ROPE", "1") != "0":
            q, gate = self._project_128(ctx, state, xn)
        else:
            q, gate = self._project(ctx, state, xn)
        if self._tensor_core_prompt(ctx, q):
            self._attend_128(ctx, state, q, gate, mixed)
        else:
            self._attend(ctx, state, q, gate, mixed)
        self.lin[1](mixed, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)

    def _project(self, ctx: StepContext, state, xn):
        """Projection, then rotation, norm and cache append.  Returns the queries' rows and the gates."""
        c, st = self.cfg, _lib.stream()
        code, ld = _lib.dtype_code(self.w_in.dtype), row_stride(self.w_in.shape[0])
        proj = rows_of(ctx.ws["proj"], ld)
        self.lin[0](xn, proj, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
        cos, sin = self.rotary.get(c.rot_dims, c.rot_base, ctx.n_pos, xn.device)
        common = (_lib.ptr(proj), ld, _lib.ptr(state.keys), _lib.ptr(state.values), _lib.ptr(ctx.tok_row), _lib.ptr(ctx.tok_pos),
                  _lib.ptr(ctx.tok_slot), _lib.ptr(cos), _lib.ptr(sin), ctx.n_pos, ctx.m_max, _lib.ptr(ctx.m_dev), c.heads, c.kv_heads, c.dim)
        max_len = state.keys.shape[2]
        if self.values_are_keys or self.unit_norm_eps is not None:
            eps = -1.0 if self.unit_norm_eps is None else self.unit_norm_eps
            _lib.call("rd_rotary_norm_append", code, *common, 0 if self.values_are_keys else c.vdim, c.rot_dims, 0, eps, max_len, st)
        else:
            _lib.call("rd_rotary_append", code, *common, c.vdim, c.rot_dims, max_len, st)
        return proj, proj[:, self.w_in.shape[0] - c.heads :] if self.gated else None

    def _heads_of_128(self) -> bool:
        """Heads whose rotation, norm and cache append ride on the projection's epilogue."""
        c, w = self.cfg, self.w_in
        if self.gated == (self.values_are_keys or self.unit_norm_eps is not None) or self.values_are_keys != (self.unit_norm_eps is not None):
            return False  # an option mix without an epilogue of its own
        return (w.dtype == torch.bfloat16 and c.dim == 128 and c.vdim == 128 and c.rot_dims % 16 == 0 and w.shape[1] >= 64
                and w.shape[1] % 8 == 0)

    def _project_128(self, ctx: StepContext, state, xn):
        c = self.cfg
        q = rows_of(ctx.ws["proj"], c.heads * 128)
        cos, sin = self.rotary.get(c.rot_dims, c.rot_base, ctx.n_pos, xn.device, head=128)
        if not self.gated:
            self.lin[0].qk_rope_norm(xn, q, state.keys, state.values, ctx.tok_row, ctx.tok_pos, ctx.tok_slot, cos, sin, c.heads, c.kv_heads,
                                     c.rot_dims, self.unit_norm_eps, ctx.m_dev, ctx.m_max, ctx.status)
            return q, None
        gate = rows_of(ctx.ws["head_gate"], row_stride(c.heads))
        self.lin[0].qkvg_rope(xn, q, state.keys, state.values, gate, ctx.tok_row, ctx.tok_pos, ctx.tok_slot, cos, sin, c.heads, c.kv_heads,
                              c.rot_dims, ctx.m_dev, ctx.m_max, ctx.status)
        return q, gate

    def _tensor_core_prompt(self, ctx: StepContext, q: torch.Tensor) -> bool:
        """Prompts and draft trees of the tcgen05 attention; few tokens take the kernel that shares keys among a group's heads."""
        c, v = self.cfg, self.visible
        tree = ctx.mode == _lib.ATTN_TREE
        return (q.dtype == torch.bfloat16 and c.dim == 128 and c.vdim == 128 and q.stride(0) == c.heads * 128 and c.scale > 0
                and (c.heads // c.kv_heads) * ctx.max_new > 32
                and not (tree and (v.kind != _lib.MASK_WINDOW or v.size < _lib.MAX_BEAM_LENGTH or ctx.mask_words > 16)))

    def _attend(self, ctx: StepContext, state, q, gate, mixed) -> None:
        c = self.cfg
        _lib.attention_masked(attention_desc(
            ctx, self.visible, c.scale, q.dtype, q=q, ldq=q.stride(0), k=state.keys, v=state.values, gate=gate,
            ld_gate=gate.stride(0) if gate is not None else 0, sink=self.sink, out=mixed, nh=c.heads, nkv=c.kv_heads, dim=c.dim, vdim=c.vdim,
            **cache_strides(state.keys, "k"), **cache_strides(state.values, "v")))

    def _attend_128(self, ctx: StepContext, state, q, gate, mixed) -> None:
        c, v = self.cfg, self.visible
        max_len = state.keys.shape[2]
        key = (q.data_ptr(), ctx.m_max, state.keys.data_ptr(), state.values.data_ptr(), ctx.batch, max_len)
        plan = self._plans.get(key, "rd_attention_plan_create", _lib.ptr(q), ctx.m_max, _lib.ptr(state.keys), _lib.ptr(state.values),
                               ctx.batch, c.heads, c.kv_heads, 128, max_len)
        _lib.call("rd_attention_tc_masked", plan, _lib.ptr(mixed), _lib.ptr(ctx.row_start), _lib.ptr(ctx.kv_begin), _lib.ptr(ctx.base_len),
                  ctx.max_new, ctx.mode, _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tree_mask), ctx.mask_words, c.scale, v.kind, v.size,
                  v.keep_first, _lib.ptr(gate), gate.stride(0) if gate is not None else 0, _lib.ptr(self.sink), _lib.ptr(ctx.status),
                  _lib.stream())

    def commit_draft(self, state: kv_cache.LayerKeyValues, kv_begin, fp, n_accepted, seq_in_beam, beam_shape) -> None:
        self._commit_planes((state.keys, state.values), kv_begin, fp, n_accepted, seq_in_beam, beam_shape)


class LatentAttention(_Mixer):
    """Attention whose keys and values are projections of one normed latent per token; a rotated key part is shared by all
    heads, and a learned score per head takes part in the softmax without a value.  The cache holds the latent and the
    rotated part only.

    Prompts of a bf16 model: the latents that their tokens see are gathered and projected up once, and attention runs on
    per-head keys and values.  Few tokens (and fp32 models): the up-projections move to the queries and to the outputs,
    so that all heads read the cached latents themselves."""

    FEW = 32  # new tokens per row up to which the projections move

    def __init__(self, cfg, width: int, eps: float, rotary: RotaryTables, scratch: "Scratch", visible: Visibility, neighbours: bool = True):
        super().__init__()
        self.cfg, self.eps, self.rotary, self.scratch, self.visible, self.neighbours = cfg, eps, rotary, scratch, visible, neighbours
        c = cfg
        self.q_rows = c.heads * (c.dim + c.rot_dim)
        self.width = c.kv_rank + c.rot_dim  # of a cached row
        # latent and key part leave the projection unrounded: they start at a multiple of 32 output features
        self.n_split = (self.q_rows + 31) // 32 * 32
        self.w_in = weight(self.n_split + self.width, width)
        self.w_up = weight(c.heads * (c.dim + c.vdim), c.kv_rank)
        self.w_out = weight(width, c.heads * c.vdim)
        self.norm = weight(c.kv_rank)
        self.sink_scores = weight(c.heads)
        self.lin: Optional[Tuple[Linear, Linear, Linear]] = None
        self.sink: Optional[torch.Tensor] = None
        self.up_k: Optional[torch.Tensor] = None  # [heads, rank, dim]
        self.up_v: Optional[torch.Tensor] = None  # [heads, vdim, rank]
        self._plans = AttentionPlans()
        self._latent_plans = AttentionPlans("rd_attention_latent_plan_destroy")

    def drop_plans(self) -> None:
        self._plans.drop()
        self._latent_plans.drop()

    def cache_spec(self) -> kv_cache.LayerSpec:
        return kv_cache.LatentSpec(self.width)

    def buffers(self, dtype: torch.dtype) -> Buffers:
        c = self.cfg
        return {"proj": (row_stride(self.n_split), dtype), "latent": (row_stride(self.width), torch.float32), "mixed": (c.heads * c.vdim, dtype)}

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.w_in.zero_()
        self.w_in[: self.q_rows].copy_(take("q"))
        self.w_in[self.n_split :].copy_(take("dkv"))
        self.w_up.copy_(torch.cat([take("uk"), take("uv")], dim=0))
        self.w_out.copy_(take("o"))
        self.norm.copy_(take("dkv.norm"))
        self.sink_scores.copy_(take("sink"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        c = self.cfg
        uk, uv = torch.split(self.w_up.detach(), [c.heads * c.dim, c.heads * c.vdim], dim=0)
        return {"q": self.w_in.detach()[: self.q_rows], "dkv": self.w_in.detach()[self.n_split :], "dkv.norm": self.norm.detach(), "uk": uk,
                "uv": uv, "sink": self.sink_scores.detach(), "o": self.w_out.detach()}

    def prepare(self) -> None:
        c = self.cfg
        self.lin = (Linear(self.w_in), Linear(self.w_out), Linear(self.w_up))
        uk, uv = torch.split(self.w_up.detach(), [c.heads * c.dim, c.heads * c.vdim], dim=0)
        self.up_k = uk.view(c.heads, c.dim, c.kv_rank).transpose(1, 2).contiguous()
        self.up_v = uv.view(c.heads, c.vdim, c.kv_rank).contiguous()
        self.sink = self.sink_scores.detach().float().contiguous()

    def run(self, ctx: StepContext, state: kv_cache.LayerLatents, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        c, ws = self.cfg, ctx.ws
        q, dkv = rows_of(ws["proj"], row_stride(self.n_split)), rows_of(ws["latent"], row_stride(self.width))
        mixed = rows_of(ws["mixed"], c.heads * c.vdim)
        self.lin[0].split(xn, q, dkv, self.n_split, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
        (self._expanded if self._expands(ctx) else self._absorbed)(ctx, state, q, dkv, mixed)
        self.lin[1](mixed, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)

    def _append(self, ctx: StepContext, state, q, dkv, q_rot: torch.Tensor, rot_head: int) -> None:
        """Latents and key parts to the cache; the queries' rotated features to q_rot (rows as q_rot's, heads rot_head apart)."""
        c = self.cfg
        cos, sin = self.rotary.get(c.rot_dims, c.rot_base, ctx.n_pos, q.device)
        _lib.call("rd_latent_append", _lib.dtype_code(q.dtype), _lib.ptr(q), q.stride(0), _lib.ptr(q_rot), q_rot.stride(0), rot_head,
                  _lib.ptr(dkv), dkv.stride(0), _lib.ptr(self.norm), self.eps, _lib.ptr(state.rows), _lib.ptr(ctx.tok_row),
                  _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tok_slot), _lib.ptr(cos), _lib.ptr(sin), ctx.n_pos, ctx.m_max, _lib.ptr(ctx.m_dev),
                  c.heads, c.dim, c.rot_dim, c.rot_dims, int(self.neighbours), c.kv_rank, state.rows.shape[2], _lib.stream())

    # ------------------------------------------------------------------------------------- few tokens
    def _absorbed(self, ctx: StepContext, state, q, dkv, mixed) -> None:
        c, code, st = self.cfg, _lib.dtype_code(q.dtype), _lib.stream()
        H, r, m = c.heads, c.kv_rank, ctx.m_max
        n_q, n_o = m * H * self.width, m * H * r
        n_q = (n_q + 7) // 8 * 8
        buf = self.scratch.get((n_q + n_o) * q.element_size(), q.device).view(q.dtype)
        wide, latent = buf[: m * H * self.width].view(m, H * self.width), buf[n_q : n_q + n_o].view(m, H * r)
        self._append(ctx, state, q, dkv, wide[:, r:], self.width)
        _lib.call("rd_head_gemm", code, _lib.ptr(q), q.stride(0), c.dim + c.rot_dim, _lib.ptr(self.up_k), _lib.ptr(wide), wide.stride(0),
                  self.width, m, _lib.ptr(ctx.m_dev), H, r, c.dim, st)
        rows = state.rows
        desc = attention_desc(ctx, self.visible, c.scale, q.dtype, q=wide, ldq=wide.stride(0), k=rows, v=rows, sink=self.sink, out=latent, nh=H,
                              nkv=1, dim=self.width, vdim=r, **cache_strides(rows, "k"), **cache_strides(rows, "v"))
        if q.dtype == torch.bfloat16 and self.width % 8 == 0 and self.width <= 576 and r <= 512:
            key = (wide.data_ptr(), m, rows.data_ptr(), rows.shape)
            plan = self._latent_plans.get(key, "rd_attention_latent_plan_create", _lib.ptr(wide), m * H, _lib.ptr(rows), rows.shape[0] * rows.shape[2],
                                          self.width)
            _lib.call("rd_attention_latent", plan, ctypes.byref(desc), _lib.ptr(ctx.status), st)
        else:
            _lib.attention_masked(desc)
        _lib.call("rd_head_gemm", code, _lib.ptr(latent), latent.stride(0), r, _lib.ptr(self.up_v), _lib.ptr(mixed), mixed.stride(0), c.vdim,
                  m, _lib.ptr(ctx.m_dev), H, c.vdim, r, st)

    # ------------------------------------------------------------------------------------- prompts
    def _expands(self, ctx: StepContext) -> bool:
        c = self.cfg
        if self.w_in.dtype != torch.bfloat16 or ctx.mode != _lib.ATTN_CAUSAL or ctx.max_new <= self.FEW:
            return False
        if c.dim % 8 or c.rot_dim % 8 or c.vdim % 8 or c.kv_rank % 8 or self.visible.keep_first:
            return False
        return self._tensor_core_sizes() or (c.dim + c.rot_dim <= 128 and c.vdim <= 128)

    def _tensor_core_sizes(self) -> bool:
        c = self.cfg
        return c.dim == 128 and c.vdim == 128 and 0 < c.rot_dim <= 64 and c.scale > 0

    def _expanded(self, ctx: StepContext, state, q, dkv, mixed) -> None:
        c, st, H = self.cfg, _lib.stream(), self.cfg.heads
        self._append(ctx, state, q, dkv, q[:, c.dim :], c.dim + c.rot_dim)
        # latents of the new tokens and, from a whole tile on, of the cached ones that the row's first new token sees
        span = min(self.visible.size - 1 + _lib.GATHER_ALIGN - 1, ctx.max_kv)
        n = (ctx.m_max + ctx.batch * span + _lib.GATHER_ALIGN - 1 + 127) // 128 * 128
        up = self.w_up.shape[0]
        head = (4 * (ctx.batch + 1) + 255) // 256 * 256
        esz = q.element_size()
        buf = self.scratch.get(head + n * (self.width + up) * esz, q.device)
        begin, n_out = buf[: 4 * ctx.batch].view(torch.int32), buf[4 * ctx.batch : 4 * ctx.batch + 4].view(torch.int32)
        rows = buf[head : head + n * self.width * esz].view(q.dtype).view(n, self.width)
        kv = buf[head + n * self.width * esz : head + n * (self.width + up) * esz].view(q.dtype).view(n, up)
        _lib.call("rd_latent_gather", _lib.dtype_code(q.dtype), _lib.ptr(state.rows), self.width, state.rows.shape[2], _lib.ptr(ctx.row_start),
                  _lib.ptr(ctx.kv_begin), _lib.ptr(ctx.base_len), ctx.batch, self.visible.kind, self.visible.size, _lib.ptr(rows), n,
                  _lib.ptr(begin), _lib.ptr(n_out), st)
        self.lin[2](rows, kv, m_dev=n_out, m_max=n, status=ctx.status)
        values, tail = kv[:, H * c.dim :], rows[:, c.kv_rank :]
        if self._tensor_core_sizes():
            key = (q.data_ptr(), q.stride(0), ctx.m_max, rows.data_ptr(), n, ctx.batch)
            plan = self._plans.get(key, "rd_attention_tail_plan_create", _lib.ptr(q), q.stride(0), ctx.m_max, _lib.ptr(kv), up, _lib.ptr(tail),
                                   self.width, _lib.ptr(values), up, n, ctx.batch, H, c.rot_dim)
            v = self.visible
            _lib.call("rd_attention_tc_masked", plan, _lib.ptr(mixed), _lib.ptr(ctx.row_start), _lib.ptr(begin), _lib.ptr(ctx.base_len), ctx.max_new,
                      ctx.mode, None, None, 0, c.scale, v.kind, v.size, v.keep_first, None, 0, _lib.ptr(self.sink), _lib.ptr(ctx.status), st)
            return
        _lib.attention_masked(attention_desc(
            ctx, self.visible, c.scale, q.dtype, q=q, ldq=q.stride(0), k=kv, k_head=c.dim, k_row=up, k_tail=tail,
            tail_row=self.width, tail_dim=c.rot_dim, v=values, v_head=c.vdim, v_row=up, sink=self.sink, out=mixed, nh=H, nkv=H,
            dim=c.dim + c.rot_dim, vdim=c.vdim, kv_begin=begin))

    def commit_draft(self, state: kv_cache.LayerLatents, kv_begin, fp, n_accepted, seq_in_beam, beam_shape) -> None:
        self._commit_planes((state.rows,), kv_begin, fp, n_accepted, seq_in_beam, beam_shape)


class MatrixMemory(_Mixer):
    """mLSTM: a matrix state per head with exponential, soft-capped gates, output normalised per head and gated."""

    def __init__(self, cfg, width: int, eps: float, scratch: "Scratch"):
        super().__init__()
        self.cfg, self.eps, self.scratch = cfg, eps, scratch
        c = cfg
        self.sizes = [c.heads * c.dim, c.heads * c.dim, c.heads * c.vdim, c.heads * c.vdim]  # q, k, v, output gate
        main = sum(self.sizes)
        # the recurrence's gates are kept in fp32 by the projection: they start at a multiple of 32 output features
        self.n_split = (main + 31) // 32 * 32
        self.w_in = weight(self.n_split + 2 * c.heads, width)
        self.w_out = weight(width, c.heads * c.vdim)
        self.norm = weight(c.heads * c.vdim)
        self.bias_i = weight(c.heads)
        self.bias_f = weight(c.heads)
        self.lin: Optional[Tuple[Linear, Linear]] = None
        self.bias: Optional[Tuple[torch.Tensor, torch.Tensor]] = None

    def cache_spec(self) -> kv_cache.LayerSpec:
        return kv_cache.MatrixStateSpec(self.cfg.heads, self.cfg.dim, self.cfg.vdim)

    def buffers(self, dtype: torch.dtype) -> Buffers:
        c = self.cfg
        return {"proj": (row_stride(self.n_split), dtype), "gates": (2 * c.heads, torch.float32), "mixed": (c.heads * c.vdim, dtype)}

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.w_in.zero_()
        main = torch.cat([take(n) for n in ("q", "k", "v", "g")], dim=0)
        self.w_in[: main.shape[0]].copy_(main)
        self.w_in[self.n_split :].copy_(torch.cat([take("i"), take("f")], dim=0))
        self.w_out.copy_(take("o"))
        self.norm.copy_(take("norm"))
        self.bias_i.copy_(take("i.b"))
        self.bias_f.copy_(take("f.b"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        w = self.w_in.detach()
        q, k, v, g = torch.split(w[: sum(self.sizes)], self.sizes, dim=0)
        i, f = torch.split(w[self.n_split :], [self.cfg.heads, self.cfg.heads], dim=0)
        return {"q": q, "k": k, "v": v, "g": g, "i": i, "f": f, "o": self.w_out.detach(), "norm": self.norm.detach(),
                "i.b": self.bias_i.detach(), "f.b": self.bias_f.detach()}

    def prepare(self) -> None:
        self.lin = (Linear(self.w_in), Linear(self.w_out))
        self.bias = (self.bias_i.detach().float().contiguous(), self.bias_f.detach().float().contiguous())

    def run(self, ctx: StepContext, state: kv_cache.LayerMatrixState, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        c, ws = self.cfg, ctx.ws
        ld = row_stride(self.n_split)
        tree = ctx.mode == _lib.ATTN_TREE
        if tree:
            # kept until the accepted path is committed
            proj, gates = state.draft_proj, state.draft_gates
            if proj is None or proj.shape[0] < ctx.m_max or proj.shape[1] < self.n_split:
                raise _lib.RedrafterError("the cache was made without room for these draft tokens")
        else:
            proj = rows_of(ws["proj"], ld)
            gates = rows_of(ws["gates"], 2 * c.heads)
        mixed = rows_of(ws["mixed"], c.heads * c.vdim)
        self.lin[0].split(xn, proj, gates, self.n_split, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
        if tree:
            self._tree(ctx, state, proj, gates, mixed)
        elif self._chunked(ctx):
            self._chunk(ctx, state, proj, gates, mixed)
        else:
            self._scan(ctx.batch, ctx.row_start, ctx.base_len, ctx.max_new, state, proj, gates, mixed)
        self.lin[1](mixed, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)

    def _chunked(self, ctx: StepContext) -> bool:
        """Prompts of a bf16 model; portions of a few tokens are run one after the other."""
        c = self.cfg
        return (self.w_in.dtype == torch.bfloat16 and ctx.max_new >= 16 and c.dim % 8 == 0 and c.dim <= 256 and c.vdim % 8 == 0
                and c.vdim <= 512)

    def _common(self, proj, gates, mixed, state, row_start, base_len):
        c = self.cfg
        return (_lib.ptr(proj), proj.stride(0), _lib.ptr(gates), gates.stride(0), _lib.ptr(self.bias[0]), _lib.ptr(self.bias[1]),
                c.gate_cap, _lib.ptr(self.norm), self.eps, _lib.ptr(mixed), _lib.ptr(state.S), _lib.ptr(state.n), _lib.ptr(state.m),
                _lib.ptr(row_start), _lib.ptr(base_len))

    def _chunk(self, ctx: StepContext, state, proj, gates, mixed) -> None:
        c = self.cfg
        need = _lib.load().rd_mlstm_chunk_workspace_bytes(ctx.m_max, ctx.batch, c.heads, c.dim, c.vdim)
        buf = self.scratch.get(need, proj.device)
        _lib.call("rd_mlstm_chunk", *self._common(proj, gates, mixed, state, ctx.row_start, ctx.base_len), ctx.batch, c.heads, c.dim,
                  c.vdim, ctx.m_max, ctx.max_new, _lib.ptr(buf), buf.numel(), _lib.ptr(ctx.status), _lib.stream())

    def _tree(self, ctx: StepContext, state, proj, gates, mixed) -> None:
        c = self.cfg
        buf = self.scratch.get(4 * ctx.m_max * c.heads * c.vdim, proj.device)
        _lib.call("rd_mlstm_tree", _lib.dtype_code(self.w_in.dtype), *self._common(proj, gates, mixed, state, ctx.row_start, ctx.base_len),
                  ctx.batch, c.heads, c.dim, c.vdim, ctx.m_max, _lib.ptr(ctx.tree_mask), ctx.mask_words, _lib.ptr(buf), buf.numel(),
                  _lib.stream())

    def _scan(self, batch, row_start, base_len, max_new, state, proj, gates, mixed, path=(None, 0, 0, None, None)) -> None:
        c = self.cfg
        p, W, Lb, seq, count = path
        _lib.call("rd_mlstm_scan", _lib.dtype_code(self.w_in.dtype), *self._common(proj, gates, mixed, state, row_start, base_len), batch,
                  c.heads, c.dim, c.vdim, max_new, _lib.ptr(p), W, Lb, _lib.ptr(seq), _lib.ptr(count), _lib.stream())

    def commit_draft(self, state: kv_cache.LayerMatrixState, kv_begin, fp, n_accepted, seq_in_beam, beam_shape) -> None:
        self._scan(fp.base_len.shape[0], fp.row_start, fp.base_len, beam_shape.length, state, state.draft_proj, state.draft_gates,
                   None, (fp.unpacker, beam_shape.width, beam_shape.length, seq_in_beam, n_accepted))


class _FeedForward(nn.Module):
    """W_down act(W_up ...), the activation in the first product's epilogue."""

    def __init__(self, width: int, ff: int, up_rows: int):
        super().__init__()
        self.ff = ff
        self.up = weight(up_rows, width)
        self.down = weight(width, ff)
        self.lin: Optional[Tuple[Linear, Linear]] = None

    def buffers(self, dtype: torch.dtype) -> Buffers:
        return {"act": (row_stride(self.ff), dtype)}

    def prepare(self) -> None:
        self.lin = (Linear(self.up), Linear(self.down))

    def linears(self) -> List[Linear]:
        return list(self.lin or ())

    def run(self, ctx: StepContext, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        act = rows_of(ctx.ws["act"], row_stride(self.ff))
        self._activate(ctx, xn, act)
        self.lin[1](act, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)


class DenseFeedForward(_FeedForward):
    """W_down xIELU(W_up h); the activation has two trained numbers."""

    def __init__(self, width: int, ff: int):
        super().__init__(width, ff, ff)
        self.act = weight(2)
        self.coeff = (0.0, 0.0)

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.up.copy_(take("up"))
        self.down.copy_(take("down"))
        self.act.copy_(take("act"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {"up": self.up.detach(), "down": self.down.detach(), "act": self.act.detach()}

    def prepare(self) -> None:
        super().prepare()
        p, q = (float(v) for v in self.act.detach().float().cpu())

        def softplus(z: float) -> float:
            return max(z, 0.0) + math.log1p(math.exp(-abs(z)))

        self.coeff = (softplus(p), 0.5 + softplus(q))

    def _activate(self, ctx: StepContext, xn: torch.Tensor, act: torch.Tensor) -> None:
        self.lin[0].xielu(xn, act, *self.coeff, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)


class ClampedGatedFeedForward(_FeedForward):
    """W_down (g sigmoid(alpha g) (u + 1)), g = W_gate h cut from above and u = W_up h cut on both sides at `limit`."""

    def __init__(self, width: int, ff: int, limit: float, alpha: float):
        super().__init__(width, ff, 2 * ff)  # gate and up rows interleaved
        self.limit, self.alpha = limit, alpha

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.up[0::2].copy_(take("gate"))
        self.up[1::2].copy_(take("up"))
        self.down.copy_(take("down"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {"gate": self.up.detach()[0::2], "up": self.up.detach()[1::2], "down": self.down.detach()}

    def _activate(self, ctx: StepContext, xn: torch.Tensor, act: torch.Tensor) -> None:
        self.lin[0].clamped_glu(xn, act, self.limit, self.alpha, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
