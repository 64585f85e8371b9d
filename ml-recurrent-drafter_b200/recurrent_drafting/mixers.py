"""Building blocks of decoders with a 32-bit residual stream: sliding-window attention with kept first tokens, the
matrix-memory recurrence, the dense xIELU feed-forward.  A block owns its weights in the layouts the kernels consume
and runs packed tokens (see StepContext); every constant is a parameter of the block."""
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


class WindowAttention(nn.Module):
    """Grouped-query attention over a sliding window plus the sequence's first tokens, rotary embedding on a part of each
    head, keys and values of different sizes, one output gate per head."""

    def __init__(self, cfg, width: int, rotary: RotaryTables):
        super().__init__()
        self.cfg = cfg
        self.rotary = rotary
        c = cfg
        self.sizes = [c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim, c.heads]  # q, k, v, gate
        self.w_in = weight(sum(self.sizes), width)
        self.w_out = weight(width, c.heads * c.vdim)
        self.lin: Optional[Tuple[Linear, Linear]] = None
        self._plans: Dict[Tuple, int] = {}  # TMA descriptors of the tcgen05 attention, by the buffers they address

    def drop_plans(self) -> None:
        plans, self._plans = self._plans, {}
        if plans:
            lib = _lib.load()
            for p in plans.values():
                lib.rd_attention_plan_destroy(p)

    def __del__(self):
        try:
            self.drop_plans()
        except Exception:
            pass

    def cache_spec(self) -> kv_cache.LayerSpec:
        return kv_cache.KeyValueSpec(self.cfg.kv_heads, self.cfg.dim, self.cfg.vdim)

    def proj_width(self) -> int:
        return sum(self.sizes)

    def out_width(self) -> int:
        return self.cfg.heads * self.cfg.vdim

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.w_in.copy_(torch.cat([take(n) for n in ("q", "k", "v", "g")], dim=0))
        self.w_out.copy_(take("o"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        q, k, v, g = torch.split(self.w_in.detach(), self.sizes, dim=0)
        return {"q": q, "k": k, "v": v, "g": g, "o": self.w_out.detach()}

    def prepare(self) -> None:
        self.lin = (Linear(self.w_in), Linear(self.w_out))

    def linears(self) -> List[Linear]:
        return list(self.lin or ())

    def run(self, ctx: StepContext, state: kv_cache.LayerKeyValues, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        """out = residual + mixer(xn); residual and out are fp32 rows, xn the normed rows in the model's dtype."""
        c, ws, st = self.cfg, ctx.ws, _lib.stream()
        if self._heads_of_128() and os.environ.get("RD_FUSED_ROPE", "1") != "0":
            self._run_128(ctx, state, xn, residual, out)
            return
        code = _lib.dtype_code(self.w_in.dtype)
        ld = row_stride(self.proj_width())
        proj = rows_of(ws["proj"], ld)
        mixed = rows_of(ws["mixed"], self.out_width())
        self.lin[0](xn, proj, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
        cos, sin = self.rotary.get(c.rot_dims, c.rot_base, ctx.n_pos, xn.device)
        max_len = state.keys.shape[2]
        _lib.call("rd_rotary_append", code, _lib.ptr(proj), ld, _lib.ptr(state.keys), _lib.ptr(state.values), _lib.ptr(ctx.tok_row),
                  _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tok_slot), _lib.ptr(cos), _lib.ptr(sin), ctx.n_pos, ctx.m_max, _lib.ptr(ctx.m_dev),
                  c.heads, c.kv_heads, c.dim, c.vdim, c.rot_dims, max_len, st)
        gate = proj[:, sum(self.sizes[:3]):]
        _lib.call("rd_attention_window", code, _lib.ptr(proj), ld, _lib.ptr(state.keys), _lib.ptr(state.values), _lib.ptr(gate), ld,
                  _lib.ptr(mixed), _lib.ptr(ctx.row_start), _lib.ptr(ctx.kv_begin), _lib.ptr(ctx.base_len), ctx.batch, c.heads, c.kv_heads,
                  c.dim, c.vdim, max_len, ctx.max_new, ctx.mode, _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tree_mask), ctx.mask_words,
                  c.scale, c.window, c.keep_first, ctx.max_kv, st)
        self.lin[1](mixed, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)

    def _heads_of_128(self) -> bool:
        c, w = self.cfg, self.w_in
        return (w.dtype == torch.bfloat16 and c.dim == 128 and c.vdim == 128 and c.rot_dims % 16 == 0 and w.shape[1] >= 64
                and w.shape[1] % 8 == 0)

    def _run_128(self, ctx: StepContext, state: kv_cache.LayerKeyValues, xn, residual, out) -> None:
        """Heads of 128 features in bf16: rotary embedding and cache append ride on the projection's epilogue, prompts and
        draft trees take the tcgen05 attention."""
        c, ws, st = self.cfg, ctx.ws, _lib.stream()
        q = rows_of(ws["proj"], c.heads * 128)
        ldg = row_stride(c.heads)
        gate = rows_of(ws["head_gate"], ldg)
        mixed = rows_of(ws["mixed"], c.heads * 128)
        cos, sin = self.rotary.get(c.rot_dims, c.rot_base, ctx.n_pos, xn.device, head=128)
        self.lin[0].qkvg_rope(xn, q, state.keys, state.values, gate, ctx.tok_row, ctx.tok_pos, ctx.tok_slot, cos, sin, c.heads, c.kv_heads,
                              c.rot_dims, ctx.m_dev, ctx.m_max, ctx.status)
        max_len = state.keys.shape[2]
        few = (c.heads // c.kv_heads) * ctx.max_new <= 32  # the kernel that shares keys among a group's heads
        tree = ctx.mode == _lib.ATTN_TREE
        if few or c.scale <= 0 or (tree and (c.window < _lib.MAX_BEAM_LENGTH or ctx.mask_words > 16)):
            _lib.call("rd_attention_window", _lib.BF16, _lib.ptr(q), c.heads * 128, _lib.ptr(state.keys), _lib.ptr(state.values), _lib.ptr(gate),
                      ldg, _lib.ptr(mixed), _lib.ptr(ctx.row_start), _lib.ptr(ctx.kv_begin), _lib.ptr(ctx.base_len), ctx.batch, c.heads,
                      c.kv_heads, 128, 128, max_len, ctx.max_new, ctx.mode, _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tree_mask),
                      ctx.mask_words, c.scale, c.window, c.keep_first, ctx.max_kv, st)
        else:
            key = (q.data_ptr(), ctx.m_max, state.keys.data_ptr(), state.values.data_ptr(), ctx.batch, max_len)
            plan = self._plans.get(key)
            if plan is None:
                plan = _lib.load().rd_attention_plan_create(_lib.ptr(q), ctx.m_max, _lib.ptr(state.keys), _lib.ptr(state.values), ctx.batch,
                                                            c.heads, c.kv_heads, 128, max_len)
                if not plan:
                    raise _lib.RedrafterError("rd_attention_plan_create failed (TMA descriptor could not be encoded)")
                if len(self._plans) >= 8:
                    self.drop_plans()
                self._plans[key] = plan
            _lib.call("rd_attention_tc_window", plan, _lib.ptr(mixed), _lib.ptr(ctx.row_start), _lib.ptr(ctx.kv_begin), _lib.ptr(ctx.base_len),
                      ctx.max_new, ctx.mode, _lib.ptr(ctx.tok_pos), _lib.ptr(ctx.tree_mask), ctx.mask_words, c.scale, c.window,
                      c.keep_first, _lib.ptr(gate), ldg, _lib.ptr(ctx.status), st)
        self.lin[1](mixed, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)

    def commit_draft(self, state: kv_cache.LayerKeyValues, kv_begin, fp, n_accepted, seq_in_beam, beam_shape) -> None:
        code = _lib.dtype_code(self.w_in.dtype)
        for plane in (state.keys, state.values):
            B, heads, max_len, dim = plane.shape
            _lib.call("rd_cache_commit", code, _lib.ptr(plane), B, heads, max_len, dim, _lib.ptr(kv_begin), _lib.ptr(fp.base_len),
                      _lib.ptr(fp.unpacker), beam_shape.width, beam_shape.length, _lib.ptr(n_accepted), _lib.ptr(seq_in_beam),
                      _lib.stream())


class MatrixMemory(nn.Module):
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

    def proj_width(self) -> int:
        return self.n_split

    def out_width(self) -> int:
        return self.cfg.heads * self.cfg.vdim

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

    def linears(self) -> List[Linear]:
        return list(self.lin or ())

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
        mixed = rows_of(ws["mixed"], self.out_width())
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


class DenseFeedForward(nn.Module):
    """W_down xIELU(W_up h); the activation has two trained numbers and sits in the first product's epilogue."""

    def __init__(self, width: int, ff: int):
        super().__init__()
        self.ff = ff
        self.up = weight(ff, width)
        self.down = weight(width, ff)
        self.act = weight(2)
        self.lin: Optional[Tuple[Linear, Linear]] = None
        self.coeff = (0.0, 0.0)

    def load(self, take: Callable[[str], torch.Tensor]) -> None:
        self.up.copy_(take("up"))
        self.down.copy_(take("down"))
        self.act.copy_(take("act"))

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {"up": self.up.detach(), "down": self.down.detach(), "act": self.act.detach()}

    def prepare(self) -> None:
        self.lin = (Linear(self.up), Linear(self.down))
        p, q = (float(v) for v in self.act.detach().float().cpu())

        def softplus(z: float) -> float:
            return max(z, 0.0) + math.log1p(math.exp(-abs(z)))

        self.coeff = (softplus(p), 0.5 + softplus(q))

    def linears(self) -> List[Linear]:
        return list(self.lin or ())

    def run(self, ctx: StepContext, xn: torch.Tensor, residual: torch.Tensor, out: torch.Tensor) -> None:
        act = rows_of(ctx.ws["act"], row_stride(self.ff))
        self.lin[0].xielu(xn, act, *self.coeff, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
        self.lin[1](act, out, _lib.EPI_RES, residual=residual, m_dev=ctx.m_dev, m_max=ctx.m_max, status=ctx.status)
