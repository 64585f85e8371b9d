"""Pre-allocated KV cache with the reference's API (recurrent_drafting/kv_cache.py).

One tensor [n_layers, 2, batch, n_kv_heads, max_length, head_dim].  The reference keeps every row
right-aligned and shifts whole rows after each decode step; here a row stays where the prompt put
it and only grows: row b occupies slots [kv_begin[b], kv_begin[b] + kv_len[b]).  kv_begin / kv_len
are device int32 vectors owned by the decode loop; the View/Cache surface below keeps the
reference's scalar `length` semantics for callers that use the cache the reference's way.
"""
from dataclasses import dataclass
from typing import List, Sequence, Tuple, Union

import torch

from . import _lib


class View:
    """Key or value cache of one layer (kv_cache.py:10-35)."""

    def __init__(self, cache: torch.Tensor, layer: int, kv: int):
        self._cache = cache
        self._layer = layer
        self._kv = kv
        self.length = 0

    @property
    def shape(self) -> Tuple[int, int, int, int]:
        _, _, batch_size, n_heads, _, head_dim = self._cache.shape
        return (batch_size, n_heads, self.length, head_dim)

    @property
    def plane(self) -> torch.Tensor:
        """[batch, n_kv_heads, max_length, head_dim] storage of this view."""
        return self._cache[self._layer, self._kv]

    def cat(self, new_kv: torch.Tensor) -> torch.Tensor:
        _, _, batch_size, n_heads, max_length, head_dim = self._cache.shape
        n = new_kv.shape[2]
        assert new_kv.shape == (batch_size, n_heads, n, head_dim)
        assert self.length + n <= max_length
        self.plane[:, :, self.length : self.length + n, :] = new_kv
        self.length += n
        return self.plane[:, :, : self.length, :]

    def slice(self, prev: int) -> torch.Tensor:
        return self.plane[:, :, prev : self.length, :]


class Cache:
    """kv_cache.py:38-98."""

    def __init__(self, batch_size: int, max_length: int, n_layers: int, n_heads: int, head_dim: int,
                 dtype: torch.dtype, device: torch.device) -> None:
        self._cache = torch.zeros([n_layers, 2, batch_size, n_heads, max_length, head_dim], dtype=dtype, device=device)
        self.sliced = tuple((View(self._cache, layer, 0), View(self._cache, layer, 1)) for layer in range(n_layers))

    @property
    def storage(self) -> torch.Tensor:
        """What the model's backbone() takes."""
        return self._cache

    @property
    def max_length(self) -> int:
        return self._cache.shape[4]

    def set_length(self, length: int) -> None:
        for k, v in self.sliced:
            k.length = v.length = length

    def unpack(self, prompt_length: int, tree_attn_index: torch.Tensor) -> None:
        """Replicates the packed-tree K/V into per-beam layout (kv_cache.py:58-98).  The decode loop
        of this package does not need it (its commit reads the packed slots directly)."""
        batch_size = tree_attn_index.shape[0]
        n_flat = tree_attn_index.shape[1] * tree_attn_index.shape[2]
        n_layers, _, cache_batch, n_heads, max_length, head_dim = self._cache.shape
        idx = tree_attn_index.reshape(batch_size, n_flat).to(torch.int64)
        if batch_size != cache_batch:
            idx = idx.expand(cache_batch, n_flat)
        idx = idx.contiguous()
        scratch = torch.empty([n_layers, 2, cache_batch, n_heads, n_flat, head_dim], dtype=self._cache.dtype,
                              device=self._cache.device)
        _lib.call("rd_cache_unpack", _lib.dtype_code(self._cache.dtype), _lib.ptr(self._cache), n_layers, cache_batch,
                  n_heads, max_length, head_dim, prompt_length, _lib.ptr(idx), n_flat, _lib.ptr(scratch), _lib.stream())
        for k, v in self.sliced:
            k.length = v.length = prompt_length + n_flat

    def unpack_static(self, prompt_length: int, tree_attn_index: torch.Tensor) -> None:
        """Cache.unpack for callers that must not allocate device memory (a host that owns all of the
        device's memory in its own arena, or a loop that forbids allocation after set-up): the staging
        copy lives in a fixed 16 MiB array inside the library instead of a fresh tensor.

        tree_attn_index must already be a contiguous int64 tensor of shape (cache batch, W, Lb) on the
        cache's device, so that this wrapper creates no tensor either.  Raises if the gathered rows
        (n_layers*2*batch*heads*W*Lb*head_dim elements) do not fit; calls that can overlap on the GPU
        share the array and must be ordered on one stream; make the first call per device at set-up.
        """
        n_layers, _, cache_batch, n_heads, max_length, head_dim = self._cache.shape
        idx = tree_attn_index
        assert idx.dtype == torch.int64 and idx.is_contiguous() and idx.shape[0] == cache_batch
        n_flat = idx.shape[1] * idx.shape[2]
        _lib.call("rd_cache_unpack_static", _lib.dtype_code(self._cache.dtype), _lib.ptr(self._cache), n_layers, cache_batch,
                  n_heads, max_length, head_dim, prompt_length, _lib.ptr(idx), n_flat, _lib.stream())
        for k, v in self.sliced:
            k.length = v.length = prompt_length + n_flat


@dataclass(frozen=True)
class KeyValueSpec:
    """A layer that keeps keys and values of every token."""

    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class MatrixStateSpec:
    """A layer that keeps a matrix state of fixed size: S [heads, dim, vdim], n [heads, dim], m [heads], fp32."""

    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class LatentSpec:
    """A layer that keeps one vector of every token, from which all heads' keys and values are formed."""

    width: int


LayerSpec = Union[KeyValueSpec, MatrixStateSpec, LatentSpec]


class LayerKeyValues:
    def __init__(self, spec: KeyValueSpec, batch: int, max_length: int, dtype: torch.dtype, device):
        self.keys = torch.zeros(batch, spec.heads, max_length, spec.dim, dtype=dtype, device=device)
        self.values = torch.zeros(batch, spec.heads, max_length, spec.vdim, dtype=dtype, device=device)


class LayerMatrixState:
    def __init__(self, spec: MatrixStateSpec, batch: int, draft_tokens: int, dtype: torch.dtype, device):
        f32 = dict(dtype=torch.float32, device=device)
        self.S = torch.zeros(batch, spec.heads, spec.dim, spec.vdim, **f32)
        self.n = torch.zeros(batch, spec.heads, spec.dim, **f32)
        self.m = torch.zeros(batch, spec.heads, **f32)
        # Projections and gates of the packed draft tokens: a verify step leaves the state alone, and the commit runs the
        # accepted path through the recurrence from here.
        width = 2 * spec.heads * (spec.dim + spec.vdim)
        self.draft_proj = torch.empty(draft_tokens, (width + 31) // 32 * 32, dtype=dtype, device=device) if draft_tokens else None
        self.draft_gates = torch.empty(draft_tokens, 2 * spec.heads, **f32) if draft_tokens else None


class LayerLatents:
    def __init__(self, spec: LatentSpec, batch: int, max_length: int, dtype: torch.dtype, device):
        self.rows = torch.zeros(batch, 1, max_length, spec.width, dtype=dtype, device=device)


class HybridCache:
    """State of a decoder whose layers differ in what they carry from token to token.  Attention layers keep keys
    [batch, heads, max_length, dim] and values [batch, heads, max_length, vdim], or latents [batch, 1, max_length, width],
    slot = position in the row; recurrent layers keep their state.  Rows are independent; a row whose length is 0 starts afresh whatever its memory holds (the
    recurrent kernels take the zero state then, and no key beyond a row's length is ever read), so giving a row back is
    setting its length to 0."""

    def __init__(self, layers: Sequence[LayerSpec], batch_size: int, max_length: int, dtype: torch.dtype, device,
                 draft_tokens: int = 0) -> None:
        self.max_length = max_length
        self.batch_size = batch_size
        self.length = 0
        self.layers: List[Union[LayerKeyValues, LayerMatrixState, LayerLatents]] = []
        for spec in layers:
            if isinstance(spec, KeyValueSpec):
                self.layers.append(LayerKeyValues(spec, batch_size, max_length, dtype, device))
            elif isinstance(spec, MatrixStateSpec):
                self.layers.append(LayerMatrixState(spec, batch_size, draft_tokens, dtype, device))
            elif isinstance(spec, LatentSpec):
                self.layers.append(LayerLatents(spec, batch_size, max_length, dtype, device))
            else:
                raise TypeError(f"unknown layer spec {spec!r}")

    @property
    def storage(self) -> "HybridCache":
        return self

    def set_length(self, length: int) -> None:
        self.length = length

    def bytes_per_token(self) -> int:
        """Memory that grows with the sequence."""
        planes = [p for l in self.layers for p in ((l.keys, l.values) if isinstance(l, LayerKeyValues) else
                                                   (l.rows,) if isinstance(l, LayerLatents) else ())]
        return sum(p[0, :, 0].numel() * p.element_size() for p in planes)
