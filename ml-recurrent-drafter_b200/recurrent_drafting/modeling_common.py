"""What the base models share: linear layers on the GEMM kernels and the language-model head."""
import os
from typing import Dict, Optional, Tuple

import torch

from . import _lib


class Linear:
    """y = epilogue(x W^T) on a fixed weight; picks the tcgen05 path for bf16 when shapes allow."""

    def __init__(self, weight: torch.Tensor, bias: Optional[torch.Tensor] = None):
        self.weight = weight
        self.bias = bias
        self._plans: Dict[Tuple, int] = {}

    MAX_PLANS = 32  # distinct (activation buffer, row capacity) pairs remembered per weight

    def drop_plans(self) -> None:
        plans, self._plans = self._plans, {}
        if plans:
            lib = _lib.load()
            for p in plans.values():
                lib.rd_gemm_plan_destroy(p)

    def __del__(self):
        try:
            self.drop_plans()
        except Exception:
            pass

    def _tc_ok(self, a: torch.Tensor, lda: int) -> bool:
        n, k = self.weight.shape
        return (
            self.weight.dtype == torch.bfloat16
            and k >= 64
            and k % 8 == 0
            and a.data_ptr() % 16 == 0
            and (lda * 2) % 16 == 0
            and self.weight.data_ptr() % 16 == 0
        )

    def _plan(self, a: torch.Tensor, lda: int, m_max: int) -> int:
        n, k = self.weight.shape
        key = (a.data_ptr(), lda, m_max)
        plan = self._plans.get(key)
        if plan is None:
            plan = _lib.load().rd_gemm_plan_create(_lib.ptr(a), lda, m_max, _lib.ptr(self.weight), self.weight.stride(0), n, k)
            if not plan:
                raise _lib.RedrafterError("rd_gemm_plan_create failed (TMA descriptor could not be encoded)")
            if len(self._plans) >= self.MAX_PLANS:
                self.drop_plans()
            self._plans[key] = plan
        return plan

    def qkv_rope(self, a: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, tok_row, tok_pos,
                 tok_slot, cos: torch.Tensor, sin: torch.Tensor, nh: int, nkv: int, hd: int, m_dev, m_max: int,
                 status: Optional[torch.Tensor], norm=None) -> None:
        """This weight as the packed QKV projection with rotary embedding and cache append in the
        GEMM epilogue (rd_gemm_bf16_tc_qkv_rope); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the fused QKV projection needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        if norm is not None:
            # `a` holds gamma-scaled, not normalised rows: the 1 / rms of each row is applied in the epilogue
            ss, dim, eps = norm
            _lib.call("rd_gemm_bf16_tc_qkv_rope_normed", plan, _lib.ptr(m_dev), _lib.ptr(q_out), _lib.ptr(k_cache),
                      _lib.ptr(v_cache), _lib.ptr(tok_row), _lib.ptr(tok_pos), _lib.ptr(tok_slot), _lib.ptr(cos), _lib.ptr(sin),
                      cos.shape[0], nh, nkv, hd, k_cache.shape[2], _lib.ptr(ss), ss.stride(0), dim // 128, dim, eps,
                      _lib.ptr(status), _lib.stream())
            return
        _lib.call("rd_gemm_bf16_tc_qkv_rope", plan, _lib.ptr(m_dev), _lib.ptr(q_out), _lib.ptr(k_cache), _lib.ptr(v_cache),
                  _lib.ptr(tok_row), _lib.ptr(tok_pos), _lib.ptr(tok_slot), _lib.ptr(cos), _lib.ptr(sin), cos.shape[0], nh, nkv,
                  hd, k_cache.shape[2], _lib.ptr(status), _lib.stream())

    def qkvg_rope(self, a: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, gate_out: torch.Tensor,
                  tok_row, tok_pos, tok_slot, cos: torch.Tensor, sin: torch.Tensor, nh: int, nkv: int, rot_dims: int, m_dev,
                  m_max: int, status: Optional[torch.Tensor]) -> None:
        """This weight as the packed q, k, v and head-gate projection of heads of 128 features, with rotary embedding on
        rot_dims of them and the cache append in the epilogue (rd_gemm_bf16_tc_qkvg_rope); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the fused QKV projection needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_qkvg_rope", plan, _lib.ptr(m_dev), _lib.ptr(q_out), _lib.ptr(k_cache), _lib.ptr(v_cache),
                  _lib.ptr(gate_out), gate_out.stride(0), _lib.ptr(tok_row), _lib.ptr(tok_pos), _lib.ptr(tok_slot), _lib.ptr(cos),
                  _lib.ptr(sin), cos.shape[0], nh, nkv, 128, rot_dims, k_cache.shape[2], _lib.ptr(status), _lib.stream())

    def qk_rope_norm(self, a: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, tok_row, tok_pos, tok_slot,
                     cos: torch.Tensor, sin: torch.Tensor, nh: int, nkv: int, rot_dims: int, eps: float, m_dev, m_max: int,
                     status: Optional[torch.Tensor]) -> None:
        """This weight as the packed q and k projection of heads of 128 features whose values are the keys: rotary embedding
        on rot_dims features, division by the head's root mean square and the append of keys and values in the epilogue
        (rd_gemm_bf16_tc_qk_rope_norm); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the fused QK projection needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_qk_rope_norm", plan, _lib.ptr(m_dev), _lib.ptr(q_out), _lib.ptr(k_cache), _lib.ptr(v_cache),
                  _lib.ptr(tok_row), _lib.ptr(tok_pos), _lib.ptr(tok_slot), _lib.ptr(cos), _lib.ptr(sin), cos.shape[0], nh, nkv, 128,
                  rot_dims, k_cache.shape[2], eps, _lib.ptr(status), _lib.stream())

    def residual_with_norm(self, a: torch.Tensor, c: torch.Tensor, residual: torch.Tensor, gamma: torch.Tensor,
                           c2: torch.Tensor, ss: torch.Tensor, m_dev, m_max: int, status: Optional[torch.Tensor]) -> None:
        """c = a @ weight^T + residual, and the producer half of the RMS norm that follows: c2 = c * gamma and the
        per-slice sums of squares ss [m_max, >= features / 128] (rd_gemm_bf16_tc_res_norm); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the folded RMS norm needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_res_norm", plan, _lib.ptr(c), c.stride(0), _lib.ptr(residual), residual.stride(0),
                  _lib.ptr(m_dev), _lib.ptr(gamma), _lib.ptr(c2), c2.stride(0), _lib.ptr(ss), ss.stride(0), _lib.ptr(status),
                  _lib.stream())

    def swiglu_normed(self, a: torch.Tensor, c: torch.Tensor, ss: torch.Tensor, dim: int, eps: float, m_dev, m_max: int,
                      status: Optional[torch.Tensor]) -> None:
        """SwiGLU projection of rows that are gamma-scaled but not normalised: each row's 1 / rms, from the sums of
        squares ss, is applied in the epilogue (rd_gemm_bf16_tc_swiglu_normed); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the folded RMS norm needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_swiglu_normed", plan, _lib.ptr(c), c.stride(0), _lib.ptr(m_dev), _lib.ptr(ss), ss.stride(0),
                  dim // 128, dim, eps, _lib.ptr(status), _lib.stream())

    def argmax(self, a: torch.Tensor, out32: Optional[torch.Tensor], workspace: torch.Tensor, m_dev, m_max: int,
               status: Optional[torch.Tensor], out64: Optional[torch.Tensor] = None) -> None:
        """out32[t] (and / or out64[t]) = argmax_n (a[t] . weight[n]) without materialising the product: the arg-max rides on
        the GEMM's epilogue (rd_gemm_bf16_tc_argmax); tensor-core path only."""
        if not self._tc_ok(a, a.stride(0)):
            raise _lib.RedrafterError("the fused LM-head arg-max needs the tensor-core GEMM path (bf16, aligned operands)")
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_argmax", plan, _lib.ptr(m_dev), _lib.ptr(workspace), workspace.numel(), _lib.ptr(out32), _lib.ptr(out64),
                  _lib.ptr(status), _lib.stream())

    def with_slice_max(self, a: torch.Tensor, c: torch.Tensor, slice_max: torch.Tensor, m_dev=None, m_max: Optional[int] = None,
                       status: Optional[torch.Tensor] = None) -> bool:
        """c = a W^T plus the per-(32 outputs, row) maxima of c in slice_max [N/32, >= m_max]
        (rd_gemm_bf16_tc_slicemax).  Returns False, doing nothing, when the shapes rule it out."""
        n, k = self.weight.shape
        m_max = a.shape[0] if m_max is None else m_max
        esz = 4 if c.dtype == torch.float32 else 2
        if not (self._tc_ok(a, a.stride(0)) and n % 32 == 0 and c.data_ptr() % 16 == 0 and (c.stride(0) * esz) % 16 == 0
                and slice_max.shape[0] * 32 == n and slice_max.stride(0) >= m_max):
            return False
        plan = self._plan(a, a.stride(0), m_max)
        _lib.call("rd_gemm_bf16_tc_slicemax", plan, _lib.dtype_code(c.dtype), _lib.ptr(c), c.stride(0), _lib.ptr(m_dev),
                  _lib.ptr(slice_max), slice_max.stride(0), _lib.ptr(status), _lib.stream())
        return True

    def xielu(self, a: torch.Tensor, c: torch.Tensor, pos: float, neg: float, m_dev=None, m_max: Optional[int] = None,
              status: Optional[torch.Tensor] = None) -> None:
        """c = xIELU(a W^T) with the activation in the epilogue."""
        n, k = self.weight.shape
        m_max = a.shape[0] if m_max is None else m_max
        if self._tc_ok(a, a.stride(0)):
            plan = self._plan(a, a.stride(0), m_max)
            _lib.call("rd_gemm_bf16_tc_xielu", plan, _lib.ptr(c), c.stride(0), _lib.ptr(m_dev), pos, neg, _lib.ptr(status),
                      _lib.stream())
        else:
            _lib.call("rd_gemm_xielu", _lib.dtype_code(self.weight.dtype), _lib.ptr(a), a.stride(0), _lib.ptr(self.weight),
                      self.weight.stride(0), _lib.ptr(c), c.stride(0), m_max, _lib.ptr(m_dev), n, k, pos, neg, _lib.stream())

    def clamped_glu(self, a: torch.Tensor, c: torch.Tensor, limit: float, alpha: float, m_dev=None, m_max: Optional[int] = None,
                    status: Optional[torch.Tensor] = None) -> None:
        """c = g sigmoid(alpha g) (u + 1) of the interleaved (gate, up) rows of this weight, g and u cut at limit, in the
        epilogue."""
        n, k = self.weight.shape
        m_max = a.shape[0] if m_max is None else m_max
        if self._tc_ok(a, a.stride(0)):
            plan = self._plan(a, a.stride(0), m_max)
            _lib.call("rd_gemm_bf16_tc_clamped_glu", plan, _lib.ptr(c), c.stride(0), _lib.ptr(m_dev), limit, alpha, _lib.ptr(status),
                      _lib.stream())
        else:
            _lib.call("rd_gemm_clamped_glu", _lib.dtype_code(self.weight.dtype), _lib.ptr(a), a.stride(0), _lib.ptr(self.weight),
                      self.weight.stride(0), _lib.ptr(c), c.stride(0), m_max, _lib.ptr(m_dev), n, k, limit, alpha, _lib.stream())

    def split(self, a: torch.Tensor, c: torch.Tensor, c_hi: torch.Tensor, n_split: int, m_dev=None,
              m_max: Optional[int] = None, status: Optional[torch.Tensor] = None) -> None:
        """Output features [0, n_split) of a W^T to c in its dtype, the rest to c_hi in fp32."""
        n, k = self.weight.shape
        m_max = a.shape[0] if m_max is None else m_max
        if self._tc_ok(a, a.stride(0)):
            plan = self._plan(a, a.stride(0), m_max)
            _lib.call("rd_gemm_bf16_tc_split", plan, _lib.ptr(c), c.stride(0), _lib.ptr(c_hi), c_hi.stride(0), n_split,
                      _lib.ptr(m_dev), _lib.ptr(status), _lib.stream())
            return
        code = _lib.dtype_code(self.weight.dtype)
        for w, out in ((self.weight[:n_split], c), (self.weight[n_split:], c_hi)):
            _lib.call("rd_gemm", code, _lib.dtype_code(out.dtype), _lib.ptr(a), a.stride(0), _lib.ptr(w), w.stride(0), _lib.ptr(out),
                      out.stride(0), None, None, 0, m_max, _lib.ptr(m_dev), w.shape[0], k, _lib.EPI_NONE, _lib.stream())

    def __call__(self, a: torch.Tensor, c: torch.Tensor, epilogue: int = _lib.EPI_NONE, residual=None,
                 m_dev: Optional[torch.Tensor] = None, lda: Optional[int] = None, ldc: Optional[int] = None,
                 ldr: Optional[int] = None, m_max: Optional[int] = None, status: Optional[torch.Tensor] = None) -> None:
        n, k = self.weight.shape
        m_max = a.shape[0] if m_max is None else m_max
        lda = a.stride(0) if lda is None else lda
        ldc = c.stride(0) if ldc is None else ldc
        if residual is not None and ldr is None:
            ldr = residual.stride(0)
        out_code = _lib.dtype_code(c.dtype)
        esz = 4 if c.dtype == torch.float32 else 2
        aligned = c.data_ptr() % 16 == 0 and (ldc * esz) % 16 == 0 and (
            residual is None or (residual.data_ptr() % 16 == 0 and (ldr * esz) % 16 == 0)
        )
        if self._tc_ok(a, lda) and aligned:
            plan = self._plan(a, lda, m_max)
            _lib.call("rd_gemm_bf16_tc", plan, out_code, _lib.ptr(c), ldc, _lib.ptr(self.bias), _lib.ptr(residual),
                      ldr or 0, _lib.ptr(m_dev), epilogue, _lib.ptr(status), _lib.stream())
        else:
            _lib.call("rd_gemm", _lib.dtype_code(self.weight.dtype), out_code, _lib.ptr(a), lda, _lib.ptr(self.weight),
                      self.weight.stride(0), _lib.ptr(c), ldc, _lib.ptr(self.bias), _lib.ptr(residual), ldr or 0, m_max,
                      _lib.ptr(m_dev), n, k, epilogue, _lib.stream())


class LMHead:
    """Mixin of a causal language model: logits, greedy tokens and slice maxima from its final hidden states.  The model
    has `config` (hidden_size, vocab_size), `dtype`, `device`, `gemm_status`, `_head_ws` and a _lin()["head"] Linear."""

    def lm_logits(self, hidden_rows: torch.Tensor, logits: torch.Tensor, m_dev=None) -> torch.Tensor:
        """fp32 logits of the given hidden rows (modeling_llama.py:272)."""
        self._lin()["head"](hidden_rows, logits, _lib.EPI_NONE, m_dev=m_dev, status=self.gemm_status)
        return logits

    def fused_head_ok(self) -> bool:
        """The LM head can run with the arg-max or the slice maxima in its epilogue (bf16 tensor-core path,
        vocabulary a multiple of 32)."""
        return (self.dtype == torch.bfloat16 and self.config.hidden_size % 64 == 0 and self.config.vocab_size % 32 == 0
                and os.environ.get("RD_FUSED_HEAD", "1") != "0")

    def _head_scratch(self, rows: int) -> torch.Tensor:
        """fp32 [vocab/32, rows rounded up to 32] scratch of the fused LM-head epilogues, grow-only."""
        slices = (self.config.vocab_size + 31) // 32
        ld = (rows + 31) // 32 * 32
        if self._head_ws is None or self._head_ws.shape[1] < ld:
            self._head_ws = torch.empty(2 * slices, ld, dtype=torch.float32, device=self.device)
        return self._head_ws

    def lm_argmax(self, hidden_rows: torch.Tensor, out32: Optional[torch.Tensor], m_dev=None,
                  out64: Optional[torch.Tensor] = None) -> None:
        """Greedy tokens of the given hidden rows, int32 and / or int64, without writing the logits (modeling_llama.py:272 +
        recurrent_drafting.py:52)."""
        rows = hidden_rows.shape[0]
        ws = self._head_scratch(rows)
        need = _lib.load().rd_gemm_argmax_workspace_bytes(rows, self.config.vocab_size)
        flat = ws.view(-1).view(torch.uint8)
        assert flat.numel() >= need
        self._lin()["head"].argmax(hidden_rows, out32, flat, m_dev, rows, self.gemm_status, out64=out64)

    def lm_logits_with_slice_max(self, hidden_rows: torch.Tensor, logits: torch.Tensor, m_dev=None) -> Optional[torch.Tensor]:
        """lm_logits() that also returns the [vocab/32, rows'] slice maxima for rd_vocab_topk_sliced, or None
        (plain logits computed) when the fused epilogue does not apply."""
        rows = hidden_rows.shape[0]
        if self.fused_head_ok():
            smax = self._head_scratch(rows)[: self.config.vocab_size // 32]
            if self._lin()["head"].with_slice_max(hidden_rows, logits, smax, m_dev=m_dev, status=self.gemm_status):
                return smax
        self.lm_logits(hidden_rows, logits, m_dev=m_dev)
        return None
