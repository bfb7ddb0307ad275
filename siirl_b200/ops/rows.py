"""Row operations of decoders with a 32-bit residual stream (``csrc/hybrid_ops.cu``): scaled embedding, residual add fused
with the following norm, gated activations, soft-capped logits.  Inference only; CPU tensors use the plain statements."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch
import torch.nn.functional as F

from . import lib as _lib

ACT = {"silu": 0, "gelu_tanh": 1}


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16), t.dtype
    return int(t.dtype == torch.float32)


def embed_scaled(ids: torch.Tensor, table: torch.Tensor, scale: float) -> torch.Tensor:
    """``table[ids] * scale`` as fp32 ``[T, W]``."""
    if not table.is_cuda:
        return F.embedding(ids, table).float() * scale
    ids = ids.to(torch.int64).contiguous()
    h = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    _lib.check(_lib.get_lib().sb_embed_scaled(_lib.ptr(ids), _lib.ptr(table), _lib.ptr(h), ids.numel(), table.shape[1],
                                              table.shape[0], ctypes.c_float(scale), _f32(table), _lib.stream()),
               "sb_embed_scaled")
    return h


def add_norm(h: torch.Tensor, delta: Optional[torch.Tensor], weight: torch.Tensor, eps: float,
             kind: str = "layer_norm") -> torch.Tensor:
    """``h += delta`` in place (fp32 ``[T, W]``; ``delta`` may be ``None``), then the norm of ``h`` times ``weight`` in the
    weight's format.  ``kind``: ``"layer_norm"`` (no bias) or ``"rms_norm"``."""
    assert h.dtype == torch.float32 and h.is_contiguous()
    if not h.is_cuda:
        if delta is not None:
            h += delta.float()
        c = h - h.mean(-1, keepdim=True) if kind == "layer_norm" else h
        return (c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * weight.float()).to(weight.dtype)
    assert delta is None or (delta.dtype == weight.dtype and delta.is_contiguous() and delta.shape == h.shape)
    y = torch.empty(h.shape, dtype=weight.dtype, device=h.device)
    _lib.check(_lib.get_lib().sb_add_norm(_lib.ptr(h), _lib.ptr(delta), _lib.ptr(weight), _lib.ptr(y), h.shape[0],
                                          h.shape[1], ctypes.c_float(eps), int(kind == "layer_norm"), _f32(weight),
                                          _lib.stream()), "sb_add_norm")
    return y


def gated_act(gate_up: torch.Tensor, act: str = "gelu_tanh") -> torch.Tensor:
    """``act(gate) * up`` for a fused projection ``[T, 2 I]`` = ``[gate | up]``."""
    T, I2 = gate_up.shape
    if not gate_up.is_cuda:
        g, u = gate_up.float().chunk(2, -1)
        return ((F.silu(g) if act == "silu" else F.gelu(g, approximate="tanh")) * u).to(gate_up.dtype)
    gate_up = gate_up.contiguous()
    out = torch.empty(T, I2 // 2, dtype=gate_up.dtype, device=gate_up.device)
    _lib.check(_lib.get_lib().sb_gated_act(_lib.ptr(gate_up), _lib.ptr(out), ctypes.c_longlong(T), I2 // 2, ACT[act],
                                           _f32(gate_up), _lib.stream()), "sb_gated_act")
    return out


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(logits / cap)`` in place on fp32 logits."""
    if not logits.is_cuda:
        return logits.copy_(cap * torch.tanh(logits / cap))
    assert logits.dtype == torch.float32 and logits.is_contiguous()
    _lib.check(_lib.get_lib().sb_softcap(_lib.ptr(logits), ctypes.c_longlong(logits.numel()), ctypes.c_float(cap),
                                         _lib.stream()), "sb_softcap")
    return logits


def gemm_simt(a: torch.Tensor, b: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """``a [M, K] @ b [N, K]^T`` with fp32 accumulation on the FMA pipes (fp32 operands stay fp32; bf16 of any pitch)."""
    assert a.dtype == b.dtype and a.stride(1) == 1 and b.stride(1) == 1 and a.shape[1] == b.shape[1]
    out = torch.empty(a.shape[0], b.shape[0], dtype=out_dtype, device=a.device)
    ll = ctypes.c_longlong
    rows = 64 * 65535
    for s in range(0, a.shape[0], rows):
        e = min(s + rows, a.shape[0])
        _lib.check(_lib.get_lib().sb_gemm_simt(_lib.ptr(a[s:e]), _lib.ptr(b), _lib.ptr(out[s:e]), e - s, b.shape[0],
                                               a.shape[1], ll(a.stride(0)), ll(b.stride(0)), ll(out.stride(0)), _f32(a),
                                               _f32(out), _lib.stream()), "sb_gemm_simt")
    return out
