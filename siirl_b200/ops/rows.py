"""Row operations of decoders with a 32-bit residual stream (``csrc/hybrid_ops.cu``): scaled embedding, residual add fused
with the following norm (and with the norm of what is added), gated residual update of two sublayers, entry of a layer
loop's pass, activations, soft-capped logits.  Inference only; CPU tensors use the plain statements."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Sequence

import torch
import torch.nn.functional as F

from . import lib as _lib

ACT = {"silu": 0, "gelu_tanh": 1, "gelu": 2, "relu2": 3, "xielu": 4}


def _act(z: torch.Tensor, act: str, numbers: Optional[torch.Tensor] = None) -> torch.Tensor:
    if act == "xielu":
        p, q = F.softplus(numbers.float())
        low = z.clamp(max=0.0)
        return torch.where(z > 0, p * z * z, (0.5 + q) * (torch.expm1(low) - low)) + 0.5 * z
    if act == "relu2":
        return F.relu(z).square()
    return F.silu(z) if act == "silu" else F.gelu(z, approximate="tanh" if act == "gelu_tanh" else "none")


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


def gated_act(gate_up: torch.Tensor, act: str = "gelu_tanh", used: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(gate) * up`` for a fused projection ``[T, 2 I]`` = ``[gate | up]``.  Rows with a negative entry in ``used``
    (int32) may be left unwritten."""
    T, I2 = gate_up.shape
    if not gate_up.is_cuda:
        g, u = gate_up.float().chunk(2, -1)
        return (_act(g, act) * u).to(gate_up.dtype)
    gate_up = gate_up.contiguous()
    out = torch.empty(T, I2 // 2, dtype=gate_up.dtype, device=gate_up.device)
    _lib.check(_lib.get_lib().sb_gated_act(_lib.ptr(gate_up), _lib.ptr(out), ctypes.c_longlong(T), I2 // 2, ACT[act],
                                           _lib.ptr(used), _f32(gate_up), _lib.stream()), "sb_gated_act")
    return out


def scaled_act(x: torch.Tensor, act: str, gain: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(gain * x)`` of a column range ``x [T, I]`` of wider rows; ``gain``: one number (a tensor)."""
    if not x.is_cuda:
        z = x.float() * (gain.float() if gain is not None else 1.0)
        return _act(z, act).to(x.dtype)
    assert x.stride(1) == 1
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    _lib.check(_lib.get_lib().sb_scaled_act(_lib.ptr(x), ctypes.c_longlong(x.stride(0)), _lib.ptr(gain), _lib.ptr(out),
                                            ctypes.c_longlong(x.shape[0]), x.shape[1], ACT[act], _f32(x), _lib.stream()),
               "sb_scaled_act")
    return out


def partial_act(x: torch.Tensor, act: str, gated: bool = False) -> torch.Tensor:
    """Activation of partial products ``x [S, T, I]`` (what :func:`siirl_b200.ops.dense.linear_partial` returns for a bf16
    model): the sum and ``act`` in one launch; ``gated``: ``act(first half) * second half`` of ``[S, T, 2 I]``."""
    S, T, N = x.shape
    I = N // 2 if gated else N
    if x.is_cuda and S > 1 and x.dtype == torch.float32:
        assert x.is_contiguous() and I % 4 == 0
        out = torch.empty(T, I, dtype=torch.bfloat16, device=x.device)
        _lib.check(_lib.get_lib().sb_partial_act(_lib.ptr(x), ctypes.c_longlong(T * N), S, _lib.ptr(out),
                                                 ctypes.c_longlong(T), I, ACT[act], int(gated), _lib.stream()),
                   "sb_partial_act")
        return out
    assert S == 1
    return gated_act(x[0], act) if gated else scaled_act(x[0], act)


def bias_act(x: torch.Tensor, act: str, dtype: torch.dtype, bias: Optional[torch.Tensor] = None,
             numbers: Optional[torch.Tensor] = None, used: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(sum of x [S, T, I] + bias)`` in ``dtype``, ``x`` as :func:`siirl_b200.ops.dense.linear_partial` returns it.
    ``numbers``: the two learned numbers of ``"xielu"`` (for ``z > 0``: ``softplus(p) z^2 + z / 2``, else
    ``(1/2 + softplus(q)) (e^z - 1 - z) + z / 2``).  Rows with a negative entry in ``used`` may be left unwritten."""
    S, T, I = x.shape
    assert (act == "xielu") == (numbers is not None)
    if not x.is_cuda:
        z = x.float().sum(0)
        return _act(z + bias.float() if bias is not None else z, act, numbers).to(dtype)
    assert x.is_contiguous() and (x.dtype == torch.float32 or (S == 1 and x.dtype == dtype))
    out = torch.empty(T, I, dtype=dtype, device=x.device)
    _lib.check(_lib.get_lib().sb_bias_act(
        _lib.ptr(x), ctypes.c_longlong(T * I), S, _f32(x), _lib.ptr(bias), _lib.ptr(numbers), _lib.ptr(out),
        ctypes.c_longlong(T), I, ACT[act], _lib.ptr(used), int(dtype == torch.float32), _lib.stream()), "sb_bias_act")
    return out


def token_gate(z: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, column: int, width: int,
               dtype: torch.dtype) -> torch.Tensor:
    """``gelu_tanh(sum of z [S, T, >= width]) * table[ids, column : column + width]``, padded columns zero."""
    S, T, I = z.shape
    if not z.is_cuda:
        e = F.embedding(ids, table)[:, column:column + width].float()
        return F.pad(_act(z.float().sum(0)[:, :width], "gelu_tanh") * e, (0, I - width)).to(dtype)
    assert z.is_contiguous() and (z.dtype == torch.float32 or (S == 1 and z.dtype == dtype)) and table.dtype == dtype
    assert ids.dtype == torch.int64 and ids.is_contiguous() and table.is_contiguous() and column + width <= table.shape[1]
    out = torch.empty(T, I, dtype=dtype, device=z.device)
    _lib.check(_lib.get_lib().sb_token_gate(
        _lib.ptr(z), ctypes.c_longlong(T * I), S, _f32(z), _lib.ptr(ids), _lib.ptr(table),
        ctypes.c_longlong(table.shape[1]), table.shape[0], column, width, _lib.ptr(out), T, I, int(dtype == torch.float32),
        _lib.stream()), "sb_token_gate")
    return out


@dataclass
class Sublayer:
    """One result waiting to enter the residual stream: ``y [S, T, W]`` (partial sums, or one tensor in the activation
    format), optionally times ``sigmoid(gain * gate + bias)`` with ``gate [T, W]`` a column range of wider rows."""
    y: torch.Tensor
    gate: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    gain: Optional[torch.Tensor] = None


class _Sub(ctypes.Structure):
    _fields_ = [("y", ctypes.c_void_p), ("slab", ctypes.c_longlong), ("slabs", ctypes.c_int), ("y_f32", ctypes.c_int),
                ("gate", ctypes.c_void_p), ("gate_stride", ctypes.c_longlong), ("bias", ctypes.c_void_p),
                ("gain", ctypes.c_void_p)]


class _Stream(ctypes.Structure):
    """Mirror of ``StreamParams`` in csrc/hybrid_ops.cu."""
    _fields_ = [("h", ctypes.c_void_p), ("rows", ctypes.c_int), ("W", ctypes.c_int), ("mult", ctypes.c_float),
                ("eps", ctypes.c_float), ("n_sub", ctypes.c_int), ("enter", ctypes.c_int), ("sub", _Sub * 2),
                ("step", ctypes.c_void_p), ("pair", ctypes.c_int), ("split", ctypes.c_int),
                ("weight", ctypes.c_void_p), ("out", ctypes.c_void_p)]


assert ctypes.sizeof(_Stream) == 176


def _sub(s: Sublayer, W: int) -> _Sub:
    assert s.y.is_contiguous() and s.y.dim() == 3 and s.y.shape[2] == W
    g = s.gate
    assert g is None or g.stride(1) == 1
    return _Sub(y=s.y.data_ptr(), slab=s.y.stride(0), slabs=s.y.shape[0], y_f32=_f32(s.y),
                gate=g.data_ptr() if g is not None else None, gate_stride=g.stride(0) if g is not None else 0,
                bias=s.bias.data_ptr() if s.bias is not None else None,
                gain=s.gain.data_ptr() if s.gain is not None else None)


def _finish_rows(h: torch.Tensor, dtype, eps: float, weight, split: bool) -> torch.Tensor:
    if split:
        if dtype == torch.float32:
            return h.clone()
        hi = h.to(dtype)
        return torch.cat([hi, (h - hi.float()).to(dtype)])
    y = h * torch.rsqrt(h.pow(2).mean(-1, keepdim=True) + eps)
    return (y * weight.float() if weight is not None else y).to(dtype)


def stream_update(h: torch.Tensor, subs: Sequence[Sublayer], mult: float, dtype: torch.dtype, eps: float,
                  weight: Optional[torch.Tensor] = None, split: bool = False) -> torch.Tensor:
    """``h += mult * (sum of at most two sublayer results)`` in place (fp32 ``[T, W]``), then ``h`` over its root mean
    square, times ``weight`` (one number) when given.  ``split``: ``h`` itself as a sum of two ``dtype`` rows instead,
    ``[2 T, W]`` (the rounded rows, then the remainders; fp32: ``h`` alone)."""
    assert h.dtype == torch.float32 and h.is_contiguous() and len(subs) <= 2
    T, W = h.shape
    if not h.is_cuda:
        for s in subs:
            y = s.y.float().sum(0)
            if s.gate is not None:
                z = s.gate.float() * (s.gain.float() if s.gain is not None else 1.0)
                y = y * torch.sigmoid(z + (s.bias.float() if s.bias is not None else 0.0))
            h += mult * y
        return _finish_rows(h, dtype, eps, weight, split)
    f32 = dtype == torch.float32
    out = torch.empty(2 * T if split and not f32 else T, W, dtype=dtype, device=h.device)
    p = _Stream(h=h.data_ptr(), rows=T, W=W, mult=mult, eps=eps, n_sub=len(subs), enter=0,
                sub=(_Sub * 2)(*[_sub(s, W) for s in subs]), split=int(split),
                weight=weight.data_ptr() if weight is not None else None, out=out.data_ptr())
    _lib.check(_lib.get_lib().sb_stream_rows(ctypes.byref(p), int(f32), _lib.stream()), "sb_stream_rows")
    return out


def enter_pass(h: torch.Tensor, mixed: torch.Tensor, base: torch.Tensor, step: torch.Tensor, eps: float) -> torch.Tensor:
    """``h = mixed + base + step`` in place, then ``h`` over its root mean square in the format of ``step [W]``.
    ``mixed [S, T or 2 T, W]`` and ``base [S, T, W]``: fp32 partial sums; ``2 T`` rows are the products of the two rows
    :func:`stream_update` splits ``h`` into."""
    T, W = h.shape
    assert mixed.dtype == base.dtype == torch.float32 and mixed.shape[1] in (T, 2 * T) and base.shape[1] == T
    if not h.is_cuda:
        m = mixed.sum(0)
        h.copy_((m[:T] + m[T:] if m.shape[0] == 2 * T and T else m) + base.sum(0) + step.float())
        return _finish_rows(h, step.dtype, eps, None, False)
    out = torch.empty(T, W, dtype=step.dtype, device=h.device)
    p = _Stream(h=h.data_ptr(), rows=T, W=W, mult=1.0, eps=eps, n_sub=2, enter=1,
                sub=(_Sub * 2)(_sub(Sublayer(mixed), W), _sub(Sublayer(base), W)), step=step.data_ptr(),
                pair=int(mixed.shape[1] == 2 * T), out=out.data_ptr())
    _lib.check(_lib.get_lib().sb_stream_rows(ctypes.byref(p), _f32(step), _lib.stream()), "sb_stream_rows")
    return out


@dataclass
class SublayerSum:
    """Result of a sublayer on its way into hyper-connected streams: ``y [S, T, W]`` (partial sums, or one tensor in the
    activation format) plus a bias, plus routed rows ``ys[pair_slot[t, j]] * pair_w[t, j]`` (slot -1: none), plus the
    sublayer's input ``x_id [T, W]`` times ``w_id [T]``; every part may be missing."""
    y: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    ys: Optional[torch.Tensor] = None
    pair_slot: Optional[torch.Tensor] = None
    pair_w: Optional[torch.Tensor] = None
    x_id: Optional[torch.Tensor] = None
    w_id: Optional[torch.Tensor] = None


class _Hyper(ctypes.Structure):
    """Mirror of ``HyperParams`` in csrc/hyper_rows.cu."""
    _fields_ = [("h", ctypes.c_void_p), ("rows", ctypes.c_int), ("S", ctypes.c_int), ("W", ctypes.c_int),
                ("vocab", ctypes.c_int), ("ids", ctypes.c_void_p), ("table", ctypes.c_void_p), ("y", ctypes.c_void_p),
                ("slab", ctypes.c_longlong), ("slabs", ctypes.c_int), ("y_f32", ctypes.c_int), ("bias", ctypes.c_void_p),
                ("ys", ctypes.c_void_p), ("pair_slot", ctypes.c_void_p), ("pair_w", ctypes.c_void_p),
                ("w_id", ctypes.c_void_p), ("x_id", ctypes.c_void_p), ("top", ctypes.c_int), ("eps", ctypes.c_float),
                ("w_mix", ctypes.c_void_p), ("w_out", ctypes.c_void_p), ("w_in", ctypes.c_void_p),
                ("norm_w", ctypes.c_void_p), ("norm_b", ctypes.c_void_p), ("out", ctypes.c_void_p)]


assert ctypes.sizeof(_Hyper) == 168


def hyper_rows(h: torch.Tensor, norm_w: torch.Tensor, norm_b: torch.Tensor, eps: float, *,
               w_in: Optional[torch.Tensor] = None, result: Optional[SublayerSum] = None,
               w_out: Optional[torch.Tensor] = None, w_mix: Optional[torch.Tensor] = None,
               ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One step between two sublayers of a decoder with hyper-connections, ``h [T, S, W]`` fp32 in place: the copies become
    ``table[ids]`` (``ids`` given), or ``h_t <- sum_s w_mix[s, t] h_s + w_out[t] * result`` (``result`` given); returns the
    layer norm (weight and bias) of ``sum_s w_in[s] h_s`` in the weight's format, ``w_in = None``: of the plain sum."""
    T, S, W = h.shape
    assert h.dtype == torch.float32 and h.is_contiguous() and not (ids is not None and result is not None)
    r = result
    if not h.is_cuda:
        if ids is not None:
            h.copy_(F.embedding(ids, table).float()[:, None].expand(T, S, W))
        elif r is not None:
            y = torch.zeros(T, W)
            if r.y is not None:
                y = y + r.y.float().sum(0)
            if r.bias is not None:
                y = y + r.bias.float()
            if r.ys is not None:
                slot, k = r.pair_slot.reshape(T, -1).long(), r.pair_w.shape[1]
                for j in range(k):
                    y = y + torch.where((slot[:, j] >= 0)[:, None],
                                        r.pair_w[:, j, None] * r.ys[slot[:, j].clamp(min=0)].float(), torch.zeros(()))
            if r.w_id is not None:
                y = y + r.w_id[:, None] * r.x_id.float()
            h.copy_(torch.einsum("st,nsw->ntw", w_mix.float(), h) + w_out.float()[None, :, None] * y[:, None])
        u = h.sum(1) if w_in is None else torch.einsum("s,nsw->nw", w_in.float(), h)
        return F.layer_norm(u, (W,), norm_w.float(), norm_b.float(), eps).to(norm_w.dtype)
    out = torch.empty(T, W, dtype=norm_w.dtype, device=h.device)
    ptr = lambda t: t.data_ptr() if t is not None else None  # noqa: E731
    p = _Hyper(h=h.data_ptr(), rows=T, S=S, W=W, eps=eps, w_in=ptr(w_in), norm_w=ptr(norm_w), norm_b=ptr(norm_b),
               out=out.data_ptr())
    if ids is not None:
        assert ids.dtype == torch.int64 and ids.is_contiguous() and table.dtype == out.dtype
        p.ids, p.table, p.vocab = ids.data_ptr(), table.data_ptr(), table.shape[0]
    if r is not None:
        p.w_mix, p.w_out, p.bias = w_mix.data_ptr(), w_out.data_ptr(), ptr(r.bias)
        if r.y is not None:
            assert r.y.is_contiguous() and r.y.shape[1:] == (T, W)
            p.y, p.slab, p.slabs, p.y_f32 = r.y.data_ptr(), T * W, r.y.shape[0], _f32(r.y)
            assert p.y_f32 or p.slabs == 1
        if r.ys is not None:
            assert r.ys.is_contiguous() and r.ys.dtype == out.dtype and r.pair_w.dtype == torch.float32
            p.ys, p.pair_slot, p.pair_w, p.top = r.ys.data_ptr(), ptr(r.pair_slot), ptr(r.pair_w), r.pair_w.shape[1]
        if r.w_id is not None:
            assert r.x_id.is_contiguous() and r.x_id.dtype == out.dtype
            p.w_id, p.x_id = r.w_id.data_ptr(), r.x_id.data_ptr()
    _lib.check(_lib.get_lib().sb_hyper_rows(ctypes.byref(p), int(out.dtype == torch.float32), _lib.stream()), "sb_hyper_rows")
    return out


class _PostNorm(ctypes.Structure):
    """Mirror of ``PostNormParams`` in csrc/post_norm_rows.cu."""
    _fields_ = [("h", ctypes.c_void_p), ("rows", ctypes.c_int), ("W", ctypes.c_int), ("vocab", ctypes.c_int),
                ("top", ctypes.c_int), ("ids", ctypes.c_void_p), ("table", ctypes.c_void_p), ("scale", ctypes.c_float),
                ("eps", ctypes.c_float), ("y", ctypes.c_void_p), ("slab", ctypes.c_longlong), ("slabs", ctypes.c_int),
                ("y_f32", ctypes.c_int), ("bias", ctypes.c_void_p), ("ys", ctypes.c_void_p), ("pair_slot", ctypes.c_void_p),
                ("pair_w", ctypes.c_void_p), ("post", ctypes.c_void_p), ("norm_w", ctypes.c_void_p),
                ("out", ctypes.c_void_p)]


assert ctypes.sizeof(_PostNorm) == 128


def post_norm_rows(h: torch.Tensor, weight: Optional[torch.Tensor], eps: float, dtype: torch.dtype, *,
                   result: Optional[SublayerSum] = None, post: Optional[torch.Tensor] = None,
                   ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None,
                   scale: float = 1.0) -> torch.Tensor:
    """One step between two sublayers of a decoder with a norm behind each, ``h [T, W]`` fp32 in place:
    ``h = table[ids] * scale`` (``ids`` given) or ``h += y / rms(y) * post`` with ``y`` the sum that ``result`` stands for;
    returns ``h / rms(h) * weight`` in ``dtype``, or ``h`` itself in ``dtype`` (``weight = None``)."""
    T, W = h.shape
    assert h.dtype == torch.float32 and h.is_contiguous() and (ids is None) != (result is None)
    r = result
    assert r is None or r.x_id is None
    if not h.is_cuda:
        if ids is not None:
            h.copy_(F.embedding(ids, table).float() * scale)
        else:
            y = torch.zeros(T, W)
            if r.y is not None:
                y = y + r.y.float().sum(0)
            if r.bias is not None:
                y = y + r.bias.float()
            if r.ys is not None:
                slot = r.pair_slot.reshape(T, -1).long()
                for j in range(r.pair_w.shape[1]):
                    y = y + torch.where((slot[:, j] >= 0)[:, None],
                                        r.pair_w[:, j, None] * r.ys[slot[:, j].clamp(min=0)].float(), torch.zeros(()))
            h += y * torch.rsqrt(y.square().mean(-1, keepdim=True) + eps) * post.float()
        x = h if weight is None else h * torch.rsqrt(h.square().mean(-1, keepdim=True) + eps) * weight.float()
        return x.to(dtype) if x is not h or dtype != torch.float32 else x.clone()
    out = torch.empty(T, W, dtype=dtype, device=h.device)
    ptr = lambda t: t.data_ptr() if t is not None else None  # noqa: E731
    p = _PostNorm(h=h.data_ptr(), rows=T, W=W, scale=scale, eps=eps, post=ptr(post), norm_w=ptr(weight), out=out.data_ptr())
    for w in (weight, post, table, r.bias if r is not None else None):
        assert w is None or (w.dtype == dtype and w.is_contiguous())
    if ids is not None:
        assert ids.dtype == torch.int64 and ids.is_contiguous()
        p.ids, p.table, p.vocab = ids.data_ptr(), table.data_ptr(), table.shape[0]
    else:
        p.bias = ptr(r.bias)
        if r.y is not None:
            assert r.y.is_contiguous() and r.y.shape[1:] == (T, W)
            p.y, p.slab, p.slabs, p.y_f32 = r.y.data_ptr(), T * W, r.y.shape[0], _f32(r.y)
            assert p.y_f32 or (p.slabs == 1 and r.y.dtype == dtype)
        if r.ys is not None:
            assert r.ys.is_contiguous() and r.ys.dtype == dtype and r.pair_w.dtype == torch.float32
            p.ys, p.pair_slot, p.pair_w, p.top = r.ys.data_ptr(), ptr(r.pair_slot), ptr(r.pair_w), r.pair_w.shape[1]
    _lib.check(_lib.get_lib().sb_post_norm_rows(ctypes.byref(p), int(dtype == torch.float32), _lib.stream()),
               "sb_post_norm_rows")
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
