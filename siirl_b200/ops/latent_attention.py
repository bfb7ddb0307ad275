"""Attention over a paged cache of latents: every token leaves one compressed row, from which all heads' keys and values
are expanded.

    c = rms_norm(W_c h) * w,   k_head = W_k[head] c,   v_head = W_v[head] c,   score = q . k * scale,   causal soft-max

Only ``c`` is cached.  One layer's cache is ``[blocks, 64 * rank]``.  Two forms of the same sums:

* expanded, for prompts: keys and values of all visible tokens are one matrix product of the latents, then ordinary
  multi-head attention on the tensor cores (``csrc/fmha_window.cu`` with the keys in packed rows);
* absorbed, for single tokens and short portions: ``q_head W_k[head]`` is a query against the latents themselves and
  ``W_v[head]`` is applied to the weighted sum of latents (``csrc/head_product.cu``, ``csrc/latent_decode.cu``), so a
  step reads one row per cached token whatever the number of heads.

The heads may be gated by the sigmoid of a projection (``g_off``).  ``gain``: one number (a tensor) that multiplies every
projected column, for norms that scale all coordinates alike.  32-bit models and sizes that are no multiple of eight run
the absorbed form on the FMA pipes; CPU tensors the plain statements below."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Optional, Sequence, Tuple

import torch

from . import lib as _lib
from .dense import linear
from .kv_cache import BLOCK
from .window_attention import KV_LATENT, KV_PACKED, QueryTiles, WindowSpec, window_params

SHORT = 16          # portions of at most this many tokens behind a cached prefix take the absorbed form
DECODE_ROWS = 1024  # rows per launch of the absorbed kernel


@dataclass
class LatentSpec:
    """Sizes of one mixer; the offsets name its columns in the projected rows (``g_off < 0``: no output gate)."""
    heads: int
    dim: int
    vdim: int
    rank: int
    q_off: int
    c_off: int
    g_off: int
    scale: float
    eps: float = 1e-6

    @property
    def block_elems(self) -> int:
        return BLOCK * self.rank

    @property
    def aligned(self) -> bool:
        """Sizes the tensor-core kernels take."""
        return self.dim % 8 == 0 and self.vdim % 8 == 0 and self.rank % 8 == 0 and self.q_off % 8 == 0 and \
            (self.g_off < 0 or self.g_off % 8 == 0) and max(self.dim, self.vdim) <= 256


class LatentPlan:
    """Prompt portions (sequence ``i``: ``lens[i]`` rows from position ``starts[i]`` of cache slot ``slots[i]``): where
    the expanded keys of every sequence begin, and the query tiles that point there."""

    def __init__(self, lens: Sequence[int], starts: Sequence[int], slots: Sequence[int], device):
        row0, at = [], 0
        for n, st in zip(lens, starts):
            row0.append(at)
            at += st + n
        self.keys = at
        self.prefix = any(starts)
        self.short = self.prefix and max(lens) <= SHORT
        self.tiles = None if self.short else QueryTiles(lens, starts, row0, device)
        if self.prefix and not self.short:
            total = torch.tensor([st + n for n, st in zip(lens, starts)])
            slot = torch.repeat_interleave(torch.tensor(slots, dtype=torch.int32), total)
            pos = torch.cat([torch.arange(int(n), dtype=torch.int32) for n in total])
            self.key_slot, self.key_pos = torch.stack([slot, pos]).to(device)


class _Params(ctypes.Structure):
    """Mirror of ``LatentParams`` in csrc/latent_params.h."""
    _fields_ = [("x", ctypes.c_void_p), ("row_stride", ctypes.c_longlong), ("c_off", ctypes.c_int), ("T", ctypes.c_int),
                ("seq_ids", ctypes.c_void_p), ("positions", ctypes.c_void_p), ("block_table", ctypes.c_void_p),
                ("cache", ctypes.c_void_p), ("num_blocks", ctypes.c_longlong), ("max_blocks", ctypes.c_int),
                ("H", ctypes.c_int), ("R", ctypes.c_int), ("scale", ctypes.c_float), ("eps", ctypes.c_float),
                ("pad_", ctypes.c_int), ("c_norm", ctypes.c_void_p), ("gain", ctypes.c_void_p),
                ("qa", ctypes.c_void_p), ("out", ctypes.c_void_p)]


assert ctypes.sizeof(_Params) == 120


class _Product(ctypes.Structure):
    """Mirror of ``HeadProduct`` in csrc/latent_params.h."""
    _fields_ = [("a", ctypes.c_void_p), ("a_head", ctypes.c_longlong), ("a_row", ctypes.c_longlong),
                ("b", ctypes.c_void_p), ("b_rows", ctypes.c_int), ("b_cols", ctypes.c_int), ("b_mn", ctypes.c_int),
                ("T", ctypes.c_int), ("H", ctypes.c_int), ("pad_", ctypes.c_int),
                ("c", ctypes.c_void_p), ("c_row", ctypes.c_longlong),
                ("gate", ctypes.c_void_p), ("gate_row", ctypes.c_longlong), ("gain", ctypes.c_void_p)]


assert ctypes.sizeof(_Product) == 96


def head_product(a: torch.Tensor, a_head: int, weight: torch.Tensor, heads: int, out: torch.Tensor, *, by_rows: bool,
                 gate: Optional[torch.Tensor] = None, gain: Optional[torch.Tensor] = None, simt: bool = False) -> None:
    """Every head times its own matrix.  ``weight [heads * m, r]`` holds ``m`` rows per head; head ``h`` of row ``t`` is
    ``a[t, h * a_head:]``.  ``by_rows``: ``out[t, h] = a[t, h, :m] @ weight_h`` (``r`` wide), else
    ``a[t, h, :r] @ weight_h^T`` (``m`` wide).  ``gate``: columns like ``out``'s whose sigmoid (times ``gain``)
    multiplies the result."""
    m, r = weight.shape[0] // heads, weight.shape[1]
    assert a.stride(1) == 1 and out.stride(1) == 1 and weight.is_contiguous() and a.dtype == weight.dtype == out.dtype
    p = _Product(a=a.data_ptr(), a_head=a_head, a_row=a.stride(0), b=weight.data_ptr(), b_rows=m, b_cols=r,
                 b_mn=int(by_rows), T=a.shape[0], H=heads, c=out.data_ptr(), c_row=out.stride(0),
                 gate=gate.data_ptr() if gate is not None else None, gate_row=gate.stride(0) if gate is not None else 0,
                 gain=gain.data_ptr() if gain is not None else None)
    L = _lib.get_lib()
    if simt or a.dtype == torch.float32:
        _lib.check(L.sb_head_product_simt(ctypes.byref(p), int(a.dtype == torch.float32), _lib.stream()),
                   "sb_head_product_simt")
    else:
        _lib.check(L.sb_head_product(ctypes.byref(p), _lib.ptr(_lib.status_word(a.device)), _lib.stream()),
                   "sb_head_product")


_workspace: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}


def _latent_params(spec: LatentSpec, x, w, seq_ids, positions, block_table, cache, qa=None, out=None) -> _Params:
    gain = w.get("gain")
    return _Params(x=x.data_ptr(), row_stride=x.stride(0), c_off=spec.c_off, T=x.shape[0], seq_ids=seq_ids.data_ptr(),
                   positions=positions.data_ptr(), block_table=block_table.data_ptr(), cache=cache.data_ptr(),
                   num_blocks=cache.shape[0], max_blocks=block_table.shape[1], H=spec.heads, R=spec.rank,
                   scale=spec.scale, eps=spec.eps, c_norm=w["c_norm"].data_ptr(),
                   gain=gain.data_ptr() if gain is not None else None, qa=qa.data_ptr() if qa is not None else None,
                   out=out.data_ptr() if out is not None else None)


def latent_append(spec: LatentSpec, x, w, seq_ids, positions, block_table, cache, plan: Optional[LatentPlan] = None):
    """Norm the rows' latents and append them to the cache.  With a ``plan`` returns the latents of every visible position
    ``[plan.keys, rank]``, sequence after sequence (portions behind a prefix read theirs back from the cache)."""
    L, f32 = _lib.get_lib(), int(x.dtype == torch.float32)
    p = _latent_params(spec, x, w, seq_ids, positions, block_table, cache)
    rows = torch.empty(plan.keys, spec.rank, dtype=x.dtype, device=x.device) if plan is not None else None
    _lib.check(L.sb_latent_append(ctypes.byref(p), _lib.ptr(rows if plan is not None and not plan.prefix else None), f32,
                                  _lib.stream()), "sb_latent_append")
    if plan is not None and plan.prefix:
        _lib.check(L.sb_latent_gather(ctypes.byref(p), _lib.ptr(plan.key_slot), _lib.ptr(plan.key_pos), _lib.ptr(rows),
                                      plan.keys, f32, _lib.stream()), "sb_latent_gather")
    return rows


def expanded_attention(spec: LatentSpec, x, gain, kv, seq_ids, positions, block_table, out, out_off, plan: LatentPlan) -> None:
    """Multi-head attention of prompt portions over expanded keys and values ``kv [plan.keys, heads * (dim + vdim)]``."""
    H = spec.heads
    ws = WindowSpec(H, H, spec.dim, spec.vdim, spec.q_off, 0, H * spec.dim, spec.scale)
    q = window_params(ws, x, seq_ids, positions, block_table, kv, out, out_off, kv_mode=KV_PACKED, gain=gain,
                      gate=x[:, spec.g_off:] if spec.g_off >= 0 else None)
    t = plan.tiles
    _lib.check(_lib.get_lib().sb_attn_window_prefill(
        ctypes.byref(q), _lib.ptr(t.row), _lib.ptr(t.rows), _lib.ptr(t.pos), _lib.ptr(t.slot), t.n,
        _lib.ptr(_lib.status_word(x.device)), _lib.stream()), "sb_attn_window_prefill")


def absorbed_attention(spec: LatentSpec, x, w, qa, seq_ids, positions, block_table, cache, mixed, *,
                       simt: bool = False) -> None:
    """Absorbed queries ``qa [T, heads * rank]`` against the cached latents: row ``t`` sees positions up to its own;
    ``mixed [T, heads * rank]`` receives the weighted sums (zero where ``seq_ids[t] < 0``)."""
    L, (T, _), H, R = _lib.get_lib(), qa.shape, spec.heads, spec.rank
    groups = 0 if simt else int(L._cdll.sb_latent_decode_groups(H, R))
    if not groups:
        ws = WindowSpec(H, 1, R, R, 0, 0, 0, spec.scale)
        q = window_params(ws, qa, seq_ids, positions, block_table, cache, mixed, 0, kv_mode=KV_LATENT, gain=w.get("gain"))
        _lib.check(L.sb_attn_window_simt(ctypes.byref(q), int(qa.dtype == torch.float32), _lib.stream()),
                   "sb_attn_window_simt")
        return
    ws = _workspace.get((x.device, H, R))
    if ws is None:      # allocated on first use, before a CUDA graph captures the launch
        per = 2 * int(L._cdll.sb_latent_decode_grid()) * (((H + groups - 1) // groups + 15) // 16 * 16)
        ws = _workspace[(x.device, H, R)] = (
            torch.empty(per * R, dtype=torch.float32, device=x.device),
            torch.empty(per + DECODE_ROWS + 1, dtype=torch.float32, device=x.device))
    for s in range(0, T, DECODE_ROWS):
        e = min(s + DECODE_ROWS, T)
        d = _latent_params(spec, x[s:e], w, seq_ids[s:e], positions[s:e], block_table, cache, qa[s:e], mixed[s:e])
        _lib.check(L.sb_latent_decode(ctypes.byref(d), _lib.ptr(ws[0]), _lib.ptr(ws[1]),
                                      _lib.ptr(_lib.status_word(x.device)), _lib.stream()), "sb_latent_decode")


def latent_attention(spec: LatentSpec, x: torch.Tensor, w: Dict[str, torch.Tensor], seq_ids: torch.Tensor,
                     positions: torch.Tensor, block_table: torch.Tensor, cache: torch.Tensor, out: torch.Tensor,
                     out_off: int, *, plan: Optional[LatentPlan] = None, simt: bool = False) -> None:
    """Append the rows' latents to ``cache`` and attend.  ``w``: ``c_norm [rank]``, ``kv_up [heads * (dim + vdim), rank]``
    (key matrices of all heads, then value matrices), ``gain`` (optional).  ``plan``: prompt portions; without it every row
    is a single token (``seq_ids[t] < 0``: idle, its result is zero).  Results go to ``out[:, out_off: ...]``; ``simt``
    forces the general kernels."""
    if not x.is_cuda:
        return _cpu(spec, x, w, seq_ids, positions, block_table, cache, out, out_off)
    T, H, R, hk, hv = x.shape[0], spec.heads, spec.rank, spec.heads * spec.dim, spec.heads * spec.vdim
    assert x.stride(1) == 1 and out.stride(1) == 1 and cache.dtype == x.dtype == out.dtype == w["kv_up"].dtype
    assert cache[0].numel() == spec.block_elems and cache.is_contiguous() and block_table.is_contiguous()
    assert seq_ids.dtype == positions.dtype == block_table.dtype == torch.int32
    tensor = x.dtype == torch.bfloat16 and not simt and spec.aligned and x.stride(0) % 8 == 0 and \
        out.stride(0) % 8 == 0 and out_off % 8 == 0
    gain = w.get("gain")
    if tensor and plan is not None and not plan.short:
        rows = latent_append(spec, x, w, seq_ids, positions, block_table, cache, plan)
        expanded_attention(spec, x, gain, linear(rows, w["kv_up"]), seq_ids, positions, block_table, out, out_off, plan)
        return
    # absorbed: queries against the latents, the weighted latents through the value matrices
    latent_append(spec, x, w, seq_ids, positions, block_table, cache)
    qa = torch.empty(T, H * R, dtype=x.dtype, device=x.device)
    mixed = torch.empty_like(qa)
    head_product(x[:, spec.q_off:], spec.dim, w["kv_up"][:hk], H, qa, by_rows=True, simt=not tensor)
    absorbed_attention(spec, x, w, qa, seq_ids, positions, block_table, cache, mixed, simt=not tensor)
    head_product(mixed, R, w["kv_up"][hk:], H, out[:, out_off:out_off + hv], by_rows=False, gain=gain,
                 gate=x[:, spec.g_off:] if spec.g_off >= 0 else None, simt=not tensor)


def _cpu(spec: LatentSpec, x, w, seq_ids, positions, block_table, cache, out, out_off) -> None:
    H, R, hk, hv = spec.heads, spec.rank, spec.heads * spec.dim, spec.heads * spec.vdim
    gain = w["gain"].float() if w.get("gain") is not None else 1.0
    pages = cache.view(-1, BLOCK, R)
    z = x[:, spec.c_off:spec.c_off + R].float() * gain
    c = (z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + spec.eps) * w["c_norm"].float()).to(cache.dtype)
    by_slot: Dict[int, list] = {}
    for t, (s, i) in enumerate(zip(seq_ids.tolist(), positions.tolist())):
        if s < 0:
            out[t, out_off:out_off + hv] = 0
        else:
            pages[int(block_table[s, i // BLOCK]), i % BLOCK] = c[t]
            by_slot.setdefault(s, []).append((t, i))
    for s, items in by_slot.items():
        ctx = max(i for _, i in items) + 1
        blocks = block_table[s, :(ctx + BLOCK - 1) // BLOCK].long()
        assert bool((blocks >= 0).all()), "a visible block was freed"
        lat = pages[blocks].reshape(-1, R)[:ctx].float()
        k = (lat @ w["kv_up"][:hk].float().t()).view(ctx, H, spec.dim)
        v = (lat @ w["kv_up"][hk:].float().t()).view(ctx, H, spec.vdim)
        tr = torch.tensor([t for t, _ in items])
        hidden = torch.arange(ctx)[None] > torch.tensor([i for _, i in items])[:, None]
        q = x[tr, spec.q_off:spec.q_off + hk].view(-1, H, spec.dim).float() * gain
        sc = torch.einsum("thd,jhd->htj", q, k) * spec.scale
        o = torch.einsum("htj,jhd->thd", torch.softmax(sc.masked_fill(hidden[None], float("-inf")), -1), v)
        o = o.reshape(len(items), hv)
        if spec.g_off >= 0:
            o = o * torch.sigmoid(x[tr, spec.g_off:spec.g_off + hv].float() * gain)
        out[tr, out_off:out_off + hv] = o.to(out.dtype)
