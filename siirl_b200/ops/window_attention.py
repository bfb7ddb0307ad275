"""Attention over a paged cache with a sliding window, kept first tokens and a linear distance bias.

Position ``i`` sees ``j <= i`` with ``i - j < window`` (``window == 0``: no limit) or ``j < keep_first``; the score is
``q . k * scale - slope_h (i - j)`` with ``slope_h = 2^(-bias_exp (h + 1) / heads)`` (``bias_exp == 0``: no bias).

One layer's cache is ``[blocks, block_elems]``: a block holds 64 tokens, keys ``[kv_heads, 64, dim]`` then values
``[kv_heads, 64, vdim]``.  CUDA: ``csrc/fmha_window.cu`` (prompt portions on the tensor cores, any size and 32-bit on a
SIMT kernel) and the windowed variant of ``csrc/fmha_decode_split.cu`` (single tokens).  CPU: the plain loop below."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, List, Sequence, Tuple

import torch

from . import lib as _lib
from .kv_cache import BLOCK

TILE = 128        # query rows per tile of the prompt kernel


@dataclass
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    q_off: int
    k_off: int
    v_off: int
    scale: float
    window: int = 0
    keep_first: int = 0
    bias_exp: float = 0.0
    out_scale: float = 1.0

    @property
    def block_elems(self) -> int:
        return self.kv_heads * BLOCK * (self.dim + self.vdim)


class _Params(ctypes.Structure):
    """Mirror of ``WinParams`` in csrc/win_params.h."""
    _fields_ = [("x", ctypes.c_void_p), ("row_stride", ctypes.c_longlong),
                ("q_off", ctypes.c_int), ("k_off", ctypes.c_int), ("v_off", ctypes.c_int), ("T", ctypes.c_int),
                ("seq_ids", ctypes.c_void_p), ("positions", ctypes.c_void_p), ("block_table", ctypes.c_void_p),
                ("cache", ctypes.c_void_p), ("num_blocks", ctypes.c_longlong), ("block_elems", ctypes.c_longlong),
                ("max_blocks", ctypes.c_int), ("Hq", ctypes.c_int), ("Hkv", ctypes.c_int), ("dk", ctypes.c_int),
                ("dv", ctypes.c_int), ("window", ctypes.c_int), ("keep_first", ctypes.c_int),
                ("scale", ctypes.c_float), ("bias_exp", ctypes.c_float), ("out_scale", ctypes.c_float),
                ("out", ctypes.c_void_p), ("out_stride", ctypes.c_longlong),
                ("out_off", ctypes.c_int), ("kv_mode", ctypes.c_int),
                ("gain", ctypes.c_void_p), ("gate", ctypes.c_void_p), ("gate_stride", ctypes.c_longlong)]


assert ctypes.sizeof(_Params) == 168
KV_PAGED, KV_PACKED, KV_LATENT = 0, 1, 2


class QueryTiles:
    """128-row query tiles of packed prompt portions (sequence ``i``: ``lens[i]`` rows from position ``starts[i]`` of
    cache slot ``slots[i]``), latest positions first so that the longest tiles start early."""

    def __init__(self, lens: Sequence[int], starts: Sequence[int], slots: Sequence[int], device):
        tiles, at = [], 0
        for n, st, slot in zip(lens, starts, slots):
            tiles += [(at + o, min(TILE, n - o), st + o, slot) for o in range(0, n, TILE)]
            at += n
        tiles.sort(key=lambda t: -t[2])
        self.n = len(tiles)
        flat = torch.tensor([t[c] for c in range(4) for t in tiles], dtype=torch.int32).to(device)
        self.row, self.rows, self.pos, self.slot = flat.split([self.n] * 4) if self.n else (flat,) * 4


def window_params(spec: WindowSpec, x, seq_ids, positions, block_table, cache, out, out_off, *, kv_mode: int = KV_PAGED,
                  gain: torch.Tensor = None, gate: torch.Tensor = None) -> _Params:
    """``kv_mode``: where keys and values are.  ``KV_PAGED``: in ``cache`` as described above.  ``KV_PACKED`` (prompts):
    ``cache`` is ``[rows, kv_heads * (dim + vdim)]``, one row per key, keys before values, and a tile's slot is the row of
    its sequence's first key.  ``KV_LATENT`` (general kernel): keys and values are the same ``dim``-wide rows of a paged
    cache.  ``gain``: one number (a tensor) that multiplies the queries and the gate.  ``gate``: columns like ``out``'s whose
    sigmoid multiplies the result (prompts)."""
    assert x.stride(1) == 1 and out.stride(1) == 1 and cache.dtype == x.dtype == out.dtype
    per_row = spec.kv_heads * (spec.dim + spec.vdim)
    elems = {KV_PAGED: spec.block_elems, KV_PACKED: per_row, KV_LATENT: BLOCK * spec.dim}[kv_mode]
    assert cache[0].numel() == elems and cache.is_contiguous() and block_table.is_contiguous()
    assert seq_ids.dtype == positions.dtype == block_table.dtype == torch.int32
    return _Params(x=x.data_ptr(), row_stride=x.stride(0), q_off=spec.q_off, k_off=spec.k_off, v_off=spec.v_off,
                   T=x.shape[0], seq_ids=seq_ids.data_ptr(), positions=positions.data_ptr(),
                   block_table=block_table.data_ptr(), cache=cache.data_ptr(), num_blocks=cache.shape[0],
                   block_elems=elems, max_blocks=block_table.shape[1], Hq=spec.heads, Hkv=spec.kv_heads,
                   dk=spec.dim, dv=spec.vdim, window=spec.window, keep_first=spec.keep_first, scale=spec.scale,
                   bias_exp=spec.bias_exp, out_scale=spec.out_scale, out=out.data_ptr(), out_stride=out.stride(0),
                   out_off=out_off, kv_mode=kv_mode, gain=gain.data_ptr() if gain is not None else None,
                   gate=gate.data_ptr() if gate is not None else None,
                   gate_stride=gate.stride(0) if gate is not None else 0)


_workspace: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}


def window_attention(spec: WindowSpec, x: torch.Tensor, seq_ids: torch.Tensor, positions: torch.Tensor,
                     block_table: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, out_off: int, *,
                     tiles: QueryTiles = None, seq_lens: torch.Tensor = None, simt: bool = False) -> None:
    """Append the rows' keys and values to ``cache`` and attend.  Prompt portions: ``tiles``.  Decoding: ``seq_lens``
    (context lengths with the current token; row ``b`` is cache slot ``b``, 0 = idle).  Results go to
    ``out[:, out_off: ...]``.  ``simt`` forces the general kernel."""
    if not x.is_cuda:
        return _cpu(spec, x, seq_ids, positions, block_table, cache, out, out_off)
    L = _lib.get_lib()
    p = window_params(spec, x, seq_ids, positions, block_table, cache, out, out_off)
    ref = ctypes.byref(p)
    f32 = int(x.dtype == torch.float32)
    _lib.check(L.sb_kv_append_split(ref, f32, _lib.stream()), "sb_kv_append_split")
    status = _lib.ptr(_lib.status_word(x.device))
    aligned = spec.dim % 8 == 0 and spec.vdim % 8 == 0 and x.stride(0) % 8 == 0 and out.stride(0) % 8 == 0 and \
        spec.q_off % 8 == 0 and out_off % 8 == 0
    if not f32 and not simt and aligned:
        if tiles is not None and max(spec.dim, spec.vdim) <= 256:
            _lib.check(L.sb_attn_window_prefill(ref, _lib.ptr(tiles.row), _lib.ptr(tiles.rows), _lib.ptr(tiles.pos),
                                                _lib.ptr(tiles.slot), tiles.n, status, _lib.stream()),
                       "sb_attn_window_prefill")
            return
        chunks = int(L._cdll.sb_attn_window_decode_chunks(ref)) if tiles is None else -1
        if chunks > 0:
            width = 128 if max(spec.dim, spec.vdim) > 64 else 64
            key = (x.device, x.shape[0], spec.heads, chunks, width)
            ws = _workspace.get(key)
            if ws is None:      # allocated on first use, before a CUDA graph captures the launch
                ws = _workspace[key] = (torch.empty(x.shape[0] * spec.heads * chunks * width, dtype=torch.float32,
                                                    device=x.device),
                                        torch.empty(x.shape[0] * spec.heads * chunks, dtype=torch.float32,
                                                    device=x.device))
            _lib.check(L.sb_attn_window_decode(ref, _lib.ptr(seq_lens), _lib.ptr(ws[0]), _lib.ptr(ws[1]), status,
                                               _lib.stream()), "sb_attn_window_decode")
            return
    _lib.check(L.sb_attn_window_simt(ref, f32, _lib.stream()), "sb_attn_window_simt")


def _cpu(spec: WindowSpec, x, seq_ids, positions, block_table, cache, out, out_off) -> None:
    H, G, dk, dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    split = G * BLOCK * dk
    kc = cache[:, :split].view(-1, G, BLOCK, dk)
    vc = cache[:, split:].view(-1, G, BLOCK, dv)
    rows = [(t, int(s), int(i)) for t, (s, i) in enumerate(zip(seq_ids.tolist(), positions.tolist()))]
    for t, s, i in rows:
        if s >= 0:
            b = int(block_table[s, i // BLOCK])
            kc[b, :, i % BLOCK] = x[t, spec.k_off:spec.k_off + G * dk].view(G, dk)
            vc[b, :, i % BLOCK] = x[t, spec.v_off:spec.v_off + G * dv].view(G, dv)
    slope = torch.tensor([2.0 ** (-spec.bias_exp * (h + 1) / H) if spec.bias_exp else 0.0 for h in range(H)])
    by_slot: Dict[int, List[Tuple[int, int]]] = {}
    for t, s, i in rows:
        if s < 0:
            out[t, out_off:out_off + H * dv] = 0
        else:
            by_slot.setdefault(s, []).append((t, i))
    for s, items in by_slot.items():
        ctx = max(i for _, i in items) + 1
        j = torch.arange(ctx)
        idx = torch.tensor([i for _, i in items])[:, None]
        seen = j[None] <= idx
        if spec.window:
            seen = seen & ((idx - j < spec.window) | (j < spec.keep_first))
        nb = (ctx + BLOCK - 1) // BLOCK
        blocks = block_table[s, :nb].long()
        used = seen.any(0)
        assert bool((blocks[torch.div(j[used], BLOCK, rounding_mode="floor")] >= 0).all()), "a visible block was freed"
        blocks = blocks.clamp(min=0)
        k = kc[blocks].permute(1, 0, 2, 3).reshape(G, nb * BLOCK, dk)[:, :ctx].float().repeat_interleave(H // G, 0)
        v = vc[blocks].permute(1, 0, 2, 3).reshape(G, nb * BLOCK, dv)[:, :ctx].float().repeat_interleave(H // G, 0)
        tr = torch.tensor([t for t, _ in items])
        q = x[tr, spec.q_off:spec.q_off + H * dk].view(-1, H, dk).float()
        sc = torch.einsum("thd,hjd->htj", q, k) * spec.scale - slope[:, None, None] * (idx - j)[None]
        pr = torch.softmax(sc.masked_fill(~seen[None], float("-inf")), -1)
        o = torch.einsum("htj,hjd->thd", pr, v) * spec.out_scale
        out[tr, out_off:out_off + H * dv] = o.reshape(len(items), H * dv).to(out.dtype)
