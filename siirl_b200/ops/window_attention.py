"""Attention over a paged cache with a sliding window, kept first tokens and a linear distance bias, or with a soft cap, a
learned distance table, a sink, pooled blocks before the window and gated heads, and what comes before it: norms and rotation
of queries and keys.

Position ``i`` sees ``j <= i`` with ``i - j < window`` (``window == 0``: no limit) or ``j < keep_first``; the score is
``q . k * scale - slope_h (i - j)`` with ``slope_h = 2^(-bias_exp (h + 1) / heads)`` (``bias_exp == 0``: no bias), or
``cap * tanh(q . k * scale / cap) + table[h, i - j]``.  A sink is one more score in the soft-max's sum, without a value: 0, or
a learned number per head.

With ``pool = P`` position ``i`` sees, beside its window, every whole block of ``P`` tokens that lies before the window
(``(b + 1) P - 1 <= i - window``) as one key and one value: the means of what the cache holds.  They are made when the block's
last token is appended and live in blocks of their own of the same cache, entry ``b`` at row ``b % 64`` of block
``pool_table[slot, b / 64]``.  Tokens between the window and the last such block are not seen.

One layer's cache is ``[blocks, block_elems]``: a block holds 64 tokens, keys ``[kv_heads, 64, dim]`` then values
``[kv_heads, 64, vdim]``.  CUDA: ``csrc/fmha_window.cu`` (prompt portions on the tensor cores, any size and 32-bit on a
SIMT kernel) and the windowed variant of ``csrc/fmha_decode_split.cu`` (single tokens); ``csrc/qkv_prepare.cu`` does
biases, norms, rotation and the append in one launch.  CPU: the plain loop below."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass, replace
from typing import Any, Dict, List, Optional, Sequence, Tuple

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
    softcap: float = 0.0
    sink: bool = False
    pool: int = 0

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
                ("gain", ctypes.c_void_p), ("gate", ctypes.c_void_p), ("gate_stride", ctypes.c_longlong),
                ("softcap", ctypes.c_float), ("sink", ctypes.c_int), ("rel", ctypes.c_void_p),
                ("rel_n", ctypes.c_longlong), ("head_gate", ctypes.c_void_p),
                ("pool", ctypes.c_int), ("pool_blocks", ctypes.c_int), ("pool_table", ctypes.c_void_p),
                ("sink_w", ctypes.c_void_p)]


assert ctypes.sizeof(_Params) == 224
KV_PAGED, KV_PACKED, KV_LATENT = 0, 1, 2


class _PrepareParams(ctypes.Structure):
    """Mirror of ``PrepareParams`` in csrc/qkv_prepare.cu."""
    _fields_ = [("x", ctypes.c_void_p), ("slab", ctypes.c_longlong), ("row_stride", ctypes.c_longlong),
                ("slabs", ctypes.c_int), ("x_f32", ctypes.c_int), ("bias", ctypes.c_void_p),
                ("q_off", ctypes.c_int), ("k_off", ctypes.c_int), ("v_off", ctypes.c_int), ("g_off", ctypes.c_int),
                ("T", ctypes.c_int), ("Hq", ctypes.c_int), ("Hkv", ctypes.c_int), ("dk", ctypes.c_int), ("dv", ctypes.c_int),
                ("norm", ctypes.c_int), ("q_norm", ctypes.c_void_p), ("k_norm", ctypes.c_void_p), ("eps", ctypes.c_float),
                ("half", ctypes.c_int), ("freq", ctypes.c_void_p), ("seq_ids", ctypes.c_void_p),
                ("positions", ctypes.c_void_p), ("block_table", ctypes.c_void_p), ("cache", ctypes.c_void_p),
                ("num_blocks", ctypes.c_longlong), ("block_elems", ctypes.c_longlong), ("max_blocks", ctypes.c_int),
                ("rel_n", ctypes.c_int), ("q_out", ctypes.c_void_p), ("q_stride", ctypes.c_longlong),
                ("gate_out", ctypes.c_void_p), ("rel", ctypes.c_void_p), ("bucket", ctypes.c_void_p),
                ("rel_out", ctypes.c_void_p), ("rot_mag", ctypes.c_float), ("pool", ctypes.c_int),
                ("pool_table", ctypes.c_void_p), ("pool_blocks", ctypes.c_int), ("pool_inline", ctypes.c_int)]


assert ctypes.sizeof(_PrepareParams) == 240
_NORMS = {"": 0, "rows": 1, "heads": 2, "head_weights": 3}


def rotary_frequencies(dims: int, base: float, scaling: Optional[Dict[str, Any]] = None) -> List[float]:
    """Angular frequency ``base^(-2 i / dims)`` of every rotated pair.  ``scaling`` (factor, low, high, original): wavelengths
    above ``original / low`` are stretched by ``factor``, those below ``original / high`` kept, the ones between blended.
    ``scaling`` (factor, original, fast, slow): YaRN, blended linearly in the pair's number between those that turn ``fast``
    and ``slow`` times within ``original`` positions."""
    out = []
    if scaling and "fast" in scaling:
        def pair_of(turns: float) -> float:
            return dims * math.log(float(scaling["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))
        first = max(math.floor(pair_of(float(scaling["fast"]))), 0)
        last = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
        for i in range(dims // 2):
            f, ramp = float(base) ** (-2.0 * i / dims), (i - first) / max(last - first, 0.001)
            ramp = min(max(ramp, 0.0), 1.0)
            out.append(f / float(scaling["factor"]) * ramp + f * (1.0 - ramp))
        return out
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            wave, length = 2.0 * math.pi / f, float(scaling["original"])
            lo, hi, factor = (float(scaling[k]) for k in ("low", "high", "factor"))
            if wave > length / lo:
                f = f / factor
            elif wave >= length / hi:
                s = (length / wave - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotary_magnitude(scaling: Optional[Dict[str, Any]] = None) -> float:
    """Factor of cosines and sines."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and "fast" in scaling else 1.0


def distance_buckets(rows: int, far: int, limit: int = 0) -> List[int]:
    """Table row of every distance from 0 on: one each for the first half of the rows, then logarithmic until ``far``.  The
    list ends at the first distance whose row is the last one (every later distance has it too), or at ``limit``."""
    half, out = rows // 2, []
    while not limit or len(out) < limit:
        n = len(out)
        if n < half:
            b = n
        elif half == 0 or far <= half:
            b = rows - 1
        else:
            b = min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))
        out.append(b)
        if b == rows - 1:
            break
    return out


@dataclass
class QkvPrepare:
    """What happens to the projected rows before the attention, see csrc/qkv_prepare.cu.  Rows may come as partial sums."""
    norm: str = ""                              # "", "rows", "heads" or "head_weights"
    eps: float = 1e-6
    freq: Optional[torch.Tensor] = None         # [pairs, 2] fp32: frequency as hi + lo
    g_off: int = -1                             # column of the per-head output gates
    bias: Optional[torch.Tensor] = None         # like a row of the projection
    q_norm: Optional[torch.Tensor] = None       # a whole projection ("rows") or one head ("head_weights")
    k_norm: Optional[torch.Tensor] = None
    magnitude: float = 1.0                      # factor of cosines and sines
    sink: Optional[torch.Tensor] = None         # [heads] learned scores
    rel: Optional[torch.Tensor] = None          # [table rows, heads]
    bucket: Optional[torch.Tensor] = None       # [distances] int32
    table: Optional[torch.Tensor] = None        # [heads, distances] fp32, filled from rel and bucket

    def run(self, spec: "WindowSpec", x: torch.Tensor, seq_ids, positions, block_table, cache, pool_table=None,
            single: bool = False):
        """``x [S, T, N]`` or ``[T, N]`` -> queries ``[T, heads * dim]`` (padded rows) and gates ``[T, heads]``; keys and
        values, and pooled entries that become whole, go to the cache.  ``single``: no two rows of one sequence."""
        x = x if x.dim() == 3 else x[None]
        S, T, N = x.shape
        assert x.stride(2) == 1 and (S == 1 or x.dtype == torch.float32) and cache.is_contiguous()
        assert self.rel is None or tuple(self.table.shape) == (spec.heads, self.bucket.numel())
        q = torch.empty(T, (spec.heads * spec.dim + 7) // 8 * 8, dtype=cache.dtype, device=x.device)
        gate = torch.empty(T, spec.heads, dtype=torch.float32, device=x.device) if self.g_off >= 0 else None
        ptr = lambda t: t.data_ptr() if t is not None else None  # noqa: E731
        p = _PrepareParams(
            x=x.data_ptr(), slab=x.stride(0), row_stride=x.stride(1), slabs=S, x_f32=int(x.dtype == torch.float32),
            bias=ptr(self.bias), q_off=spec.q_off, k_off=spec.k_off, v_off=spec.v_off, g_off=self.g_off, T=T, Hq=spec.heads,
            Hkv=spec.kv_heads, dk=spec.dim, dv=spec.vdim, norm=_NORMS[self.norm], q_norm=ptr(self.q_norm),
            k_norm=ptr(self.k_norm), eps=self.eps, half=self.freq.shape[0] if self.freq is not None else 0,
            freq=ptr(self.freq), seq_ids=seq_ids.data_ptr(), positions=positions.data_ptr(),
            block_table=block_table.data_ptr(), cache=cache.data_ptr(), num_blocks=cache.shape[0],
            block_elems=spec.block_elems, max_blocks=block_table.shape[1],
            rel_n=self.bucket.numel() if self.rel is not None else 0, q_out=q.data_ptr(), q_stride=q.stride(0),
            gate_out=ptr(gate), rel=ptr(self.rel), bucket=ptr(self.bucket), rel_out=ptr(self.table),
            rot_mag=self.magnitude, pool=spec.pool, pool_table=ptr(pool_table),
            pool_blocks=pool_table.shape[1] if pool_table is not None else 0, pool_inline=int(single and spec.pool > 0))
        assert not spec.pool or (pool_table is not None and pool_table.is_contiguous() and pool_table.dtype == torch.int32)
        _lib.check(_lib.get_lib().sb_qkv_prepare(ctypes.byref(p), int(cache.dtype == torch.float32), _lib.stream()),
                   "sb_qkv_prepare")
        if spec.pool and not single:
            _lib.check(_lib.get_lib().sb_kv_pool(ctypes.byref(p), int(cache.dtype == torch.float32), _lib.stream()),
                       "sb_kv_pool")
        return q, gate

    def plain(self, spec: "WindowSpec", x: torch.Tensor, positions: torch.Tensor):
        """The same on the CPU: rows like ``x`` with queries, keys and values as the attention takes them, and the gates."""
        x = (x.float().sum(0) if x.dim() == 3 else x.float())
        if self.bias is not None:
            x = x + self.bias.float()
        T, H, G, dk = x.shape[0], spec.heads, spec.kv_heads, spec.dim
        out = x.clone()
        if spec.v_off == spec.k_off:        # the values are the keys as projected: they keep a place of their own
            out = torch.cat([out, x[:, spec.v_off:spec.v_off + G * spec.vdim]], 1)
        for off, n, w in ((spec.q_off, H, self.q_norm), (spec.k_off, G, self.k_norm)):
            y = x[:, off:off + n * dk]
            if self.norm == "rows":
                y = y * torch.rsqrt(y.square().mean(-1, keepdim=True) + self.eps) * w.float()
            y = y.reshape(T, n, dk)
            if self.norm == "head_weights":
                y = y * torch.rsqrt(y.square().mean(-1, keepdim=True) + self.eps) * w.float()
            if self.freq is not None:
                half = self.freq.shape[0]
                a = positions.double()[:, None] * self.freq.double().sum(-1)[None]
                c, s = (self.magnitude * torch.cos(a)).float()[:, None], (self.magnitude * torch.sin(a)).float()[:, None]
                u, v = y[..., :half], y[..., half:2 * half]
                y = torch.cat([u * c - v * s, v * c + u * s, y[..., 2 * half:]], -1)
            if self.norm == "heads":
                y = y * torch.rsqrt(y.square().mean(-1, keepdim=True) + self.eps)
            out[:, off:off + n * dk] = y.reshape(T, n * dk)
        gate = torch.sigmoid(x[:, self.g_off:self.g_off + H]) if self.g_off >= 0 else None
        return out, gate


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
                  gain: torch.Tensor = None, gate: torch.Tensor = None, rel: torch.Tensor = None,
                  head_gate: torch.Tensor = None, pool_table: torch.Tensor = None, sink: torch.Tensor = None) -> _Params:
    """``kv_mode``: where keys and values are.  ``KV_PAGED``: in ``cache`` as described above.  ``KV_PACKED`` (prompts):
    ``cache`` is ``[rows, kv_heads * (dim + vdim)]``, one row per key, keys before values, and a tile's slot is the row of
    its sequence's first key.  ``KV_LATENT`` (general kernel): keys and values are the same ``dim``-wide rows of a paged
    cache.  ``gain``: one number (a tensor) that multiplies the queries and the gate.  ``gate``: columns like ``out``'s whose
    sigmoid multiplies the result (prompts).  ``rel [heads, distances]``: bias by distance.  ``head_gate [T, heads]``: factors
    of the result.  ``pool_table``: blocks of the pooled entries.  ``sink [heads]``: learned scores of the sink."""
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
                   gate_stride=gate.stride(0) if gate is not None else 0, softcap=spec.softcap, sink=int(spec.sink),
                   rel=rel.data_ptr() if rel is not None else None, rel_n=rel.shape[1] if rel is not None else 0,
                   head_gate=head_gate.data_ptr() if head_gate is not None else None,
                   pool=spec.pool, pool_blocks=pool_table.shape[1] if pool_table is not None else 0,
                   pool_table=pool_table.data_ptr() if pool_table is not None else None,
                   sink_w=sink.data_ptr() if sink is not None else None)


_workspace: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}


def window_attention(spec: WindowSpec, x: torch.Tensor, seq_ids: torch.Tensor, positions: torch.Tensor,
                     block_table: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, out_off: int, *,
                     tiles: QueryTiles = None, seq_lens: torch.Tensor = None, simt: bool = False,
                     prepare: Optional[QkvPrepare] = None, pool_table: torch.Tensor = None) -> None:
    """Append the rows' keys and values to ``cache`` and attend.  Prompt portions: ``tiles``.  Decoding: ``seq_lens``
    (context lengths with the current token; row ``b`` is cache slot ``b``, 0 = idle).  Results go to
    ``out[:, out_off: ...]``.  ``prepare``: biases, norms, rotation, gates and distance table of the branch; ``x`` may then
    be partial sums ``[S, T, N]``.  ``pool_table`` (with ``spec.pool``): blocks of the pooled entries.  ``simt`` forces the
    general kernel."""
    if spec.pool and (spec.window < 1 or prepare is None or pool_table is None):
        raise ValueError("pooled blocks: a window, blocks to keep them in and a prepare step that makes them")
    if spec.pool and (spec.softcap or spec.keep_first or spec.bias_exp or prepare.rel is not None):
        raise ValueError("pooled blocks: no kept first tokens, biases by distance or soft-capped scores")
    if not x.is_cuda:
        gate = None
        if prepare is not None:
            if spec.v_off == spec.k_off:
                spec = replace(spec, v_off=x.shape[-1])
                x, gate = prepare.plain(replace(spec, v_off=spec.k_off), x, positions)
            else:
                x, gate = prepare.plain(spec, x, positions)
        return _cpu(spec, x, seq_ids, positions, block_table, cache, out, out_off, prepare, gate, pool_table)
    L = _lib.get_lib()
    if prepare is not None:
        x, gate = prepare.run(spec, x, seq_ids, positions, block_table, cache, pool_table, single=tiles is None)
        spec = replace(spec, q_off=0)
        p = window_params(spec, x, seq_ids, positions, block_table, cache, out, out_off,
                          rel=prepare.table if prepare.rel is not None else None, head_gate=gate,
                          pool_table=pool_table if spec.pool else None, sink=prepare.sink)
    else:
        p = window_params(spec, x, seq_ids, positions, block_table, cache, out, out_off)
    ref = ctypes.byref(p)
    f32 = int(x.dtype == torch.float32)
    if prepare is None:
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


def _cpu(spec: WindowSpec, x, seq_ids, positions, block_table, cache, out, out_off, prepare=None, gate=None,
         pool_table=None) -> None:
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
    for _, s, i in rows:
        if s >= 0 and spec.pool and (i + 1) % spec.pool == 0:
            j = torch.arange(i + 1 - spec.pool, i + 1)
            b, e = block_table[s, torch.div(j, BLOCK, rounding_mode="floor")].long(), i // spec.pool
            to = int(pool_table[s, e // BLOCK])
            assert bool((b >= 0).all()) and to >= 0, "a block of a pooled run was freed, or there is none for its mean"
            for c in (kc, vc):
                c[to, :, e % BLOCK] = c[b, :, j % BLOCK].float().mean(0).to(c.dtype)
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
        if spec.softcap:
            sc = spec.softcap * torch.tanh(sc / spec.softcap)
        if prepare is not None and prepare.rel is not None:
            far = prepare.bucket.numel() - 1
            sc = sc + prepare.rel.float()[prepare.bucket[(idx - j).clamp(0, far)].long()].permute(2, 0, 1)
        sc = sc.masked_fill(~seen[None], float("-inf"))
        if spec.pool and int(idx.max()) >= spec.window + spec.pool - 1:
            n = (int(idx.max()) - spec.window + 1) // spec.pool
            e = torch.arange(n)
            b = pool_table[s, torch.div(e, BLOCK, rounding_mode="floor")].long()
            assert bool((b >= 0).all()), "a block of pooled entries was freed"
            kp, vp = (c[b, :, e % BLOCK].float().permute(1, 0, 2).repeat_interleave(H // G, 0) for c in (kc, vc))
            sp = torch.einsum("thd,hjd->htj", q, kp) * spec.scale
            sc = torch.cat([sc, sp.masked_fill(((e + 1) * spec.pool - 1 > idx - spec.window)[None], float("-inf"))], -1)
            v = torch.cat([v, vp], 1)
        if prepare is not None and prepare.sink is not None:
            last = prepare.sink.float()[:, None, None].expand(H, sc.shape[1], 1)
            pr = torch.softmax(torch.cat([sc, last], -1), -1)[..., :-1]
        elif spec.sink:
            pr = torch.softmax(torch.cat([sc, torch.zeros(*sc.shape[:2], 1)], -1), -1)[..., :-1]
        else:
            pr = torch.softmax(sc, -1)
        o = torch.einsum("htj,hjd->thd", pr, v) * spec.out_scale
        if gate is not None:
            o = o * gate[tr][:, :, None]
        out[tr, out_off:out_off + H * dv] = o.reshape(len(items), H * dv).to(out.dtype)
