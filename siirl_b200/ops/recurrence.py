"""Gated outer-product recurrences (linear attention with a matrix state) with a per-sequence state in cache slots.

    S_t = diag(a_t) S_(t-1) + w_t k_t v_t^T,    o_t = S_t^T q_t

Three gate forms: ``"channel"`` (gated linear attention: ``a_t = sigmoid(W2 e_t + b)^(1 / tau)`` per key channel),
``"delta"`` (generalized delta rule, below) and
``"head"`` (the stabilised matrix memory of xLSTM: exponential input gate, sigmoid forget gate, running maximum ``m`` and
a normaliser that is kept as one more value column).  The output is RMS-normed per head, weighted, gated and scaled.

Delta form, with the unit key ``u_t = k_t / sqrt(|k_t|^2 + 1e-6)``, decay ``a_t = exp(-e^(-1/2) sigmoid(W2 tanh(e_t) + b))``
and removal rate ``f_t = sigmoid(f + b_f)`` per key channel:

    S_t = diag(a_t) S_(t-1) - (f_t u_t) (u_t^T S_(t-1)) + k_t v_t^T,    o_t = S_t^T q_t

State of a branch, all in 32-bit floats: ``S [slots, heads, vdim (+1), dim]`` and, for the head form, ``m [slots, heads]``.
A portion that begins at position 0 starts from zero whatever its slot holds.

CUDA tensors run ``csrc/recurrence.cu`` (delta form: ``csrc/delta_rule.cu``): decoding and 32-bit models the token-by-token
kernel, bf16 prompts the chunked tensor-core kernels.  CPU tensors run the plain loop below."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn.functional as F

from . import lib as _lib

CHUNK = 16      # tokens per tile of the chunked kernels (kChunk in csrc/recurrence.cu)


@dataclass
class RecurrenceSpec:
    """Sizes and constants of one branch; the offsets name its columns in the projected rows."""
    gate: str                      # "channel", "head" or "delta"
    heads: int
    dim: int
    vdim: int
    q_off: int
    k_off: int
    v_off: int
    g_off: int
    e_off: int                     # "channel", "delta": low-rank row; "head": input-gate pre-activations
    f_off: int = 0                 # "head": forget-gate pre-activations; "delta": those of the removal rates
    rank: int = 0
    tau: float = 1.0
    cap: float = 1.0
    eps: float = 1e-6
    out_scale: float = 1.0
    gate_act: str = "silu"         # output gate: "silu" or "sigmoid"
    norm_per_head: bool = False    # norm weight per head, or one shared by the heads

    @property
    def rows(self) -> int:
        return self.vdim + (1 if self.gate == "head" else 0)

    @property
    def q_scale(self) -> float:
        return 1.0 if self.gate == "delta" else self.dim ** -0.5

    def state_shapes(self) -> Dict[str, tuple]:
        out = {"S": (self.heads, self.rows, self.dim)}
        if self.gate == "head":
            out["m"] = (self.heads,)
        return out


class _Params(ctypes.Structure):
    """Mirror of ``RecParams`` in csrc/recurrence.cu."""
    _fields_ = [("x", ctypes.c_void_p), ("row_stride", ctypes.c_longlong),
                ("q_off", ctypes.c_int), ("k_off", ctypes.c_int), ("v_off", ctypes.c_int), ("g_off", ctypes.c_int),
                ("e_off", ctypes.c_int), ("f_off", ctypes.c_int),
                ("kind", ctypes.c_int), ("rank", ctypes.c_int), ("norm_per_head", ctypes.c_int),
                ("gate_act", ctypes.c_int),
                ("w2", ctypes.c_void_p), ("b_e", ctypes.c_void_p), ("b_f", ctypes.c_void_p),
                ("norm_w", ctypes.c_void_p),
                ("inv_tau", ctypes.c_float), ("cap", ctypes.c_float), ("q_scale", ctypes.c_float),
                ("eps", ctypes.c_float), ("out_scale", ctypes.c_float),
                ("S", ctypes.c_void_p), ("m", ctypes.c_void_p), ("out", ctypes.c_void_p),
                ("out_stride", ctypes.c_longlong),
                ("out_off", ctypes.c_int), ("H", ctypes.c_int), ("dk", ctypes.c_int), ("dv", ctypes.c_int)]


assert ctypes.sizeof(_Params) == 160


class PortionPlan:
    """Row ranges of a packed batch of prompt portions and their 16-token chunks, on the device."""

    def __init__(self, lens: Sequence[int], starts: Sequence[int], slots: Sequence[int], device):
        self.lens, self.starts, self.slots = list(lens), list(starts), list(slots)
        row0, chunk_row, chunk_len, at = [], [], [], 0
        for n in self.lens:
            row0.append(at)
            for c in range(0, n, CHUNK):
                chunk_row.append(at + c)
                chunk_len.append(min(CHUNK, n - c))
            at += n
        self.row0_cpu, self.n_seq, self.n_chunks, self.total = row0, len(row0), len(chunk_row), at
        self.device = device
        self._segments: Dict[int, Tuple[torch.Tensor, int]] = {}
        # one copy to the device: the pieces are views
        parts = [row0, self.lens, self.slots, self.starts, chunk_row, chunk_len]
        flat = torch.tensor([v for p in parts for v in p], dtype=torch.int32).to(device)
        self.row0, self.nrow, self.slot, self.pos0, self.chunk_row, self.chunk_len = flat.split([len(p) for p in parts])

    def segments(self, blocks: int) -> Tuple[torch.Tensor, int]:
        """Runs of chunks that work in parallel, about ``blocks`` of them in all, equal within a sequence:
        ``[5 n + sequences + 1]`` ints (sequence, first chunk, first row, tokens, flags; first segment per sequence)."""
        want = max(4, -(-self.n_chunks // max(blocks, 1)))
        if want not in self._segments:
            seq, chunk0, row, tokens, flags, first, base = [], [], [], [], [], [0], 0
            for i, n in enumerate(self.lens):
                chunks = -(-n // CHUNK)
                per = -(-chunks // max(1, chunks // want)) if chunks else 1
                for c in range(0, chunks, per):
                    seq.append(i)
                    chunk0.append(base + c)
                    row.append(self.row0_cpu[i] + c * CHUNK)
                    tokens.append(min(per * CHUNK, n - c * CHUNK))
                    flags.append((1 if c == 0 else 0) | (2 if c + per >= chunks else 0))
                base += chunks
                first.append(len(seq))
            flat = torch.tensor(seq + chunk0 + row + tokens + flags + first, dtype=torch.int32)
            self._segments[want] = (flat.to(self.device), len(seq))
        return self._segments[want]


def _params(spec: RecurrenceSpec, x, weights, state, out, out_off) -> _Params:
    assert x.stride(1) == 1 and out.stride(1) == 1 and state["S"].dtype == torch.float32
    kinds = {"channel": 0, "head": 1, "delta": 2}
    addr = lambda t: None if t is None else t.data_ptr()  # noqa: E731
    for w in weights.values():
        assert w.dtype == x.dtype and w.is_contiguous()
    return _Params(
        x=x.data_ptr(), row_stride=x.stride(0), q_off=spec.q_off, k_off=spec.k_off, v_off=spec.v_off, g_off=spec.g_off,
        e_off=spec.e_off, f_off=spec.f_off, kind=kinds[spec.gate], rank=spec.rank,
        norm_per_head=int(spec.norm_per_head), gate_act=1 if spec.gate_act == "sigmoid" else 0,
        w2=addr(weights.get("w2")), b_e=addr(weights["b_e"]), b_f=addr(weights.get("b_f")),
        norm_w=addr(weights["norm"]), inv_tau=1.0 / spec.tau, cap=spec.cap, q_scale=spec.q_scale, eps=spec.eps,
        out_scale=spec.out_scale, S=state["S"].data_ptr(), m=addr(state.get("m")), out=out.data_ptr(),
        out_stride=out.stride(0), out_off=out_off, H=spec.heads, dk=spec.dim, dv=spec.vdim)


def recurrence_prefill(spec: RecurrenceSpec, x: torch.Tensor, weights: Dict[str, torch.Tensor],
                       state: Dict[str, torch.Tensor], plan: PortionPlan, out: torch.Tensor, out_off: int,
                       stepwise: bool = False, segments: Optional[int] = None) -> None:
    """Run packed portions through the recurrence: rows ``x [T, width]``, results in ``out[:, out_off: ...]``, states
    read from and left in the portions' slots.  ``weights``: ``norm`` and ``w2``/``b_e`` (channel form) or ``b_e``/``b_f``
    (head form).  ``stepwise`` forces the token-by-token kernel; ``segments`` (delta form): about that many segments run in
    parallel."""
    if not x.is_cuda:
        rows = [list(range(r, r + n)) for r, n in zip(plan.row0_cpu, plan.lens)]
        _run_cpu(spec, x, weights, state, rows, plan.slots, plan.starts, out, out_off)
        return
    L = _lib.get_lib()
    p = _params(spec, x, weights, state, out, out_off)
    ref = ctypes.byref(p)
    if x.dtype == torch.bfloat16 and not stepwise and spec.gate == "delta":
        fn = L._cdll.sb_delta_workspace
        fn.restype = ctypes.c_longlong
        blocks = int(L._cdll.sb_delta_resident(ref)) // spec.heads if segments is None else segments
        segs, n_seg = plan.segments(blocks)
        if segments is None and n_seg < 3 * plan.n_seq:     # a segment costs two passes over its chunks
            segs, n_seg = plan.segments(plan.n_seq)
        nbytes = int(fn(ref, plan.n_chunks, n_seg, x.shape[0]))
        if nbytes >= 0:
            ws = torch.empty(max(nbytes, 16), dtype=torch.uint8, device=x.device)
            _lib.check(L.sb_delta_prefill(
                ref, _lib.ptr(plan.slot), _lib.ptr(plan.pos0), plan.n_seq, _lib.ptr(plan.chunk_row),
                _lib.ptr(plan.chunk_len), plan.n_chunks, _lib.ptr(segs), n_seg, x.shape[0], _lib.ptr(ws), _lib.stream()),
                "sb_delta_prefill")
            _lib.add_launches(2 if n_seg > plan.n_seq else 0)
            return
    elif x.dtype == torch.bfloat16 and not stepwise:
        fn = L._cdll.sb_recurrence_workspace
        fn.restype = ctypes.c_longlong
        segs, n_seg = plan.segments(int(L._cdll.sb_recurrence_resident(ref)) // spec.heads)
        nbytes = int(fn(ref, plan.n_chunks, n_seg, x.shape[0]))
        if nbytes >= 0:
            ws = torch.empty(max(nbytes, 16), dtype=torch.uint8, device=x.device)
            _lib.check(L.sb_recurrence_prefill(
                ref, _lib.ptr(plan.row0), _lib.ptr(plan.nrow), _lib.ptr(plan.slot), _lib.ptr(plan.pos0), plan.n_seq,
                _lib.ptr(plan.chunk_row), _lib.ptr(plan.chunk_len), plan.n_chunks, _lib.ptr(segs), n_seg, x.shape[0],
                _lib.ptr(ws), _lib.stream()), "sb_recurrence_prefill")
            # counted as two kernels (chunk preparation or gate scan, chunk scan): segment states come on top
            _lib.add_launches(2 if n_seg > plan.n_seq else 0)
            return
    step = L.sb_delta_step if spec.gate == "delta" else L.sb_recurrence_step
    _lib.check(step(ref, _lib.ptr(plan.row0), _lib.ptr(plan.nrow), _lib.ptr(plan.slot),
                                    _lib.ptr(plan.pos0), plan.n_seq, int(x.dtype == torch.float32), _lib.stream()),
               "sb_recurrence_step")


def recurrence_decode(spec: RecurrenceSpec, x: torch.Tensor, weights: Dict[str, torch.Tensor],
                      state: Dict[str, torch.Tensor], slots: torch.Tensor, positions: torch.Tensor, out: torch.Tensor,
                      out_off: int) -> None:
    """One token per row: row ``b`` advances the state in slot ``slots[b]`` (int32; -1: idle, its output is zero)."""
    if not x.is_cuda:
        rows = [[b] for b in range(x.shape[0])]
        _run_cpu(spec, x, weights, state, rows, slots.tolist(), positions.tolist(), out, out_off)
        return
    L = _lib.get_lib()
    p = _params(spec, x, weights, state, out, out_off)
    step = L.sb_delta_step if spec.gate == "delta" else L.sb_recurrence_step
    _lib.check(step(ctypes.byref(p), None, None, _lib.ptr(slots), _lib.ptr(positions), x.shape[0],
                                    int(x.dtype == torch.float32), _lib.stream()), "sb_recurrence_step")


def _run_cpu(spec: RecurrenceSpec, x, weights, state, rows: List[List[int]], slots, starts, out, out_off) -> None:
    H, dk, dv = spec.heads, spec.dim, spec.vdim
    for idx, slot, start in zip(rows, slots, starts):
        if not idx:
            continue
        if slot < 0:
            out[idx, out_off:out_off + H * dv] = 0
            continue
        r = x[idx].float()
        n = len(idx)
        q = r[:, spec.q_off:spec.q_off + H * dk].reshape(n, H, dk) * spec.q_scale
        k = r[:, spec.k_off:spec.k_off + H * dk].reshape(n, H, dk)
        v = r[:, spec.v_off:spec.v_off + H * dv].reshape(n, H, dv)
        g = r[:, spec.g_off:spec.g_off + H * dv]
        S = torch.zeros_like(state["S"][slot]) if start == 0 else state["S"][slot].clone()
        o = torch.empty(n, H, dv)
        if spec.gate == "channel":
            z = r[:, spec.e_off:spec.e_off + spec.rank] @ weights["w2"].float().t() + weights["b_e"].float()
            a = torch.exp(F.logsigmoid(z) / spec.tau).reshape(n, H, 1, dk)
            for t in range(n):
                S = S * a[t] + v[t][:, :, None] * k[t][:, None, :]
                o[t] = torch.einsum("hvd,hd->hv", S, q[t])
        elif spec.gate == "delta":
            z = torch.tanh(r[:, spec.e_off:spec.e_off + spec.rank]) @ weights["w2"].float().t() + weights["b_e"].float()
            a = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).reshape(n, H, 1, dk)
            f = torch.sigmoid(r[:, spec.f_off:spec.f_off + H * dk] + weights["b_f"].float()).reshape(n, H, dk)
            u = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
            for t in range(n):
                seen = torch.einsum("hvd,hd->hv", S, u[t])
                S = S * a[t] - seen[:, :, None] * (f[t] * u[t])[:, None, :] + v[t][:, :, None] * k[t][:, None, :]
                o[t] = torch.einsum("hvd,hd->hv", S, q[t])
        else:
            i = spec.cap * torch.tanh((r[:, spec.e_off:spec.e_off + H] + weights["b_e"].float()) / spec.cap)
            f = F.logsigmoid(spec.cap * torch.tanh((r[:, spec.f_off:spec.f_off + H] + weights["b_f"].float())
                                                   / spec.cap))
            m = torch.zeros(H) if start == 0 else state["m"][slot].clone()
            v1 = torch.cat([v, torch.ones(n, H, 1)], -1)
            for t in range(n):
                mn = torch.maximum(f[t] + m, i[t])
                S = S * torch.exp(f[t] + m - mn)[:, None, None] + \
                    torch.exp(i[t] - mn)[:, None, None] * v1[t][:, :, None] * k[t][:, None, :]
                m = mn
                y = torch.einsum("hvd,hd->hv", S, q[t])
                o[t] = y[:, :dv] / (torch.maximum(y[:, dv:].abs(), torch.exp(-m)[:, None]) + 1e-6)
            state["m"][slot] = m
        state["S"][slot] = S
        w = weights["norm"].float()
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + spec.eps)
        o = (o.reshape(n, H * dv) * w if spec.norm_per_head else (o * w).reshape(n, H * dv))
        gate = torch.sigmoid(g) if spec.gate_act == "sigmoid" else F.silu(g)
        out[idx, out_off:out_off + H * dv] = (o * gate * spec.out_scale).to(out.dtype)


def copy_states(state: Dict[str, torch.Tensor], src: torch.Tensor, dst: torch.Tensor) -> None:
    """Slots ``dst`` receive the states of slots ``src`` (samples of one prompt)."""
    for t in state.values():
        t.index_copy_(0, dst.long(), t.index_select(0, src.long()))


def empty_state(spec: Optional[RecurrenceSpec], slots: int, device) -> Dict[str, torch.Tensor]:
    return {k: torch.zeros(slots, *s, dtype=torch.float32, device=device) for k, s in spec.state_shapes().items()}
