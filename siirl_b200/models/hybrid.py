"""Hybrid decoder: layers that mix window attention, latent attention and matrix-state recurrences, with the residual
stream in 32-bit.

Every layer is a list of branches over one normed input (``DecoderConfig.hybrid``): their projections are one fused
matrix (``in_proj``), each branch writes its (scaled) heads into its columns of one row, and one matrix (``o_proj``) adds
the branches up.  In the parallel arrangement the feed-forward reads the same stream and the residual gates read the
sublayers' inputs, so their matrices join ``in_proj``: the norms there are one number each, which commutes with the
projections, and one row (the stream over its root mean square) feeds them all; the numbers are applied by the kernels
behind.  In the hyper arrangement several copies of the stream are mixed between sublayers, the mixers are attention of
several kinds and a feed-forward may be routed.  In the sandwich arrangement every sublayer's result passes a second norm
before it is added, and a second embedding table feeds every layer.  A run of layers may be repeated (``HybridSpec.loop``).

The serving path is the one of :class:`DecoderLM`: ``forward_cached`` over the engine's paged blocks, plus the engine's
per-slot recurrent states.  A prompt portion appends its keys and values and reads everything it sees back from the
cache, so whole prompts, portions and single tokens use the same memory.

bf16 models run the tensor-core kernels; fp32 models run true 32-bit kernels (FMA-pipe matrix products).  Weights keep
the checkpoint's values; fused matrices are padded with zero rows / columns to multiples of eight.  Scoring
(``logprobs``) is supported; there is no backward pass on CUDA."""
from __future__ import annotations

import ctypes
from dataclasses import replace
from typing import Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops import kv_cache as kvc
from ..ops import rows as R
from ..ops.attention import SeqInfo
from ..ops.dense import linear_partial
from ..ops.latent_attention import LatentPlan, LatentSpec, latent_attention
from ..ops.lm_head import lm_head_logits
from ..ops.recurrence import PortionPlan, RecurrenceSpec, empty_state, recurrence_decode, recurrence_prefill
from ..ops.moe import route_grouped, routed_experts
from ..ops.window_attention import (QkvPrepare, QueryTiles, WindowSpec, distance_buckets, rotary_frequencies,
                                    rotary_magnitude, window_attention)
from .config import DecoderConfig, ExpertSpec, MixerBranch
from .decoder import _Init, _param


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def branch_segments(b: MixerBranch) -> List[Tuple[str, int]]:
    """(name, rows) of a branch's projections in ``in_proj``, in order."""
    hk, hv = b.heads * b.dim, b.heads * b.vdim
    if b.kind == "attention":
        seg = [("q", hk), ("k", b.kv_heads * b.dim)] + ([] if b.key_values else [("v", b.kv_heads * b.vdim)])
        return seg + ([("g", b.heads)] if b.head_gate else [])
    if b.kind == "general_delta":
        return [("r", hk), ("k", hk), ("v", hv), ("g", hv), ("a", hk), ("w1", b.rank)]
    if b.kind == "latent_attention":
        return [("q", hk), ("c", b.kv_rank)] + ([("g", hv)] if b.output_gate else [])
    seg = [("q", hk), ("k", hk), ("v", hv), ("g", hv)]
    return seg + ([("a1", b.rank)] if b.kind == "gated_linear" else [("i", b.heads), ("f", b.heads)])


class HybridBranch(nn.Module):
    """Small parameters of one branch and its place in the layer's fused rows."""

    def __init__(self, b: MixerBranch, cfg: DecoderConfig, in_off: int, out_off: int, dtype, device, gen):
        super().__init__()
        self.b = b
        self.out_off = out_off
        self.cols: Dict[str, Tuple[int, int]] = {}
        for name, n in branch_segments(b):
            self.cols[name] = (in_off, n)
            in_off += _pad8(n)
        self.in_end = in_off
        off = {k: v[0] for k, v in self.cols.items()}
        if b.kind == "attention":
            if b.key_values and b.vdim != b.dim:
                raise ValueError("attention: values that are the keys have their width")
            self.spec = WindowSpec(b.heads, b.kv_heads, b.dim, b.vdim, off["q"], off["k"], off.get("v", off["k"]), b.scale,
                                   b.window, b.keep_first, b.bias_exp, b.out_scale, b.softcap, b.sink, b.pool)
            if b.sink_weight:
                self.sink = _param((b.heads,), dtype, device, 1.0, gen)
            self.prepare = self._prepare(cfg, in_off, off, dtype, device, gen)
            return
        hk, hv = b.heads * b.dim, b.heads * b.vdim
        if b.kind == "latent_attention":
            if b.kv_rank < 1 or b.out_scale != 1.0:
                raise ValueError("latent_attention: a latent width and no output scale")
            self.c_norm = _param((b.kv_rank,), dtype, device, -1, gen)
            self.kv_up_weight = _param((hk + hv, b.kv_rank), dtype, device, b.kv_rank ** -0.5, gen)
            self.spec = LatentSpec(b.heads, b.dim, b.vdim, b.kv_rank, off["q"], off["c"], off.get("g", -1), b.scale,
                                   cfg.rms_norm_eps)
            return
        common = dict(heads=b.heads, dim=b.dim, vdim=b.vdim, q_off=off["r" if b.kind == "general_delta" else "q"],
                      k_off=off["k"], v_off=off["v"], g_off=off["g"], eps=cfg.rms_norm_eps, out_scale=b.out_scale)
        if b.kind == "gated_linear":
            if b.rank < 1:
                raise ValueError("gated_linear: the decay's low-rank width is not set")
            self.norm = _param((b.vdim,), dtype, device, -1, gen)
            self.w2 = _param((hk, b.rank), dtype, device, b.rank ** -0.5, gen)
            self.b_e = _param((hk,), dtype, device, 1.0, gen)
            self.spec = RecurrenceSpec("channel", e_off=off["a1"], rank=b.rank, tau=b.tau, gate_act="silu", **common)
        elif b.kind == "matrix_memory":
            self.norm = _param((hv,), dtype, device, -1, gen)
            self.b_e = _param((b.heads,), dtype, device, 0, gen)
            self.b_f = _param((b.heads,), dtype, device, 1.0, gen)
            self.spec = RecurrenceSpec("head", e_off=off["i"], f_off=off["f"], cap=b.gate_cap, gate_act="sigmoid",
                                       norm_per_head=True, **common)
        elif b.kind == "general_delta":
            if b.rank < 1 or b.vdim != b.dim:
                raise ValueError("general_delta: the decay's low-rank width is not set, or unequal key and value widths")
            self.norm = _param((hv,), dtype, device, -1, gen)
            self.w2 = _param((hk, b.rank), dtype, device, b.rank ** -0.5, gen)
            self.b_e = _param((hk,), dtype, device, 1.0, gen)
            self.b_f = _param((hk,), dtype, device, 1.0, gen)
            self.spec = RecurrenceSpec("delta", e_off=off["w1"], f_off=off["a"], rank=b.rank, gate_act="sigmoid",
                                       norm_per_head=True, **common)
        else:
            raise ValueError(f"unknown mixer {b.kind!r}")

    def _prepare(self, cfg: DecoderConfig, rows: int, off: Dict[str, int], dtype, device, gen) -> Optional[QkvPrepare]:
        """Parameters and tables of what an attention branch does to its projections; ``None``: nothing."""
        b = self.b
        if not (b.proj_bias or b.qk_norm or b.rot_dims or b.rel_max or b.head_gate or b.pool or b.sink_weight or b.key_values):
            return None
        if b.rot_dims % 2 or b.rot_dims > b.dim or b.heads % b.kv_heads or \
                b.qk_norm not in ("", "rows", "heads", "head_weights"):
            raise ValueError("attention: rotated dimensions, head counts or query / key norm")
        pr = QkvPrepare(norm=b.qk_norm, eps=cfg.rms_norm_eps, g_off=off.get("g", -1))
        if b.proj_bias:
            self.bias = _param((rows - off["q"],), dtype, device, 0, gen)
        if b.qk_norm == "rows":
            self.q_norm = _param((b.heads * b.dim,), dtype, device, -1, gen)
            self.k_norm = _param((b.kv_heads * b.dim,), dtype, device, -1, gen)
        if b.qk_norm == "head_weights":
            self.q_norm = _param((b.dim,), dtype, device, -1, gen)
            self.k_norm = _param((b.dim,), dtype, device, -1, gen)
        if b.rot_dims:
            pr.magnitude = rotary_magnitude(b.rot_scaling)
            f = torch.tensor(rotary_frequencies(b.rot_dims, b.rot_base, b.rot_scaling), dtype=torch.float64)
            hi = f.float()
            pr.freq = torch.stack([hi, (f - hi.double()).float()], 1).to(device)
        if b.rel_max:
            if b.rel_rows < 1:
                raise ValueError("attention: the rows of the distance table are not set")
            self.rel = _param((b.rel_rows, b.heads), dtype, device, 1.0, gen)
            pr.bucket = torch.tensor(distance_buckets(b.rel_rows, b.rel_max, b.window), dtype=torch.int32).to(device)
            pr.table = torch.empty(b.heads, pr.bucket.numel(), dtype=torch.float32, device=device)
        return pr

    @property
    def recurrent(self) -> bool:
        return self.b.recurrent

    def weights(self) -> Dict[str, torch.Tensor]:
        return {k: getattr(self, k).detach() for k in ("norm", "w2", "b_e", "b_f") if hasattr(self, k)}

    def run(self, p: torch.Tensor, io: "_Batch", out: torch.Tensor, gain: Optional[torch.Tensor] = None) -> None:
        """The branch's heads of the projected rows ``p`` into its columns of ``out``; ``gain``: one number that the
        projections still have to be multiplied by (latent attention only)."""
        if self.b.kind == "latent_attention":
            w = {"c_norm": self.c_norm.detach(), "kv_up": self.kv_up_weight.detach(), "gain": gain}
            latent_attention(self.spec, p, w, io.seq_ids, io.positions, io.block_table, io.next_cache(), out,
                             self.out_off, plan=io.latent)
        elif self.b.kind == "attention":
            window_attention(self.spec, p, io.seq_ids, io.positions, io.block_table, io.next_cache(), out, self.out_off,
                             tiles=io.tiles, seq_lens=io.seq_lens, pool_table=io.pool_table,
                             prepare=self.prepare and replace(self.prepare, **{
                                 k: getattr(self, k).detach() for k in ("bias", "q_norm", "k_norm", "rel", "sink")
                                 if hasattr(self, k)}))
        elif io.plan is not None:
            recurrence_prefill(self.spec, p, self.weights(), io.next_state(), io.plan, out, self.out_off)
        else:
            recurrence_decode(self.spec, p, self.weights(), io.next_state(), io.seq_ids, io.positions, out, self.out_off)


class HybridLayer(nn.Module):
    def __init__(self, cfg: DecoderConfig, index: int, dtype, device, gen):
        super().__init__()
        lay, W, std = cfg.hybrid.layers[index], cfg.hidden_size, cfg.initializer_range
        self.cfg, self.ff = cfg, lay.ff
        in_off = out_off = 0
        branches = []
        for b in lay.branches:
            br = HybridBranch(b, cfg, in_off, out_off, dtype, device, gen)
            in_off, out_off = br.in_end, out_off + _pad8(b.heads * b.vdim)
            branches.append(br)
        self.branches = nn.ModuleList(branches)
        self.padded_out = any(b.heads * b.vdim % 8 for b in lay.branches)
        self.norm1 = _param((W,), dtype, device, -1, gen)
        self.in_proj_weight = _param((in_off, W), dtype, device, std, gen)
        self.o_proj_weight = _param((W, out_off), dtype, device, std, gen)
        with torch.no_grad():
            for br in self.branches:
                for at, n in br.cols.values():
                    self.in_proj_weight[at + n:at + _pad8(n)] = 0
                n = br.b.heads * br.b.vdim
                self.o_proj_weight[:, br.out_off + n:br.out_off + _pad8(n)] = 0
        if self.ff:
            self.ffp = _pad8(self.ff)
            self.norm2 = _param((W,), dtype, device, -1, gen)
            self.gate_up_proj_weight = _param((2 * self.ffp, W), dtype, device, std, gen)
            self.down_proj_weight = _param((W, self.ffp), dtype, device, std, gen)
            with torch.no_grad():
                self.gate_up_proj_weight[self.ff:self.ffp] = 0
                self.gate_up_proj_weight[self.ffp + self.ff:] = 0
                self.down_proj_weight[:, self.ff:] = 0

    def mix(self, x: torch.Tensor, io: "_Batch") -> torch.Tensor:
        p = ops.linear(x, self.in_proj_weight)
        alloc = torch.zeros if self.padded_out else torch.empty
        out = alloc(x.shape[0], self.o_proj_weight.shape[1], dtype=x.dtype, device=x.device)
        for br in self.branches:
            br.run(p, io, out)
        return ops.linear(out, self.o_proj_weight)

    def mlp(self, x: torch.Tensor) -> torch.Tensor:
        return ops.linear(R.gated_act(ops.linear(x, self.gate_up_proj_weight), self.cfg.hybrid.act),
                          self.down_proj_weight)


class ParallelLayer(nn.Module):
    """Mixer and feed-forward side by side on one stream (see :class:`HybridSpec`)."""

    def __init__(self, cfg: DecoderConfig, index: int, dtype, device, gen):
        super().__init__()
        hy, W, std = cfg.hybrid, cfg.hidden_size, cfg.initializer_range
        lay = hy.layers[index]
        if hy.norm != "rms_norm" or any(b.kind != "latent_attention" for b in lay.branches):
            raise ValueError("parallel layers: RMS norms of one number and latent attention")
        self.cfg, self.ff, self.ffp = cfg, lay.ff, _pad8(lay.ff)
        at = out_off = 0
        branches, used = [], []
        for b in lay.branches:
            br = HybridBranch(b, cfg, at, out_off, dtype, device, gen)
            used += list(br.cols.values())
            at, out_off = br.in_end, out_off + _pad8(b.heads * b.vdim)
            branches.append(br)
        self.branches = nn.ModuleList(branches)

        def place(n: int) -> int:
            nonlocal at
            used.append((at, n))
            at += _pad8(n)
            return at - _pad8(n)
        self.norm1 = _param((), dtype, device, -1, gen)
        self.rg1_off = place(W) if hy.residual_gate else -1
        if self.ff:
            self.norm2 = _param((), dtype, device, -1, gen)
            self.up_off = place(self.ff)
            self.rg2_off = place(W) if hy.residual_gate else -1
            self.down_proj_weight = _param((W, self.ffp), dtype, device, std, gen)
        self.in_proj_weight = _param((at, W), dtype, device, std, gen)
        self.o_proj_weight = _param((W, out_off), dtype, device, std, gen)
        if hy.residual_gate:
            self.rg1_bias = _param((W,), dtype, device, 0, gen)
            self.rg2_bias = _param((W,), dtype, device, 0, gen) if self.ff else None
        self.padded_out = any(b.heads * b.vdim % 8 for b in lay.branches)
        with torch.no_grad():
            for o, n in used:
                self.in_proj_weight[o + n:o + _pad8(n)] = 0
            if self.ff:
                self.down_proj_weight[:, self.ff:] = 0
            for br in self.branches:
                n = br.b.heads * br.b.vdim
                self.o_proj_weight[:, br.out_off + n:br.out_off + _pad8(n)] = 0

    def run(self, x: torch.Tensor, io: "_Batch") -> List[R.Sublayer]:
        """Both sublayers of rows ``x`` (the stream over its root mean square), not yet added to the stream."""
        W = self.cfg.hidden_size
        p = ops.linear(x, self.in_proj_weight)
        alloc = torch.zeros if self.padded_out else torch.empty
        heads = alloc(x.shape[0], self.o_proj_weight.shape[1], dtype=x.dtype, device=x.device)
        g1 = self.norm1.detach()
        for br in self.branches:
            br.run(p, io, heads, g1)

        def result(y, off, name, gain):
            if off < 0:
                return R.Sublayer(y)
            return R.Sublayer(y, p[:, off:off + W], getattr(self, name).detach(), gain)
        out = [result(linear_partial(heads, self.o_proj_weight.detach()), self.rg1_off, "rg1_bias", g1)]
        if self.ff:
            g2 = self.norm2.detach()
            u = R.scaled_act(p[:, self.up_off:self.up_off + self.ffp], self.cfg.hybrid.act, g2)
            out.append(result(linear_partial(u, self.down_proj_weight.detach()), self.rg2_off, "rg2_bias", g2))
        return out


class Connection(nn.Module):
    """Hyper-connection and norm of one sublayer: what it reads from the copies of the stream and how they change."""

    def __init__(self, cfg: DecoderConfig, dtype, device, gen):
        super().__init__()
        S, W = cfg.hybrid.streams, cfg.hidden_size
        self.norm = _param((W,), dtype, device, -1, gen)
        self.norm_bias = _param((W,), dtype, device, 0, gen)
        self.w_in = _param((S,), dtype, device, 0, gen)
        self.w_out = _param((S,), dtype, device, -1, gen)
        self.w_mix = _param((S, S), dtype, device, 0, gen)
        with torch.no_grad():
            self.w_in.fill_(1.0 / S)
            self.w_mix.copy_(torch.eye(S))


class RoutedFeedForward(nn.Module):
    """Router, gated experts, identity experts and an expert that takes every token (:class:`ExpertSpec`)."""

    def __init__(self, e: ExpertSpec, W: int, std: float, dtype, device, gen):
        super().__init__()
        if not 1 <= e.top <= e.outputs or e.outputs % e.groups or not 1 <= e.keep <= e.groups or e.top > e.keep * (e.outputs // e.groups):
            raise ValueError(f"{e.top} of {e.outputs} router outputs in {e.keep} of {e.groups} groups")
        self.spec, ffp, sp = e, _pad8(e.ff), _pad8(e.shared_ff)
        self.router_weight = _param((_pad8(e.outputs), W), dtype, device, std, gen)
        if e.corrected:
            self.correction = _param((e.outputs,), dtype, device, 0, gen)
        self.down_weight = _param((e.experts, W, ffp), dtype, device, std, gen)
        pads = []
        if e.gated:
            self.gate_up_weight = _param((e.experts, 2 * ffp, W), dtype, device, std, gen)
            pads.append((self.gate_up_weight, self.down_weight, e.ff, ffp))
        else:
            self.up_weight = _param((e.experts, ffp, W), dtype, device, std, gen)
            pads.append((self.up_weight, self.down_weight, e.ff, ffp))
        if e.shared_ff:
            self.shared_gate_up_weight = _param((2 * sp, W), dtype, device, std, gen)
            self.shared_down_weight = _param((W, sp), dtype, device, std, gen)
            pads.append((self.shared_gate_up_weight, self.shared_down_weight, e.shared_ff, sp))
        with torch.no_grad():
            self.router_weight[e.outputs:] = 0
            for gate_up, down, ff, pad in pads:
                gate_up[..., ff:pad, :] = 0
                if gate_up.shape[-2] > pad:
                    gate_up[..., pad + ff:, :] = 0
                down[..., ff:] = 0

    def run(self, x: torch.Tensor) -> R.SublayerSum:
        e = self.spec
        z = linear_partial(x, self.router_weight.detach(), f32=True, max_splits=12)
        w, ids, w_id = route_grouped(z, self.correction.detach() if e.corrected else None, e.experts, e.top, e.groups, e.keep,
                                     e.scale, outputs=e.outputs, renormalize=e.renormalize)
        up = (self.gate_up_weight if e.gated else self.up_weight).detach()
        ys, slots = routed_experts(x, ids, up, self.down_weight.detach(), e.act, gated=e.gated)
        out = R.SublayerSum(ys=ys, pair_slot=slots, pair_w=w)
        if e.identity:
            out.x_id, out.w_id = x, w_id
        if e.shared_ff:
            a = R.partial_act(linear_partial(x, self.shared_gate_up_weight.detach()), e.act, gated=True)
            out.y = linear_partial(a, self.shared_down_weight.detach())
        return out


class HyperLayer(nn.Module):
    """Attention and a dense or routed feed-forward around copies of the stream (see :class:`HybridSpec`)."""

    def __init__(self, cfg: DecoderConfig, index: int, dtype, device, gen):
        super().__init__()
        hy, W, std = cfg.hybrid, cfg.hidden_size, cfg.initializer_range
        lay = hy.layers[index]
        if len(lay.branches) != 1 or lay.branches[0].kind != "attention" or hy.norm != "layer_norm" or hy.streams < 1:
            raise ValueError("hyper-connected layers: one attention branch and layer norms")
        self.cfg, self.ff, self.ffp = cfg, lay.ff, _pad8(lay.ff)
        b = lay.branches[0]
        br = HybridBranch(b, cfg, 0, 0, dtype, device, gen)
        self.branches = nn.ModuleList([br])
        heads = b.heads * b.vdim
        self.in_proj_weight = _param((br.in_end, W), dtype, device, std, gen)
        self.o_proj_weight = _param((W, _pad8(heads)), dtype, device, std, gen)
        self.o_proj_bias = _param((W,), dtype, device, 0, gen) if b.proj_bias else None
        self.mixer_connection = Connection(cfg, dtype, device, gen)
        self.ff_connection = Connection(cfg, dtype, device, gen) if lay.has_ff else None
        self.moe = RoutedFeedForward(lay.moe, W, std, dtype, device, gen) if lay.moe is not None else None
        if self.ff:
            self.up_proj_weight = _param((self.ffp, W), dtype, device, std, gen)
            self.down_proj_weight = _param((W, self.ffp), dtype, device, std, gen)
        with torch.no_grad():
            for at, n in br.cols.values():
                self.in_proj_weight[at + n:at + _pad8(n)] = 0
            self.o_proj_weight[:, heads:] = 0
            if self.ff:
                self.up_proj_weight[self.ff:] = 0
                self.down_proj_weight[:, self.ff:] = 0

    def connections(self) -> List[Connection]:
        return [self.mixer_connection] + ([self.ff_connection] if self.ff_connection is not None else [])

    def sublayers(self):
        """``(connection, function of its normed rows)`` in order."""
        yield self.mixer_connection, self.mix
        if self.ff_connection is not None:
            yield self.ff_connection, self.feed_forward

    def mix(self, x: torch.Tensor, io: "_Batch") -> R.SublayerSum:
        br, = self.branches
        p = linear_partial(x, self.in_proj_weight.detach())
        alloc = torch.zeros if br.b.heads * br.b.vdim % 8 else torch.empty
        heads = alloc(x.shape[0], self.o_proj_weight.shape[1], dtype=x.dtype, device=x.device)
        br.run(p, io, heads)
        return R.SublayerSum(linear_partial(heads, self.o_proj_weight.detach()),
                             self.o_proj_bias.detach() if self.o_proj_bias is not None else None)

    def feed_forward(self, x: torch.Tensor, io: "_Batch") -> R.SublayerSum:
        if self.moe is not None:
            return self.moe.run(x)
        a = R.partial_act(linear_partial(x, self.up_proj_weight.detach()), self.cfg.hybrid.act)
        return R.SublayerSum(linear_partial(a, self.down_proj_weight.detach()))


class SandwichLayer(nn.Module):
    """One mixer and a dense or routed feed-forward, each between two norms, then the layer's own token vectors (see
    :class:`HybridSpec`)."""

    def __init__(self, cfg: DecoderConfig, index: int, dtype, device, gen):
        super().__init__()
        hy, W, std = cfg.hybrid, cfg.hidden_size, cfg.initializer_range
        lay = hy.layers[index]
        if len(lay.branches) != 1 or lay.branches[0].kind == "latent_attention" or hy.norm != "rms_norm":
            raise ValueError("layers between two norms: one branch with heads of its own and RMS norms")
        self.cfg, self.index, self.ff, self.ffp, self.has_ff = cfg, index, lay.ff, _pad8(lay.ff), lay.has_ff
        b = lay.branches[0]
        br = HybridBranch(b, cfg, 0, 0, dtype, device, gen)
        self.branches = nn.ModuleList([br])
        heads = b.heads * b.vdim
        vector = lambda: _param((W,), dtype, device, -1, gen)  # noqa: E731
        self.norm1, self.norm1b = vector(), vector()
        self.in_proj_weight = _param((br.in_end, W), dtype, device, std, gen)
        self.o_proj_weight = _param((W, _pad8(heads)), dtype, device, std, gen)
        if self.has_ff:
            self.norm2, self.norm2b = vector(), vector()
        self.moe = RoutedFeedForward(lay.moe, W, std, dtype, device, gen) if lay.moe is not None else None
        self.up_proj_bias = self.down_proj_bias = self.act_numbers = None
        if self.ff:
            self.up_proj_weight = _param((self.ffp, W), dtype, device, std, gen)
            self.down_proj_weight = _param((W, self.ffp), dtype, device, std, gen)
            if hy.ff_bias:
                self.up_proj_bias = _param((self.ffp,), dtype, device, 0, gen)
                self.down_proj_bias = _param((W,), dtype, device, 0, gen)
            if hy.act == "xielu":
                self.act_numbers = _param((2,), dtype, device, 0, gen)
        self.side = hy.token_side
        if self.side:
            sp = _pad8(self.side)
            self.side_gate_weight = _param((sp, W), dtype, device, std, gen)
            self.side_proj_weight = _param((W, sp), dtype, device, std, gen)
            self.side_norm = vector()
        with torch.no_grad():
            for at, n in br.cols.values():
                self.in_proj_weight[at + n:at + _pad8(n)] = 0
            self.o_proj_weight[:, heads:] = 0
            if self.ff:
                self.up_proj_weight[self.ff:] = 0
                self.down_proj_weight[:, self.ff:] = 0
            if self.side:
                self.side_gate_weight[self.side:] = 0
                self.side_proj_weight[:, self.side:] = 0

    def mix(self, x: torch.Tensor, io: "_Batch") -> R.SublayerSum:
        br, = self.branches
        # a recurrence reads its rows several times: they come as one tensor
        p = ops.linear(x, self.in_proj_weight) if br.recurrent else linear_partial(x, self.in_proj_weight.detach())
        alloc = torch.zeros if br.b.heads * br.b.vdim % 8 else torch.empty
        heads = alloc(x.shape[0], self.o_proj_weight.shape[1], dtype=x.dtype, device=x.device)
        br.run(p, io, heads)
        return R.SublayerSum(linear_partial(heads, self.o_proj_weight.detach()))

    def feed_forward(self, x: torch.Tensor) -> R.SublayerSum:
        if self.moe is not None:
            return self.moe.run(x)
        data = lambda t: t.detach() if t is not None else None  # noqa: E731
        a = R.bias_act(linear_partial(x, self.up_proj_weight.detach()), self.cfg.hybrid.act, x.dtype,
                       bias=data(self.up_proj_bias), numbers=data(self.act_numbers))
        return R.SublayerSum(linear_partial(a, self.down_proj_weight.detach()), data(self.down_proj_bias))

    def token_input(self, x: torch.Tensor, ids: torch.Tensor, table: torch.Tensor) -> R.SublayerSum:
        """``x``: rows of the stream itself."""
        z = linear_partial(x, self.side_gate_weight.detach(), max_splits=12)
        g = R.token_gate(z, ids, table, self.index * self.side, self.side, x.dtype)
        return R.SublayerSum(linear_partial(g, self.side_proj_weight.detach()))


class _Batch:
    """What one forward pass needs besides the rows: places in the cache, prompt portions or decode lengths."""

    def __init__(self, seq_ids, positions, block_table, cache, states, plan=None, tiles=None, latent=None, seq_lens=None,
                 pool_table=None):
        self.seq_ids, self.positions, self.block_table, self.pool_table = seq_ids, positions, block_table, pool_table
        self.plan, self.tiles, self.latent, self.seq_lens = plan, tiles, latent, seq_lens
        self._cache, self._states = iter(cache), iter(states or ())

    def next_cache(self):
        return next(self._cache)

    def next_state(self):
        return next(self._states)


class HybridLM(nn.Module):
    def __init__(self, cfg: DecoderConfig, dtype=torch.bfloat16, device="cpu", seed: int = 0,
                 gradient_checkpointing: bool = False):
        super().__init__()
        if cfg.value_head or cfg.lora_rank > 0:
            raise NotImplementedError("hybrid decoders have no value head and no adapters")
        self.cfg, self.dtype = cfg, dtype
        self.gradient_checkpointing = gradient_checkpointing
        self.vision = None
        gen = _Init(seed, device)
        std = cfg.initializer_range
        self.embed_tokens = _param((cfg.vocab_size, cfg.hidden_size), dtype, device, std, gen)
        kinds = {"sequential": HybridLayer, "parallel": ParallelLayer, "hyper": HyperLayer, "sandwich": SandwichLayer}
        self.arrangement = cfg.hybrid.arrangement
        self.parallel = self.arrangement == "parallel"
        if self.arrangement not in kinds or (cfg.hybrid.loop is not None and self.arrangement in ("sequential", "sandwich")):
            raise ValueError("layer arrangements: sequential or sandwich, or parallel or hyper with an optional loop")
        self.layers = nn.ModuleList([kinds[self.arrangement](cfg, i, dtype, device, gen) for i in range(cfg.num_layers)])
        if cfg.hybrid.loop is not None and self.parallel:
            W = cfg.hidden_size
            self.loop_in_weight = _param((W, 2 * W), dtype, device, (2 * W) ** -0.5, gen)
            self.loop_step = _param((cfg.hybrid.loop.times, W), dtype, device, std, gen)
        self.norm = _param(() if self.parallel else (cfg.hidden_size,), dtype, device, -1, gen)
        if self.arrangement == "hyper":
            self.norm_bias = _param((cfg.hidden_size,), dtype, device, 0, gen)
        if cfg.hybrid.token_side:
            self.side_embed = _param((cfg.vocab_size, cfg.num_layers * cfg.hybrid.token_side), dtype, device, std, gen)
        self.lm_head = None
        if not cfg.tie_word_embeddings:
            self.lm_head = _param((cfg.vocab_size, cfg.hidden_size), dtype, device, std, gen)

    @property
    def head_weight(self) -> torch.Tensor:
        return self.lm_head if self.lm_head is not None else self.embed_tokens

    # ---- state description for the cache manager ---------------------------------------------------
    def recurrent_branches(self) -> List[HybridBranch]:
        return [br for layer in self.layers for br in layer.branches if br.recurrent]

    def new_states(self, slots: int) -> List[Dict[str, torch.Tensor]]:
        """Recurrent states of ``slots`` sequences, one dictionary per recurrent branch."""
        return [empty_state(br.spec, slots, self.embed_tokens.device) for br in self.recurrent_branches()]

    # ---- forward -----------------------------------------------------------------------------------
    def _layers(self, ids: torch.Tensor, io: _Batch) -> torch.Tensor:
        cfg = self.cfg
        if self.parallel:
            return self._parallel_layers(ids, io)
        if self.arrangement == "hyper":
            return self._hyper_layers(ids, io)
        if self.arrangement == "sandwich":
            return self._sandwich_layers(ids, io)
        kind, eps = cfg.hybrid.norm, cfg.rms_norm_eps
        h = R.embed_scaled(ids, self.embed_tokens.detach(), cfg.hybrid.embed_scale)
        delta = None
        for layer in self.layers:
            delta = layer.mix(R.add_norm(h, delta, layer.norm1, eps, kind), io)
            if layer.ff:
                delta = layer.mlp(R.add_norm(h, delta, layer.norm2, eps, kind))
        return R.add_norm(h, delta, self.norm, eps, kind)

    def _parallel_layers(self, ids: torch.Tensor, io: _Batch) -> torch.Tensor:
        hy, eps, dtype = self.cfg.hybrid, self.cfg.rms_norm_eps, self.embed_tokens.dtype
        W, mult = self.cfg.hidden_size, hy.residual_mult
        h = R.embed_scaled(ids, self.embed_tokens.detach(), hy.embed_scale)
        if hy.loop is not None:
            # a pass begins with W_in [h; embedding]: the embedding's half is the same in every pass, and h keeps its 32
            # bits as a sum of two rows of the activation format
            w_in = self.loop_in_weight.detach()
            x0 = R.stream_update(h, [], mult, dtype, eps, split=True)[:h.shape[0]]
            base = linear_partial(x0, w_in[:, W:], f32=True)
        subs: List[R.Sublayer] = []
        for i, t in hy.runs():
            if t is None:
                x = R.stream_update(h, subs, mult, dtype, eps)
            else:
                parts = R.stream_update(h, subs, mult, dtype, eps, split=True)
                x = R.enter_pass(h, linear_partial(parts, w_in[:, :W], f32=True), base, self.loop_step.detach()[t], eps)
            subs = self.layers[i].run(x, io)
        return R.stream_update(h, subs, mult, dtype, eps, weight=self.norm.detach())

    def _hyper_layers(self, ids: torch.Tensor, io: _Batch) -> torch.Tensor:
        hy, eps, W = self.cfg.hybrid, self.cfg.rms_norm_eps, self.cfg.hidden_size
        h = torch.empty(ids.shape[0], hy.streams, W, dtype=torch.float32, device=ids.device)
        step = dict(ids=ids.to(torch.int64).contiguous(), table=self.embed_tokens.detach())
        for i, _ in hy.runs():
            for conn, fn in self.layers[i].sublayers():
                x = R.hyper_rows(h, conn.norm.detach(), conn.norm_bias.detach(), eps, w_in=conn.w_in.detach(), **step)
                step = dict(result=fn(x, io), w_out=conn.w_out.detach(), w_mix=conn.w_mix.detach())
        return R.hyper_rows(h, self.norm.detach(), self.norm_bias.detach(), eps, **step)

    def _sandwich_layers(self, ids: torch.Tensor, io: _Batch) -> torch.Tensor:
        hy, eps, W = self.cfg.hybrid, self.cfg.rms_norm_eps, self.cfg.hidden_size
        ids = ids.to(torch.int64).contiguous()
        h = torch.empty(ids.shape[0], W, dtype=torch.float32, device=ids.device)
        dtype = self.embed_tokens.dtype

        def rows(weight, step):
            return R.post_norm_rows(h, weight.detach() if weight is not None else None, eps, dtype, **step)
        step = dict(ids=ids, table=self.embed_tokens.detach(), scale=hy.embed_scale)
        for layer in self.layers:
            step = dict(result=layer.mix(rows(layer.norm1, step), io), post=layer.norm1b.detach())
            if layer.has_ff:
                step = dict(result=layer.feed_forward(rows(layer.norm2, step)), post=layer.norm2b.detach())
            if layer.side:
                step = dict(result=layer.token_input(rows(None, step), ids, self.side_embed.detach()),
                            post=layer.side_norm.detach())
        return rows(self.norm, step)

    @torch.no_grad()
    def forward_cached(self, input_ids: torch.Tensor, positions: torch.Tensor, cache: Sequence[torch.Tensor],
                       block_table: torch.Tensor, seq_ids: torch.Tensor, *, states=None,
                       prefill_info: Optional[SeqInfo] = None, seq_lens: Optional[torch.Tensor] = None,
                       rope_positions=None, prefix_lens=None, prefill_slots=None, pool_table=None) -> torch.Tensor:
        """Final-norm hidden states of new tokens (see :meth:`DecoderLM.forward_cached`).  ``states``: one dictionary
        per recurrent branch, indexed by slot; ``prefill_slots[i]`` / ``prefix_lens[i]``: the slot of portion ``i`` and
        the tokens it holds already; ``pool_table``: like ``block_table``, the blocks that hold pooled keys and values."""
        pos = positions.to(torch.int32).contiguous()
        seq = seq_ids.to(torch.int32).contiguous()
        if prefill_info is None:
            return self._layers(input_ids, _Batch(seq, pos, block_table, cache, states, seq_lens=seq_lens,
                                                  pool_table=pool_table))
        lens = prefill_info.seqlens
        starts = list(prefix_lens) if prefix_lens is not None else [0] * len(lens)
        dev = input_ids.device
        kinds = {b.kind for layer in self.cfg.hybrid.layers for b in layer.branches}
        recurrent = kinds - {"attention", "latent_attention"}
        io = _Batch(seq, pos, block_table, cache, states, pool_table=pool_table,
                    plan=PortionPlan(lens, starts, prefill_slots, dev) if recurrent else None,
                    tiles=QueryTiles(lens, starts, prefill_slots, dev) if "attention" in kinds else None,
                    latent=LatentPlan(lens, starts, prefill_slots, dev) if "latent_attention" in kinds else None)
        return self._layers(input_ids, io)

    @torch.no_grad()
    def _score_hidden(self, input_ids: torch.Tensor, info: SeqInfo) -> torch.Tensor:
        """Packed whole sequences through the prompt path: one scratch arena serves every attention layer (each layer
        writes before it reads), the recurrent states are dropped."""
        cfg, dev = self.cfg, input_ids.device
        pools, at = cfg.hybrid.pools(), 0

        def place(counts):
            nonlocal at
            table = torch.full((max(len(counts), 1), max(max(counts, default=1), 1)), -1, dtype=torch.int32)
            for i, n in enumerate(counts):
                table[i, :n] = torch.arange(at, at + n, dtype=torch.int32)
                at += n
            return table.to(dev)
        nb = [(n + kvc.BLOCK - 1) // kvc.BLOCK for n in info.seqlens]
        table = place(nb)
        pool_table = place([kvc.pool_blocks(n, pools[0]) for n in info.seqlens]) if pools else None
        paged = cfg.paged_layers()
        elems = [g * kvc.BLOCK * (dk + dv) for g, dk, dv in paged]
        arena = torch.zeros(at * max(elems, default=0), dtype=self.embed_tokens.dtype, device=dev)
        cache = [arena[:at * e].view(at, e) for e in elems]
        seq_ids = torch.repeat_interleave(torch.arange(len(nb), dtype=torch.int32), torch.tensor(info.seqlens)).to(dev)
        return self.forward_cached(input_ids, info.positions, cache, table, seq_ids,
                                   states=self.new_states(len(nb)), prefill_info=info,
                                   prefill_slots=list(range(len(nb))), pool_table=pool_table)

    def forward_hidden(self, input_ids: torch.Tensor, positions: torch.Tensor, info: SeqInfo, **mm) -> torch.Tensor:
        if torch.is_grad_enabled() and self.head_weight.requires_grad:
            raise NotImplementedError("hybrid decoders are served and scored; they have no backward pass")
        if any(v is not None for v in mm.values()):
            raise ValueError("hybrid decoders take token ids only")
        return self._score_hidden(input_ids, info)

    def token_logprobs(self, hidden: torch.Tensor, labels: torch.Tensor, temperature: float = 1.0,
                       with_entropy: bool = True):
        """``log p(label)`` and entropy of the capped, tempered distribution, a bounded block of rows at a time."""
        from ..ops import lib as _lib
        T, V = hidden.shape[0], self.cfg.vocab_size
        labels = labels.to(torch.int64).contiguous()
        logp = torch.empty(T, dtype=torch.float32, device=hidden.device)
        ent = torch.empty_like(logp)
        step = max(128, (1 << 28) // V // 128 * 128)
        for s in range(0, T, step):
            e = min(T, s + step)
            z = self.logits_of(hidden[s:e])
            if z.is_cuda:
                if V % 4:       # the statistics kernel reads vectors of four: columns without weight
                    z = torch.nn.functional.pad(z, (0, -V % 4), value=-1e30)
                ws = torch.empty_like(logp[s:e])
                _lib.check(_lib.get_lib().sb_lmhead_stats(
                    _lib.ptr(z), ctypes.c_longlong(z.shape[1]), _lib.ptr(labels[s:e]), ctypes.c_float(1.0 / temperature),
                    _lib.ptr(logp[s:e]), _lib.ptr(ent[s:e]), _lib.ptr(ws), e - s, z.shape[1], _lib.stream()), "sb_lmhead_stats")
            else:
                lp = torch.log_softmax(z / temperature, -1)
                logp[s:e] = lp.gather(1, labels[s:e, None])[:, 0]
                ent[s:e] = -(lp.exp() * lp).sum(-1)
        return logp, (ent if with_entropy else None)

    def logits_of(self, hidden: torch.Tensor) -> torch.Tensor:
        """Capped fp32 logits of final-norm hidden states."""
        return lm_head_logits(hidden, self.head_weight.detach(), self.cfg.logit_softcap)

    def logprobs(self, input_ids, positions, info: SeqInfo, labels, temperature: float = 1.0,
                 with_entropy: bool = True, **mm):
        return self.token_logprobs(self.forward_hidden(input_ids, positions, info, **mm), labels, temperature,
                                   with_entropy)

    def logits(self, input_ids, positions, info: SeqInfo, **mm) -> torch.Tensor:
        return self.logits_of(self.forward_hidden(input_ids, positions, info, **mm))

    def named_flat_order(self):
        return list(self.named_parameters())
