"""Mechanisms of the Rizitar decoder one by one against the plain statements of ``rizitar_oracle``: windowed attention with pooled
runs, learned sinks, weighted heads and scaled rotation; the generalized delta rule; plain routed experts; xIELU; token vectors;
norms around sublayers.  The same cases run on the framework's CPU path, its 32-bit and its bf16 CUDA kernels."""
import math

import pytest
import rizitar_oracle as O
import torch

from siirl_b200.ops import rows as R
from siirl_b200.ops.moe import route_grouped, routed_experts
from siirl_b200.ops.recurrence import PortionPlan, RecurrenceSpec, empty_state, recurrence_decode, recurrence_prefill
from siirl_b200.ops.window_attention import (QkvPrepare, QueryTiles, WindowSpec, rotary_frequencies, rotary_magnitude,
                                             window_attention)

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]
EPS = 1e-4


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def close(got, want, dtype, what="", f32=2e-5, bf16=1.5e-2):
    got, want = got.detach().double().cpu(), want.double()
    err = (got - want).abs().max().item()
    lim = (f32 if dtype == torch.float32 else bf16) * max(want.abs().max().item(), 1e-6)
    assert err <= lim, f"{what}: {err:.3e} > {lim:.3e}"


def finish(device):
    if device == "cuda":
        from siirl_b200.ops import lib
        torch.cuda.synchronize()
        lib.check_status()


def rounded(t):
    return t.bfloat16().double()


# ---- positions --------------------------------------------------------------------------------------------------------------
def test_scaled_frequencies():
    full = dict(factor=6.0, fast=16.0, original=500, slow=0.5)
    cases = [dict(dims=64, base=1e6, scaling=full), dict(dims=20, base=2e4, scaling=dict(full, slow=16.0)),
             dict(dims=2, base=10.0, scaling=full), dict(dims=32, base=1e4, scaling=dict(full, fast=1e4, slow=1e-9)),
             dict(dims=16, base=100.0, scaling=dict(full, factor=1.0)), dict(dims=24, base=5e4)]
    for rot in cases:
        want, mag = O.frequencies(rot)
        assert rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling")) == pytest.approx(want, rel=1e-12)
        assert rotary_magnitude(rot.get("scaling")) == pytest.approx(mag, rel=1e-12)
    ratio = [a / b for a, b in zip(O.frequencies(cases[0])[0], O.frequencies(dict(cases[0], scaling=None))[0])]
    # all three bands are there
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 6) and any(0.17 < r < 0.99 for r in ratio)
    assert rotary_magnitude(full) == pytest.approx(1 + 0.1 * math.log(6.0))


# ---- attention --------------------------------------------------------------------------------------------------------------
YARN = dict(factor=4.0, fast=8.0, original=100, slow=1.0)
ATT = {
    # (heads, kv_heads, dim), window, pool, then the rotation
    "plain": dict(size=(6, 2, 32), window=37, pool=5, rot=dict(dims=16, base=5e3, scaling=YARN)),
    "wide": dict(size=(4, 1, 128), window=70, pool=16, rot=dict(dims=32, base=1e5, scaling=YARN)),
    "whole_head": dict(size=(8, 8, 64), window=20, pool=8, rot=dict(dims=64, base=1e6)),
    "middle": dict(size=(3, 3, 80), window=33, pool=7, rot=dict(dims=80, base=3e4, scaling=YARN)),
    "page": dict(size=(4, 2, 64), window=64, pool=64, rot=dict(dims=16, base=1e4)),
    "pool_over_window": dict(size=(4, 2, 40), window=10, pool=70, rot=dict(dims=8, base=1e4)),
    "one": dict(size=(2, 2, 32), window=1, pool=1, rot=dict(dims=32, base=1e4)),
    "pairs": dict(size=(5, 1, 48), window=3, pool=2, rot=dict(dims=16, base=1e4)),
    "no_pool": dict(size=(4, 2, 24), window=50, pool=0, rot=dict(dims=8, base=1e4)),
    "open": dict(size=(4, 1, 32), window=0, pool=0, rot=dict(dims=16, base=1e4)),
    "no_rotation": dict(size=(4, 2, 32), window=21, pool=4, rot=None),
    "many_heads": dict(size=(40, 2, 64), window=60, pool=9, rot=dict(dims=32, base=1e4)),
    "group_of_24": dict(size=(24, 1, 32), window=30, pool=6, rot=dict(dims=32, base=1e4)),
    "very_wide": dict(size=(2, 1, 192), window=45, pool=12, rot=dict(dims=64, base=1e4)),
    "odd": dict(size=(3, 1, 21), window=29, pool=10, rot=dict(dims=6, base=1e3)),
    "odd_pairs": dict(size=(2, 2, 18), window=17, pool=3, rot=dict(dims=18, base=1e3)),
    "single": dict(size=(1, 1, 8), window=9, pool=4, rot=dict(dims=2, base=10.0)),
}


class Case:
    """Raw projections whose queries single out one token or one pooled run at the edges of what they see and just beyond, the
    oracle's answer and the framework's description of the branch."""

    def __init__(self, name, T, seed=0, sink=None):
        c = self.c = ATT[name]
        H, G, d = c["size"]
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.scale, self.T = 16.0 / d, T
        w, P = c["window"], c["pool"]
        # tokens of a run resemble each other, so that a query can single their mean out
        run = max(P, 1)
        k = (0.8 * rnd(T // run + 1, G, d).repeat_interleave(run, 0)[:T] + 0.6 * rnd(T, G, d)).double()
        self.k = rounded(k.reshape(T, -1))
        self.wq, self.wk = rounded(1 + 0.3 * rnd(d)), rounded(1 + 0.3 * rnd(d))
        self.sink = rounded(rnd(H) + 2.0) if sink is None else rounded(torch.full((H,), float(sink)))
        pos = torch.arange(T)
        kr = self.turned(O.rms(self.k.view(T, G, d), EPS) * self.wk, pos)
        runs = O.pooled(kr, P) if P else None
        q = rnd(T, H, d).double()
        for i in range(T):
            spots = [i - w + 1, i - w, 0, i, i // 64 * 64, i - 1, i // 2]
            n = (i - w + 1) // P if P and i - w + 1 > 0 else 0
            blocks = [n - 1, n, 0, n // 2, n + 1] if P else []
            pick = i % (len(spots) + len(blocks))
            target = None
            if pick < len(spots):
                target = kr[spots[pick]] if 0 <= spots[pick] <= i else None
            else:
                b = blocks[pick - len(spots)]
                target = runs[b] if 0 <= b < (i + 1) // P else None
            if target is not None:      # what gives, weighted and turned at i, the target's direction
                t = target.repeat_interleave(H // G, 0)[None]
                q[i] = self.turned(t, -torch.tensor([i]))[0] / self.wq
        self.q = rounded(q.reshape(T, -1))
        up = lambda n: (n + 7) // 8 * 8  # noqa: E731
        self.offs = [8, 8 + up(H * d)]
        self.width = self.offs[1] + up(G * d) + 8

    def turned(self, x, pos):
        return O.rotate(x, pos, self.c["rot"]) if self.c["rot"] else x

    def want(self, first=0):
        """The oracle's heads of rows ``first ..``."""
        H, G, d = self.c["size"]
        pos = torch.arange(self.T)
        v = self.k.view(self.T, G, d)
        q = self.turned(O.rms(self.q.view(self.T, H, d), EPS) * self.wq, pos)
        k = self.turned(O.rms(v, EPS) * self.wk, pos)
        return O.attend(q, k, v, self.sink, self.scale, self.c["window"], self.c["pool"]).reshape(self.T, -1)[first:]

    def branch(self, dtype, device):
        H, G, d = self.c["size"]
        to = lambda t: t.to(dtype).to(device)  # noqa: E731
        spec = WindowSpec(H, G, d, d, self.offs[0], self.offs[1], self.offs[1], self.scale, self.c["window"],
                          pool=self.c["pool"])
        pr = QkvPrepare(norm="head_weights", eps=EPS, q_norm=to(self.wq), k_norm=to(self.wk), sink=to(self.sink))
        if self.c["rot"]:
            r = self.c["rot"]
            f = torch.tensor(rotary_frequencies(r["dims"], r["base"], r.get("scaling")), dtype=torch.float64)
            pr.freq = torch.stack([f.float(), (f - f.float().double()).float()], 1).to(device)
            pr.magnitude = rotary_magnitude(r.get("scaling"))
        x = torch.full((self.T, self.width), 7.0, dtype=torch.float64)
        for off, t in zip(self.offs, (self.q, self.k)):
            x[:, off:off + t.shape[1]] = t
        return spec, pr, x.to(dtype).to(device)


class Pages:
    def __init__(self, spec, slots, max_len, dtype, device, seed=3):
        g = torch.Generator().manual_seed(seed)
        nb, npool = (max_len + 63) // 64, (max_len // spec.pool + 63) // 64 if spec.pool else 0
        total = slots * (nb + npool)
        order = torch.randperm(total + 3, generator=g)[:total].to(torch.int32)
        self.table = order[:slots * nb].view(slots, nb).contiguous().to(device)
        self.pool_table = order[slots * nb:].view(slots, npool).contiguous().to(device) if npool else None
        # blocks hold what earlier sequences left: finite values that must not matter
        self.cache = (torch.randn(total + 3, spec.block_elems, generator=g) * 30).to(dtype).to(device)


def prompts(spec, pr, xs, pages, slots, starts, simt=False):
    """Portions ``xs[i]`` from position ``starts[i]`` of slot ``slots[i]``, one batch."""
    dev, lens = xs[0].device, [x.shape[0] for x in xs]
    pos = torch.cat([torch.arange(s, s + n, dtype=torch.int32) for s, n in zip(starts, lens)]).to(dev)
    ids = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, n in zip(slots, lens)]).to(dev)
    x = torch.cat(xs)
    out = torch.full((x.shape[0], 16 + (spec.heads * spec.vdim + 7) // 8 * 8), 9.0, dtype=x.dtype, device=dev)
    window_attention(spec, x, ids, pos, pages.table, pages.cache, out, 16, tiles=QueryTiles(lens, starts, slots, dev),
                     simt=simt, prepare=pr, pool_table=pages.pool_table)
    assert (out[:, :16] == 9).all()
    return out[:, 16:16 + spec.heads * spec.vdim].split(lens)


def single(spec, pr, x, pages, slot, at, slabs=1):
    """One decode row in a batch with idle slots; ``slabs``: the projection as partial sums."""
    S, dev = pages.table.shape[0], x.device
    rows = torch.zeros(S, x.shape[1], dtype=x.dtype, device=dev)
    rows[slot] = x[at]
    if slabs > 1:
        parts = torch.randn(slabs, *rows.shape, device=dev)
        parts[0] = rows.float() - parts[1:].sum(0)
        rows = parts
    ids = torch.full((S,), -1, dtype=torch.int32, device=dev)
    pos, lens = torch.zeros(S, dtype=torch.int32, device=dev), torch.zeros(S, dtype=torch.int32, device=dev)
    ids[slot], pos[slot], lens[slot] = slot, at, at + 1
    o = torch.full((S, 16 + (spec.heads * spec.vdim + 7) // 8 * 8), 5.0, dtype=x.dtype, device=dev)
    window_attention(spec, rows, ids, pos, pages.table, pages.cache, o, 16, seq_lens=lens, prepare=pr,
                     pool_table=pages.pool_table)
    o = o[:, 16:16 + spec.heads * spec.vdim]
    assert o[[s for s in range(S) if s != slot]].abs().max().item() == 0
    return o[slot]


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(ATT))
def test_attention_of_prompts_portions_and_single_tokens(name, device, dtype):
    T = 203
    case = Case(name, T)
    want = case.want()
    spec, pr, x = case.branch(dtype, device)
    for cuts in ([T], [2, 62, 64, 1, 66, 8], [128, 75], [2] * 30 + [143]):
        pages, at, got = Pages(spec, 3, 256, dtype, device), 0, []
        for n in cuts:
            got += prompts(spec, pr, [x[at:at + n]], pages, [1], [at])
            at += n
        finish(device)
        close(torch.cat(got), want, dtype, f"portions {cuts[:6]}", f32=5e-5)
    pages = Pages(spec, 3, 256, dtype, device)
    got = [prompts(spec, pr, [x[:37]], pages, [2], [0])[0]]
    got += [single(spec, pr, x, pages, 2, at, slabs=1 + at % 3)[None] for at in range(37, T)]
    finish(device)
    close(torch.cat(got), want, dtype, "single tokens", f32=1e-4)


def test_edges_of_windows_and_runs_show():
    """The cases above tell a window or a run that is one token off: the oracle's own answers differ visibly."""
    for name, c in ATT.items():
        if name == "one":       # runs of one token are the tokens themselves: every window is the same
            continue
        case = Case(name, 203)
        want, was = case.want(), (c["window"], c["pool"])
        for window, pool in ((was[0] + 1, was[1]), (was[0] - 1, was[1]), (was[0], 0), (was[0], was[1] + 1)):
            if was[0] == 0 or window < 1 or (pool, window) == (was[1], was[0]) or (was[1] == 0 and pool):
                continue
            c["window"], c["pool"] = window, pool
            try:
                assert (case.want() - want).abs().max() > 0.1 * want.abs().max(), (name, window, pool)
            finally:
                c["window"], c["pool"] = was
        sink, case.sink = case.sink, case.sink + 1.0
        assert (case.want() - want).abs().max() > 0.03 * want.abs().max()
        case.sink = sink


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["plain", "wide", "pool_over_window", "odd"])
def test_attention_of_unequal_sequences_in_one_batch(name, device, dtype):
    lens, starts, slots = [1, 130, 64, 7], [0, 65, 2, 70], [3, 2, 1, 0]
    cases = [Case(name, s + n, seed=i) for i, (n, s) in enumerate(zip(lens, starts))]
    spec, pr, _ = cases[0].branch(dtype, device)
    pages = Pages(spec, 4, 256, dtype, device)
    # the branch's weights are the first case's: the others only lend their rows
    for c in cases[1:]:
        c.wq, c.wk, c.sink = (getattr(cases[0], k) for k in ("wq", "wk", "sink"))
    xs = [c.branch(dtype, device)[2] for c in cases]
    for x, s, slot in zip(xs, starts, slots):
        if s:
            prompts(spec, pr, [x[:s]], pages, [slot], [0])
    got = prompts(spec, pr, [x[s:] for x, s in zip(xs, starts)], pages, slots, starts)
    finish(device)
    for o, c, s in zip(got, cases, starts):
        close(o, c.want()[s:], dtype, f32=5e-5)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 25.0])
def test_small_and_large_sinks(sink, device, dtype):
    """A sink that takes nothing and one that takes nearly everything."""
    case = Case("plain", 150, sink=sink)
    spec, pr, x = case.branch(dtype, device)
    pages = Pages(spec, 2, 192, dtype, device)
    got = [prompts(spec, pr, [x[:140]], pages, [0], [0])[0]]
    got += [single(spec, pr, x, pages, 0, at)[None] for at in range(140, 150)]
    finish(device)
    close(torch.cat(got), case.want(), dtype, f32=5e-5)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_a_long_context_in_several_work_items(device, dtype):
    """More than 1024 visible entries: decoding cuts them into chunks and joins them, the sink once; several blocks of pooled
    entries, and runs that lie across page borders."""
    T = 2300 if device == "cuda" else 300
    for extra in (dict(size=(4, 2, 64), window=300, pool=3, rot=dict(dims=32, base=1e5, scaling=YARN)),
                  dict(size=(12, 1, 32), window=1100, pool=7, rot=dict(dims=32, base=1e5))):
        ATT["long"] = extra
        case = Case("long", T)
        first = T - 9
        spec, pr, x = case.branch(dtype, device)
        pages = Pages(spec, 2, T + 64, dtype, device)
        prompts(spec, pr, [x[:first]], pages, [0], [0])
        got = torch.stack([single(spec, pr, x, pages, 0, at) for at in range(first, T)])
        again = prompts(spec, pr, [x], Pages(spec, 2, T + 64, dtype, device), [1], [0])[0]
        finish(device)
        close(got, case.want(first), dtype, "single tokens", f32=1e-4)
        close(again, case.want(), dtype, "prompt", f32=1e-4)
    del ATT["long"]


@pytest.mark.parametrize("device,dtype", WHERE)
def test_attention_is_the_same_wherever_blocks_lie(device, dtype):
    """Other slots and other blocks, and the general kernel beside the tensor-core one."""
    for name in ("plain", "wide", "no_rotation"):
        case = Case(name, 150)
        spec, pr, x = case.branch(dtype, device)
        a = prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device, seed=1), [0], [0])[0]
        b = prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device, seed=2), [2], [0])[0]
        assert torch.equal(a, b)
        close(prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device), [1], [0], simt=True)[0], a.double().cpu(), dtype)
    finish(device)


def test_pooled_runs_need_a_window_and_blocks():
    case = Case("plain", 8)
    spec, pr, x = case.branch(torch.float32, "cpu")
    pages = Pages(spec, 1, 64, torch.float32, "cpu")
    out = torch.zeros(8, 16 + spec.heads * spec.vdim)
    args = (x, torch.zeros(8, dtype=torch.int32), torch.arange(8, dtype=torch.int32), pages.table, pages.cache, out, 16)
    from dataclasses import replace
    for kw in (dict(prepare=pr), dict(pool_table=pages.pool_table)):
        with pytest.raises(ValueError):
            window_attention(spec, *args, **kw)
    for bad in (dict(window=0), dict(softcap=9.0), dict(keep_first=2), dict(bias_exp=8.0)):
        with pytest.raises(ValueError):
            window_attention(replace(spec, **bad), *args, prepare=pr, pool_table=pages.pool_table)


# ---- generalized delta rule -------------------------------------------------------------------------------------------------
DELTA = {  # heads, dim, rank
    "small": (3, 16, 8), "narrow": (2, 8, 3), "middle": (2, 24, 16), "three": (1, 48, 5), "usual": (4, 64, 64),
    "uneven": (2, 40, 33), "wide": (1, 96, 24), "widest": (2, 128, 130), "rank_one": (1, 32, 1),
    "beyond": (1, 144, 16), "odd": (2, 13, 7), "one": (1, 1, 1), "quad": (2, 20, 10),
}


class Delta:
    """Projected rows of one branch.  ``kind``: "random"; "same_key" (one key over and over: the removal does the work);
    "keep" (slow decay, no removal), "drop" (fast decay, full removal)."""

    def __init__(self, name, T, kind="random", seed=0):
        H, d, rank = self.size = DELTA[name]
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.T = T
        k = rnd(T, H * d) * (0.3 + rnd(T, 1).abs())
        if kind == "same_key":
            k = k[:1] * torch.where(rnd(T, 1) > 0, 1.0, -1.0) + 0.05 * rnd(T, H * d)
        self.r, self.k, self.v, self.g = (rounded(t) for t in (rnd(T, H * d), k, rnd(T, H * d), 2 * rnd(T, H * d)))
        self.a, self.e = rounded(rnd(T, H * d)), rounded(2 * rnd(T, rank))
        shift = {"random": (0.0, 0.0), "same_key": (3.0, -2.0), "keep": (-9.0, -9.0), "drop": (9.0, 9.0)}[kind]
        self.ab, self.w0 = rounded(rnd(H * d) + shift[0]), rounded(rnd(H * d) + shift[1])
        self.w2, self.norm = rounded(rnd(H * d, rank) * rank ** -0.5), rounded(1 + 0.3 * rnd(H * d))
        up = lambda n: (n + 7) // 8 * 8  # noqa: E731
        self.offs, at = [], 8
        for n in [H * d] * 5 + [rank]:
            self.offs.append(at)
            at += up(n)
        self.width = at

    def want(self):
        H, d, _ = self.size
        w = {"w1": torch.eye(self.e.shape[1]).double(), "w2": self.w2, "w0": self.w0,
             "a": torch.zeros(1, 1).double(), "a.b": self.ab}
        decay, _ = O.delta_gates(self.e, dict(w, a=torch.zeros(H * d, self.e.shape[1]).double()))
        split = lambda x: x.reshape(self.T, H, d)  # noqa: E731
        o, S = O.delta_scan(split(self.r), split(self.k), split(self.v), split(decay), split(O.sigmoid(self.a + self.ab)))
        return O.rms(o, EPS).reshape(self.T, H * d) * self.norm * O.sigmoid(self.g), S.transpose(1, 2)

    def branch(self, dtype, device):
        H, d, rank = self.size
        r, k, v, g, a, e = self.offs
        spec = RecurrenceSpec("delta", heads=H, dim=d, vdim=d, q_off=r, k_off=k, v_off=v, g_off=g, e_off=e, f_off=a, rank=rank,
                              eps=EPS, gate_act="sigmoid", norm_per_head=True)
        to = lambda t: t.to(dtype).to(device)  # noqa: E731
        w = {"norm": to(self.norm), "w2": to(self.w2), "b_e": to(self.w0), "b_f": to(self.ab)}
        x = torch.full((self.T, self.width), 3.0, dtype=torch.float64)
        for off, t in zip(self.offs, (self.r, self.k, self.v, self.g, self.a, self.e)):
            x[:, off:off + t.shape[1]] = t
        return spec, w, to(x)


def dirty(spec, slots, device):
    state = empty_state(spec, slots, device)
    state["S"].fill_(11.0)      # what an earlier sequence left
    return state


def scan(spec, w, xs, state, slots, starts, stepwise=False, segments=None):
    dev, lens = xs[0].device, [x.shape[0] for x in xs]
    x = torch.cat(xs)
    out = torch.full((x.shape[0], 16 + (spec.heads * spec.vdim + 7) // 8 * 8), 9.0, dtype=x.dtype, device=dev)
    recurrence_prefill(spec, x, w, state, PortionPlan(lens, starts, slots, dev), out, 16, stepwise=stepwise,
                       segments=segments)
    assert (out[:, :16] == 9).all()
    return out[:, 16:16 + spec.heads * spec.vdim].split(lens)


def one_token(spec, w, x, state, slot, at):
    S, dev = state["S"].shape[0], x.device
    rows = torch.zeros(S, x.shape[1], dtype=x.dtype, device=dev)
    rows[slot] = x[at]
    ids, pos = torch.full((S,), -1, dtype=torch.int32, device=dev), torch.zeros(S, dtype=torch.int32, device=dev)
    ids[slot], pos[slot] = slot, at
    out = torch.full((S, 16 + (spec.heads * spec.vdim + 7) // 8 * 8), 5.0, dtype=x.dtype, device=dev)
    recurrence_decode(spec, rows, w, state, ids, pos, out, 16)
    o = out[:, 16:16 + spec.heads * spec.vdim]
    assert o[[s for s in range(S) if s != slot]].abs().max().item() == 0
    return o[slot]


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(DELTA))
def test_delta_rule_in_prompts_portions_and_single_tokens(name, device, dtype):
    T = 83
    case = Delta(name, T)
    want, last = case.want()
    spec, w, x = case.branch(dtype, device)
    for cuts in ([T], [2] * 10 + [63], [16, 32, 1, 34], [17, 15, 3, 48]):
        state, at, got = dirty(spec, 3, device), 0, []
        for n in cuts:
            got += scan(spec, w, [x[at:at + n]], state, [2], [at])
            at += n
        finish(device)
        close(torch.cat(got), want, dtype, f"portions {cuts[:4]}", f32=2e-4)
        close(state["S"][2], last, dtype, f"state after portions {cuts[:4]}", f32=1e-4, bf16=1e-3)
        assert (state["S"][:2] == 11).all()
    state = dirty(spec, 3, device)
    got = [one_token(spec, w, x, state, 1, at)[None] for at in range(40)]
    got += scan(spec, w, [x[40:60]], state, [1], [40])
    got += [one_token(spec, w, x, state, 1, at)[None] for at in range(60, T)]
    finish(device)
    close(torch.cat(got), want, dtype, "single tokens", f32=2e-4)
    close(state["S"][1], last, dtype, "state after single tokens", f32=1e-4, bf16=1e-3)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("kind", ["same_key", "keep", "drop"])
@pytest.mark.parametrize("name", ["usual", "middle", "widest"])
def test_delta_rule_with_extreme_gates(name, kind, device, dtype):
    T = 150
    case = Delta(name, T, kind)
    want, last = case.want()
    spec, w, x = case.branch(dtype, device)
    for stepwise in (False, True):
        state = dirty(spec, 1, device)
        got, = scan(spec, w, [x], state, [0], [0], stepwise=stepwise)
        finish(device)
        close(got, want, dtype, kind, f32=5e-4, bf16=2e-2)
        close(state["S"][0], last, dtype, kind + " state", f32=2e-4, bf16=2e-3)


def test_what_the_delta_rule_removes_shows():
    """Without the removal, or with the removal read from the decayed state, the answers above are far off."""
    for name in ("small", "usual"):
        case = Delta(name, 60, "same_key")
        want, _ = case.want()
        case.ab = case.ab - 20
        assert (case.want()[0] - want).abs().max() > 0.2 * want.abs().max()


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["usual", "odd"])
def test_delta_rule_of_unequal_sequences_in_one_batch(name, device, dtype):
    lens, starts, slots = [1, 130, 16, 33, 5], [0, 20, 3, 0, 16], [4, 2, 1, 3, 0]
    cases = [Delta(name, s + n, seed=i) for i, (n, s) in enumerate(zip(lens, starts))]
    spec, w, _ = cases[0].branch(dtype, device)
    for c in cases[1:]:
        c.w2, c.w0, c.ab, c.norm = (getattr(cases[0], k) for k in ("w2", "w0", "ab", "norm"))
    xs = [c.branch(dtype, device)[2] for c in cases]
    state = dirty(spec, 6, device)
    for x, s, slot in zip(xs, starts, slots):
        if s:
            scan(spec, w, [x[:s]], state, [slot], [0])
    got = scan(spec, w, [x[s:] for x, s in zip(xs, starts)], state, slots, starts)
    finish(device)
    for o, c, s, slot in zip(got, cases, starts, slots):
        want, last = c.want()
        close(o, want[s:], dtype, f32=2e-4)
        close(state["S"][slot], last, dtype, f32=1e-4, bf16=1e-3)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["small", "narrow", "middle", "uneven", "usual", "wide", "widest"])
def test_segments_of_the_delta_rule_that_run_in_parallel(name, device, dtype):
    """Long portions cut into segments, beside one of a single segment; from zero and from a state."""
    lens, starts, slots = [470, 3, 200], [30, 0, 0], [2, 0, 1]
    cases = [Delta(name, s + n, "same_key" if i else "keep", seed=i) for i, (n, s) in enumerate(zip(lens, starts))]
    spec, w, _ = cases[0].branch(dtype, device)
    for c in cases[1:]:
        c.w2, c.w0, c.ab, c.norm = (getattr(cases[0], k) for k in ("w2", "w0", "ab", "norm"))
    xs = [c.branch(dtype, device)[2] for c in cases]
    for segments in (4, 9, 40):
        state = dirty(spec, 4, device)
        scan(spec, w, [xs[0][:30]], state, [2], [0])
        got = scan(spec, w, [x[s:] for x, s in zip(xs, starts)], state, slots, starts, segments=segments)
        finish(device)
        for o, c, s, slot in zip(got, cases, starts, slots):
            want, last = c.want()
            close(o, want[s:], dtype, f"{segments}", f32=2e-3, bf16=2e-2)
            close(state["S"][slot], last, dtype, f"{segments} state", f32=2e-4, bf16=2e-3)
        assert (state["S"][3] == 11).all()


@pytest.mark.parametrize("device,dtype", WHERE)
def test_a_long_delta_rule_keeps_its_state_in_32_bits(device, dtype):
    """A value written at the start is read at the end, past many weak writes."""
    T = 1500 if device == "cuda" else 300
    case = Delta("middle", T, "keep")
    case.k[1:] *= 0.02
    case.k = rounded(case.k)
    want, last = case.want()
    spec, w, x = case.branch(dtype, device)
    state = dirty(spec, 2, device)
    got = [scan(spec, w, [x[:T - 40]], state, [0], [0])[0]]
    got += [one_token(spec, w, x, state, 0, at)[None] for at in range(T - 40, T)]
    finish(device)
    close(torch.cat(got), want, dtype, f32=1e-3, bf16=2e-2)
    close(state["S"][0], last, dtype, "state", f32=1e-4, bf16=1e-3)


# ---- experts ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("E,top", [(7, 3), (1, 1), (64, 8), (200, 6), (300, 32)])
def test_router_without_correction(E, top, device, dtype):
    """Weights are the scores as they are, not over their sum."""
    T, g = 50, torch.Generator().manual_seed(E)
    z = torch.randn(T, E, generator=g) * 2
    parts = torch.full((3, T, E + 3), 50.0)
    parts[1:, :, :E] = torch.randn(2, T, E, generator=g)
    parts[0, :, :E] = z - parts[1:, :, :E].sum(0)
    w, ids, w_id = route_grouped(parts.to(device), None, E, top, 1, 1, 1.0, outputs=E, renormalize=False)
    finish(device)
    want_w, want_ids = O.route(parts.double().sum(0)[:, :E], top)
    assert torch.equal(ids.cpu().sort(-1).values.long(), want_ids.sort(-1).values)
    order, want_order = ids.cpu().long().argsort(-1), want_ids.argsort(-1)
    close(w.cpu().gather(1, order), want_w.gather(1, want_order), torch.float32, f32=1e-5)
    assert w_id.abs().max().item() == 0
    if E > 1 and top < E:
        assert (want_w.sum(-1) < 0.95).any()


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,W,I", [(1, 64, 24), (5, 72, 40), (300, 128, 64), (97, 51, 13), (33, 40, 20),
                                   (1050, 72, 16)])
def test_plain_experts_and_their_normed_sum(T, W, I, device, dtype):
    """Rows reach their experts and come back weighted, and the sum is normed before it enters the stream."""
    E, top, pad = 6, 3, (I + 7) // 8 * 8
    g = torch.Generator().manual_seed(T)
    ups, downs = torch.zeros(E, pad, W), torch.zeros(E, W, pad)
    ups[:, :I] = torch.randn(E, I, W, generator=g) * W ** -0.5
    downs[:, :, :I] = torch.randn(E, W, I, generator=g) * I ** -0.5
    ups, downs, x = rounded(ups), rounded(downs), rounded(torch.randn(T, W, generator=g))
    post, norm = rounded(1 + 0.3 * torch.randn(W, generator=g)), rounded(1 + 0.3 * torch.randn(W, generator=g))
    to = lambda t: t.to(dtype).to(device)  # noqa: E731
    for kind in ("random", "same"):
        ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
        if kind == "same":
            ids[:] = torch.tensor([4, 1, 0], dtype=torch.int32)
        w = torch.rand(T, top, generator=g) + 0.1
        ys, slots = routed_experts(to(x), ids.to(device), to(ups), to(downs), "relu2", gated=False)
        h0 = torch.randn(T, W, generator=g)
        h = h0.clone().to(device)
        row = R.post_norm_rows(h, to(norm), EPS, dtype, post=to(post),
                               result=R.SublayerSum(ys=ys, pair_slot=slots, pair_w=w.to(device)))
        finish(device)
        want = h0.double() + O.rms(O.experts(x, w.double(), ids, ups, downs), EPS) * post
        close(h, want, dtype, kind, bf16=1e-2)
        close(row, O.rms(want, EPS) * norm, dtype, kind, bf16=1.5e-2)


# ---- rows -------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W,T", [(64, 7), (40, 3), (1024, 5), (1536, 4), (2056, 300), (96, 1300), (51, 4), (4096, 3), (4104, 2),
                                 (5000, 2), (1000, 1025), (1536, 1024), (2048, 1026)])
def test_rows_between_two_norms(W, T, device, dtype):
    g = torch.Generator().manual_seed(W)
    rnd = lambda *s: rounded(torch.randn(*s, generator=g))  # noqa: E731
    to = lambda t: t.to(dtype).to(device)  # noqa: E731
    table, ids = rnd(11, W), torch.randint(0, 11, (T,), generator=g)
    norms = [rounded(1 + 0.3 * rnd(W)) for _ in range(3)]
    posts = [rounded(1 + 0.3 * rnd(W)) for _ in range(3)]
    h = torch.full((T, W), float("nan"), device=device)
    row = R.post_norm_rows(h, to(norms[0]), EPS, dtype, ids=ids.to(device), table=to(table), scale=4.25)
    x = table[ids] * 4.25
    close(h, x, torch.float32, "embedding", f32=1e-6)
    close(row, O.rms(x, EPS) * norms[0], dtype, "first", bf16=1e-2)
    # partial sums and a bias; small, so that the epsilon inside the root shows
    y, b = 0.01 * torch.randn(3, T, W, generator=g), rounded(0.01 * rnd(W))
    row = R.post_norm_rows(h, to(norms[1]), EPS, dtype, post=to(posts[0]), result=R.SublayerSum(y.to(device), to(b)))
    x = x + O.rms(y.double().sum(0) + b, EPS) * posts[0]
    close(h, x, torch.float32, "stream")
    close(row, O.rms(x, EPS) * norms[1], dtype, "second", bf16=1e-2)
    # one tensor in the activation format; the stream itself comes back
    y = rnd(T, W)
    row = R.post_norm_rows(h, None, EPS, dtype, post=to(posts[1]), result=R.SublayerSum(to(y)[None]))
    x = x + O.rms(y, EPS) * posts[1]
    close(h, x, torch.float32, "stream")
    close(row, x, dtype, "raw", bf16=5e-3)
    assert row.data_ptr() != h.data_ptr()
    # nothing but zeros
    R.post_norm_rows(h, to(norms[2]), EPS, dtype, post=to(posts[2]), result=R.SublayerSum(to(0 * y)[None]))
    finish(device)
    close(h, x, torch.float32, "no change")


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("n,layers", [(16, 3), (24, 2), (5, 4), (1, 1), (13, 3)])
def test_token_vectors(n, layers, device, dtype):
    """The layer's part of the table, gated by the stream."""
    T, W, V, pad = 70, 48, 19, (n + 7) // 8 * 8
    g = torch.Generator().manual_seed(n)
    table, ids = rounded(torch.randn(V, n * layers, generator=g)), torch.randint(0, V, (T,), generator=g)
    z = torch.full((T, pad), 0.0)
    z[:, :n] = 2 * torch.randn(T, n, generator=g)
    for i in range(layers):
        e = table[ids][:, i * n:(i + 1) * n]
        zz = rounded(z)
        got = R.token_gate(zz.to(dtype).to(device)[None], ids.to(device), table.to(dtype).to(device), i * n, n, dtype)
        close(got[:, :n], O.gelu_tanh(zz[:, :n]) * e, dtype, f"layer {i}", bf16=6e-3)
        assert (got[:, n:] == 0).all()
        parts = torch.randn(3, T, pad, generator=g)
        parts[0] = z - parts[1:].sum(0)
        got = R.token_gate(parts.to(device), ids.to(device), table.to(dtype).to(device), i * n, n, dtype)
        close(got[:, :n], O.gelu_tanh(parts.double().sum(0)[:, :n]) * e, dtype, f"layer {i}, partial sums", bf16=6e-3)
        assert (got[:, n:] == 0).all()
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_activations(device, dtype):
    g = torch.Generator().manual_seed(0)
    to = lambda t: t.to(dtype).to(device)  # noqa: E731
    for I, T in ((40, 9), (13, 5), (2056, 30)):
        for p, q in ((0.3, -1.2), (2.5, 3.0), (-4.0, 0.0)):
            num = rounded(torch.tensor([p, q]))
            b = rounded(torch.randn(I, generator=g))
            z = rounded(torch.randn(T, I, generator=g) * torch.tensor([0.01, 1.0, 6.0, 0.3, 2.0]).repeat(T)[:T, None])
            want = O.xielu(z + b, *num)
            got = R.bias_act(to(z)[None], "xielu", dtype, bias=to(b), numbers=to(num))
            close(got, want, dtype, bf16=6e-3)
            small = (z + b).abs() < 0.05
            if small.any():      # no cancellation next to zero
                close(got.cpu()[small], want[small], dtype, "small", f32=1e-5, bf16=6e-3)
            parts = torch.randn(3, T, I, generator=g)
            parts[0] = z.float() - parts[1:].sum(0)
            close(R.bias_act(parts.to(device), "xielu", dtype, bias=to(b), numbers=to(num)),
                  O.xielu(parts.double().sum(0) + b, *num), dtype, "partial sums", bf16=6e-3)
        z = rounded(3 * torch.randn(T, I, generator=g))
        used = torch.tensor([0, -1, 5, 3, -1, 2, 2, 1, 0] * 4, dtype=torch.int32)[:T].to(device)
        got = R.bias_act(to(z)[None], "relu2", dtype, used=used)
        keep = [i for i in range(T) if used[i] >= 0]
        close(got[keep], (torch.clamp(z, min=0) ** 2)[keep], dtype, bf16=6e-3)
    finish(device)
