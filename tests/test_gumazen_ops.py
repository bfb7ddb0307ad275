"""Mechanisms of the Gumazen decoder one by one against the plain statements of ``gumazen_oracle``: rotation and norms in front
of attention with a sink, a soft cap, a distance table and gated heads; the grouped router and the routed feed-forward; the
hyper-connected residual.  The same cases run on the framework's CPU path, its 32-bit and its bf16 CUDA kernels."""
import math

import gumazen_oracle as O
import pytest
import torch

from siirl_b200.ops import rows as R
from siirl_b200.ops.moe import route_grouped, routed_experts
from siirl_b200.ops.window_attention import (QkvPrepare, QueryTiles, WindowSpec, distance_buckets, rotary_frequencies,
                                             window_attention)

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]


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
def test_frequencies_and_buckets():
    scaling = {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 300}
    for rot in (dict(dims=20, base=2e4), dict(dims=64, base=1e6, scaling=scaling), dict(dims=2, base=10.0, scaling=scaling)):
        want = O.frequencies(rot)
        assert rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling")) == pytest.approx(want, rel=1e-12)
    full = O.frequencies(dict(dims=64, base=1e6, scaling=scaling))
    plain = O.frequencies(dict(dims=64, base=1e6))
    ratio = [a / b for a, b in zip(full, plain)]
    # all three bands are there
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 6) and any(0.17 < r < 0.99 for r in ratio)
    for rows, far in ((16, 90), (32, 128), (6, 7), (8, 1000), (2, 40), (10, 33)):
        b = distance_buckets(rows, far)
        assert b[-1] == rows - 1 and b == sorted(b) and b[:rows // 2] == list(range(rows // 2))
        assert [b[min(n, len(b) - 1)] for n in range(2000)] == [O.bucket(n, rows, far) for n in range(2000)]
        assert distance_buckets(rows, far, 5) == b[:5]
    assert distance_buckets(1, 30) == [0]


# ---- attention -------------------------------------------------------------------------------------------------------------
ATT = {
    # heads, kv_heads, dk, dv, then what is special
    "sink": dict(size=(6, 2, 32, 24), norm="heads", rot=dict(dims=16, base=5e3), sink=True),
    "sink_one_kv": dict(size=(5, 1, 48, 48), norm="heads", rot=dict(dims=48, base=1e4), sink=True),
    "sink_wide": dict(size=(4, 4, 128, 96), norm="heads", rot=dict(dims=32, base=1e5), sink=True),
    "table": dict(size=(6, 2, 40, 72), norm="rows", window=37, cap=18.0, rel=(16, 30), gate=True),
    "table_far": dict(size=(8, 1, 64, 64), norm="rows", window=130, cap=30.0, rel=(12, 40), gate=True),
    "table_open": dict(size=(4, 2, 24, 16), norm="rows", window=0, cap=25.0, rel=(8, 60), gate=True),
    "table_many_heads": dict(size=(20, 2, 64, 32), norm="rows", window=90, cap=18.0, rel=(32, 200), gate=True),
    "window_one": dict(size=(2, 2, 32, 32), norm="rows", window=1, cap=10.0, rel=(4, 9), gate=True),
    "page_window": dict(size=(3, 1, 96, 80), norm="rows", window=64, cap=20.0, rel=(2, 64), gate=True),
    "bias": dict(size=(6, 3, 64, 40), norm="rows", bias=True,
                 rot=dict(dims=24, base=1e4, scaling={"factor": 4.0, "low": 1.0, "high": 4.0, "original": 60})),
    "bias_whole": dict(size=(4, 1, 128, 128), norm="rows", bias=True, rot=dict(dims=128, base=1e6)),
    "very_wide": dict(size=(2, 1, 192, 256), norm="rows", bias=True, rot=dict(dims=96, base=1e4)),
    "many_columns": dict(size=(33, 11, 192, 16), norm="heads", rot=dict(dims=16, base=1e4), sink=True),
    "odd_units": dict(size=(5, 5, 24, 8), norm="heads", rot=dict(dims=16, base=1e4), sink=True),
    "odd": dict(size=(3, 3, 21, 13), norm="rows", window=50, cap=15.0, rel=(10, 33), gate=True),
    "odd_sink": dict(size=(3, 1, 18, 11), norm="heads", rot=dict(dims=6, base=1e3), sink=True),
    "odd_bias": dict(size=(5, 5, 10, 7), norm="rows", bias=True, rot=dict(dims=10, base=1e3)),
    "single": dict(size=(1, 1, 8, 8), norm="heads", rot=dict(dims=2, base=10.0), sink=True),
}
EPS = 1e-4


class Case:
    """Raw projections with queries that single out keys at the edges of what they see and just beyond, the oracle's answer
    and the framework's description of the branch."""

    def __init__(self, name, T, seed=0):
        c = self.c = ATT[name]
        H, G, dk, dv = c["size"]
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.scale = 14.0 / dk
        k, v = rnd(T, G, dk), rnd(T, G, dv)
        wq, wk = (1 + 0.3 * rnd(H * dk), 1 + 0.3 * rnd(G * dk)) if c["norm"] == "rows" else (torch.ones(H * dk), torch.ones(G * dk))
        self.wq, self.wk = rounded(wq), rounded(wk)
        w, q = c.get("window", 0), rnd(T, H, dk)
        for i in range(T):
            spots = [i - w + 1, i - w, 0, i, i - 64, i // 64 * 64, i - 1, i // 2]
            j = spots[i % len(spots)]
            if 0 <= j <= i:
                # what gives, weighted and turned at i, the key at j weighted and turned there
                kk = (k[j] * self.wk.view(G, dk).float()).repeat_interleave(H // G, 0)[None]
                if "rot" in c:
                    kk = O.rotate(kk.double(), torch.tensor([j - i]), c["rot"]).float()
                q[i] = kk[0] / self.wq.view(H, dk).float()
        self.bq, self.bk, self.bv = (rounded(0.3 * rnd(H * dk)), rounded(0.3 * rnd(G * dk)), rounded(0.3 * rnd(G * dv))) \
            if c.get("bias") else (torch.zeros(H * dk).double(), torch.zeros(G * dk).double(), torch.zeros(G * dv).double())
        self.q = rounded(q.reshape(T, -1) - self.bq.float())
        self.k = rounded(k.reshape(T, -1) - self.bk.float())
        self.v = rounded(v.reshape(T, -1))
        self.z = rounded(2 * rnd(T, H))
        self.rel = rounded(2 * rnd(c["rel"][0], H)) if "rel" in c else None
        up = lambda n: (n + 7) // 8 * 8  # noqa: E731
        self.offs = [8, 8 + up(H * dk), 8 + up(H * dk) + up(G * dk), 8 + up(H * dk) + up(G * dk) + up(G * dv)]
        self.width = self.offs[3] + up(H) + 8
        self.T = T

    def want(self, first=0):
        """The oracle's heads of rows ``first ..``."""
        H, G, dk, dv = self.c["size"]
        c, pos = self.c, torch.arange(self.T)
        q, k, v = self.q + self.bq, self.k + self.bk, (self.v + self.bv).view(self.T, G, dv)
        if c["norm"] == "rows":
            q, k = O.rms(q, EPS) * self.wq, O.rms(k, EPS) * self.wk
        q, k = q.view(self.T, H, dk), k.view(self.T, G, dk)
        if "rot" in c:
            q, k = O.rotate(q, pos, c["rot"]), O.rotate(k, pos, c["rot"])
        if c["norm"] == "heads":
            q, k = O.rms(q, EPS), O.rms(k, EPS)
        bias = None
        if self.rel is not None:
            bias = self.rel[torch.tensor([O.bucket(n, *c["rel"]) for n in range(self.T)])]
        o = O.attend(q[first:], k, v, self.scale, start=first, window=c.get("window", 0), cap=c.get("cap", 0.0), bias=bias,
                     sink=c.get("sink", False))
        if c.get("gate"):
            o = o * O.sigmoid(self.z[first:])[:, :, None]
        return o.reshape(self.T - first, -1)

    def branch(self, dtype, device):
        H, G, dk, dv = self.c["size"]
        c, to = self.c, lambda t: t.to(dtype).to(device)  # noqa: E731
        spec = WindowSpec(H, G, dk, dv, *self.offs[:3], self.scale, c.get("window", 0), softcap=c.get("cap", 0.0),
                          sink=c.get("sink", False))
        pr = QkvPrepare(norm=c["norm"], eps=EPS, g_off=self.offs[3] if c.get("gate") else -1)
        if c["norm"] == "rows":
            pr.q_norm, pr.k_norm = to(self.wq), to(self.wk)
        if c.get("bias"):
            pr.bias = torch.zeros(self.width, dtype=dtype, device=device)
            for off, b in zip(self.offs, (self.bq, self.bk, self.bv)):
                pr.bias[off:off + b.numel()] = b.to(dtype)
        if "rot" in c:
            f = torch.tensor(rotary_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling")), dtype=torch.float64)
            pr.freq = torch.stack([f.float(), (f - f.float().double()).float()], 1).to(device)
        if self.rel is not None:
            pr.rel = to(self.rel)
            pr.bucket = torch.tensor(distance_buckets(*c["rel"], c.get("window", 0)), dtype=torch.int32, device=device)
            pr.table = torch.full((H, pr.bucket.numel()), float("nan"), device=device)
        x = torch.full((self.T, self.width), 7.0, dtype=torch.float64)
        for off, t in zip(self.offs, (self.q, self.k, self.v, self.z)):
            x[:, off:off + t.shape[1]] = t
        return spec, pr, x.to(dtype).to(device)


class Pages:
    def __init__(self, spec, slots, max_len, dtype, device, seed=3):
        g = torch.Generator().manual_seed(seed)
        nb = (max_len + 63) // 64
        order = torch.randperm(slots * nb + 3, generator=g)[: slots * nb].to(torch.int32)
        self.table = order.view(slots, nb).to(device)
        # blocks hold what earlier sequences left: finite values that must not matter
        self.cache = (torch.randn(slots * nb + 3, spec.block_elems, generator=g) * 30).to(dtype).to(device)


def prompts(spec, pr, xs, pages, slots, starts, simt=False):
    """Portions ``xs[i]`` from position ``starts[i]`` of slot ``slots[i]``, one batch."""
    dev, lens = xs[0].device, [x.shape[0] for x in xs]
    pos = torch.cat([torch.arange(s, s + n, dtype=torch.int32) for s, n in zip(starts, lens)]).to(dev)
    ids = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, n in zip(slots, lens)]).to(dev)
    x = torch.cat(xs)
    out = torch.full((x.shape[0], 16 + (spec.heads * spec.vdim + 7) // 8 * 8), 9.0, dtype=x.dtype, device=dev)
    window_attention(spec, x, ids, pos, pages.table, pages.cache, out, 16, tiles=QueryTiles(lens, starts, slots, dev),
                     simt=simt, prepare=pr)
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
    window_attention(spec, rows, ids, pos, pages.table, pages.cache, o, 16, seq_lens=lens, prepare=pr)
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
    for cuts in ([T], [2, 62, 64, 1, 66, 8], [128, 75]):
        pages, at, got = Pages(spec, 3, 256, dtype, device), 0, []
        for n in cuts:
            got += prompts(spec, pr, [x[at:at + n]], pages, [1], [at])
            at += n
        finish(device)
        close(torch.cat(got), want, dtype, f"portions {cuts}")
    pages = Pages(spec, 3, 256, dtype, device)
    got = [prompts(spec, pr, [x[:97]], pages, [2], [0])[0]]
    got += [single(spec, pr, x, pages, 2, at, slabs=1 + at % 3)[None] for at in range(97, T)]
    finish(device)
    close(torch.cat(got), want, dtype, "single tokens", f32=1e-4)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["sink", "table", "bias"])
def test_attention_of_unequal_sequences_in_one_batch(name, device, dtype):
    lens, starts, slots = [1, 130, 64, 7], [0, 65, 2, 70], [3, 2, 1, 0]
    cases = [Case(name, s + n, seed=i) for i, (n, s) in enumerate(zip(lens, starts))]
    spec, _, _ = cases[0].branch(dtype, device)
    pages = Pages(spec, 4, 256, dtype, device)
    # the branch's weights are the first case's: the others only lend their rows
    for c in cases[1:]:
        c.wq, c.wk, c.bq, c.bk, c.bv, c.rel = (getattr(cases[0], k) for k in ("wq", "wk", "bq", "bk", "bv", "rel"))
    _, pr, _ = cases[0].branch(dtype, device)
    xs = [c.branch(dtype, device)[2] for c in cases]
    for x, s, slot in zip(xs, starts, slots):
        if s:
            prompts(spec, pr, [x[:s]], pages, [slot], [0])
    got = prompts(spec, pr, [x[s:] for x, s in zip(xs, starts)], pages, slots, starts)
    finish(device)
    for o, c, s in zip(got, cases, starts):
        close(o, c.want()[s:], dtype)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_a_long_context_in_several_work_items(device, dtype):
    """More than 1024 visible tokens: decoding cuts them into chunks and joins them, the sink and the gates once."""
    T = 2300 if device == "cuda" else 200
    for extra in (dict(size=(4, 2, 64, 64), norm="heads", rot=dict(dims=32, base=1e5), sink=True),
                  dict(size=(4, 2, 64, 64), norm="rows", window=1500, cap=20.0, rel=(32, 1400), gate=True)):
        ATT["long"] = extra
        case = Case("long", T)
        first = T - 6
        spec, pr, x = case.branch(dtype, device)
        pages = Pages(spec, 2, T + 64, dtype, device)
        prompts(spec, pr, [x[:first]], pages, [0], [0])
        got = torch.stack([single(spec, pr, x, pages, 0, at) for at in range(first, T)])
        again = prompts(spec, pr, [x], Pages(spec, 2, T + 64, dtype, device), [1], [0])[0][first:]
        finish(device)
        close(got, case.want(first), dtype, "single tokens", f32=1e-4)
        close(again, case.want(first), dtype, "prompt", f32=1e-4)
    del ATT["long"]


@pytest.mark.parametrize("device,dtype", WHERE)
def test_attention_is_the_same_wherever_blocks_lie(device, dtype):
    """Other slots and other blocks, and the general kernel beside the tensor-core one."""
    for name in ("sink", "table", "bias"):
        case = Case(name, 150)
        spec, pr, x = case.branch(dtype, device)
        a = prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device, seed=1), [0], [0])[0]
        b = prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device, seed=2), [2], [0])[0]
        assert torch.equal(a, b)
        close(prompts(spec, pr, [x], Pages(spec, 3, 192, dtype, device), [1], [0], simt=True)[0], a.double().cpu(), dtype)
    finish(device)


# ---- router and routed feed-forward ----------------------------------------------------------------------------------------
ROUTER = {  # experts, identity, top, groups, keep, scale
    "grouped": (12, 4, 3, 4, 2, 2.5), "one_group": (6, 3, 2, 1, 1, 1.0), "all_groups": (8, 1, 4, 3, 3, 0.7),
    "no_identity": (10, 0, 1, 5, 1, 1.3), "mostly_identity": (2, 30, 5, 8, 3, 1.0), "many": (200, 56, 8, 8, 4, 2.0),
    "very_many": (300, 20, 6, 10, 2, 1.5), "everything": (4, 0, 4, 2, 2, 1.0), "one": (1, 0, 1, 1, 1, 3.0),
    "wide_groups": (60, 10, 32, 2, 1, 1.0),
}


def router_case(name, T, seed=0):
    n, ident, top, groups, keep, scale = ROUTER[name]
    g = torch.Generator().manual_seed(seed)
    E = n + ident
    z = torch.randn(T, E, generator=g) * 2
    corr = rounded(torch.randn(E, generator=g) * 0.4)       # most choice scores are negative
    spec = dict(experts=n, identity=ident, top=top, scale=scale, groups=dict(count=groups, keep=keep))
    return z, corr, spec


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(ROUTER))
def test_router(name, device, dtype):
    T = 70
    z, corr, spec = router_case(name, T)
    E = z.shape[1]
    parts = torch.full((3, T, E + 5), 50.0)                  # partial sums in wider rows
    parts[1:, :, :E] = torch.randn(2, T, E)
    parts[0, :, :E] = z - parts[1:, :, :E].sum(0)
    z = parts.double().sum(0)[:, :E]
    args = (spec["experts"], spec["top"], spec["groups"]["count"], spec["groups"]["keep"], spec["scale"])
    w, ids, w_id = route_grouped(parts.to(device), corr.to(dtype).to(device), *args)
    finish(device)
    for t in range(T):
        want_ids, want_w = O.route(z[t], corr, spec)
        want = {}
        for i, x in zip(want_ids, want_w.tolist()):
            key = -1 if i >= spec["experts"] else i
            want[key] = want.get(key, 0.0) + x
        got = {}
        for i, x in zip(ids[t].tolist(), w[t].tolist()):
            got[i] = got.get(i, 0.0) + x
        assert set(got) == set(want)
        assert all(abs(got[i] - want[i]) < 1e-4 * max(want.values()) for i in want)
        assert abs(w_id[t].item() - want.get(-1, 0.0)) < 1e-4 * max(want.values())


def test_router_refuses_impossible_choices():
    z, corr = torch.zeros(1, 2, 12), torch.zeros(12)
    for args in ((12, 5, 3, 1, 1.0), (12, 2, 5, 1, 1.0), (12, 2, 3, 4, 1.0), (13, 2, 3, 1, 1.0)):
        with pytest.raises(ValueError):
            route_grouped(z, corr, *args)


def gated_weights(E, W, I, g):
    up = (I + 7) // 8 * 8
    gate_up, down = torch.zeros(E, 2 * up, W), torch.zeros(E, W, up)
    gate_up[:, :I] = torch.randn(E, I, W, generator=g) * W ** -0.5
    gate_up[:, up:up + I] = torch.randn(E, I, W, generator=g) * W ** -0.5
    down[:, :, :I] = torch.randn(E, W, I, generator=g) * I ** -0.5
    return rounded(gate_up), rounded(down)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,W,I", [(1, 64, 24), (5, 72, 40), (300, 128, 64), (97, 51, 13), (33, 40, 20)])
def test_routed_experts_and_their_sum(T, W, I, device, dtype):
    """Rows reach their experts and come back weighted, with identity experts and a shared part, into one stream."""
    E, top = 6, 3
    g = torch.Generator().manual_seed(T)
    gate_up, down = gated_weights(E, W, I, g)
    x = rounded(torch.randn(T, W, generator=g))
    for kind in ("random", "same", "nobody"):
        ids = torch.randint(-1, E, (T, top), generator=g).to(torch.int32)
        if kind == "same":
            ids[:] = torch.tensor([4, -1, 0], dtype=torch.int32)
        if kind == "nobody":
            ids[:] = -1
        w = torch.rand(T, top, generator=g)
        to = lambda t: t.to(dtype).to(device)  # noqa: E731
        ys, slots = routed_experts(to(x), ids.to(device), to(gate_up), to(down), "silu")
        h0 = torch.randn(T, 2, W, generator=g)
        shared = torch.randn(2, T, W, generator=g)
        w_id = torch.rand(T, generator=g)
        mix, out, bias = rounded(torch.randn(2, 2, generator=g)), rounded(torch.randn(2, generator=g)), rounded(torch.randn(W, generator=g))
        h = h0.clone().to(device)
        R.hyper_rows(h, to(torch.ones(W)), to(torch.zeros(W)), 1e-5, w_in=to(torch.ones(2)), w_mix=to(mix), w_out=to(out),
                     result=R.SublayerSum(shared.to(device), to(bias), ys, slots, w.to(device), to(x), w_id.to(device)))
        finish(device)
        half = gate_up.shape[1] // 2
        y = shared.double().sum(0) + bias + w_id[:, None].double() * x
        for t in range(T):
            for e, a in zip(ids[t].tolist(), w[t].tolist()):
                if e >= 0:
                    parts = {"e.gate": gate_up[e, :half], "e.up": gate_up[e, half:], "e.down": down[e]}
                    y[t] += a * O.expert(x[t:t + 1], parts, "e.")[0]
        want = torch.stack([sum(mix[s, t] * h0[:, s].double() for s in range(2)) + out[t] * y for t in range(2)], 1)
        close(h, want, dtype, kind, bf16=8e-3)


# ---- hyper-connected residual ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("S,W,T", [(2, 64, 7), (1, 40, 3), (4, 2056, 5), (3, 96, 300), (2, 51, 4), (5, 72, 6), (16, 24, 2),
                                   (2, 4100, 3), (2, 5000, 2), (4, 3584, 2)])
def test_hyper_connected_rows(S, W, T, device, dtype):
    g = torch.Generator().manual_seed(S * W)
    rnd = lambda *s: rounded(torch.randn(*s, generator=g))  # noqa: E731
    to = lambda t: t.to(dtype).to(device)  # noqa: E731
    table, ids = rnd(11, W), torch.randint(0, 11, (T,), generator=g)
    norms = [(1 + 0.3 * rnd(W), 0.5 * rnd(W)) for _ in range(3)]
    norms = [(rounded(a), rounded(b)) for a, b in norms]
    w_in, w_out, w_mix = [rnd(S), rnd(S)], [rnd(S), rnd(S)], [rnd(S, S), rnd(S, S)]
    h = torch.full((T, S, W), float("nan"), device=device)
    eps = 1e-3
    # first sublayer, from the table
    row = R.hyper_rows(h, *map(to, norms[0]), eps, w_in=to(w_in[0]), ids=ids.to(device), table=to(table))
    xs = [table[ids]] * S
    read = lambda xs, w: sum(w[s] * xs[s] for s in range(S))  # noqa: E731
    close(row, O.layer_norm(read(xs, w_in[0]), *norms[0], eps), dtype, "first", bf16=1e-2)
    # between two sublayers: partial sums
    y = torch.randn(3, T, W, generator=g)
    row = R.hyper_rows(h, *map(to, norms[1]), eps, w_in=to(w_in[1]), w_out=to(w_out[0]), w_mix=to(w_mix[0]),
                       result=R.SublayerSum(y.to(device)))
    step = lambda xs, mix, out, y: [sum(mix[s, t] * xs[s] for s in range(S)) + out[t] * y for t in range(S)]  # noqa: E731
    xs = step(xs, w_mix[0], w_out[0], y.double().sum(0))
    close(h, torch.stack(xs, 1), torch.float32, "streams")
    close(row, O.layer_norm(read(xs, w_in[1]), *norms[1], eps), dtype, "second", f32=1e-4, bf16=1e-2)
    # the end: one tensor in the activation format, plain sum
    y = rnd(T, W)
    row = R.hyper_rows(h, *map(to, norms[2]), eps, w_out=to(w_out[1]), w_mix=to(w_mix[1]), result=R.SublayerSum(to(y)[None]))
    xs = step(xs, w_mix[1], w_out[1], y)
    finish(device)
    close(h, torch.stack(xs, 1), torch.float32, "streams at the end")
    close(row, O.layer_norm(sum(xs), *norms[2], eps), dtype, "last", f32=1e-4, bf16=1e-2)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_activations(device, dtype):
    g = torch.Generator().manual_seed(0)
    for I in (40, 13):
        z = rounded(3 * torch.randn(9, I, generator=g))
        close(R.scaled_act(z.to(dtype).to(device), "relu2"), torch.relu(z) ** 2, dtype, bf16=6e-3)
        gu = rounded(3 * torch.randn(9, 2 * I, generator=g))
        used = torch.tensor([0, -1, 5, 3, -1, 2, 2, 1, 0], dtype=torch.int32, device=device)
        got = R.gated_act(gu.to(dtype).to(device), "silu", used)
        keep = [i for i in range(9) if used[i] >= 0]
        close(got[keep], (gu[:, :I] * O.sigmoid(gu[:, :I]) * gu[:, I:])[keep], dtype, bf16=6e-3)
    finish(device)


@pytest.mark.gpu
def test_activation_of_partial_products():
    """Few rows split the contraction; the activation adds the parts up itself."""
    from siirl_b200.ops.dense import linear_partial
    g = torch.Generator().manual_seed(1)
    for T, W, I in ((5, 2048, 96), (200, 1024, 72), (700, 512, 40)):
        x, w = rounded(torch.randn(T, W, generator=g)), rounded(torch.randn(2 * I, W, generator=g) * W ** -0.5)
        y = x @ w.T
        parts = linear_partial(x.bfloat16().cuda(), w.bfloat16().cuda())
        assert (parts.shape[0] > 1) == (T < 512)
        close(R.partial_act(parts, "silu", gated=True), y[:, :I] * O.sigmoid(y[:, :I]) * y[:, I:], torch.bfloat16)
        close(R.partial_act(parts, "relu2"), torch.relu(y) ** 2, torch.bfloat16)
        z = linear_partial(x.bfloat16().cuda(), w.bfloat16().cuda(), f32=True, max_splits=12)
        close(z.sum(0), y, torch.float32, f32=1e-5)
    finish("cuda")


def test_angles_keep_their_remainder():
    """Far positions: the two-float frequency gives the double-precision angle where one float is off."""
    f = torch.tensor(rotary_frequencies(64, 1e6), dtype=torch.float64)
    hi = f.float()
    lo = (f - hi.double()).float()
    n = torch.tensor(100003.0)
    a = n * hi
    rest = torch.addcmul(-a.double(), n.double(), hi.double()).float() + n * lo
    err = (a.double() + rest.double() - 100003.0 * f).abs().max().item()
    assert err < 1e-7 < (a.double() - 100003.0 * f).abs().max().item()
    assert math.isclose(rotary_frequencies(64, 1e6)[1], 1e6 ** (-2 / 64))
