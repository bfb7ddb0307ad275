"""The Gumazen decoder through the framework: checkpoint loading, the rollout engine's prefill / decode / scheduler, its block
allocator and prefix cache, scoring, export and the command line, against the plain forward of ``gumazen_oracle`` (CPU path,
32-bit CUDA kernels, bf16 CUDA kernels)."""
import copy
import json
import os
import subprocess
import sys

import gumazen_oracle as O
import pytest
import torch

from siirl_b200.engine.rollout.native_engine import RolloutEngine, SamplingParams
from siirl_b200.engine.rollout.trace_replay import TraceReplay, load_engine
from siirl_b200.models.config import DecoderConfig, get_config
from siirl_b200.ops.attention import SeqInfo

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def sink(heads, kv, dim, vdim, mlp, dims=8, base=1e4, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim,
                                           "scale": scale or 2.0 * dim ** -0.5, "rot": {"base": base, "dims": dims}}, "mlp": mlp}


def table(heads, kv, dim, vdim, mlp, window, rows, far, cap=20.0, scale=None):
    return {"type": "attention_2", "rel_rows": rows,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5,
                      "softcap": cap, "bias_max": far, "mask": {"size": window}}, "mlp": mlp}


def bias(heads, kv, dim, vdim, mlp, dims=8, base=1e4, scaling=None, scale=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention_3", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim,
                                             "scale": scale or 1.2 * dim ** -0.5, "rot": rot}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, ff, top, groups, keep, identity, scale, shared):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale,
                                                         "groups": {"count": groups, "keep": keep}}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


MODELS = {
    # unequal widths everywhere, a layer without feed-forward, a loop in the middle, three streams
    "mixed": dict(vocab=203, width=72, eps=1e-4, streams=3, loop=loop(1, 4, 2), layers=[
        table(6, 3, 24, 16, moe(7, 24, 3, 3, 2, 2, 1.7, 40), window=21, rows=12, far=19),
        bias(4, 2, 32, 40, dense(104), dims=16, scaling=(5.0, 1.0, 3.0, 40)),
        sink(3, 1, 16, 48, None, dims=16), sink(5, 5, 24, 8, moe(5, 16, 2, 2, 1, 1, 0.8, 0), dims=6),
        table(2, 1, 64, 32, dense(40), window=70, rows=20, far=66)]),
    # sizes that are equal, constants that are one, the loop over everything, once, one stream
    "ones": dict(vocab=128, width=64, eps=1e-5, streams=1, loop=loop(0, 3, 1), layers=[
        bias(1, 1, 64, 64, dense(64), dims=64, scale=1.0), sink(1, 1, 64, 64, moe(1, 64, 1, 1, 1, 0, 1.0, 64), dims=64, scale=1.0),
        table(1, 1, 64, 64, moe(2, 64, 1, 1, 1, 1, 1.0, 64), window=1, rows=2, far=2, scale=1.0)]),
    # windows only: blocks leave them; two streams, no loop, every output kept
    "windows": dict(vocab=96, width=40, eps=1e-2, streams=2, loop=None, layers=[
        table(4, 2, 16, 24, moe(6, 8, 4, 2, 2, 2, 2.0, 16), window=64, rows=8, far=30),
        table(2, 2, 8, 8, None, window=33, rows=16, far=100)]),
    # a loop at the end, one layer many times, four streams, many outputs
    "tail": dict(vocab=64, width=96, eps=1e-3, streams=4, loop=loop(1, 2, 4), layers=[
        sink(17, 1, 8, 24, dense(48), dims=4, base=500.0),
        bias(4, 1, 48, 32, moe(33, 24, 5, 4, 2, 15, 1.2, 24), dims=24, scaling=(8.0, 1.0, 4.0, 100))]),
    # a loop at the start
    "head": dict(vocab=80, width=48, eps=1e-5, streams=2, loop=loop(0, 2, 3), layers=[
        table(3, 1, 40, 16, dense(56), window=100, rows=32, far=90, cap=8.0), sink(2, 2, 16, 24, dense(24), dims=2),
        bias(4, 4, 8, 8, moe(4, 40, 2, 1, 1, 0, 3.0, 8))]),
    # sizes no vector access or tensor map takes
    "odd": dict(vocab=101, width=51, eps=1e-5, streams=2, loop=loop(1, 3, 2), layers=[
        table(3, 1, 13, 11, moe(5, 21, 2, 3, 2, 1, 1.5, 13), window=37, rows=10, far=29),
        bias(2, 1, 10, 7, dense(37), dims=6), sink(1, 1, 5, 3, moe(3, 9, 1, 1, 1, 1, 1.0, 0), dims=4)]),
}


def make(tmp, name):
    """Checkpoint folder, parsed config and weights of one of the models above."""
    from safetensors.torch import save_file
    m = copy.deepcopy(MODELS[name])
    cfg = {"architecture": "Gumazen", "vocab": m["vocab"], "width": m["width"], "norm": {"eps": m["eps"]},
           "streams": m["streams"], "layers": m["layers"]}
    if m["loop"]:
        cfg["loop"] = m["loop"]
    W = O.random_checkpoint(cfg, seed=len(name))
    for layer in cfg["layers"]:
        layer.pop("rel_rows", None)
    path = os.path.join(str(tmp), name)
    os.makedirs(path, exist_ok=True)
    save_file(W, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return path, cfg, W


def tokens_of(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def routed(cfg):
    return any(x["mlp"] and x["mlp"]["kind"] == "moe" for x in cfg["layers"])


def check(got, want, dtype, what="", cfg=None):
    """Root mean square over the vocabulary, relative to the logits' own.  With 16-bit rounding some token of a routed model
    takes another expert on a close call: a few positions may be off, most may not."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == torch.float32:
        assert err.max().item() < 1e-4, f"{what}: {err.max().item():.2e} at row {int(err.argmax())}"
    else:
        worst = err.sort().values[max(0, int(0.8 * (len(err) - 1)))] if cfg is not None and routed(cfg) else err.max()
        assert worst.item() < 8e-2, f"{what}: {worst.item():.2e}, largest at row {int(err.argmax())}"


def replay(path, dtype, device, max_tokens=1024, slots=8):
    return TraceReplay(load_engine(path, dtype, max_tokens, slots=slots, device=device), max_slots=slots)


def finish(device):
    if device == "cuda":
        from siirl_b200.ops import lib
        torch.cuda.synchronize()
        lib.check_status()


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(MODELS))
def test_prompts_portions_and_decoding_equal_the_plain_forward(name, device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, name)
    n = 150
    toks = tokens_of(cfg, n, 1)
    want = O.forward(cfg, W, toks)
    rp = replay(path, dtype, device)
    check(rp.step([("whole", toks, list(range(n)))]), want, dtype, "whole prompt", cfg)
    for i, cuts in enumerate([[2] * 20 + [110], [3, 61, 64, 22], [65, 64, 21], [130, 20]]):
        got, at = [], 0
        for c in cuts:
            got.append(rp.step([(f"p{i}", toks[at:at + c], list(range(c)))]))
            at += c
        check(torch.cat(got), want, dtype, f"portions {cuts[:4]}", cfg)
    for i, start in enumerate((1, 63, 100)):
        got = [rp.step([(f"d{i}", toks[:start], list(range(start)))])]
        got += [rp.step([(f"d{i}", [t], [0])]) for t in toks[start:]]
        check(torch.cat(got), want, dtype, f"decoding from {start}", cfg)
    finish(device)


def test_the_sum_of_streams_after_every_layer_run(tmp_path):
    """Layer by layer, the loop's passes included, on the CPU path."""
    from siirl_b200.ops import rows as R
    for name in ("mixed", "tail", "head"):
        path, cfg, W = make(tmp_path, name)
        toks = tokens_of(cfg, 9, 2)
        want = []
        O.forward(cfg, W, toks, want)
        rp = replay(path, torch.float32, "cpu")
        seen, step = [], R.hyper_rows

        def spy(h, *a, **kw):
            out = step(h, *a, **kw)
            if kw.get("result") is not None:
                seen.append(h.sum(1))
            return out
        R.hyper_rows = spy
        try:
            rp.step([("x", toks, [])])
        finally:
            R.hyper_rows = step
        order = O.run_order(cfg)
        ends, at = [], 0
        for i in order:
            at += 1 + int(cfg["layers"][i]["mlp"] is not None)
            ends.append(at - 1)
        assert len(seen) == at and len(rp.engine.cache) == len(order) == len(want)
        for i, (e, b) in enumerate(zip(ends, want)):
            assert (seen[e] - b).abs().max() < 1e-4 * b.abs().max(), i


FAULTS = ["passes", "sink", "window", "cap", "table", "gate", "mix", "out", "bias", "frequencies", "rows_norm", "correction",
          "groups", "identity", "shared", "router_scale", "relu", "norm_bias", "pairing"]


@pytest.mark.parametrize("fault", FAULTS)
def test_a_misread_design_is_far_outside_the_tolerance(fault, tmp_path, monkeypatch):
    """Mistakes planted in the plain forward move the logits far beyond what the 32-bit comparisons above allow."""
    path, cfg, W = make(tmp_path, "mixed")
    toks = tokens_of(cfg, 60, 3)
    right = O.forward(cfg, W, toks)
    W, cfg = {k: v.double() for k, v in W.items()}, copy.deepcopy(cfg)
    attend, route = O.attend, O.route
    if fault == "passes":
        cfg["loop"]["times"] = 1
    elif fault == "sink":
        monkeypatch.setattr(O, "attend", lambda *a, **kw: attend(*a, **dict(kw, sink=False)))
    elif fault == "window":
        cfg["layers"][0]["mixer"]["mask"]["size"] += 1
    elif fault == "cap":
        monkeypatch.setattr(O, "attend", lambda *a, **kw: attend(*a, **dict(kw, cap=0.0)))
    elif fault == "table":          # one distance off
        monkeypatch.setattr(O, "bucket", lambda n, rows, far, real=O.bucket: real(n + 1, rows, far))
    elif fault == "gate":
        W["l0.mix.g"] *= 0
    elif fault == "mix":
        W = {k: v.T if k.endswith(".mix") and "hc" in k else v for k, v in W.items()}
    elif fault == "out":
        W["l1.hc2.out"] = W["l1.hc2.out"].roll(1, 0)
    elif fault == "bias":
        W["l1.mix.k.b"] *= 0
    elif fault == "frequencies":
        del cfg["layers"][1]["mixer"]["rot"]["scaling"]
    elif fault == "rows_norm":      # after the split into heads
        W["l1.mix.q.norm"] = W["l1.mix.q.norm"].roll(1, 0)
    elif fault == "correction":
        W["l0.mlp.correction"] *= 0
    elif fault == "groups":         # every group allowed
        monkeypatch.setattr(O, "route", lambda z, c, r: route(z, c, dict(r, groups={"count": r["groups"]["count"],
                                                                                       "keep": r["groups"]["count"]})))
    elif fault == "identity":       # identity experts that give nothing
        monkeypatch.setattr(O, "route", lambda z, c, r: tuple(zip(*[(i, w * (i < r["experts"])) for i, w in zip(*route(z, c, r))])))
    elif fault == "shared":
        del cfg["layers"][0]["mlp"]["shared"]
    elif fault == "router_scale":
        cfg["layers"][0]["mlp"]["router"]["scale"] *= 1.1
    elif fault == "relu":
        monkeypatch.setattr(O, "dense", lambda h, W, p: torch.relu(h @ W[p + "up"].T) @ W[p + "down"].T)
    elif fault == "norm_bias":
        W["l2.norm1.b"] *= 0
    elif fault == "pairing":        # neighbours instead of halves
        def rotate(x, positions, rot, real=O.rotate):
            d = rot["dims"]
            perm = torch.tensor([i // 2 + (i % 2) * (d // 2) for i in range(d)] + list(range(d, x.shape[-1])))
            return real(x[..., torch.argsort(perm)], positions, rot)[..., perm]
        monkeypatch.setattr(O, "rotate", rotate)
    err = (O.forward(cfg, W, toks) - right).pow(2).mean(-1).sqrt().max() / right.pow(2).mean().sqrt()
    assert err > 5e-3, err


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "ones", "windows"])
def test_batches_and_reused_slots(name, device, dtype, tmp_path):
    """Unequal requests together, ended at different times; later ones take their slots and blocks."""
    path, cfg, W = make(tmp_path, name)
    rp = replay(path, dtype, device, max_tokens=700, slots=8)
    lens = {"a": 1, "b": 64, "c": 131, "d": 70, "e": 2}
    for again in range(2):
        toks = {k: tokens_of(cfg, n + 30, 10 * again + i) for i, (k, n) in enumerate(lens.items())}
        want = {k: O.forward(cfg, W, t) for k, t in toks.items()}
        got = {k: [] for k in lens}
        out = rp.step([(k, toks[k][:n], list(range(n))) for k, n in lens.items()])
        for k, part in zip(lens, out.split(list(lens.values()))):
            got[k].append(part)
        live = list(lens)
        for s in range(30):
            if s in (4, 9, 20):
                rp.end([live.pop(s % 2)])
            out = rp.step([(k, [toks[k][lens[k] + s]], [0]) for k in live])
            for k, row in zip(live, out):
                got[k].append(row[None])
        rp.end(live)
        for k in lens:
            z = torch.cat(got[k])
            check(z, want[k][:z.shape[0]], dtype, f"pass {again} request {k}", cfg)
        assert rp.engine.alloc.num_free == rp.engine.alloc.num_blocks and len(rp.free) == 8
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["head", "windows"])
def test_long_decoding(name, device, dtype, tmp_path):
    """Blocks that left every window go back while the sequence runs, when no layer sees everything."""
    path, cfg, W = make(tmp_path, name)
    n = 420 if device == "cuda" else 200
    toks = tokens_of(cfg, n, 5)
    rp = replay(path, dtype, device)
    got = [rp.step([("x", toks[:7], list(range(7)))])]
    got += [rp.step([("x", [t], [0])]) for t in toks[7:]]
    check(torch.cat(got), O.forward(cfg, W, toks), dtype, "", cfg)
    held = [b for b in rp.live["x"].blocks if b >= 0]
    assert len(held) == ((n + 63) // 64 if name == "head" else 2 if (n - 64) % 64 else 1)
    rp.end(["x"])
    assert rp.engine.alloc.num_free == rp.engine.alloc.num_blocks
    finish(device)


def greedy_is_consistent(cfg, W, prompt, new, logprobs, dtype):
    """Every generated token is the oracle's best one up to rounding, with the oracle's log-probability."""
    z = O.forward(cfg, W, prompt + new[:-1])[len(prompt) - 1:]
    tol = 1e-4 if dtype == torch.float32 else 0.3
    best = torch.stack([row.max() - row[t] - tol * row.std() for t, row in zip(new, z)])
    lp = torch.log_softmax(z, -1)[torch.arange(len(new)), torch.tensor(new)]
    off = (lp - torch.tensor(logprobs).double()).abs()
    if dtype == torch.float32:
        assert best.max() <= 1e-9 and off.max() < 2e-3
    else:       # a close call of a router moves single tokens
        assert (best > 0).float().mean() <= 0.2 and off.median() < 0.3


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "windows"])
def test_greedy_generation_through_the_scheduler(name, device, dtype, tmp_path):
    """More sequences than slots, two samples per prompt, chunked prompts: greedy tokens are the plain forward's."""
    path, cfg, W = make(tmp_path, name)
    model = load_engine(path, dtype, 256, device=device).model
    prompts = [tokens_of(cfg, n, 40 + n) for n in (5, 64, 130, 1, 77)]
    sp = SamplingParams(n=2, temperature=0.0, max_new_tokens=10, ignore_eos=True)
    runs = []
    for kw in (dict(max_num_seqs=16), dict(max_num_seqs=4, enable_chunked_prefill=True, max_num_batched_tokens=33),
               dict(max_num_seqs=8, use_cuda_graph=False)):
        eng = RolloutEngine(model, max_model_len=256, num_blocks=40, sync_interval=4, **kw)
        outs = eng.generate(prompts, sp)
        assert len(outs) == 10
        for o in outs:
            greedy_is_consistent(cfg, W, prompts[o.prompt_index], o.token_ids, o.logprobs, dtype)
        assert eng.alloc.num_free == eng.alloc.num_blocks
        runs.append([o.token_ids for o in outs])
        assert eng.generate(prompts[:2], sp)[0].token_ids is not None       # slots and blocks again
    if dtype == torch.float32:
        assert runs[0] == runs[1] == runs[2]
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_prompts_that_share_a_prefix_reuse_its_blocks(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "tail")
    eng = load_engine(path, dtype, 512, device=device)
    stem = tokens_of(cfg, 130, 7)
    sp = SamplingParams(n=1, temperature=0.0, max_new_tokens=6, ignore_eos=True)
    eng.generate([stem], sp)
    for p in (stem[:128] + tokens_of(cfg, 40, 8), stem[:128] + tokens_of(cfg, 3, 9)):
        before = eng.stats.get("prefix_cache_hit_tokens", 0)
        o, = eng.generate([p], sp)
        assert eng.stats["prefix_cache_hit_tokens"] - before == 128
        greedy_is_consistent(cfg, W, p, o.token_ids, o.logprobs, dtype)
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_sleep_and_wake_and_sampling(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "tail")
    model = load_engine(path, dtype, 256, device=device).model
    eng = RolloutEngine(model, max_num_seqs=8, max_model_len=128, num_blocks=24, sync_interval=4)
    sp = SamplingParams(n=4, temperature=1.0, max_new_tokens=9, ignore_eos=True, seed=3)
    first = eng.generate([tokens_of(cfg, 20, 1)], sp)
    eng.sleep()
    assert eng.cache is None
    eng.wake_up()
    again = eng.generate([tokens_of(cfg, 20, 1)], sp)
    if device == "cuda":
        assert [o.token_ids for o in first] == [o.token_ids for o in again]
    assert len({tuple(o.token_ids) for o in again}) > 1
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_weights_that_change_reach_the_next_call(device, dtype, tmp_path):
    """Tables derived from weights (biases by distance) follow a reload, and parameters may move to other storage."""
    from siirl_b200.models.hf_io import load_hf_weights
    path, cfg, W = make(tmp_path, "head")
    rp = replay(path, dtype, device)
    toks = tokens_of(cfg, 40, 4)
    rp.step([("a", toks, [39])])
    W2 = dict(W, **{"l0.mix.rel": W["l0.mix.rel"].flip(0).contiguous(), "l2.mix.q.b": W["l2.mix.q.b"] * -2})
    from safetensors.torch import save_file
    save_file(W2, os.path.join(path, "model.safetensors"))
    for p in rp.engine.model.parameters():
        p.data = p.data.clone()
    load_hf_weights(rp.engine.model, path)
    got = torch.cat([rp.step([("b", toks[:30], list(range(30)))])] + [rp.step([("b", [t], [0])]) for t in toks[30:]])
    check(got, O.forward(cfg, W2, toks), dtype, "", cfg)
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_scoring_equals_the_plain_forward(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "head")
    model = load_engine(path, dtype, 256, device=device).model
    lens = [70, 1, 133]
    toks = [tokens_of(cfg, n, n) for n in lens]
    info = SeqInfo(lens, device=device)
    ids = torch.tensor(sum(toks, []), device=device)
    labels = torch.roll(ids, -1)
    lp, ent = model.logprobs(ids, info.positions, info, labels, temperature=0.7)
    z = torch.cat([O.forward(cfg, W, t) for t in toks]) / 0.7
    ref = torch.log_softmax(z, -1)
    err = (lp.double().cpu() - ref.gather(1, labels.cpu()[:, None])[:, 0]).abs()
    err2 = (ent.double().cpu() + (ref.exp() * ref).sum(-1)).abs()
    if dtype == torch.float32:
        assert max(err.max(), err2.max()) < 2e-3
    else:
        assert max(err.quantile(0.8), err2.quantile(0.8)) < 0.3
    finish(device)


def test_configuration_and_checkpoint_round_trip(tmp_path):
    from safetensors.torch import load_file

    from siirl_b200.models.decoder import build_model
    from siirl_b200.models.hf_io import load_hf_weights, save_hf_model
    for name in MODELS:
        path, cfg, W = make(tmp_path, name)
        c = get_config(path)
        assert c.to_hf_config() == cfg
        assert DecoderConfig.from_dict(json.loads(json.dumps(c.to_dict()))) == c
        assert len(c.paged_layers()) == len(O.run_order(cfg))
        model = build_model(c, dtype=torch.bfloat16)
        load_hf_weights(model, path)
        out = os.path.join(str(tmp_path), name + "_out")
        save_hf_model(model, out)
        back = load_file(os.path.join(out, "model.safetensors"))
        assert set(back) == set(W) and all(torch.equal(back[k], W[k]) for k in W)
        assert get_config(out).to_dict() == c.to_dict()
        assert c.num_parameters() == sum(t.numel() for t in W.values())
    lay = cfg["layers"]
    for bad in (dict(cfg, layers=[dict(lay[0], type="unknown")]), dict(cfg, loop=loop(2, 4, 1)),
                dict(cfg, layers=[dict(lay[0], mlp={"kind": "sparse", "ff": 8})])):
        with pytest.raises(ValueError):
            DecoderConfig.from_hf_config(bad)
    # a router that cannot choose that many, a rotation wider than the head
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["router"]["top"] = 30
    bad2 = copy.deepcopy(cfg)
    bad2["layers"][1]["mixer"]["rot"]["dims"] = 12
    for c in (bad, bad2):
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(c, f)
        with pytest.raises(ValueError):
            build_model(get_config(path), dtype=torch.float32)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(dict(cfg, width=cfg["width"] + 8), f)
    with pytest.raises(ValueError):
        load_hf_weights(build_model(get_config(path), dtype=torch.float32), path)


def test_cache_free_generation_is_the_same(tmp_path):
    from siirl_b200.engine.rollout.recompute_engine import RecomputeEngine
    path, cfg, W = make(tmp_path, "ones")
    eng = load_engine(path, torch.float32, 256, device="cpu")
    prompts = [tokens_of(cfg, n, n) for n in (4, 70)]
    sp = SamplingParams(n=1, temperature=0.0, max_new_tokens=6, ignore_eos=True)
    a = eng.generate(prompts, sp)
    b = RecomputeEngine(eng.model, max_num_seqs=4, max_model_len=256).generate(prompts, sp)
    assert [o.token_ids for o in a] == [o.token_ids for o in b]


def test_command_line_serves_the_design():
    """A validation-only run of the launcher on the preset: rollout, reward and metrics through the worker's engine."""
    env = dict(os.environ, OMP_NUM_THREADS="2")
    cmd = [sys.executable, "-m", "siirl_b200.main_dag", "algorithm.adv_estimator=grpo", "data.synthetic=arith",
           "data.synthetic_size=8", "data.train_batch_size=4", "data.max_prompt_length=16", "data.max_response_length=8",
           "actor_rollout_ref.model.arch_preset=tiny-gumazen", "actor_rollout_ref.model.random_init=True",
           "actor_rollout_ref.rollout.n=2", "actor_rollout_ref.actor.ppo_mini_batch_size=4",
           "actor_rollout_ref.actor.ppo_micro_batch_size_per_gpu=2", "trainer.n_gpus_per_node=1", "trainer.device=cpu",
           "trainer.val_before_train=True", "trainer.val_only=True", "trainer.logger=[console]",
           "trainer.resume_mode=disable"]
    r = subprocess.run(cmd, cwd=ROOT, env=env, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "val" in r.stdout + r.stderr


@GPU
def test_trace_run_program(tmp_path):
    """The replay program on a folder, both formats."""
    import numpy as np
    path, cfg, W = make(tmp_path, "head")
    toks = tokens_of(cfg, 80, 9)
    lines = [{"step": 0, "entries": [{"id": "u", "tokens": toks[:70], "want": [3, 69]},
                                     {"id": "v", "tokens": toks[:2], "want": []}], "end": ["v"]},
             {"step": 1, "entries": [{"id": "u", "tokens": toks[70:71], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "u", "tokens": toks[71:72], "want": [0]}], "end": ["u"]}]
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "200"], input="\n".join(json.dumps(x) for x in lines) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
        z = O.forward(cfg, W, toks[:72])
        got = torch.from_numpy(np.concatenate([np.fromfile(out / f, dtype="<f4") for f in ("0.f32", "2.f32")]))
        check(got.view(3, -1), z[[3, 69, 71]], getattr(torch, dtype), "", cfg)
