"""The Rizitar decoder through the framework: checkpoint loading, the rollout engine's prefill / decode / scheduler, its block
allocator with blocks of pooled entries, recurrent states, scoring, export and the command line, against the plain forward of
``rizitar_oracle`` (CPU path, 32-bit CUDA kernels, bf16 CUDA kernels)."""
import copy
import json
import os
import subprocess
import sys

import pytest
import rizitar_oracle as O
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


def att(heads, kv, dim, mlp, window, pool, dims=8, base=1e4, scaling=None, scale=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "fast", "original", "slow"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim,
                                           "scale": scale or 1.5 * dim ** -0.5, "rot": rot,
                                           "mask": {"size": window, "pool": pool}}, "mlp": mlp}


def delta(heads, dim, mlp, rank):
    return {"type": "general_delta", "rank": rank, "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, ff, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


MODELS = {
    # unequal widths everywhere, two pools, a layer without feed-forward
    "mixed": dict(vocab=203, width=72, eps=1e-4, scale=3.7, side=10, layers=[
        delta(3, 24, moe(7, 24, 3), rank=5),
        att(6, 3, 24, dense(104), window=21, pool=5, dims=16, scaling=(5.0, 4.0, 60, 0.5)),
        att(4, 2, 32, None, window=45, pool=14, dims=32), delta(2, 16, dense(40), rank=16)]),
    # sizes that are equal, constants that are one
    "ones": dict(vocab=128, width=64, eps=1e-5, scale=1.0, side=64, layers=[
        att(1, 1, 64, moe(1, 64, 1), window=1, pool=1, dims=64, scale=1.0, scaling=(1.0, 1.0, 64, 1.0)),
        delta(1, 64, dense(64), rank=64), att(1, 1, 64, dense(64), window=64, pool=64, dims=64, scale=1.0)]),
    # attention only: blocks leave the windows, pooled entries stay; a pool wider than its window and than a page
    "windows": dict(vocab=96, width=40, eps=1e-2, scale=0.5, side=8, layers=[
        att(4, 2, 16, moe(6, 8, 4), window=33, pool=7), att(2, 2, 8, None, window=20, pool=70, dims=4)]),
    # short pools: several blocks of pooled entries, full ones shared by the samples of a prompt
    "short": dict(vocab=64, width=48, eps=1e-3, scale=2.0, side=8, layers=[
        att(2, 1, 16, dense(24), window=9, pool=2), delta(3, 16, None, rank=4), att(2, 2, 16, None, window=30, pool=3)]),
    # recurrences only, wide and narrow heads
    "deltas": dict(vocab=64, width=96, eps=1e-3, scale=9.8, side=24, layers=[
        delta(1, 128, dense(48), rank=24), delta(5, 8, moe(33, 24, 5), rank=3), delta(2, 48, None, rank=32)]),
    # sizes no vector access or tensor map takes
    "odd": dict(vocab=101, width=51, eps=1e-5, scale=7.1, side=5, layers=[
        att(3, 1, 13, moe(5, 21, 2), window=37, pool=11, dims=6), delta(3, 7, dense(37), rank=3),
        att(2, 2, 10, dense(9), window=5, pool=3, dims=10, base=500.0, scaling=(8.0, 32.0, 100, 1.0))]),
}


def make(tmp, name):
    """Checkpoint folder, parsed config and weights of one of the models above."""
    from safetensors.torch import save_file
    m = copy.deepcopy(MODELS[name])
    cfg = {"architecture": "Rizitar", "vocab": m["vocab"], "width": m["width"], "norm": {"eps": m["eps"]},
           "embedding": {"scale": m["scale"]}, "token_side": {"dim": m["side"]}, "layers": m["layers"]}
    W = O.random_checkpoint(cfg, seed=len(name))
    for layer in cfg["layers"]:
        layer.pop("rank", None)
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
    """Root mean square over the vocabulary, relative to the logits' own.  With 16-bit rounding most positions are close; a few
    of these small models are further off, because a head's short result is divided by its length, or because a routed token
    takes another expert on a close call."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == torch.float32:
        assert err.max().item() < 1e-4, f"{what}: {err.max().item():.2e} at row {int(err.argmax())}"
        return
    most = err.sort().values[max(0, int(0.8 * (len(err) - 1)))].item()
    assert most < 8e-2, f"{what}: {most:.2e}"
    if cfg is None or not routed(cfg):
        assert err.max().item() < 0.2, f"{what}: {err.max().item():.2e} at row {int(err.argmax())}"


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
    n = 170
    toks = tokens_of(cfg, n, 1)
    want = O.forward(cfg, W, toks)
    rp = replay(path, dtype, device)
    check(rp.step([("whole", toks, list(range(n)))]), want, dtype, "whole prompt", cfg)
    for i, cuts in enumerate([[2] * 20 + [130], [3, 61, 64, 42], [65, 64, 41], [130, 40], [17, 16, 2, 5, 130]]):
        got, at = [], 0
        for c in cuts:
            got.append(rp.step([(f"p{i}", toks[at:at + c], list(range(c)))]))
            at += c
        rp.end([f"p{i}"])
        check(torch.cat(got), want, dtype, f"portions {cuts[:4]}", cfg)
    for i, start in enumerate((1, 63, 100)):
        got = [rp.step([(f"d{i}", toks[:start], list(range(start)))])]
        got += [rp.step([(f"d{i}", [t], [0])]) for t in toks[start:]]
        check(torch.cat(got), want, dtype, f"decoding from {start}", cfg)
    # a prompt, single tokens, another portion, single tokens
    got = [rp.step([("m", toks[:40], list(range(40)))])]
    got += [rp.step([("m", [t], [0])]) for t in toks[40:59]]
    got += [rp.step([("m", toks[59:140], list(range(81)))])]
    got += [rp.step([("m", [t], [0])]) for t in toks[140:]]
    check(torch.cat(got), want, dtype, "mixed", cfg)
    finish(device)


def test_the_stream_after_every_layer(tmp_path):
    """Layer by layer on the CPU path."""
    from siirl_b200.ops import rows as R
    for name in ("mixed", "windows", "odd"):
        path, cfg, W = make(tmp_path, name)
        toks = tokens_of(cfg, 50, 2)
        want = []
        O.forward(cfg, W, toks, want)
        rp = replay(path, torch.float32, "cpu")
        seen, step = [], R.post_norm_rows

        def spy(h, *a, **kw):
            out = step(h, *a, **kw)
            seen.append(h.clone())
            return out
        R.post_norm_rows = spy
        try:
            rp.step([("x", toks, [])])
        finally:
            R.post_norm_rows = step
        at, ends = 0, []
        for c in cfg["layers"]:
            at += 3 if c["mlp"] else 2
            ends.append(at)
        assert len(seen) == at + 1
        for i, (e, b) in enumerate(zip(ends, want)):
            assert (seen[e] - b).abs().max() < 1e-4 * b.abs().max(), i


FAULTS = ["sink", "sink_scaled", "window", "pool_early", "pool_late", "no_pool", "pool_one_token", "values_after_norm",
          "norm_after_rotation", "frequencies", "magnitude", "pairing", "post_norm", "side_first", "side_next_layer", "scale",
          "unit_key", "old_state", "decay", "rate", "head_norm", "gate", "tanh", "relu", "act", "bias", "head"]


@pytest.mark.parametrize("fault", FAULTS)
def test_a_misread_design_is_far_outside_the_tolerance(fault, tmp_path, monkeypatch):
    """Mistakes planted in the plain forward move the logits far beyond what the 32-bit comparisons above allow."""
    path, cfg, W = make(tmp_path, "mixed")
    toks = tokens_of(cfg, 90, 3)
    right = O.forward(cfg, W, toks)
    W, cfg = {k: v.double() for k, v in W.items()}, copy.deepcopy(cfg)
    a = [i for i, x in enumerate(cfg["layers"]) if x["type"] == "attention"]
    attend, pooled, scan, gates = O.attend, O.pooled, O.delta_scan, O.delta_gates
    if fault == "sink":
        monkeypatch.setattr(O, "attend", lambda q, k, v, s, *r: attend(q, k, v, None, *r))
    elif fault == "sink_scaled":
        monkeypatch.setattr(O, "attend", lambda q, k, v, s, scale, *r: attend(q, k, v, s * scale, scale, *r))
    elif fault == "window":
        cfg["layers"][a[0]]["mixer"]["mask"]["size"] += 1
    elif fault in ("pool_early", "pool_late"):      # a block is seen one position too early or too late
        def scores(q, k, scale, window, pool, by=1 if fault == "pool_late" else -1):
            T = q.shape[0]
            i, j, b = torch.arange(T)[:, None], torch.arange(T)[None], torch.arange(T // pool)[None]
            s = (q @ k.t() * scale).masked_fill((j > i) | (i - j >= window), float("-inf"))
            sb = q @ pooled(k[:, None], pool)[:, 0].t() * scale
            return torch.cat([s, sb.masked_fill((b + 1) * pool - 1 > i - window - by, float("-inf"))], 1)
        monkeypatch.setattr(O, "window_scores", scores)
    elif fault == "no_pool":
        for i in a:
            cfg["layers"][i]["mixer"]["mask"]["pool"] = 0
    elif fault == "pool_one_token":
        monkeypatch.setattr(O, "pooled", lambda x, n: x[n - 1::n])
    elif fault == "values_after_norm":
        monkeypatch.setattr(O, "attend", lambda q, k, v, *r: attend(q, k, k, *r))
    elif fault == "norm_after_rotation":
        for i in a:
            for x in ("q", "k"):
                W[f"l{i}.mix.{x}.norm"] = W[f"l{i}.mix.{x}.norm"].flip(0)
    elif fault == "frequencies":
        monkeypatch.setattr(O, "frequencies", lambda rot, f=O.frequencies: (f(dict(rot, scaling=None))[0], f(rot)[1]))
    elif fault == "magnitude":
        monkeypatch.setattr(O, "frequencies", lambda rot, f=O.frequencies: (f(rot)[0], 1.0))
    elif fault == "pairing":        # neighbours instead of halves
        def rotate(x, positions, rot, real=O.rotate):
            d = rot["dims"]
            perm = torch.tensor([i // 2 + (i % 2) * (d // 2) for i in range(d)] + list(range(d, x.shape[-1])))
            return real(x[..., torch.argsort(perm)], positions, rot)[..., perm]
        monkeypatch.setattr(O, "rotate", rotate)
    elif fault == "post_norm":
        W["l0.norm1b"], W["l0.norm1"] = W["l0.norm1"], W["l0.norm1b"]
    elif fault == "side_first":     # gated by the normed stream
        monkeypatch.setattr(O, "token_side", lambda x, e, w, eps, f=O.token_side: f(O.rms(x, eps), e, w, eps))
    elif fault == "side_next_layer":
        W["side.embed"] = W["side.embed"].roll(10, 1)
    elif fault == "scale":          # the head takes the embedding's scale too
        W["embed"] = W["embed"] * cfg["embedding"]["scale"]
        cfg["embedding"]["scale"] = 1.0
    elif fault == "unit_key":       # the removal reads the key as it is
        monkeypatch.setattr(O, "delta_scan", lambda r, k, v, w, f: scan(r, k / 3, v * 3, w, f * 3))
    elif fault == "old_state":      # the removal reads the decayed state
        def after(r, k, v, w, f):
            S, out = torch.zeros(*k.shape[1:], v.shape[2], dtype=r.dtype), []
            for t in range(r.shape[0]):
                u = k[t] / torch.sqrt((k[t] * k[t]).sum(-1, keepdim=True) + 1e-6)
                S = w[t][:, :, None] * S
                S = S - (f[t] * u)[:, :, None] * torch.einsum("hk,hkv->hv", u, S)[:, None] + k[t][:, :, None] * v[t][:, None]
                out.append(torch.einsum("hk,hkv->hv", r[t], S))
            return torch.stack(out), S
        monkeypatch.setattr(O, "delta_scan", after)
    elif fault == "decay":
        monkeypatch.setattr(O, "delta_gates", lambda h, w: (gates(h, w)[0] ** 1.1, gates(h, w)[1]))
    elif fault == "rate":
        monkeypatch.setattr(O, "delta_gates", lambda h, w: (gates(h, w)[0], gates(h, dict(w, **{"a.b": 0 * w["a.b"]}))[1]))
    elif fault == "head_norm":
        W["l0.mix.norm"] = W["l0.mix.norm"].view(3, 24)[0].repeat(3)
    elif fault == "gate":
        W["l0.mix.g"] *= 0
    elif fault == "tanh":
        monkeypatch.setattr(O, "delta_gates", lambda h, w: gates(h, dict(w, w1=w["w1"] * 0.8)))
    elif fault == "relu":
        monkeypatch.setattr(O, "experts", lambda h, w, ids, u, d: sum_of_relu(h, w, ids, u, d))
    elif fault == "act":
        W["l1.mlp.act"] = W["l1.mlp.act"].flip(0)
    elif fault == "bias":
        W["l1.mlp.down.b"] *= 0
    elif fault == "head":
        W["final.norm"] = W["final.norm"].roll(1, 0)
    err = (O.forward(cfg, W, toks) - right).pow(2).mean(-1).sqrt().max() / right.pow(2).mean().sqrt()
    assert err > 5e-3, err


def sum_of_relu(h, w, ids, ups, downs):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for x, e in zip(w[t], ids[t].tolist()):
            out[t] += x * (downs[e] @ torch.relu(ups[e] @ h[t]))
    return out


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "ones", "windows"])
def test_batches_and_reused_slots(name, device, dtype, tmp_path):
    """Unequal requests together, ended at different times; later ones take their slots, states and blocks."""
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
@pytest.mark.parametrize("name", ["mixed", "windows", "deltas"])
def test_long_decoding(name, device, dtype, tmp_path):
    """Blocks that left every window go back while the sequence runs; the pooled entries, more than one block of them, stay."""
    path, cfg, W = make(tmp_path, name)
    n = 540 if device == "cuda" else 400
    toks = tokens_of(cfg, n, 5)
    rp = replay(path, dtype, device)
    got = [rp.step([("x", toks[:7], list(range(7)))])]
    got += [rp.step([("x", [t], [0])]) for t in toks[7:]]
    check(torch.cat(got), O.forward(cfg, W, toks), dtype, "", cfg)
    seq = rp.live["x"]
    if name != "deltas":
        span, pool = {"mixed": (45, 5), "windows": (70, 7)}[name]
        assert len([b for b in seq.blocks if b >= 0]) <= (span + 62) // 64 + 1
        assert len(seq.pool_blocks) == (n // pool + 63) // 64 and all(b >= 0 for b in seq.pool_blocks)
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
@pytest.mark.parametrize("name", ["mixed", "windows", "short"])
def test_greedy_generation_through_the_scheduler(name, device, dtype, tmp_path):
    """More sequences than slots, two samples per prompt (which share full blocks of tokens and of pooled entries), chunked
    prompts: greedy tokens are the plain forward's."""
    path, cfg, W = make(tmp_path, name)
    model = load_engine(path, dtype, 640, device=device).model
    lens = (5, 64, 130, 1, 77) if device == "cpu" and name == "mixed" else (5, 64, 130, 1, 77, 390)
    prompts = [tokens_of(cfg, n, 40 + n) for n in lens]
    sp = SamplingParams(n=2, temperature=0.0, max_new_tokens=12, ignore_eos=True)
    runs = []
    for kw in (dict(max_num_seqs=16), dict(max_num_seqs=4, enable_chunked_prefill=True, max_num_batched_tokens=33),
               dict(max_num_seqs=8, use_cuda_graph=False)):
        eng = RolloutEngine(model, max_model_len=512, num_blocks=80, sync_interval=4, **kw)
        assert not eng.enable_prefix_caching
        outs = eng.generate(prompts, sp)
        assert len(outs) == 2 * len(prompts)
        for o in outs:
            greedy_is_consistent(cfg, W, prompts[o.prompt_index], o.token_ids, o.logprobs, dtype)
        assert eng.alloc.num_free == eng.alloc.num_blocks
        runs.append([o.token_ids for o in outs])
        assert eng.generate(prompts[:2], sp)[0].token_ids is not None       # slots and blocks again
    if dtype == torch.float32:
        assert runs[0] == runs[1] == runs[2]
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_sleep_and_wake_and_sampling(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "mixed")
    model = load_engine(path, dtype, 256, device=device).model
    eng = RolloutEngine(model, max_num_seqs=8, max_model_len=128, num_blocks=24, sync_interval=4)
    sp = SamplingParams(n=4, temperature=1.0, max_new_tokens=9, ignore_eos=True, seed=3)
    first = eng.generate([tokens_of(cfg, 20, 1)], sp)
    eng.sleep()
    assert eng.cache is None and not eng.states
    eng.wake_up()
    again = eng.generate([tokens_of(cfg, 20, 1)], sp)
    if device == "cuda":
        assert [o.token_ids for o in first] == [o.token_ids for o in again]
    assert len({tuple(o.token_ids) for o in again}) > 1
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_scoring_equals_the_plain_forward(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "mixed")
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
        assert max(err.max(), err2.max()) < 5e-3
    else:
        assert max(err.quantile(0.8), err2.quantile(0.8)) < 0.5
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
        assert len(c.paged_layers()) == sum(x["type"] == "attention" for x in cfg["layers"])
        model = build_model(c, dtype=torch.bfloat16)
        load_hf_weights(model, path)
        out = os.path.join(str(tmp_path), name + "_out")
        save_hf_model(model, out)
        back = load_file(os.path.join(out, "model.safetensors"))
        assert set(back) == set(W) and all(torch.equal(back[k], W[k]) for k in W)
        assert get_config(out).to_dict() == c.to_dict()
        assert c.num_parameters() == sum(t.numel() for t in W.values())
    lay = cfg["layers"]
    two_widths, no_window = copy.deepcopy(lay[0]), copy.deepcopy(lay[0])
    two_widths["mixer"]["vdim"] = 4
    no_window["mixer"]["mask"]["size"] = 0
    for bad in (dict(lay[0], type="unknown"), dict(lay[0], mlp={"kind": "sparse", "ff": 8}), two_widths, no_window):
        with pytest.raises(ValueError):
            DecoderConfig.from_hf_config(dict(cfg, layers=[bad]))
    # a router that cannot choose that many, a rotation wider than the head
    bad, bad2 = copy.deepcopy(cfg), copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["router"]["top"] = 30
    bad2["layers"][0]["mixer"]["rot"]["dims"] = 14
    for c in (bad, bad2):
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(c, f)
        with pytest.raises(ValueError):
            build_model(get_config(path), dtype=torch.float32)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(dict(cfg, width=cfg["width"] + 8), f)
    with pytest.raises(ValueError):
        load_hf_weights(build_model(get_config(path), dtype=torch.float32), path)


def test_optional_parts_may_be_missing(tmp_path):
    """Attention without a window, without pooled runs or without a rotation; no second embedding table."""
    from safetensors.torch import save_file
    path, cfg, W = make(tmp_path, "windows")
    for drop in ("pool", "mask", "rot"):
        c = copy.deepcopy(cfg)
        for x in c["layers"]:
            if drop == "pool":
                del x["mixer"]["mask"]["pool"]
            else:
                del x["mixer"][drop]
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(c, f)
        assert get_config(path).to_hf_config() == c
        toks = tokens_of(cfg, 100, 2)
        rp = replay(path, torch.float32, "cpu")
        got = torch.cat([rp.step([("x", toks[:80], list(range(80)))])] + [rp.step([("x", [t], [0])]) for t in toks[80:]])
        check(got, O.forward(c, W, toks), torch.float32, drop)
    c = {k: v for k, v in cfg.items() if k != "token_side"}
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(c, f)
    save_file({k: v for k, v in W.items() if "side" not in k}, os.path.join(path, "model.safetensors"))
    rp = replay(path, torch.float32, "cpu")
    z = rp.step([("x", [1, 2, 3], [0, 1, 2])])
    zero = {k: (v * 0 if k.endswith("side.norm") else v) for k, v in W.items()}
    check(z, O.forward(cfg, zero, [1, 2, 3]), torch.float32, "no token vectors")


def test_cache_free_generation_is_the_same(tmp_path):
    from siirl_b200.engine.rollout.recompute_engine import RecomputeEngine
    path, cfg, W = make(tmp_path, "mixed")
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
           "actor_rollout_ref.model.arch_preset=tiny-rizitar", "actor_rollout_ref.model.random_init=True",
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
    path, cfg, W = make(tmp_path, "mixed")
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
