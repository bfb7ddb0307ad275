"""The Poralorn decoder through the framework: checkpoint loading, the rollout engine's prefill / decode / scheduler, its
block allocator and prefix cache, scoring, export and the command line, against the plain forward of ``poralorn_oracle``
(CPU path, 32-bit CUDA kernels, bf16 CUDA kernels)."""
import copy
import json
import os
import subprocess
import sys

import poralorn_oracle as O
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


def lay(heads, dim, vdim, rank, ff, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or 1.2 * dim ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


MODELS = {
    # unequal widths everywhere, a layer without feed-forward, a loop in the middle
    "mixed": dict(vocab=203, width=72, cap=9.0, eps=1e-4, mult=0.8, loop=loop(1, 3, 3), layers=[
        lay(3, 24, 16, 40, 88), lay(5, 16, 40, 24, 0), lay(2, 48, 24, 136, 104), lay(1, 32, 8, 16, 56)]),
    # sizes that are equal, constants that are one, the loop over everything, once
    "ones": dict(vocab=128, width=64, cap=20.0, eps=1e-5, mult=1.0, loop=loop(0, 2, 1), layers=[
        lay(1, 64, 64, 64, 64, 1.0), lay(1, 64, 64, 64, 64, 1.0)]),
    # the loop at the end, one layer many times, no cap worth mentioning
    "tail": dict(vocab=96, width=40, cap=200.0, eps=1e-2, mult=0.4, loop=loop(1, 2, 4), layers=[
        lay(4, 8, 24, 32, 24), lay(17, 8, 8, 48, 40)]),
    # the loop at the start, the others after it
    "head": dict(vocab=64, width=96, cap=3.0, eps=1e-3, mult=1.3, loop=loop(0, 1, 2), layers=[
        lay(2, 40, 32, 72, 48), lay(3, 32, 48, 56, 0)]),
    # no loop
    "straight": dict(vocab=80, width=48, cap=12.0, eps=1e-5, mult=0.6, loop=None, layers=[
        lay(2, 16, 24, 64, 56), lay(4, 8, 8, 8, 32)]),
    # sizes no vector access or tensor map takes
    "odd": dict(vocab=101, width=51, cap=10.0, eps=1e-5, mult=0.7, loop=loop(1, 3, 2), layers=[
        lay(3, 13, 11, 21, 37), lay(2, 9, 7, 19, 29), lay(1, 5, 3, 10, 0)]),
}


def make(tmp, name):
    """Checkpoint folder, parsed config and weights of one of the models above."""
    from safetensors.torch import save_file
    m = MODELS[name]
    cfg = {"architecture": "Poralorn", "vocab": m["vocab"], "width": m["width"], "norm": {"eps": m["eps"]},
           "residual_mult": m["mult"], "logit_softcap": m["cap"], "layers": m["layers"]}
    if m["loop"]:
        cfg["loop"] = m["loop"]
    W = O.random_checkpoint(cfg, seed=len(name))
    path = os.path.join(str(tmp), name)
    os.makedirs(path, exist_ok=True)
    save_file(W, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return path, cfg, W


def tokens_of(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def check(got, want, dtype, what=""):
    """Root mean square over the vocabulary, relative to the logits' own."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    lim = 3e-5 if dtype == torch.float32 else 8e-2
    assert err.max().item() < lim, f"{what}: {err.max().item():.2e} at row {int(err.argmax())}"


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
    check(rp.step([("whole", toks, list(range(n)))]), want, dtype, "whole prompt")
    for i, cuts in enumerate([[2] * 20 + [110], [3, 61, 64, 22], [65, 64, 21], [130, 20]]):
        got, at = [], 0
        for c in cuts:
            got.append(rp.step([(f"p{i}", toks[at:at + c], list(range(c)))]))
            at += c
        check(torch.cat(got), want, dtype, f"portions {cuts[:4]}")
    for i, start in enumerate((1, 63, 100)):
        got = [rp.step([(f"d{i}", toks[:start], list(range(start)))])]
        got += [rp.step([(f"d{i}", [t], [0])]) for t in toks[start:]]
        check(torch.cat(got), want, dtype, f"decoding from {start}")
    finish(device)


def test_the_residual_stream_after_every_layer_run(tmp_path):
    """Layer by layer: what each run adds, the passes' entries included, on the CPU path."""
    from siirl_b200.ops import rows as R
    for name in ("mixed", "head"):
        path, cfg, W = make(tmp_path, name)
        toks = tokens_of(cfg, 9, 2)
        want = []
        O.forward(cfg, W, toks, want)
        rp = replay(path, torch.float32, "cpu")
        seen, update = [], R.stream_update

        def spy(h, subs, *a, **kw):
            out = update(h, subs, *a, **kw)
            if subs:
                seen.append(h.clone())
            return out
        R.stream_update = spy
        try:
            rp.step([("x", toks, [])])
        finally:
            R.stream_update = update
        assert len(seen) == len(want) == len(rp.engine.cache) == len(O.run_order(cfg))
        for i, (a, b) in enumerate(zip(seen, want)):
            assert (a - b).abs().max() < 1e-4 * b.abs().max(), i


@pytest.mark.parametrize("fault", ["passes", "step", "halves", "embedding", "gate_input", "mult", "tanh_gelu", "output_gate"])
def test_a_misread_design_is_far_outside_the_tolerance(fault, tmp_path, monkeypatch):
    """Mistakes planted in the plain forward move the logits far beyond what the 32-bit comparisons above allow."""
    path, cfg, W = make(tmp_path, "mixed")
    toks = tokens_of(cfg, 40, 3)
    right = O.forward(cfg, W, toks)
    W, cfg, width = {k: v.double() for k, v in W.items()}, copy.deepcopy(cfg), cfg["width"]
    if fault == "passes":
        cfg["loop"]["times"] = 2
    elif fault == "step":
        W["loop.step"] = W["loop.step"].roll(1, 0)
    elif fault == "halves":
        W["loop.in"] = W["loop.in"].roll(width, 1)
    elif fault == "embedding":
        W["loop.in"][:, width:] = 0
    elif fault == "gate_input":         # the feed-forward's gate on the mixer's input
        W["l0.rg2"] *= W["l0.norm1"] / W["l0.norm2"]
    elif fault == "mult":
        cfg["residual_mult"] *= 0.9
    elif fault == "tanh_gelu":
        monkeypatch.setattr(O, "gelu_erf", lambda z: torch.nn.functional.gelu(z, approximate="tanh"))
    else:
        W["l0.mix.g"] *= 0
    err = (O.forward(cfg, W, toks) - right).pow(2).mean(-1).sqrt().max() / right.pow(2).mean().sqrt()
    assert err > (2e-4 if fault == "tanh_gelu" else 2e-2), err


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "ones", "tail"])
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
            check(z, want[k][:z.shape[0]], dtype, f"pass {again} request {k}")
        assert rp.engine.alloc.num_free == rp.engine.alloc.num_blocks and len(rp.free) == 8
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_long_decoding(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "head")
    n = 420 if device == "cuda" else 200
    toks = tokens_of(cfg, n, 5)
    rp = replay(path, dtype, device)
    got = [rp.step([("x", toks[:7], list(range(7)))])]
    got += [rp.step([("x", [t], [0])]) for t in toks[7:]]
    check(torch.cat(got), O.forward(cfg, W, toks), dtype)
    assert len(rp.live["x"].blocks) == (n + 63) // 64
    rp.end(["x"])
    assert rp.engine.alloc.num_free == rp.engine.alloc.num_blocks
    finish(device)


def greedy_is_consistent(cfg, W, prompt, new, logprobs, dtype):
    """Every generated token is the oracle's best one up to rounding, with the oracle's log-probability."""
    z = O.forward(cfg, W, prompt + new[:-1])[len(prompt) - 1:]
    tol = 1e-4 if dtype == torch.float32 else 0.2
    for t, row in zip(new, z):
        assert row[t].item() >= row.max().item() - tol * row.std().item() - 1e-9
    lp = torch.log_softmax(z, -1)[torch.arange(len(new)), torch.tensor(new)]
    assert (lp - torch.tensor(logprobs).double()).abs().max() < (2e-3 if dtype == torch.float32 else 0.4)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "straight"])
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
    path, cfg, W = make(tmp_path, "mixed")
    eng = load_engine(path, dtype, 512, device=device)
    stem = tokens_of(cfg, 130, 7)
    sp = SamplingParams(n=1, temperature=0.0, max_new_tokens=4, ignore_eos=True)
    eng.generate([stem], sp)
    # far behind the shared blocks (expanded form) and right behind them (a few tokens: absorbed form)
    prompts = [stem[:128] + tokens_of(cfg, 40, 8), stem[:128] + tokens_of(cfg, 3, 9)]
    for p in prompts:
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
    tol = 2e-3 if dtype == torch.float32 else 0.4
    assert (lp.double().cpu() - ref.gather(1, labels.cpu()[:, None])[:, 0]).abs().max() < tol
    assert (ent.double().cpu() + (ref.exp() * ref).sum(-1)).abs().max() < tol
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
    for bad in (dict(cfg, layers=[dict(cfg["layers"][0], type="unknown")]), dict(cfg, loop=loop(2, 4, 1)),
                dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "sparse", "ff": 8})])):
        with pytest.raises(ValueError):
            DecoderConfig.from_hf_config(bad)
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
           "actor_rollout_ref.model.arch_preset=tiny-poralorn", "actor_rollout_ref.model.random_init=True",
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
        check(got.view(3, -1), z[[3, 69, 71]], getattr(torch, dtype))
