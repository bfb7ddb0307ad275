"""The Domavik decoder through the framework: checkpoint loading, the rollout engine's prefill / decode / scheduler, its
block allocator and recurrent slots, scoring, export and the command line, against the plain forward of
``domavik_oracle`` (CPU path, 32-bit CUDA kernels, bf16 CUDA kernels)."""
import json
import os
import subprocess
import sys

import domavik_oracle as O
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


def att(heads, kv, dim, vdim, size, first):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.2 * dim ** -0.5,
            "mask": {"size": size, "keep_first": first}}


def par(left, right, ls, rs, ff):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mem(heads, dim, vdim, cap, ff):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


MODELS = {
    # unequal widths everywhere, a layer without feed-forward, memory first
    "mixed": dict(vocab=203, width=72, scale=1.7, cap=9.0, eps=1e-4, rank=6, layers=[
        mem(3, 24, 16, 11.0, 88), par(att(6, 3, 16, 24, 9, 3), gla(2, 40, 24, 5.0), 0.8, 1.3, 0),
        par(att(2, 1, 48, 32, 70, 66), gla(3, 8, 16, 16.0), 1.0, 0.4, 104), mem(1, 16, 40, 5.0, 0)]),
    # constants that are one, single heads, sizes that are equal
    "ones": dict(vocab=128, width=64, scale=1.0, cap=20.0, eps=1e-5, rank=16, layers=[
        par(att(1, 1, 64, 64, 64, 64), gla(1, 64, 64, 1.0), 1.0, 1.0, 64), mem(1, 64, 64, 1.0, 64)]),
    # attention of one kind only, no kept token, window of a few tokens
    "narrow": dict(vocab=96, width=40, scale=0.5, cap=3.0, eps=1e-3, rank=3, layers=[
        par(att(4, 2, 8, 8, 3, 0), gla(2, 16, 8, 2.0), 1.5, 0.7, 24), par(att(4, 4, 24, 16, 5, 1), gla(4, 8, 8, 32.0),
                                                                          0.6, 1.1, 40)]),
    # recurrences only
    "memory": dict(vocab=64, width=48, scale=2.0, cap=12.0, eps=1e-5, rank=4, layers=[mem(2, 16, 24, 15.0, 56),
                                                                                      mem(4, 8, 8, 8.0, 32)]),
    # sizes no vector access or tensor map takes
    "odd": dict(vocab=101, width=51, scale=1.1, cap=10.0, eps=1e-5, rank=5, layers=[
        par(att(3, 1, 13, 11, 17, 4), gla(2, 9, 7, 3.0), 1.1, 0.9, 37), mem(3, 10, 15, 6.0, 29)]),
}


def make(tmp, name):
    """Checkpoint folder, parsed config and weights of one of the models above."""
    from safetensors.torch import save_file
    m = MODELS[name]
    cfg = {"architecture": "Domavik", "vocab": m["vocab"], "width": m["width"], "embedding": {"scale": m["scale"]},
           "norm": {"eps": m["eps"]}, "logit_softcap": m["cap"], "layers": m["layers"]}
    W = O.random_checkpoint(cfg, seed=len(name), gate_rank=m["rank"])
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
    lim = 2e-4 if dtype == torch.float32 else 8e-2
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


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "ones"])
def test_batches_and_reused_slots(name, device, dtype, tmp_path):
    """Unequal requests together, ended at different times; later ones take their slots and blocks."""
    path, cfg, W = make(tmp_path, name)
    rp = replay(path, dtype, device, max_tokens=700, slots=8)
    lens = {"a": 1, "b": 64, "c": 131, "d": 70, "e": 2}
    for again in range(3):
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
def test_long_decoding_gives_back_blocks_that_left_the_windows(device, dtype, tmp_path):
    path, cfg, W = make(tmp_path, "narrow")
    n = 420 if device == "cuda" else 300
    toks = tokens_of(cfg, n, 5)
    want = O.forward(cfg, W, toks)
    rp = replay(path, dtype, device)
    got = [rp.step([("x", toks[:7], list(range(7)))])]
    got += [rp.step([("x", [t], [0])]) for t in toks[7:]]
    check(torch.cat(got), want, dtype)
    held = sum(b >= 0 for b in rp.live["x"].blocks)
    assert held <= 3 and len(rp.live["x"].blocks) == (n + 63) // 64      # the kept first token's block and the window's
    rp.end(["x"])
    assert rp.engine.alloc.num_free == rp.engine.alloc.num_blocks
    finish(device)


def greedy_is_consistent(cfg, W, prompt, new, dtype):
    """Every generated token is the oracle's best one up to rounding."""
    z = O.forward(cfg, W, prompt + new[:-1])[len(prompt) - 1:]
    tol = 1e-4 if dtype == torch.float32 else 0.15
    for t, row in zip(new, z):
        assert row[t].item() >= row.max().item() - tol * row.std().item() - 1e-9


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", ["mixed", "narrow", "memory"])
def test_greedy_generation_through_the_scheduler(name, device, dtype, tmp_path):
    """More sequences than slots, two samples per prompt, chunked prompts: greedy tokens are the plain forward's."""
    path, cfg, W = make(tmp_path, name)
    model = load_engine(path, dtype, 256, device=device).model
    prompts = [tokens_of(cfg, n, 40 + n) for n in (5, 64, 130, 1, 77)]
    sp = SamplingParams(n=2, temperature=0.0, max_new_tokens=12, ignore_eos=True)
    runs = []
    for kw in (dict(max_num_seqs=16), dict(max_num_seqs=4, enable_chunked_prefill=True, max_num_batched_tokens=33),
               dict(max_num_seqs=8, use_cuda_graph=False)):
        eng = RolloutEngine(model, max_model_len=256, num_blocks=40, sync_interval=4, **kw)
        outs = eng.generate(prompts, sp)
        assert len(outs) == 10
        for o in outs:
            greedy_is_consistent(cfg, W, prompts[o.prompt_index], o.token_ids, dtype)
            z = O.forward(cfg, W, prompts[o.prompt_index] + o.token_ids[:-1])[len(prompts[o.prompt_index]) - 1:]
            lp = torch.log_softmax(z, -1)[torch.arange(12), torch.tensor(o.token_ids)]
            assert (lp - torch.tensor(o.logprobs).double()).abs().max() < (2e-3 if dtype == torch.float32 else 0.35)
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
    tol = 2e-3 if dtype == torch.float32 else 0.4
    assert (lp.double().cpu() - ref.gather(1, labels.cpu()[:, None])[:, 0]).abs().max() < tol
    assert (ent.double().cpu() + (ref.exp() * ref).sum(-1)).abs().max() < tol
    with pytest.raises(NotImplementedError):
        for p in model.parameters():
            p.requires_grad_(True)
        model.forward_hidden(ids, info.positions, info)
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
        model = build_model(c, dtype=torch.bfloat16)
        load_hf_weights(model, path)
        out = os.path.join(str(tmp_path), name + "_out")
        save_hf_model(model, out)
        back = load_file(os.path.join(out, "model.safetensors"))
        assert set(back) == set(W) and all(torch.equal(back[k], W[k]) for k in W)
        assert get_config(out).to_dict() == c.to_dict()
        assert c.num_parameters() == sum(t.numel() for t in W.values())
    bad = dict(cfg, layers=[dict(cfg["layers"][0], type="unknown")])
    with pytest.raises(ValueError):
        DecoderConfig.from_hf_config(bad)
    wrong = dict(cfg, width=cfg["width"] + 8)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(wrong, f)
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
           "actor_rollout_ref.model.arch_preset=tiny-domavik", "actor_rollout_ref.model.random_init=True",
           "actor_rollout_ref.rollout.n=2", "actor_rollout_ref.actor.ppo_mini_batch_size=4",
           "actor_rollout_ref.actor.ppo_micro_batch_size_per_gpu=2", "trainer.n_gpus_per_node=1", "trainer.device=cpu",
           "trainer.val_before_train=True", "trainer.val_only=True", "trainer.logger=[console]",
           "trainer.resume_mode=disable"]
    r = subprocess.run(cmd, cwd=ROOT, env=env, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "val" in r.stdout + r.stderr


@GPU
def test_trace_run_program(tmp_path):
    """The replay program on a folder: exit code, answer files, refusal of 32-bit for a bf16-only family."""
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
    other = tmp_path / "qwen"
    other.mkdir()
    (other / "config.json").write_text(json.dumps(get_config("tiny").to_hf_config()))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(other), "--dtype", "float32", "--out",
                        str(tmp_path)], input="", capture_output=True, text=True, timeout=600)
    assert r.returncode == 3
