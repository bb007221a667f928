"""Taralix through the engine on CPU tensors: reading of checkpoints, every schedule of steps
against the plain restatement, and that mistakes would be noticed (planted in the restatement)."""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import taralix_oracle as oracle
import taralix_util as u
from arcticinference_b200 import LLM, SamplingParams
from arcticinference_b200.config import EngineArgs, ModelConfig
from arcticinference_b200.ops import latent_ops as lat

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module", params=sorted(u.CONFIGS))
def model(request, tmp_path_factory):
    cfg = u.CONFIGS[request.param]
    w = u.weights(cfg, seed=3, peak=1.0)
    return cfg, w, u.save(tmp_path_factory.mktemp(request.param), cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_schedules(model, dtype):
    cfg, w, path = model
    u.check_schedules(cfg, path, dtype, "cpu", w)


def test_expanded_form_agrees(tmp_path, monkeypatch):
    """Long chunks through expanded keys and values beside absorbed decode rows."""
    cfg = u.CONFIGS["wide_latents"]
    w = u.weights(cfg, seed=4, peak=1.0)
    path = u.save(tmp_path, cfg, w)
    sess = u.session(path, "bfloat16", 64 * 9, "cpu")
    m = sess.engine.runner.model
    assert m.expand_min_tokens is not None
    m.expand_min_tokens = 20
    seqs = {"a": u.tokens(cfg, 100, 1), "b": u.tokens(cfg, 90, 2), "c": u.tokens(cfg, 30, 3)}
    steps = [[("a", 30), ("b", 2)], [("a", 68), ("b", 40), ("c", 3)],
             [("c", 26), ("b", 48), ("a", 1)], [("c", 1), ("a", 1)]]
    u.compare(cfg, w, u.run(sess, seqs, steps), seqs, "bfloat16")


def test_greedy_generation_through_the_scheduler(model):
    cfg, w, path = model
    llm = LLM(model=path, device="cpu", dtype="float32", num_gpu_blocks_override=40, block_size=16,
              max_model_len=256, max_num_batched_tokens=32)
    prompts = [u.tokens(cfg, n, 10 + n) for n in (40, 3, 17)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))
    for p, ro in zip(prompts, outs):
        seq = list(p) + ro.outputs[0].token_ids
        z = oracle.forward(cfg, w, seq[:-1])[len(p) - 1:]
        chosen = z.gather(1, torch.tensor(ro.outputs[0].token_ids).unsqueeze(1)).squeeze(1)
        # the largest logit at every step (a tie within rounding counts)
        assert float((z.max(-1).values - chosen).max()) < 1e-4
        assert len(ro.outputs[0].token_ids) == 9


def test_prefix_cache_and_preemption(tmp_path):
    """A prompt served from cached latents, and requests recomputed after their pages were taken,
    generate what they generate alone."""
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg, seed=5)
    path = u.save(tmp_path, cfg, w)
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    prompts = [u.tokens(cfg, 70, 1)[:48] + u.tokens(cfg, n, n) for n in (1, 9, 20)]
    roomy = LLM(model=path, device="cpu", dtype="float32", num_gpu_blocks_override=64,
                block_size=16, max_model_len=128)
    alone = [roomy.generate({"prompt_token_ids": p}, sp)[0] for p in prompts]
    assert alone[2].num_cached_tokens == 48
    tight = LLM(model=path, device="cpu", dtype="float32", num_gpu_blocks_override=12,
                block_size=16, max_model_len=128, enable_prefix_caching=False)
    for a, b in zip(alone, tight.generate([{"prompt_token_ids": p} for p in prompts], sp)):
        assert a.outputs[0].token_ids == b.outputs[0].token_ids


# ---------------------------------------------------------------- mistakes planted in the oracle
def _logits(cfg, w, toks, **patch):
    saved = {k: getattr(oracle, k) for k in patch}
    try:
        for k, v in patch.items():
            setattr(oracle, k, v)
        return oracle.forward(cfg, w, toks)
    finally:
        for k, v in saved.items():
            setattr(oracle, k, v)


def test_planted_mistakes_show(tmp_path):
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg, seed=3, peak=1.0)
    toks = u.tokens(cfg, 130, 7)
    sess = u.session(u.save(tmp_path, cfg, w), "float32", 256, "cpu")
    got = u.run(sess, {"a": toks}, [[("a", n)] for n in u.portions(130, [64, 2, 31, 1])])["a"]
    assert u.error(got, oracle.forward(cfg, w, toks)) < u.TOLERANCE["float32"]

    def plus_one(x, weight, eps):
        return oracle.rms(x, eps) * oracle.f64(weight)

    def eps_outside(x, eps):
        return x / (torch.sqrt((x * x).mean(-1, keepdim=True)) + eps)

    def all_logits(h, w_router, bias, top):
        z = oracle.apply(w_router, h) + oracle.f64(bias)
        chosen = torch.argsort(z, dim=-1, descending=True)[:, :top]
        return chosen, torch.softmax(z, -1).gather(1, chosen)

    no_bias = lambda h, w_router, bias, top: _route(h, w_router, torch.zeros_like(bias), top)
    _route = oracle.route

    def one_key_short(h, c, *a):
        return _attend(h, torch.cat([c[1:2], c[1:]]), *a)
    _attend = oracle.attend_latent

    tol = 10 * u.TOLERANCE["float32"]
    for patch in ({"zero_centred_norm": plus_one}, {"rms": eps_outside}, {"route": all_logits},
                  {"route": no_bias}, {"gelu_tanh": oracle.silu}, {"attend_latent": one_key_short},
                  {"latent": lambda h, a, b, eps: oracle.apply(a, h)}):
        assert u.error(got, _logits(cfg, w, toks, **patch)) > tol, list(patch)
    for change in (lambda c: c.update(postln_alpha=2.4), lambda c: c["norm"].update(eps=0.04),
                   lambda c: c["layers"][1]["mixer"].update(scale=0.2),
                   lambda c: c["layers"][4]["mixer"].update(kv_from=2) or
                   c["layers"][5]["mixer"].update(scale=0.1)):
        other = copy.deepcopy(cfg)
        change(other)
        assert u.error(got, oracle.forward(other, w, toks)) > tol / 5


# ---------------------------------------------------------------- configuration and loading
def test_config_is_read_from_the_checkpoint(tmp_path):
    cfg = u.CONFIGS["mixed"]
    path = u.save(tmp_path, cfg, u.weights(cfg))
    m = ModelConfig.from_pretrained(path)
    assert m.architecture == "Taralix" and m.hidden_size == 160 and m.vocab_size == 211
    assert m.postln_alpha == 2.5 and m.rms_norm_eps == 0.03 and len(m.layer_specs) == 6
    assert m.layer_specs[1].mixer.kv_from == 0 and m.layer_specs[2].mlp is None
    assert m.layer_specs[3].mlp.experts == 7 and m.layer_specs[3].mlp.top == 1
    from arcticinference_b200.plugin import supported_architectures
    assert "Taralix" in supported_architectures()


def test_refused_configurations(tmp_path):
    def broken(change):
        c = copy.deepcopy(u.CONFIGS["mixed"])
        change(c)
        p = tmp_path / "c"
        os.makedirs(p, exist_ok=True)
        (p / "config.json").write_text(json.dumps(c))
        return EngineArgs(model=str(p)).create_engine_config()

    with pytest.raises(NotImplementedError):
        broken(lambda c: c["layers"][0].update(type="other"))
    with pytest.raises(NotImplementedError):
        broken(lambda c: c["layers"][0]["mlp"].update(kind="other"))
    with pytest.raises(ValueError):
        broken(lambda c: c["layers"][1]["mixer"].update(kv_from=1))
    with pytest.raises(ValueError):
        broken(lambda c: c["layers"][3]["mixer"].update(kv_from=1))       # not an owner
    with pytest.raises(ValueError):
        broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    path = u.save(tmp_path / "ok", u.CONFIGS["mixed"], u.weights(u.CONFIGS["mixed"]))
    for kw in ({"tensor_parallel_size": 2}, {"quantization": "fp8"}, {"dtype": "float16"},
               {"forest_cascade_attn_configs": "{}"}):
        with pytest.raises(NotImplementedError):
            EngineArgs(model=path, **kw).create_engine_config()
    with pytest.raises(NotImplementedError):
        EngineArgs(model="llama-tiny", dtype="float32").create_engine_config()


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    cfg = u.CONFIGS["single"]
    w = u.weights(cfg)
    missing = {k: v for k, v in w.items() if k != "l0.mix.uv"}
    with pytest.raises(ValueError, match="l0.mix.uv"):
        u.session(u.save(tmp_path / "a", cfg, missing), "float32", 64, "cpu")
    with pytest.raises(ValueError, match="unexpected"):
        u.session(u.save(tmp_path / "b", cfg, {**w, "l0.mix.extra": w["embed"]}), "float32", 64, "cpu")
    with pytest.raises(ValueError, match="shape"):
        u.session(u.save(tmp_path / "c", cfg, {**w, "l0.mix.o": w["embed"]}), "float32", 64, "cpu")


def test_shared_latents_take_no_memory(tmp_path):
    cfg = u.CONFIGS["mixed"]
    sess = u.session(u.save(tmp_path, cfg, u.weights(cfg)), "float32", 256, "cpu")
    kv, m = sess.engine.runner.kv, sess.engine.runner.model
    assert kv.of(1) is kv.of(0) and kv.of(5) is kv.of(0) and kv.of(4) is kv.of(2)
    assert m.kv_bytes_per_block(64) == (56 + 72) * 64 * 4


def test_weight_sync_is_refused(tmp_path):
    from arcticinference_b200.server.weight_sync.receiver import (engine_sync_weights,
                                                                  engine_weights_info)
    cfg = u.CONFIGS["single"]
    engine = u.session(u.save(tmp_path, cfg, u.weights(cfg)), "float32", 64, "cpu").engine
    with pytest.raises(NotImplementedError):
        engine_weights_info(engine)
    with pytest.raises(NotImplementedError):
        engine_sync_weights(engine, {"master_addr": "ipc://nothing"})


def test_kernel_set_names_existing_sources():
    from arcticinference_b200 import build
    stems = {p.stem for p in build.kernel_sources()}
    for names in build.KERNEL_SETS.values():
        assert set(names) <= stems


# ---------------------------------------------------------------- planning of the latent kernel
@pytest.mark.parametrize("heads,q_lens,kv_lens", [
    (16, [1] * 5, [1, 128, 129, 5000, 64]), (5, [3, 1, 130], [3, 700, 400]),
    (40, [1] * 300, list(range(1, 301))), (130, [2, 0, 1], [2, 5, 4096])])
@pytest.mark.parametrize("cap", [1, 3, 16])
def test_latent_work_covers_every_row_and_key_once(heads, q_lens, kv_lens, cap):
    nr = lat.LatentShape(heads, 256, "latent").tile_rows
    work, tok_splits, ms = lat.plan_latent_work(q_lens, kv_lens, heads, nr, max_splits_cap=cap)
    assert ms <= cap and (work[:, 2] <= nr).all() and (work[:, 2] > 0).all()
    tok0 = np.cumsum(q_lens) - q_lens
    seen = {}
    for seq, row0, n, pos0, ks, ke, piece, pieces in work.tolist():
        assert ks % lat.KEY_TILE == 0 and ks < ke <= kv_lens[seq]
        for r in range(row0, row0 + n):
            t = r // heads
            assert tok0[seq] <= t < tok0[seq] + q_lens[seq]
            assert pos0 + t == kv_lens[seq] - q_lens[seq] + (t - tok0[seq])
            assert tok_splits[t] == pieces
            seen.setdefault(r, []).append((ks, ke))
    assert len(seen) == sum(q_lens) * heads
    for r, spans in seen.items():
        spans.sort()
        assert spans[0][0] == 0 and all(a[1] == b[0] for a, b in zip(spans, spans[1:]))
        seq = int(np.searchsorted(np.cumsum(q_lens), r // heads, side="right"))
        assert spans[-1][1] == kv_lens[seq]


def test_decode_capacity_holds_every_plan():
    for heads, rank in ((7, 64), (16, 512), (40, 256), (130, 128)):
        shape = lat.LatentShape.of(heads, rank, torch.bfloat16)
        for bucket in (1, 2, 8, 40, 136, 256, 512):
            cap, splits = shape.decode_capacity(bucket, 1, 64)
            for kl in (1, 500, 9000):
                lens = [kl] * max(1, bucket // 2)
                q = [1] * len(lens)
                if len(lens) < bucket:
                    q.append(bucket - len(lens))
                    lens.append(bucket - len(lens))
                work, _, ms = shape.plan(q, lens, max_splits_cap=splits)
                assert work.shape[0] <= cap and ms <= splits, (heads, rank, bucket, kl)


# ---------------------------------------------------------------- the trace runner as a program
def test_trace_run_program(tmp_path):
    cfg = u.CONFIGS["single"]
    w = u.weights(cfg, seed=9)
    path = u.save(tmp_path / "m", cfg, w)
    out = tmp_path / "out"
    toks = u.tokens(cfg, 9)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:5], "want": [4, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[5:7], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": toks[:1], "want": [0]},
                                     {"id": "x", "tokens": toks[7:], "want": [1]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", path, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128", "--device", "cpu"],
                       input="".join(json.dumps(l) + "\n" for l in lines), text=True,
                       capture_output=True, timeout=300,
                       env={**os.environ, "PATH": os.path.dirname(sys.executable) + ":" +
                            os.environ["PATH"]})
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    z = oracle.forward(cfg, w, toks)
    read = lambda n: torch.from_numpy(np.fromfile(out / ("%d.f32" % n), "<f4").copy()).double() \
        .reshape(-1, cfg["vocab"])
    assert u.error(read(0), z[[4, 0]]) < u.TOLERANCE["float32"]
    assert u.error(read(2), z[[0, 8]]) < u.TOLERANCE["float32"]
    assert not (out / "1.f32").exists()


def test_trace_run_refuses_float32_for_other_models(tmp_path):
    from arcticinference_b200.entrypoints.trace_run import main
    assert main(["--model", "llama-tiny", "--dtype", "float32", "--out", str(tmp_path),
                 "--max-tokens", "64"]) == 3
