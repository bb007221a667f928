"""Zatirax through the engine on CPU tensors: reading of checkpoints, every mechanism and every
schedule of steps against the plain restatement, and that mistakes would be noticed (planted in
the restatement)."""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zatirax_oracle as oracle
import zatirax_util as u
from arcticinference_b200 import LLM, SamplingParams, ops
from arcticinference_b200.config import EngineArgs, MaskSpec, ModelConfig, RotarySpec
from arcticinference_b200.ops import head_ops as hd
from arcticinference_b200.ops import latent_ops as lat
from arcticinference_b200.ops import stream_ops as st

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module", params=sorted(u.CONFIGS))
def model(request, tmp_path_factory):
    cfg = u.CONFIGS[request.param]
    w = u.weights(cfg, seed=3, peak=u.PEAK[request.param])
    return cfg, w, u.save(tmp_path_factory.mktemp(request.param), cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_schedules(model, dtype):
    cfg, w, path = model
    u.check_schedules(cfg, path, dtype, "cpu", w)


def test_expanded_form_agrees(tmp_path):
    """Long chunks through expanded keys and values beside absorbed decode rows."""
    cfg = u.EXPANDED
    w = u.weights(cfg, seed=4, peak=1.0)
    sess = u.session(u.save(tmp_path, cfg, w), "bfloat16", 64 * 10, "cpu")
    m = sess.engine.runner.model
    assert {x.expand for x in m.mixers} >= {(64, 64), (128, 128), (192, 128)}
    m.expand_min_tokens = 20
    seqs = {"a": u.tokens(cfg, 200, 1), "b": u.tokens(cfg, 190, 2), "c": u.tokens(cfg, 30, 3)}
    steps = [[("a", 130), ("b", 2)], [("a", 68), ("b", 40), ("c", 3)],
             [("c", 26), ("b", 148), ("a", 1)], [("c", 1), ("a", 1)]]
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
    """A prompt served from cached blocks, and requests recomputed after their pages were taken,
    generate what they generate alone."""
    cfg = u.CONFIGS["mixed"]
    path = u.save(tmp_path, cfg, u.weights(cfg, seed=5))
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


def test_a_pass_of_the_loop_has_its_own_cache(tmp_path):
    cfg = u.CONFIGS["mixed"]
    sess = u.session(u.save(tmp_path, cfg, u.weights(cfg)), "float32", 256, "cpu")
    kv, m = sess.engine.runner.kv, sess.engine.runner.model
    assert [l for l, _ in m.runs] == [0, 1, 2, 1, 2, 3, 4]
    assert [t for _, t in m.runs] == [None, 0, None, 1, None, None, None]
    caches = [t.data_ptr() for run in kv.runs for t in run]
    assert len(kv.runs) == 7 and len(set(caches)) == len(caches) == 4 * 2 + 3
    per_token = 2 * (40 + 24) + 2 * (40 + 8) + 2 * (4 * 128) + (100 + 32) + (16 + 8)
    assert m.kv_bytes_per_block(64) == per_token * 64 * 4


# ---------------------------------------------------------------- mechanisms by themselves
@pytest.mark.parametrize("rot", [u.rotary(2), u.rotary(48, 700.0), u.rotary(
    64, 10000.0, (8.0, 1.0, 4.0, 256)), u.rotary(10, 20.0, (3.0, 2.0, 5.0, 40))])
def test_rotation(rot):
    s = rot.get("scaling")
    spec = RotarySpec(rot["base"], rot["dims"], None if s is None else
                      (s["factor"], s["low"], s["high"], s["original"]))
    assert np.allclose(spec.frequencies(), oracle.frequencies(rot), rtol=1e-12)
    pos = torch.tensor([0, 1, 77, 4000])
    x = torch.randn(4, 3, rot["dims"] + 5)
    got = hd.rotate_ref(x, hd.rotary_table(pos, torch.tensor(spec.frequencies()).float()))
    for h in range(3):
        assert float((got[:, h] - oracle.rotate(x[:, h].double(), pos, rot)).abs().max()) < 2e-3
        assert torch.equal(got[:, h, rot["dims"]:], x[:, h, rot["dims"]:])


def test_masks():
    for size in (1, 2, 7, 64):
        for kind, seen in (("window", oracle.in_window), ("chunk", oracle.in_chunk)):
            first = MaskSpec(kind, size).first_key(np.arange(150))
            for i in range(150):
                assert first[i] == min(j for j in range(i + 1) if seen(i, j, size))
                assert MaskSpec(kind, size).first_key(i) == first[i]


def test_clamped_swish():
    g, up = torch.linspace(-9, 9, 61).repeat(61), torch.linspace(-9, 9, 61).repeat_interleave(61)
    for limit in (0.5, 1.0, 7.0):
        got = st.Gate("clamped_swish", limit).join(g.double(), up.double())
        assert float((got - oracle.clamped_swish(g.double(), up.double(), limit)).abs().max()) < 1e-12


def test_stream_sandwich():
    x0, y, w1, w2, v = (torch.randn(*s) for s in ((5, 33), (5, 33), (33,), (33,), (33,)))
    x, act = x0.clone(), torch.empty(5, 33)
    st.stream_sandwich(x, y, w1, v, w2, act, eps=0.3)
    want = x0.double() + oracle.norm(y.double(), w1, 0.3) + v.double()
    assert float((x - want).abs().max()) < 1e-5
    assert float((act - oracle.norm(want, w2, 0.3)).abs().max()) < 1e-5


# ---------------------------------------------------------------- mistakes planted in the oracle
def _logits(cfg, w, toks, **patch):
    saved = {k: getattr(oracle, k) for k in patch}
    oracle.visible.cache_clear()
    try:
        for k, v in patch.items():
            setattr(oracle, k, v)
        return oracle.forward(cfg, w, toks)
    finally:
        for k, v in saved.items():
            setattr(oracle, k, v)
        oracle.visible.cache_clear()


def test_planted_mistakes_show(tmp_path):
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg, seed=3, peak=1.0)
    toks = u.tokens(cfg, 170, 7)
    sess = u.session(u.save(tmp_path, cfg, w), "float32", 256, "cpu")
    got = u.run(sess, {"a": toks}, [[("a", n)] for n in u.portions(170, [64, 2, 31, 1])])["a"]
    assert u.error(got, oracle.forward(cfg, w, toks)) < u.TOLERANCE["float32"]

    _weights_of, _rotate, _window, _chunk = (oracle.weights_of, oracle.rotate, oracle.in_window,
                                             oracle.in_chunk)

    def eps_outside(x, weight, eps):
        return x / (torch.sqrt((x * x).mean(-1, keepdim=True)) + eps) * oracle.f64(weight)

    def interleaved(x, pos, rot):
        n = rot["dims"]
        a = pos.double().unsqueeze(1) * torch.tensor(oracle.frequencies(rot), dtype=torch.float64)
        p, q = x[:, 0:n:2], x[:, 1:n:2]
        out = torch.stack([p * a.cos() - q * a.sin(), q * a.cos() + p * a.sin()], -1).flatten(1)
        return torch.cat([out, x[:, n:]], 1)

    def no_last_run(cfg):
        return [(i, None) for i, _ in _runs(cfg)]
    _runs = oracle.runs

    tol = 10 * u.TOLERANCE["float32"]
    for patch in (
            {"norm": eps_outside}, {"rotate": lambda x, p, r: x}, {"rotate": interleaved},
            {"rotate": lambda x, p, r: _rotate(x, -p, r)},
            {"stretched": lambda f, s: f},
            {"stretched": lambda f, s: f if s is None else f / s["factor"]},
            {"weights_of": lambda s, m, sink=None: _weights_of(s, m)},
            {"in_window": lambda i, j, n: _window(i, j, n + 1)},
            {"in_window": lambda i, j, n: _window(i, j, n - 1)},
            {"in_window": lambda i, j, n: j <= i},
            {"in_chunk": lambda i, j, n: _chunk(i, j, n + 1)},
            {"in_chunk": lambda i, j, n: _window(i, j, n)},
            {"in_chunk": lambda i, j, n: j <= i},
            {"gated_output": lambda o, h, g: o},
            {"gated_output": lambda o, h, g: o * torch.tanh(oracle.apply(g, h))},
            {"clamped_swish": lambda g, up, n: g / (1 + torch.exp(-1.702 * g)) * (up + 1)},
            {"clamped_swish": lambda g, up, n: g.clamp(max=n) / (1 + torch.exp(-g.clamp(max=n)))
             * (up.clamp(-n, n) + 1)},
            {"clamped_swish": lambda g, up, n: g.clamp(-n, n) / (1 + torch.exp(-1.702 * g.clamp(-n, n)))
             * (up.clamp(-n, n) + 1)},
            {"runs": no_last_run}):
        assert u.error(got, _logits(cfg, w, toks, **patch)) > tol, list(patch)
    for change in (lambda c: c["embedding"].update(scale=1.6), lambda c: c["norm"].update(eps=0.03),
                   lambda c: c["layers"][1]["mixer"].update(scale=0.2),
                   lambda c: c["layers"][4]["mixer"].update(scale=0.3),
                   lambda c: c["layers"][3]["mixer"]["rot"].update(base=310.0),
                   lambda c: c["layers"][3]["mlp"].update(limit=2.0),
                   lambda c: c["loop"].update(times=1), lambda c: c["loop"].update(stop=2)):
        other = copy.deepcopy(cfg)
        change(other)
        assert u.error(got, oracle.forward(other, w, toks)) > tol / 5


# ---------------------------------------------------------------- planning under a mask
MASKS = [MaskSpec("window", 1), MaskSpec("window", 100), MaskSpec("window", 3000),
         MaskSpec("chunk", 1), MaskSpec("chunk", 96), MaskSpec("chunk", 2048)]
BATCHES = [([1] * 5, [1, 128, 129, 5000, 64]), ([3, 1, 130], [3, 700, 400]),
           ([1] * 300, list(range(1, 301))), ([2, 0, 1], [2, 5, 4096]), ([600], [5000])]


def _covered(pieces, first, last):
    """The spans cover first .. last without a gap and overlap nowhere."""
    pieces = sorted(p for p in pieces if p[1] > first)
    assert pieces[0][0] <= first and all(a[1] == b[0] for a, b in zip(pieces, pieces[1:]))
    assert pieces[-1][1] > last


@pytest.mark.parametrize("mask", MASKS)
@pytest.mark.parametrize("q_lens,kv_lens", BATCHES)
@pytest.mark.parametrize("cap", [1, 3, 16])
def test_head_work_covers_every_visible_key_once(mask, q_lens, kv_lens, cap):
    for G, Hkv in ((1, 2), (8, 1)):
        work, tok_splits, ms = ops.plan_attention_work(q_lens, kv_lens, G, True, Hkv=Hkv,
                                                       max_splits_cap=cap, mask=mask, align=16)
        assert ms <= cap
        tok0, seen = np.cumsum(q_lens) - q_lens, {}
        for seq, t0, n, pos0, ks, ke, piece, pieces in work.tolist():
            assert ks % 16 == 0
            for t in range(t0, t0 + n):
                assert pos0 + t - t0 == kv_lens[seq] - q_lens[seq] + t - tok0[seq]
                assert tok_splits[t] == pieces
                seen.setdefault((seq, pos0 + t - t0), []).append((ks, ke))
        assert len(seen) == sum(q_lens)
        for (seq, pos), spans in seen.items():
            _covered(spans, int(mask.first_key(pos)), pos)
        # nothing far before the window is read
        for seq, t0, n, pos0, ks, ke, _, pieces in work.tolist():
            if pieces == 1:
                assert ks >= int(mask.first_key(pos0)) - 16


@pytest.mark.parametrize("mask", MASKS)
@pytest.mark.parametrize("q_lens,kv_lens", BATCHES)
@pytest.mark.parametrize("heads", [5, 16, 130])
def test_latent_work_covers_every_visible_key_once(mask, q_lens, kv_lens, heads):
    for cap in (1, 16):
        nr = lat.LatentShape(heads, 256, "latent").tile_rows
        work, tok_splits, ms = lat.plan_latent_work(q_lens, kv_lens, heads, nr, max_splits_cap=cap,
                                                    mask=mask, align=16)
        assert ms <= cap
        seen = {}
        for seq, row0, n, pos0, ks, ke, piece, pieces in work.tolist():
            assert ks % 16 == 0 and ke <= kv_lens[seq]
            for r in range(row0, row0 + n):
                assert tok_splits[r // heads] == pieces
                seen.setdefault((seq, r, pos0 + r // heads), []).append((ks, ke))
        assert len(seen) == sum(q_lens) * heads
        for (seq, r, pos), spans in seen.items():
            _covered(spans, int(mask.first_key(pos)), pos)


@pytest.mark.parametrize("mask", MASKS)
def test_decode_capacity_holds_every_plan(mask):
    shapes = [hd.HeadShape.of(8, 2, 128, 128, torch.bfloat16, mask),
              lat.LatentShape.of(16, 512, torch.bfloat16, 64, mask),
              lat.LatentShape.of(7, 64, torch.bfloat16, 0, mask)]
    for shape in shapes:
        for bucket in (1, 2, 8, 40, 136, 512):
            cls = hd.HeadDecodePlan if isinstance(shape, hd.HeadShape) else lat.LatentDecodePlan
            plan = cls(shape, bucket, 1, 64)
            for kl in (1, 500, 9000):
                lens = [kl] * max(1, bucket // 2)
                q = [1] * len(lens)
                if len(lens) < bucket:
                    q.append(bucket - len(lens))
                    lens.append(bucket - len(lens))
                work, _, ms = plan.plan(q, lens)
                assert work.shape[0] <= plan.work_cap and ms <= plan.splits


# ---------------------------------------------------------------- configuration and loading
def test_config_is_read_from_the_checkpoint(tmp_path):
    cfg = u.CONFIGS["mixed"]
    m = ModelConfig.from_pretrained(u.save(tmp_path, cfg, u.weights(cfg)))
    assert m.architecture == "Zatirax" and m.hidden_size == 160 and m.vocab_size == 211
    assert m.embedding_scale == 1.7 and m.rms_norm_eps == 0.02 and m.loop.times == 2
    a, b = m.layer_specs[0].mixer, m.layer_specs[3].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim) == (6, 2, 40, 24) and a.mask == MaskSpec("chunk", 37)
    assert a.rotary.scaling == (4.0, 1.0, 4.0, 64.0) and a.sink and a.output_gate and a.qk_norm
    assert (b.kv_rank, b.rot_dim) == (100, 32) and b.mask == MaskSpec("window", 65)
    assert m.layer_specs[2].mlp is None and m.layer_specs[1].mlp.limit == 0.7
    from arcticinference_b200.plugin import supported_architectures
    assert "Zatirax" in supported_architectures()


def test_rows_of_the_latent_cache():
    of = lambda *a: lat.LatentLayout.of(*a, torch.bfloat16)
    assert of(40, 8, 5) == lat.LatentLayout(64, 0, 40)
    assert of(100, 20, 5) == lat.LatentLayout(128, 0, 100)
    assert of(100, 32, 5) == lat.LatentLayout(128, 64, 128)
    assert of(512, 64, 5) == lat.LatentLayout(512, 64, 512)
    assert of(256, 96, 5) == lat.LatentLayout(384, 0, 256)
    assert lat.LatentLayout.of(100, 32, 5, torch.float32) == lat.LatentLayout(100, 32, 100)


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
        broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    for change in (lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=42),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
                   lambda c: c["layers"][1]["mixer"].update(rot_dim=6),
                   lambda c: c["layers"][0]["mlp"].update(limit=0.0),
                   lambda c: c["loop"].update(stop=6), lambda c: c["loop"].update(start=3)):
        with pytest.raises(ValueError):
            broken(change)
    path = u.save(tmp_path / "ok", u.CONFIGS["mixed"], u.weights(u.CONFIGS["mixed"]))
    for kw in ({"tensor_parallel_size": 2}, {"quantization": "fp8"}, {"dtype": "float16"}):
        with pytest.raises(NotImplementedError):
            EngineArgs(model=path, **kw).create_engine_config()


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    cfg = u.CONFIGS["all_looped"]
    w = u.weights(cfg)
    for name in ("l1.mix.sink", "loop.step", "l2.norm2b"):
        missing = {k: v for k, v in w.items() if k != name}
        with pytest.raises(ValueError, match=name):
            u.session(u.save(tmp_path / "a", cfg, missing), "float32", 64, "cpu")
    with pytest.raises(ValueError, match="unexpected"):
        u.session(u.save(tmp_path / "b", cfg, {**w, "l1.norm2": w["l0.norm2"]}), "float32", 64, "cpu")
    with pytest.raises(ValueError, match="shape"):
        u.session(u.save(tmp_path / "c", cfg, {**w, "l0.mix.o": w["embed"]}), "float32", 64, "cpu")


def test_preset_generates():
    llm = LLM(model="zatirax-tiny", device="cpu", num_gpu_blocks_override=16, max_model_len=256)
    out = llm.generate([{"prompt_token_ids": [5, 6, 7, 8]}],
                       SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 4


# ---------------------------------------------------------------- the trace runner as a program
def test_trace_run_program(tmp_path):
    cfg = u.CONFIGS["all_looped"]
    w = u.weights(cfg, seed=9)
    path, out = u.save(tmp_path / "m", cfg, w), tmp_path / "out"
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
