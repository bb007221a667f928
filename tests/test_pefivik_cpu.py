"""Pefivik through the engine on CPU tensors: reading of checkpoints, every mechanism and every
schedule of steps against the plain restatement, and that mistakes would be noticed (planted in the
restatement)."""

import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pefivik_oracle as oracle
import pefivik_util as u
from arcticinference_b200 import LLM, SamplingParams
from arcticinference_b200.config import BigramSpec, EngineArgs, LoopSpec, ModelConfig
from arcticinference_b200.engine.model_runner import pack_tokens
from arcticinference_b200.engine.request import Request
from arcticinference_b200.engine.scheduler import ScheduledRequest
from arcticinference_b200.ops import latent_ops as lat
from arcticinference_b200.ops import state_ops as states
from arcticinference_b200.ops import stream_ops as st

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, ignore_eos=True)


@pytest.fixture(scope="module", params=sorted(u.CONFIGS))
def model(request, tmp_path_factory):
    name, cfg = request.param, u.CONFIGS[request.param]
    out = {}
    for dtype in ("float32", "bfloat16"):
        w = u.weights(cfg, seed=3, peak=u.peak(name, dtype))
        out[dtype] = (cfg, w, u.save(tmp_path_factory.mktemp(name + dtype), cfg, w))
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_schedules(model, dtype):
    cfg, w, path = model[dtype]
    u.check_schedules(cfg, path, dtype, "cpu", w)


def test_residual_stream_after_every_run(model):
    cfg, w, path = model["float32"]
    toks, want, got = u.tokens(cfg, 50, 8), [], []
    oracle.forward(cfg, w, toks, want)
    sess = u.session(path, "float32", 128, "cpu")
    forward = sess.engine.runner.model.forward
    sess.engine.runner.model.forward = lambda b, kv: forward(b, kv, layers_out=got)
    sess.step([{"id": "a", "tokens": toks, "want": [0]}], ["a"])
    assert len(got) == len(want) == len(oracle.order_of_runs(cfg))
    for a, b in zip(got, want):
        assert float((a.double() - b).abs().max()) < 1e-4 * float(b.abs().max())


def greedy_gaps(cfg, w, prompt, generated):
    """How far each generated token's logit lies below the largest one."""
    seq = list(prompt) + generated
    z = oracle.forward(cfg, w, seq[:-1])[len(prompt) - 1:]
    return z.max(-1).values - z.gather(1, torch.tensor(generated).unsqueeze(1)).squeeze(1)


@pytest.mark.parametrize("ahead", [True, False])
def test_greedy_generation_through_the_scheduler(model, ahead):
    """Chunked prompts, decode steps queued ahead of their tokens (whose previous tokens are known
    all the same), requests that finish at different times."""
    cfg, w, path = model["float32"]
    llm = LLM(model=path, device="cpu", dtype="float32", num_gpu_blocks_override=40, block_size=16,
              max_model_len=256, max_num_batched_tokens=32, async_scheduling=ahead)
    prompts = [u.tokens(cfg, n, 10 + n) for n in (40, 3, 17, 1)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        [SamplingParams(max_tokens=n, **GREEDY) for n in (9, 12, 5, 9)])
    for p, n, ro in zip(prompts, (9, 12, 5, 9), outs):
        toks = ro.outputs[0].token_ids
        assert len(toks) == n and float(greedy_gaps(cfg, w, p, toks).max()) < 1e-3


def test_preemption_recomputes_states(tmp_path):
    cfg = u.CONFIGS["mixed"]
    path = u.save(tmp_path, cfg, u.weights(cfg, seed=5))
    sp = SamplingParams(max_tokens=12, **GREEDY)
    prompts = [u.tokens(cfg, 70, 1)[:48] + u.tokens(cfg, n, n) for n in (1, 9, 20)]
    kw = dict(model=path, device="cpu", dtype="float32", block_size=16, max_model_len=128)
    roomy = LLM(num_gpu_blocks_override=64, **kw)
    alone = [roomy.generate({"prompt_token_ids": p}, sp)[0] for p in prompts]
    assert all(r.num_cached_tokens == 0 for r in alone)
    for more in (dict(num_gpu_blocks_override=12), dict(num_gpu_blocks_override=64, max_num_seqs=2),
                 dict(num_gpu_blocks_override=12, async_scheduling=False)):
        llm = LLM(**kw, **more)
        for a, b in zip(alone, llm.generate([{"prompt_token_ids": p} for p in prompts], sp)):
            assert a.outputs[0].token_ids == b.outputs[0].token_ids
        kv = llm.engine.kv_manager
        assert len(kv.states.free) == kv.states.num_slots - 1


def test_cached_prefixes_without_states(tmp_path):
    """Without recurrent layers prompts share cached blocks; the first token behind them still knows
    the one before it."""
    cfg = u.CONFIGS["wide_latents"]
    w = u.weights(cfg, seed=5)
    path = u.save(tmp_path, cfg, w)
    sp = SamplingParams(max_tokens=6, **GREEDY)
    head = u.tokens(cfg, 32, 1)
    prompts = [head + u.tokens(cfg, n, n) for n in (1, 9, 20)]
    kw = dict(model=path, device="cpu", dtype="float32", block_size=16, max_model_len=128,
              num_gpu_blocks_override=64)
    cold = [LLM(enable_prefix_caching=False, **kw).generate({"prompt_token_ids": p}, sp)[0] for p in prompts]
    llm = LLM(**kw)
    warm = [llm.generate({"prompt_token_ids": p}, sp)[0] for p in prompts]
    assert [r.num_cached_tokens for r in warm] == [0, 32, 32]
    for a, b, p in zip(cold, warm, prompts):
        assert a.outputs[0].token_ids == b.outputs[0].token_ids
        assert float(greedy_gaps(cfg, w, p, b.outputs[0].token_ids).max()) < 1e-3


def test_drafts_know_the_tokens_before_them(tmp_path):
    """Suffix speculation (models without recurrent layers) changes no token."""
    cfg = u.CONFIGS["wide_latents"]
    path = u.save(tmp_path, cfg, u.weights(cfg, seed=5))
    sp = SamplingParams(max_tokens=24, **GREEDY)
    prompt = {"prompt_token_ids": u.tokens(cfg, 12, 1) * 3}
    kw = dict(model=path, device="cpu", dtype="float32", block_size=16, max_model_len=128,
              num_gpu_blocks_override=32)
    want = LLM(**kw).generate(prompt, sp)[0].outputs[0].token_ids
    llm = LLM(speculative_config={"method": "suffix", "num_speculative_tokens": 4}, **kw)
    assert llm.generate(prompt, sp)[0].outputs[0].token_ids == want
    assert llm.engine.get_stats()["draft_tokens"] > 0


def test_every_run_has_its_own_cache_and_state(tmp_path):
    cfg = u.CONFIGS["mixed"]
    sess = u.session(u.save(tmp_path, cfg, u.weights(cfg)), "float32", 256, "cpu")
    kv, m = sess.engine.runner.kv, sess.engine.runner.model
    assert m.runs == [(0, None)] + [(1, 0), (2, None), (3, None)] + [(1, 1), (2, None), (3, None)] + \
        [(1, 2), (2, None), (3, None)] + [(4, None)]
    assert [len(t) for t in kv.runs] == [1] + [0, 1, 0] * 3 + [1]
    assert [len(t) for t in kv.states] == [0] + [1, 0, 1] * 3 + [0]
    every = [t.data_ptr() for run in kv.runs + kv.states for t in run]
    assert len(set(every)) == len(every)
    assert m.state_bytes_per_slot() == 3 * 4 * (3 * 40 * 24 + 6 * 24 * 56)
    assert m.kv_bytes_per_block(64) == (56 + 3 * 72 + 72) * 64 * 4


# ---------------------------------------------------------------- mechanisms by themselves
def step_of(table):
    return states.StateStep.build(np.asarray(table, dtype=np.int32), "cpu")


def forget_case(H, d, dv, T, seed=0, gap=0):
    """(shape, projection, weights): parts of the projection ``gap`` columns apart."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    nk, nv = H * d, H * dv
    s = states.ForgetShape(H, d, dv, 0, nk + gap, 2 * (nk + gap))
    w = dict(f_bias=torch.rand(nk, generator=g) * 10 - 4, lower=torch.rand(nk, generator=g) * 0.9,
             norm=rnd(dv))
    w["lower"][::3] = 0.0
    return s, rnd(T, 2 * (nk + gap) + nv), w


def forget_want(s, proj, w, eps):
    """One whole sequence by the restatement."""
    H, d, dv, p = s.heads, s.dim, s.vdim, oracle.f64(proj)
    q = oracle.silu(p[:, s.q_at:s.q_at + H * d])
    f = oracle.forget_gates(p[:, s.f_at:s.f_at + H * d] + oracle.f64(w["f_bias"]), w["lower"])
    v = p[:, s.v_at:s.v_at + H * dv]
    return torch.cat([oracle.rms(oracle.hgrn2_scan(
        q[:, a * d:(a + 1) * d], f[:, a * d:(a + 1) * d], v[:, a * dv:(a + 1) * dv]), eps) *
        oracle.f64(w["norm"]) for a in range(H)], 1)


@pytest.mark.parametrize("H,d,dv", [(3, 6, 5), (1, 1, 1), (2, 16, 12)])
def test_forget_scan(H, d, dv):
    s, proj, w = forget_case(H, d, dv, 31, seed=d, gap=2)
    want = forget_want(s, proj, w, 0.01)
    for cuts in ([31], [1] * 31, [2, 1, 17, 2, 9]):
        state = torch.full((3, H, d, s.state_cols), 9.0)
        at, phase, got = 0, 0, []
        for n in cuts:
            got.append(states.forget_scan(proj[at:at + n], *w.values(), s, state,
                                          step_of([(0, n, 2, at, phase)]), 0.01))
            at, phase = at + n, phase ^ 1
        assert float((torch.cat(got) - want).abs().max()) < 1e-4 * float(want.abs().max())
        assert bool((state[1] == 9).all())
    out = states.forget_scan(proj[:5], *w.values(), s, state, step_of([(0, 2, 1, 0, 0), (2, 3, 0, 0, 0)]),
                             0.01)
    assert float(out[2:].abs().max()) == 0 and bool((state[0] == 9).all())


def test_latent_attention_with_sink_and_gate():
    H, R, n, kl = 3, 8, 4, 21
    shape = lat.LatentShape.of(H, R, torch.float32)
    cache, bt = torch.randn(3, 1, 16, R), torch.tensor([[2, 1]], dtype=torch.int32)
    q, gate, sink = torch.randn(n, H * R), torch.randn(n, H), torch.tensor([-30.0, 1.0, 6.0])
    meta = lat.build_plan(shape, [n], [kl], bt, 16, "cpu")
    got = lat.latent_attention(q, cache, meta, shape, 0.3, sink=sink, gate=gate).view(n, H, R)
    c = torch.cat([cache[2, 0], cache[1, 0]])[:kl].double()
    for h in range(H):
        s = torch.full((kl, kl), -1e9, dtype=torch.float64)
        s[kl - n:] = q.view(n, H, R)[:, h].double() @ c.t() * 0.3
        want = oracle.weights_of(s, float(sink[h]))[kl - n:] @ c * oracle.sigmoid(gate[:, h:h + 1].double())
        assert float((got[:, h] - want).abs().max()) < 1e-5


@pytest.mark.parametrize("experts,top,count,keep", [(12, 3, 4, 2), (6, 2, 3, 1), (5, 2, 5, 3), (8, 8, 2, 2),
                                                    (4, 1, 1, 1)])
def test_grouped_router(experts, top, count, keep):
    g = torch.Generator().manual_seed(top)
    x, w = torch.randn(60, 24, generator=g), torch.randn(experts, 24, generator=g) * 0.4
    r, rows = st.route(x, x, w, None, top, 0, 1.3, (count, keep))
    ids, weights, lead = oracle.route(x.double(), w, {"top": top, "scale": 1.3,
                                                      "groups": {"count": count, "keep": keep}})
    sure = lead > 1e-5
    assert bool(sure.sum() > 50) and torch.equal(r.ids.long()[sure], ids[sure])
    assert float((r.weights - weights)[sure].abs().max()) < 1e-5
    assert torch.equal(rows[r.rows.flatten().long()], x.repeat_interleave(top, 0))


def test_stream_pre():
    f = lambda t: t.double()
    x0, y, y2, base = (torch.randn(6, 33) for _ in range(4))
    bias, step, gain, vec = torch.randn(33), torch.randn(33), torch.tensor([0.8]), torch.randn(33)
    rows = torch.tensor([[0, 1], [5, 2], [3, 3], [1, 3], [4, 4], [2, 0]], dtype=torch.int32)
    r = st.Routing(rows, torch.rand(6, 2), rows, 2, 6)
    mix = sum(f(r.weights[:, j:j + 1]) * f(y)[rows[:, j].long()] for j in range(2)) + f(y2)
    for kw, out in (({}, torch.zeros(6, 33)), (dict(y=y), f(y)), (dict(y=y, bias=bias), f(y) + f(bias)),
                    (dict(y=y, experts=r, shared=y2), mix)):
        for more in ({}, dict(base=base, step=step), dict(step=step)):
            for w in (gain, vec):
                x, act = x0.clone(), torch.empty(6, 33)
                st.stream_pre(x, 0.3, 0.02, w_in=w, act=act, **kw, **more)
                want = oracle.residual(f(x0), out, 0.3) + sum(f(t) for t in more.values())
                assert float((x - want).abs().max()) < 1e-5
                assert float((act - oracle.stream_norm(want, w, 0.02)).abs().max()) < 1e-5


def test_poly_norm_and_soft_cap():
    z, bias, coef = torch.randn(5, 24) * 3, torch.randn(24), torch.tensor([0.6, -0.5, 0.4, 0.3])
    got = st.poly_norm(z, bias, coef, 21, 0.02)
    want = oracle.poly_norm(z[:, :21].double() + bias[:21].double(), coef, 0.02)
    assert float((got[:, :21] - want).abs().max()) < 1e-5 and float(got[:, 21:].abs().max()) == 0
    cap = st.soft_cap(torch.tensor([[1.0, -50.0, 0.0]]), 4.0)
    assert cap.dtype == torch.float32
    assert torch.allclose(cap, torch.tensor([[4 * math.tanh(0.25), -4.0, 0.0]]))


def test_pairs_of_tokens():
    spec, table, second = BigramSpec(7, 5, 3), torch.randn(10, 6), torch.randn(8, 6)
    toks = [3, 9, 0, 0, 4]
    ids, prev = torch.tensor(toks), torch.tensor([-1] + toks[:-1])
    keep = torch.empty(5, 6)
    x, _ = st.stream_embedding(ids, table, rounded=False, pairs=(prev, second, spec), keep=keep)
    rows = oracle.bigram_rows(toks, {"buckets": 7, "mul_prev": 5, "mul_cur": 3})
    assert rows == [7, (15 + 27) % 7, 45 % 7, 0, 12 % 7]
    assert torch.equal(x, table[ids] + second[rows]) and torch.equal(x, keep)


def test_previous_tokens_of_a_batch():
    def request(prompt, out, spec=()):
        r = Request("r", prompt, SamplingParams())
        r.output_token_ids, r.spec_token_ids, r.block_ids = out, list(spec), [1, 2]
        return r
    sched = [ScheduledRequest(request([5, 6, 7], []), 0, 3, 0, True),
             ScheduledRequest(request([5, 6, 7], []), 2, 1, 0, True),
             ScheduledRequest(request([4], []), 0, 1, 0, True),
             ScheduledRequest(request([1, 2], [3, -1]), 3, 1, 0, True),     # newest one not read yet
             ScheduledRequest(request([1, 2], [8], (9, 3)), 2, 3, 2, True),
             ScheduledRequest(request(list(range(20)), []), 17, 2, 0, False)]
    n = sum(s.num_tokens for s in sched)
    ids, pos, slots, prev = (np.zeros(n, np.int64) for _ in range(4))
    pack_tokens(sched, 16, ids, pos, slots, np.zeros((len(sched), 2), np.int32), prev)
    assert ids.tolist() == [5, 6, 7, 7, 4, -1, 8, 9, 3, 17, 18]
    assert prev.tolist() == [-1, 5, 6, 6, -1, 3, 2, 8, 9, 16, 17]


# ---------------------------------------------------------------- mistakes planted in the oracle
def _logits(cfg, w, toks, **patch):
    saved = {k: getattr(oracle, k) for k in patch}
    mixers = dict(oracle.MIXERS)
    try:
        for k, v in patch.items():
            setattr(oracle, k, v)
        return oracle.forward(cfg, w, toks)
    finally:
        for k, v in saved.items():
            setattr(oracle, k, v)
        oracle.MIXERS.update(mixers)


def test_planted_mistakes_show(tmp_path):
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg, seed=3, peak=3.0)
    toks = u.tokens(cfg, 150, 7)
    sess = u.session(u.save(tmp_path, cfg, w), "float32", 256, "cpu")
    got = u.run(sess, {"a": toks}, [[("a", n)] for n in u.portions(150, [64, 2, 31, 1])])["a"]
    tol = u.TOLERANCE["float32"]
    assert u.error(got, oracle.forward(cfg, w, toks)) < tol

    _rows, _weights, _gates, _forget, _scan, _route, _poly, _enter, _rms = (
        oracle.bigram_rows, oracle.weights_of, oracle.head_gates, oracle.forget_gates,
        oracle.hgrn2_scan, oracle.route, oracle.poly_norm, oracle.enter_pass, oracle.rms)

    def cut_rows(t, b):        # the token before a portion forgotten
        return _rows(t[:64], b) + _rows(t[64:], b)

    def pieces(q, f, v):       # a state that is lost after 64 tokens
        return torch.cat([_scan(q[i:i + 64], f[i:i + 64], v[i:i + 64]) for i in range(0, q.shape[0], 64)])

    def late_read(q, f, v):
        return torch.cat([torch.zeros_like(v[:1]), _scan(q, f, v)[:-1]])

    def no_groups(h, wr, r):
        return _route(h, wr, {**r, "groups": {"count": 1, "keep": 1}})

    def best_of_group(h, wr, r):      # groups scored by their best expert alone
        s = oracle.sigmoid(oracle.apply(wr, h))
        n, c = s.shape[0], r["groups"]["count"]
        kept = s.view(n, c, -1).max(-1).values.topk(r["groups"]["keep"]).indices
        open_ = torch.zeros(n, c, dtype=torch.bool).scatter_(1, kept, True)
        s = s.masked_fill(~open_.repeat_interleave(s.shape[1] // c, 1), -1.0)
        top = s.topk(r["top"])
        return top.indices, top.values / top.values.sum(-1, keepdim=True) * r["scale"], None

    def unnormalised(h, wr, r):
        i, v, lead = _route(h, wr, r)
        return i, oracle.sigmoid(oracle.apply(wr, h)).gather(1, i) * r["scale"], lead

    def softmax_weights(h, wr, r):
        i, v, lead = _route(h, wr, r)
        return i, oracle.apply(wr, h).gather(1, i).softmax(-1) * r["scale"], lead

    def powers_of_norm(z, act, eps):
        a, b, c, e = (float(x) for x in act)
        n = _rms(z, eps)
        return a * n + b * n ** 2 + c * n ** 3 + e

    for patch in (
            {"bigram_rows": lambda t, b: _rows(t, {**b, "mul_prev": b["mul_cur"], "mul_cur": b["mul_prev"]})},
            {"bigram_rows": lambda t, b: [0] + _rows(t, b)[1:]}, {"bigram_rows": cut_rows},
            {"enter_pass": lambda x, x0, s, t: _enter(x, 0 * x0, s, t)},
            {"enter_pass": lambda x, x0, s, t: _enter(x, x0, s, t) + (x0 if t == 0 else 0)},
            {"enter_pass": lambda x, x0, s, t: _enter(x, x0, s.flip(0), t)},
            {"enter_pass": lambda x, x0, s, t: _enter(x, x0, 0 * s, t)},
            {"stream_norm": lambda x, g, e: _rms(x, e)},
            {"residual": lambda x, y, m: x + y}, {"residual": lambda x, y, m: m * x + y},
            {"sees": lambda i, j: j < i or i == 0}, {"sees": lambda i, j: j <= i and i - j < 64},
            {"sees": lambda i, j: 0 < j <= i or i == j},
            {"weights_of": lambda s, k: _weights(s, -1e9)},
            {"weights_of": lambda s, k: _weights(s, k * 0.3)},
            {"weights_of": lambda s, k: _weights(s, k + math.log(2.0))},
            {"head_gates": lambda h, w, p: torch.ones_like(_gates(h, w, p))},
            {"head_gates": lambda h, w, p: _gates(h, w, p).roll(1, -1)},
            {"latent": lambda h, w, p, e: oracle.rms(oracle.apply(w[p + "dkv"], h), e)},
            {"forget_gates": lambda z, l: _forget(z, 0 * l)},
            {"forget_gates": lambda z, l: torch.maximum(oracle.sigmoid(z), oracle.f64(l).expand_as(z))},
            {"hgrn2_scan": pieces}, {"hgrn2_scan": late_read},
            {"hgrn2_scan": lambda q, f, v: _scan(q, f, v) * q.shape[1] ** -0.5},
            {"silu": lambda z: z},
            {"poly_norm": powers_of_norm},
            {"poly_norm": lambda z, a, e: _poly(z, a * torch.tensor([1, 1, 1, 0]), e)},
            {"poly_norm": lambda z, a, e: _poly(z, a[[0, 2, 1, 3]], e)},
            {"route": no_groups}, {"route": best_of_group}, {"route": unnormalised},
            {"route": softmax_weights},
            {"rms": lambda x, e: x / (torch.sqrt((x * x).mean(-1, keepdim=True)) + e)}):
        assert u.error(got, _logits(cfg, w, toks, **patch)) > 10 * tol, list(patch)
    router = lambda c, i: c["layers"][i]["mlp"]["router"]
    for change in (lambda c: c["norm"].update(eps=0.011), lambda c: c.update(residual_mult=0.41),
                   lambda c: c.update(logit_softcap=3.1), lambda c: c["loop"].update(stop=3),
                   lambda c: c["loop"].update(times=2),
                   lambda c: c["embedding"]["bigram"].update(mul_cur=11),
                   lambda c: c["layers"][0]["mixer"].update(scale=0.31),
                   lambda c: router(c, 0).update(scale=1.6), lambda c: router(c, 0).update(top=2),
                   lambda c: router(c, 3).update(groups={"count": 3, "keep": 2}),
                   lambda c: c["layers"][0]["mlp"].update(shared=None), lambda c: c["layers"].pop()):
        other = copy.deepcopy(cfg)
        change(other)
        assert u.error(got, oracle.forward(other, w, toks)) > 5 * tol
    for name in ("l1.mlp.up.b", "l1.mlp.down.b", "l0.mix.dkv.norm", "l1.mix.norm", "l3.mix.f.b"):
        assert u.error(got, oracle.forward(cfg, {**w, name: w[name] * 0}, toks)) > 10 * tol, name


# ---------------------------------------------------------------- configuration and loading
def test_config_is_read_from_the_checkpoint(tmp_path):
    cfg = u.CONFIGS["mixed"]
    m = ModelConfig.from_pretrained(u.save(tmp_path, cfg, u.weights(cfg)))
    assert m.architecture == "Pefivik" and m.hidden_size == 160 and m.vocab_size == 211
    assert m.rms_norm_eps == 0.01 and not m.tie_word_embeddings and m.has_state
    assert m.bigram == BigramSpec(97, 5, 12) and m.loop == LoopSpec(1, 4, 3, True)
    assert (m.residual_mult, m.logit_softcap) == (0.4, 3.0)
    a, b = (m.layer_specs[i].mixer for i in (0, 1))
    assert (a.heads, a.dim, a.vdim, a.kv_rank, a.scale, a.sink, a.head_gate) == \
        (6, 24, 40, 56, 0.3, "learned", True)
    assert (b.heads, b.dim, b.vdim) == (3, 40, 24)
    f, g = (m.layer_specs[i].mlp for i in (0, 1))
    assert (f.ff, f.act, f.experts, f.top, f.router_scale, f.scoring, f.groups, f.keep_groups) == \
        (40, "silu", 12, 3, 1.7, "sigmoid", 4, 2)
    assert f.shared.ff == 72 and (g.ff, g.act, g.experts) == (136, "poly_norm", 0)
    assert m.layer_specs[2].mlp is None
    from arcticinference_b200.plugin import supported_architectures
    assert "Pefivik" in supported_architectures()
    e = EngineArgs(model=str(tmp_path)).create_engine_config()
    assert not e.cache.enable_prefix_caching
    other = u.CONFIGS["wide_latents"]
    e = EngineArgs(model=u.save(tmp_path / "b", other, u.weights(other))).create_engine_config()
    assert e.cache.enable_prefix_caching and not e.model.has_state


def test_refused_configurations(tmp_path):
    def broken(change, **kw):
        c = copy.deepcopy(u.CONFIGS["mixed"])
        change(c)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return EngineArgs(model=str(tmp_path), **kw).create_engine_config()

    layer = lambda c, i: c["layers"][i]
    for change in (lambda c: layer(c, 0).update(type="other"),
                   lambda c: layer(c, 0)["mlp"].update(kind="other")):
        with pytest.raises(NotImplementedError):
            broken(change)
    router = lambda c: layer(c, 0)["mlp"]["router"]
    for change in (lambda c: layer(c, 1)["mixer"].update(dim=0),
                   lambda c: layer(c, 0)["mixer"].update(kv_rank=0),
                   lambda c: layer(c, 1)["mlp"].update(ff=0),
                   lambda c: router(c).update(groups={"count": 5, "keep": 2}),
                   lambda c: router(c).update(groups={"count": 4, "keep": 5}),
                   lambda c: router(c).update(groups={"count": 4, "keep": 0}),
                   lambda c: router(c).update(top=7),
                   lambda c: c["loop"].update(stop=6), lambda c: c["loop"].update(times=0),
                   lambda c: c["embedding"]["bigram"].update(buckets=0),
                   lambda c: c.update(logit_softcap=-1.0)):
        with pytest.raises(ValueError):
            broken(change)
    for kw in ({"tensor_parallel_size": 2}, {"quantization": "fp8"}, {"dtype": "float16"},
               {"speculative_config": {"method": "suffix"}}):
        with pytest.raises(NotImplementedError):
            broken(lambda c: None, **kw)


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg)
    for name in ("bigram", "loop.step", "l0.mix.sink", "l0.mix.g", "l1.mix.lower", "l1.mix.f.b",
                 "l1.mlp.act", "l1.mlp.down.b", "l0.mlp.shared.up", "head"):
        missing = {k: v for k, v in w.items() if k != name}
        with pytest.raises(ValueError, match=name):
            u.session(u.save(tmp_path / "a", cfg, missing), "float32", 64, "cpu")
    for name in ("l2.norm2", "l0.norm1b", "l1.mlp.gate", "l0.mlp.router.b", "l1.mix.g"):
        with pytest.raises(ValueError, match="unexpected"):
            u.session(u.save(tmp_path / "b", cfg, {**w, name: w["l0.norm1"]}), "float32", 64, "cpu")
    for name in ("l0.norm1", "bigram", "l0.mix.sink"):
        with pytest.raises(ValueError, match="shape"):
            u.session(u.save(tmp_path / "c", cfg, {**w, name: w["l1.mix.norm"]}), "float32", 64, "cpu")


def test_preset_generates():
    llm = LLM(model="pefivik-tiny", device="cpu", num_gpu_blocks_override=16, max_model_len=256,
              max_num_seqs=4)
    out = llm.generate([{"prompt_token_ids": [5, 6, 7, 8]}], SamplingParams(max_tokens=4, **GREEDY))
    assert len(out[0].outputs[0].token_ids) == 4


# ---------------------------------------------------------------- the trace runner as a program
def test_trace_run_program(tmp_path):
    cfg = u.CONFIGS["ones"]
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
