"""Pererax through the engine on CPU tensors: reading of checkpoints, every mechanism and every
schedule of steps against the plain restatement, state slots, and that mistakes would be noticed
(planted in the restatement)."""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pererax_oracle as oracle
import pererax_util as u
from arcticinference_b200 import LLM, SamplingParams
from arcticinference_b200.config import EngineArgs, MaskSpec, ModelConfig
from arcticinference_b200.engine.kv_cache import KVCacheManager
from arcticinference_b200.engine.request import Request
from arcticinference_b200.ops import head_ops as hd
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
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert float((a.double() - b).abs().max()) < 1e-4 * float(b.abs().max())


def greedy_gaps(cfg, w, prompt, generated):
    """How far each generated token's logit lies below the largest one."""
    seq = list(prompt) + generated
    z = oracle.forward(cfg, w, seq[:-1])[len(prompt) - 1:]
    return z.max(-1).values - z.gather(1, torch.tensor(generated).unsqueeze(1)).squeeze(1)


def test_greedy_generation_through_the_scheduler(model):
    cfg, w, path = model["float32"]
    llm = LLM(model=path, device="cpu", dtype="float32", num_gpu_blocks_override=40, block_size=16,
              max_model_len=256, max_num_batched_tokens=32)
    prompts = [u.tokens(cfg, n, 10 + n) for n in (40, 3, 17)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(max_tokens=9, **GREEDY))
    for p, ro in zip(prompts, outs):
        toks = ro.outputs[0].token_ids
        assert len(toks) == 9 and float(greedy_gaps(cfg, w, p, toks).max()) < 1e-3


def test_preemption_recomputes_states(tmp_path):
    """Requests recomputed after their pages and slots were taken generate what they generate alone,
    also from a prompt that another request began with (nothing is served from cached blocks)."""
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


def test_state_slots():
    kv = KVCacheManager(8, 16, False, num_state_slots=3)
    a, b, c = (Request(n, [1], SamplingParams()) for n in "abc")
    for r in (a, b):
        kv.allocate(r, 1)
    assert {a.state_slot, b.state_slot} == {1, 2} and not kv.can_allocate(c, 1)
    with pytest.raises(RuntimeError):
        kv.allocate(c, 1)
    kv.free(c)
    a.state_phase, gone = 1, a.state_slot
    kv.allocate(a, 30)                   # keeps its slot
    assert a.state_slot == gone
    kv.free(a)
    assert a.state_slot == 0 and kv.can_allocate(c, 1)
    kv.allocate(c, 1)
    assert c.state_slot == gone and c.state_phase == 0
    plain = KVCacheManager(8, 16, False)
    plain.allocate(a, 1)
    assert a.state_slot == 0


def test_every_run_has_its_own_cache_and_state(tmp_path):
    cfg = u.CONFIGS["mixed"]
    sess = u.session(u.save(tmp_path, cfg, u.weights(cfg)), "float32", 256, "cpu")
    kv, m = sess.engine.runner.kv, sess.engine.runner.model
    assert [l for l, _ in m.runs] == [0, 1, 2, 3, 2, 0, 1]
    assert [len(t) for t in kv.runs] == [0, 2, 2, 2, 2, 0, 2]
    assert [len(t) for t in kv.states] == [2, 2, 0, 2, 0, 2, 2]
    every = [t.data_ptr() for run in kv.runs + kv.states for t in run]
    assert len(set(every)) == len(every)
    slots = sess.engine.kv_manager.states.num_slots
    assert slots == 5 and all(t.shape[0] == slots for run in kv.states for t in run)
    assert m.state_bytes_per_slot() == sum(t[0].numel() * t.element_size()
                                           for run in kv.states for t in run)
    per_token = 2 * 2 * (40 + 24) + 2 * 2 * (32 + 32) + (64 + 48)
    assert m.kv_bytes_per_block(64) == per_token * 64 * 4
    assert [l is None for l in m.layers] == [False] * 4 + [True] * 3
    assert m.embed is m.lm_head


# ---------------------------------------------------------------- mechanisms by themselves
def step_of(table):
    return states.StateStep.build(np.asarray(table, dtype=np.int32), "cpu")


def delta_case(H, G, d, dv, taps, lens, seed=0):
    """(shape, projections, decay, gate, weights, per-sequence oracle outputs before the norm)."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    T, nk, nv = sum(lens), G * d, H * dv
    proj = rnd(T, 2 * nk + nv + H)
    s = states.DeltaShape(H, G, d, dv, taps, 0, nk, 2 * nk, 2 * nk + nv)
    w = dict(conv=rnd(taps, s.channels), a_exp=(torch.rand(H, generator=g) * 5 - 3).exp(),
             dt_bias=torch.rand(H * d, generator=g) * 6 - 5, norm=rnd(dv))
    return s, proj, rnd(T, H * d), rnd(T, nv), w


def delta_want(s, proj, decay, gate, w, eps):
    """One whole sequence by the restatement."""
    H, G, d, dv = s.heads, s.kv_heads, s.dim, s.vdim
    f = lambda t: t.detach().cpu().double()
    parts = [oracle.short_conv(f(proj)[:, a:a + n], w["conv"][:, c:c + n].t()) for a, n, c in
             ((s.q_at, G * d, 0), (s.k_at, G * d, G * d), (s.v_at, H * dv, 2 * G * d))]
    beta = oracle.sigmoid(f(proj)[:, s.b_at:s.b_at + H])
    g = oracle.decays(f(decay), w["a_exp"].log(), w["dt_bias"], H)
    out = []
    for a in range(H):
        b = a // (H // G)
        o = oracle.delta_scan(oracle.unit(parts[0][:, b * d:(b + 1) * d]) * d ** -0.5,
                              oracle.unit(parts[1][:, b * d:(b + 1) * d]),
                              parts[2][:, a * dv:(a + 1) * dv], g[:, a], beta[:, a])
        out.append(oracle.norm(o, w["norm"], eps))
    return torch.cat(out, 1) * oracle.sigmoid(f(gate))


@pytest.mark.parametrize("H,G,d,dv,taps", [(4, 2, 6, 5, 3), (1, 1, 1, 1, 1), (3, 1, 8, 12, 5)])
def test_delta_rule(H, G, d, dv, taps):
    s, proj, decay, gate, w = delta_case(H, G, d, dv, taps, [23])
    want = delta_want(s, proj, decay, gate, w, 0.01)
    for cuts in ([23], [1] * 23, [2, 1, 7, 2, 11]):
        state, conv = torch.full((3, H, d, s.state_cols), 9.0), torch.full((3, 2, taps - 1, s.channels), 9.0)
        at, phase, got = 0, 0, []
        for n in cuts:
            rows = slice(at, at + n)
            got.append(states.delta_scan(proj[rows], decay[rows], gate[rows], *w.values(), s, state,
                                         conv, step_of([(0, n, 2, at, phase)]), 0.01))
            at, phase = at + n, phase ^ 1
        assert float((torch.cat(got) - want).abs().max()) < 1e-4 * float(want.abs().max())
        assert bool((state[1] == 9).all()) and bool((conv[1] == 9).all())


@pytest.mark.parametrize("H,d,dv", [(3, 6, 5), (1, 1, 1), (2, 16, 12)])
def test_matrix_memory(H, d, dv):
    g = torch.Generator().manual_seed(d)
    rnd = lambda *s: torch.randn(*s, generator=g)
    T, nk, nv = 31, H * d, H * dv
    s = states.MemoryShape(H, d, dv, 4.0, 0, nk, 2 * nk, 2 * nk + nv, 2 * nk + nv + H)
    proj, gate, norm = rnd(T, 2 * nk + nv + 2 * H), rnd(T, nv), rnd(nv)
    ib, fb = rnd(H) * 3, rnd(H) * 3 + 2
    p = proj.double()
    i, f = oracle.memory_gates(p[:, s.i_at:s.i_at + H] + ib, p[:, s.f_at:s.f_at + H] + fb, 4.0)
    want = torch.cat([oracle.rms(oracle.memory_scan(
        p[:, a * d:(a + 1) * d] * d ** -0.5, p[:, nk + a * d:nk + (a + 1) * d],
        p[:, 2 * nk + a * dv:2 * nk + (a + 1) * dv], i[:, a], f[:, a]), 0.01) for a in range(H)], 1)
    want = want * norm.double() * oracle.sigmoid(gate.double())
    for cuts in ([31], [1] * 31, [2, 1, 17, 2, 9]):
        state, top = torch.full((2, H, d, s.state_cols), 9.0), torch.full((2, 2, H), 9.0)
        at, phase, got = 0, 0, []
        for n in cuts:
            rows = slice(at, at + n)
            got.append(states.memory_scan(proj[rows], gate[rows], ib, fb, norm, s, state, top,
                                          step_of([(0, n, 1, at, phase)]), 0.01))
            at, phase = at + n, phase ^ 1
        assert float((torch.cat(got) - want).abs().max()) < 1e-4 * float(want.abs().max())


def test_padding_rows_touch_no_state():
    s, proj, decay, gate, w = delta_case(2, 1, 4, 4, 3, [5])
    state, conv = torch.full((2, 2, 4, 4), 9.0), torch.full((2, 2, 2, s.channels), 9.0)
    out = states.delta_scan(proj, decay, gate, *w.values(), s, state, conv,
                            step_of([(0, 2, 1, 0, 0), (2, 3, 0, 0, 0)]), 0.01)
    assert float(out[2:].abs().max()) == 0 and float((state[0] - 9).abs().max()) == 0


def test_norm_over_the_projection_and_values_that_are_keys():
    H, G, d, T = 4, 2, 6, 3
    shape = hd.HeadShape.of(H, G, d, d, torch.float32, MaskSpec("window", 5))
    proj = torch.randn(T, (H + G) * d)
    raw, wq, wk = proj.clone().double(), torch.randn(H * d), torch.randn(G * d)
    k, v = torch.zeros(2, G, 16, d), torch.zeros(2, G, 16, d)
    pos, rot = torch.tensor([0, 7, 300]), {"base": 50.0, "dims": 4}
    freq = torch.tensor([1.0, 50.0 ** -0.5])
    hd.head_rope_cache(proj, shape, d, wq, wk, hd.rotary_table(pos, freq), 0.01,
                       torch.tensor([3, 20, -1]), k, v, whole=True, shared_kv=True)
    q = oracle.projection_norm(raw[:, :H * d], wq, 0.01)
    kk = oracle.projection_norm(raw[:, H * d:], wk, 0.01)
    for h in range(H):
        want = oracle.rotate(q[:, h * d:(h + 1) * d], pos, rot)
        assert float((proj[:, h * d:(h + 1) * d] - want).abs().max()) < 1e-4
    for g in range(G):
        cols = slice(g * d, (g + 1) * d)
        want = oracle.rotate(kk[:, cols], pos, rot)
        assert float((k[0, g, 3] - want[0]).abs().max()) < 1e-5
        assert float((k[1, g, 4] - want[1]).abs().max()) < 1e-5
        assert torch.equal(v[0, g, 3].double(), raw[0, H * d:][cols])
        assert torch.equal(v[1, g, 4].double(), raw[1, H * d:][cols])


@pytest.mark.parametrize("experts,identity,top", [(5, 3, 2), (4, 0, 4), (1, 6, 3), (3, 2, 5)])
def test_router_over_all_outputs(experts, identity, top):
    g = torch.Generator().manual_seed(top)
    x, w = torch.randn(40, 24, generator=g), torch.randn(experts + identity, 24, generator=g) * 0.4
    corr = torch.rand(experts + identity, generator=g)
    r, rows = st.route(x, x, w, corr, top, identity, 1.3)
    ids, weights, lead = oracle.route(x.double(), w, corr, top, 1.3)
    sure = lead > 1e-5
    assert bool(sure.sum() > 30) and torch.equal(r.ids.long()[sure], ids[sure])
    assert float((r.weights - weights)[sure].abs().max()) < 1e-5
    assert rows.shape[0] == int((r.ids < experts).sum())
    for t in range(40):
        for j in range(top):
            k = int(r.rows[t, j])
            assert (k < 0) == (int(r.ids[t, j]) >= experts)
            if k >= 0:
                assert torch.equal(rows[k], x[t])


def test_stream_add():
    x0, y, y2, w, w1, w2 = (torch.randn(*s) for s in ((6, 33), (6, 33), (6, 33), (33,), (33,), (33,)))
    f = lambda t: t.double()
    x, act = x0.clone(), torch.empty(6, 33)
    st.stream_add(x, act, w, 0.02, y)
    want = f(x0) + oracle.norm(f(y), w, 0.02)
    assert float((x - want).abs().max()) < 1e-5 and torch.equal(act, x)
    x = x0.clone()
    st.stream_add(x, x, w, 0.02, y, pair=(y2, w1, w2))
    both = 0.5 * (oracle.norm(f(y), w1, 0.02) + oracle.norm(f(y2), w2, 0.02))
    assert float((x - f(x0) - oracle.norm(both, w, 0.02)).abs().max()) < 1e-5
    rows = torch.tensor([[0, -1], [5, 2], [-1, -1], [1, 3], [4, 4], [2, -1]], dtype=torch.int32)
    r = st.Routing(rows.clamp(min=0), torch.rand(6, 2), rows, 2, 6)
    for shared in (None, y2):
        x = x0.clone()
        st.stream_add(x, x, w, 0.02, y, experts=r, shared=shared)
        s = torch.zeros(6, 33, dtype=torch.float64) if shared is None else f(shared)
        s = s + sum(f(r.weights[:, j:j + 1]) * torch.where(rows[:, j:j + 1] < 0, f(x0), f(y)[rows[:, j].long()])
                    for j in range(2))
        assert float((x - f(x0) - oracle.norm(s, w, 0.02)).abs().max()) < 1e-5


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
    w = u.weights(cfg, seed=3, peak=1.5)
    toks = u.tokens(cfg, 150, 7)
    sess = u.session(u.save(tmp_path, cfg, w), "float32", 256, "cpu")
    got = u.run(sess, {"a": toks}, [[("a", n)] for n in u.portions(150, [64, 2, 31, 1])])["a"]
    tol = u.TOLERANCE["float32"]
    assert u.error(got, oracle.forward(cfg, w, toks)) < tol

    _weights_of, _rotate, _sees, _conv, _delta, _memory, _gates, _route, _decays = (
        oracle.weights_of, oracle.rotate, oracle.sees, oracle.short_conv, oracle.delta_scan,
        oracle.memory_scan, oracle.memory_gates, oracle.route, oracle.decays)

    def per_head_norm(x, weight, eps):
        n = x.shape[1] // 8
        return (oracle.rms(x.reshape(x.shape[0], n, 8), eps)).reshape(x.shape) * oracle.f64(weight)

    def pieces(scan, n):      # a state that is lost after n tokens
        return lambda *a: torch.cat([scan(*(t[i:i + n] for t in a)) for i in range(0, a[0].shape[0], n)])

    def conv_cut(x, taps):    # inputs of an earlier portion forgotten
        return torch.cat([_conv(x[:64], taps), _conv(x[64:], taps)])

    def late_read(q, k, v, g, beta):
        return torch.cat([torch.zeros_like(v[:1]), _delta(q, k, v, g, beta)[:-1]])

    def swapped_route(h, wr, c, top, scale):
        z = oracle.apply(wr, h)
        i = z.argsort(-1, descending=True)[:, :top]
        return i, z.softmax(-1).gather(1, i) * scale, None

    def weighted_with_correction(h, wr, c, top, scale):
        i, s, lead = _route(h, wr, c, top, scale)
        return i, s + oracle.f64(c)[i] * scale, lead

    def renormalised(h, wr, c, top, scale):
        i, s, lead = _route(h, wr, c, top, scale)
        return i, s / s.sum(-1, keepdim=True) * scale, lead

    ident = lambda x, *a: x
    for patch in (
            {"rotate": ident}, {"rotate": lambda x, p, r: _rotate(x, -p, r)},
            {"projection_norm": per_head_norm}, {"projection_norm": lambda x, w, e: oracle.rms(x, e)},
            {"weights_of": lambda s, m, sink: _weights_of(s, m, False)},
            {"weights_of": lambda s, m, sink: _weights_of(s, m, True)},
            {"sees": lambda i, j, n: _sees(i, j, n and n + 1)},
            {"sees": lambda i, j, n: _sees(i, j, n and n - 1)}, {"sees": lambda i, j, n: j <= i},
            {"capped": ident},
            {"short_conv": lambda x, t: _conv(x, t.flip(1))}, {"short_conv": conv_cut},
            {"unit": ident}, {"delta_scan": pieces(_delta, 64)}, {"delta_scan": late_read},
            {"decays": lambda z, a, b, h: _decays(z, a, b, h).mean(-1, keepdim=True).expand(
                -1, -1, z.shape[1] // h)},
            {"softplus": lambda z: torch.clamp(z, min=0.0)},
            {"memory_scan": pieces(_memory, 64)},
            {"memory_gates": lambda i, f, c: (_gates(i, f, 1e6)[0], _gates(i, f, c)[1])},
            {"memory_gates": lambda i, f, c: (_gates(i, f, c)[0], _gates(i, f, 1e6)[1])},
            {"route": swapped_route}, {"route": weighted_with_correction}, {"route": renormalised},
            {"clamped_swish": lambda g, x, n: g * oracle.sigmoid(1.702 * g) * (x + 1)},
            {"clamped_swish": lambda g, x, n: g.clamp(max=n) * oracle.sigmoid(g.clamp(max=n)) *
             (x.clamp(-n, n) + 1)},
            {"residual": lambda x, y, n, s, e: x + oracle.norm(y, n, e)},
            {"residual": lambda x, y, n, s, e: x + y * oracle.f64(s)},
            {"rms": lambda x, e: x / (torch.sqrt((x * x).mean(-1, keepdim=True)) + e)}):
        oracle.visible.cache_clear()
        assert u.error(got, _logits(cfg, w, toks, **patch)) > 10 * tol, list(patch)
    oracle.visible.cache_clear()
    right = lambda c, i: c["layers"][i]["mixer"]["right"]
    left = lambda c, i: c["layers"][i]["mixer"]["left"]
    for change in (lambda c: c["norm"].update(eps=0.02), lambda c: left(c, 1).update(scale=0.33),
                   lambda c: left(c, 3).update(softcap=14.0), lambda c: right(c, 3).update(gate_cap=11.0),
                   lambda c: left(c, 1)["rot"].update(base=400.0),
                   lambda c: c["layers"][2]["mixer"].update(scale=0.2),
                   lambda c: c["layers"][0]["mlp"]["router"].update(scale=1.6),
                   lambda c: c["layers"][0]["mlp"].update(shared=None),
                   lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.5),
                   lambda c: c["layers"][2]["mlp"]["expert"].update(limit=1.5),
                   lambda c: c["layers"].pop()):
        other = copy.deepcopy(cfg)
        change(other)
        assert u.error(got, oracle.forward(other, w, toks)) > 2 * tol


# ---------------------------------------------------------------- configuration and loading
def test_config_is_read_from_the_checkpoint(tmp_path):
    cfg = u.CONFIGS["mixed"]
    m = ModelConfig.from_pretrained(u.save(tmp_path, cfg, u.weights(cfg)))
    assert m.architecture == "Pererax" and m.hidden_size == 160 and m.vocab_size == 211
    assert m.rms_norm_eps == 0.01 and m.tie_word_embeddings and m.has_state
    a, b, c = (m.layer_specs[i].mixer for i in (0, 1, 2))
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.conv) == (6, 2, 40, 24, 3)
    assert b.left.softcap == 4.0 and b.left.sink == "zero" and not b.left.values_are_keys
    assert (b.right.heads, b.right.dim, b.right.vdim, b.right.gate_cap) == (3, 24, 56, 5.0)
    assert c.mask == MaskSpec("window", 37) and c.values_are_keys and c.sink is None
    assert b.left.qk_norm == c.qk_norm == "projection"
    f = m.layer_specs[0].mlp
    assert (f.ff, f.experts, f.identity, f.top, f.limit, f.router_scale) == (40, 5, 2, 3, 1.5, 1.7)
    assert (f.shared.ff, f.shared.limit) == (72, 0.9) and m.layer_specs[1].mlp is None
    assert [l for l, _ in m.layer_runs] == [0, 1, 2, 3, 2, 0, 1]
    from arcticinference_b200.plugin import supported_architectures
    assert "Pererax" in supported_architectures()
    e = EngineArgs(model=str(tmp_path)).create_engine_config()
    assert not e.cache.enable_prefix_caching


def test_refused_configurations(tmp_path):
    def broken(change, **kw):
        c = copy.deepcopy(u.CONFIGS["mixed"])
        change(c)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return EngineArgs(model=str(tmp_path), **kw).create_engine_config()

    layer = lambda c, i: c["layers"][i]
    for change in (lambda c: layer(c, 0).update(type="other"),
                   lambda c: layer(c, 0)["mlp"].update(kind="dense")):
        with pytest.raises(NotImplementedError):
            broken(change)
    for change in (lambda c: layer(c, 0)["mixer"].update(kv_heads=4),
                   lambda c: layer(c, 0)["mixer"].update(conv=0),
                   lambda c: layer(c, 2)["mixer"]["mask"].update(size=0),
                   lambda c: layer(c, 2)["mixer"]["rot"].update(dims=34),
                   lambda c: layer(c, 1)["mixer"]["right"].update(gate_cap=0.0),
                   lambda c: layer(c, 0)["mlp"]["router"].update(top=8),
                   lambda c: layer(c, 0)["mlp"]["expert"].update(limit=0.0),
                   lambda c: layer(c, 4).update(weights_of=3),
                   lambda c: layer(c, 4).update(weights_of=4),
                   lambda c: layer(c, 2).update(weights_of=4)):
        with pytest.raises(ValueError):
            broken(change)
    for kw in ({"tensor_parallel_size": 2}, {"quantization": "fp8"}, {"dtype": "float16"},
               {"speculative_config": {"method": "suffix"}}):
        with pytest.raises(NotImplementedError):
            broken(lambda c: None, **kw)


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg)
    for name in ("l1.mix.left.out", "l0.ls2", "l0.mlp.correction", "l2.mix.k.norm", "l0.mlp.shared.up"):
        missing = {k: v for k, v in w.items() if k != name}
        with pytest.raises(ValueError, match=name):
            u.session(u.save(tmp_path / "a", cfg, missing), "float32", 64, "cpu")
    for name in ("l4.norm1", "l1.norm2", "head", "l2.mix.v"):
        with pytest.raises(ValueError, match="unexpected"):
            u.session(u.save(tmp_path / "b", cfg, {**w, name: w["l0.norm1"]}), "float32", 64, "cpu")
    with pytest.raises(ValueError, match="shape"):
        u.session(u.save(tmp_path / "c", cfg, {**w, "l0.mix.o": w["embed"]}), "float32", 64, "cpu")


def test_preset_generates():
    llm = LLM(model="pererax-tiny", device="cpu", num_gpu_blocks_override=16, max_model_len=256,
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
