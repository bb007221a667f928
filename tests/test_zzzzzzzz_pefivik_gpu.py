"""Pefivik on a GPU: each kernel against the fp64 restatement, then the model through the engine's
step function, captured decode steps and scheduler."""

import numpy as np
import pytest
import torch

import pefivik_oracle as oracle
import pefivik_util as u
from arcticinference_b200 import LLM, SamplingParams, ops
from arcticinference_b200.config import BigramSpec, MaskSpec
from arcticinference_b200.ops import latent_ops as lat
from arcticinference_b200.ops import state_ops as states
from arcticinference_b200.ops import stream_ops as st
from test_pefivik_cpu import forget_case, forget_want, greedy_gaps
from test_zzzzzz_zatirax_gpu import close, place
from test_zzzzzzz_pererax_gpu import LENS, check_scan

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32


def rnd(*shape, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, device=DEV) * scale).to(dtype)


def f64(t):
    return t.detach().double().cpu()


# ------------------------------------------------------------------ recurrence
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,d,dv,gap", [
    (4, 32, 48, 0), (3, 64, 64, 0), (2, 128, 128, 8), (6, 24, 40, 0), (3, 7, 11, 0), (1, 1, 1, 3),
    (2, 200, 72, 0), (1, 256, 300, 0), (2, 96, 170, 2), (8, 16, 16, 0), (2, 64, 128, 1), (3, 33, 6, 0)])
def test_forget_scan(H, d, dv, gap, strong, dtype):
    s, proj, w = forget_case(H, d, dv, sum(LENS), seed=d, gap=gap)
    if strong:      # channels that are erased within a token, or within a few
        w["f_bias"] -= 9.0
        w["lower"] *= torch.arange(H * d) % 2 == 0
    proj = proj.to(dtype)
    want, a = [], 0
    for n in LENS:
        want.append(forget_want(s, proj[a:a + n], w, 0.01))
        a += n
    proj, wd = proj.to(DEV), [t.to(DEV) for t in w.values()]
    state = torch.full((4, H, d, s.state_cols), float("nan"), device=DEV)
    check_scan(lambda rows, step: states.forget_scan(proj[rows], *wd, s, state, step, 0.01),
               torch.cat(want), LENS, dtype)
    assert bool(torch.isnan(state[0]).all())


@pytest.mark.parametrize("rows", [1, 20])
def test_padding_rows_put_out_zeros(rows):
    s, proj, w = forget_case(2, 32, 200, 2 * rows)
    state = torch.ones(2, 2, 32, s.state_cols, device=DEV)
    step = states.StateStep.build(np.asarray([(0, rows, 1, 0, 0), (rows, rows, 0, 0, 0)],
                                             dtype=np.int32), DEV)
    out = states.forget_scan(proj.to(DEV), *(t.to(DEV) for t in w.values()), s, state, step, 0.01)
    assert float(out[rows:].abs().max()) == 0 < float(out[:rows].abs().max())
    assert bool((state[0] == 1).all())
    ops.check_status()


def test_states_after_portions_and_after_single_tokens_agree():
    n = 70
    s, proj, w = forget_case(2, 64, 96, n, seed=5)
    proj, w = proj.to(BF16).to(DEV), [t.to(DEV) for t in w.values()]
    left, out = [], []
    for cuts in ([n], [1] * n, [2, 33, 16, 19]):
        S, at, got = torch.zeros(2, 2, 64, 96, device=DEV), 0, []
        for k in cuts:
            step = states.StateStep.build(np.asarray([(0, k, 1, at, 0)], dtype=np.int32), DEV)
            got.append(states.forget_scan(proj[at:at + k], *w, s, S, step, 1e-6))
            at += k
        left.append(S[1])
        out.append(torch.cat(got))
    ops.check_status()
    for a, o in zip(left[1:], out[1:]):
        assert float((a - left[0]).abs().max()) < 1e-4 * float(left[0].abs().max())
        close(o, out[0], BF16)


def test_the_split_of_a_head_does_not_matter():
    s, proj, w = forget_case(2, 64, 128, 70)
    proj, w, outs = proj.to(DEV), [t.to(DEV) for t in w.values()], []
    for n in (1, 8):
        state = torch.zeros(2, 2, 64, s.state_cols, device=DEV)
        step = states.StateStep.build(np.asarray([(0, 70, 1, 0, 0)], dtype=np.int32), DEV)
        saved, states.slices_for = states.slices_for, lambda *a: n
        try:
            outs.append((states.forget_scan(proj, *w, s, state, step, 0.01), state))
        finally:
            states.slices_for = saved
    for a, b in zip(*outs):
        close(a, b, F32)


# ------------------------------------------------------------------ embedding, stream, feed-forward
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("W", [8, 101, 2048])
def test_pairs_of_tokens(W, dtype):
    spec, table, second = BigramSpec(1009, 100003, 77), rnd(50, W, dtype=dtype), rnd(1010, W, dtype=dtype)
    toks = torch.randint(0, 50, (300,)).tolist()
    ids, prev = torch.tensor(toks, device=DEV), torch.tensor([-1] + toks[:-1], device=DEV)
    prev[17] = -1
    rows = oracle.bigram_rows(toks, {"buckets": 1009, "mul_prev": 100003, "mul_cur": 77})
    rows[17] = 1009
    keep = torch.empty(300, W, device=DEV)
    x, act = st.stream_embedding(ids, table, 0.5, pairs=(prev, second, spec), keep=keep)
    want = table[ids].float() * 0.5 + second[rows].float()
    assert torch.equal(x, want) and torch.equal(keep, want) and torch.equal(act, want.to(dtype))
    ops.check_status()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W", [(1, 8), (37, 101), (5, 2048), (3, 6148), (2, 9000), (4, 320)])
def test_stream_pre(T, W, dtype):
    torch.manual_seed(W)
    x0, y, y2, rows_y = rnd(T, W, dtype=F32), *(rnd(n, W, dtype=dtype) for n in (T, T, 3 * T))
    base, bias, step, vec = (rnd(*s, dtype=F32) for s in ((T, W), (W,), (W,), (W,)))
    gain = torch.tensor([0.8], device=DEV)
    rows = torch.randint(0, 3 * T, (T, 3), device=DEV, dtype=torch.int32)
    r = st.Routing(rows, torch.rand(T, 3, device=DEV), rows, 3, 4)
    mix = sum(f64(r.weights)[:, j:j + 1] * f64(rows_y)[rows[:, j].long().cpu()] for j in range(3))
    for kw, out in (({}, torch.zeros(T, W)), (dict(y=y), f64(y)), (dict(y=y, bias=bias), f64(y) + f64(bias)),
                    (dict(y=rows_y, experts=r), mix), (dict(y=rows_y, experts=r, shared=y2), mix + f64(y2))):
        for more in ({}, dict(base=base, step=step), dict(step=step)):
            for w in (gain, vec, None):
                x = x0.clone()
                act = None if w is None else torch.empty(T, W, dtype=dtype, device=DEV)
                st.stream_pre(x, 0.3, 0.02, w_in=w, act=act, **kw, **more)
                want = oracle.residual(f64(x0), out, 0.3) + sum(f64(t) for t in more.values())
                close(x.cpu(), want, F32)
                if act is not None:
                    close(act.cpu(), oracle.stream_norm(want, w, 0.02), dtype)
    ops.check_status()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,n,ff", [(1, 8, 3), (300, 104, 101), (5, 2048, 2048), (3, 14336, 14336),
                                    (300, 28672, 28668), (2, 40000, 40000), (2, 70000, 70000), (7, 37, 37), (4, 136, 136)])
def test_poly_norm(T, n, ff, dtype):
    torch.manual_seed(ff)
    z, bias = rnd(T, n, dtype=dtype), rnd(n, dtype=dtype)
    z[0] *= 1e-3      # powers below the root of eps
    if T > 1:
        z[1] *= 50.0
    coef = torch.tensor([0.6, -0.5, 0.4, 0.3], device=DEV)
    for b in (bias, bias * 1e-3):
        got = st.poly_norm(z, b, coef, ff, 0.02)
        want = oracle.poly_norm(f64(z)[:, :ff] + f64(b)[:ff], coef, 0.02)
        close(got[:, :ff].cpu(), want, dtype)
        assert not ff < n or float(got[:, ff:].abs().max()) == 0
    ops.check_status()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,V,ld", [(1, 53, 56), (3, 1000, 1000), (300, 130, 136), (2, 128256, 128256)])
def test_soft_cap(T, V, ld, dtype):
    z = rnd(T, ld, scale=20.0, dtype=dtype)
    got = st.soft_cap(z[:, :V], 15.0)
    assert got.dtype == F32
    close(got.cpu(), 15.0 * torch.tanh(f64(z)[:, :V] / 15.0), F32)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W,experts,top,count,keep,ff", [
    (3, 96, 12, 3, 4, 2, 40), (300, 264, 64, 6, 8, 3, 72), (1500, 136, 8, 2, 4, 1, 64), (40, 77, 5, 2, 5, 3, 9),
    (1, 64, 4, 4, 2, 2, 16), (7, 128, 160, 8, 40, 4, 24), (5, 2048, 256, 8, 8, 4, 16), (9, 64, 1, 1, 1, 1, 8)])
def test_grouped_router(T, W, experts, top, count, keep, ff, dtype):
    torch.manual_seed(T)
    act = rnd(T, W, dtype=dtype)
    router = rnd(experts, W, scale=1.5 * W ** -0.5, dtype=dtype)
    want = oracle.route(f64(act), router, {"top": top, "scale": 1.4,
                                           "groups": {"count": count, "keep": keep}})
    sure = want[2] > 1e-5
    assert float(sure.double().mean()) > 0.8
    for x in (act, act.float()):
        r, rows = st.route(x, act, router, None, top, 0, 1.4, (count, keep))
        assert torch.equal(r.ids.cpu().long()[sure], want[0][sure])
        assert float((r.weights.cpu() - want[1])[sure].abs().max()) < 1e-5
        flat = r.rows.flatten().long()
        assert torch.equal(flat.sort().values.cpu(), torch.arange(T * top))
        assert torch.equal(rows[flat], act.repeat_interleave(top, 0))
    gate, up, down = (rnd(experts, *s, scale=s[-1] ** -0.5, dtype=dtype) for s in ((ff, W), (ff, W), (W, ff)))
    h = st.grouped_linear(rows, st.interleave_gate_up(gate, up), r, act="silu")
    y = st.grouped_linear(h, torch.nn.functional.pad(down, (0, -ff % st.GATE_BLOCK)).contiguous(), r)
    for e in range(0, experts, max(1, experts // 8)):
        t, j = torch.nonzero(r.ids.cpu() == e, as_tuple=True)
        if t.numel():
            w = {"gate": gate[e], "up": up[e], "down": down[e]}
            close(y[r.rows.cpu()[t, j].long().to(DEV)].cpu(), oracle.expert(f64(act)[t], w, ""), dtype, 2.0)
    ops.check_status()


# ------------------------------------------------------------------ attention in latent space
CASES = [
    (9, 64, 64, [1, 1, 1], [1, 64, 65]),
    (5, 64, 16, [30, 1, 2], [30, 500, 129]),
    (12, 64, 64, [100], [300]),
    (8, 64, 64, [1], [4000]),
    (1, 128, 16, [1, 3], [257, 128]),
    (16, 512, 64, [1] * 4, [2000, 1, 127, 128]),
    (16, 512, 64, [7, 1], [700, 3000]),
    (5, 256, 64, [33, 1, 2], [33, 385, 130]),
    (20, 384, 32, [2, 1], [140, 999]),
    (40, 256, 128, [1, 1], [300, 5]),
    (130, 128, 64, [1, 2], [200, 70]),
    (3, 100, 16, [4, 1], [60, 40]),
]


def standing_out(q, c, H, R, q_lens, kv_lens, bs):
    """Single keys that stand out: the first ones, the token itself, block borders."""
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        for j in range(n):
            pos = kl - n + j
            for h in range(H):
                key = (0, pos, pos // bs * bs, max(0, pos // bs * bs - 1), min(1, pos), pos // 2)[h % 6]
                v = q[t + j].view(H, R)
                v[h] = v[h] * 0.3 + c[o + key] * 0.35
        o, t = o + kl, t + n


def attention_want(q, c, sink, gate, H, R, q_lens, kv_lens, scale):
    out, o, t = [], 0, 0
    for n, kl in zip(q_lens, kv_lens):
        cs = c[o:o + kl].double()
        s = torch.einsum("thr,kr->htk", q[t:t + n].reshape(n, H, R).double(), cs) * scale
        hidden = torch.arange(kl, device=DEV) > torch.arange(kl - n, kl, device=DEV).unsqueeze(1)
        s = s.masked_fill(hidden, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.double().view(H, 1, 1).expand(H, n, 1)], -1)
        w = torch.softmax(s, -1)[..., :kl]
        x = torch.einsum("htk,kr->thr", w, cs)
        if gate is not None:
            x = x * torch.sigmoid(gate[t:t + n].double()).unsqueeze(-1)
        out.append(x.reshape(n, H * R))
        o, t = o + kl, t + n
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,R,bs,q_lens,kv_lens", CASES)
def test_latent_attention_with_sinks_and_head_gates(H, R, bs, q_lens, kv_lens, dtype):
    torch.manual_seed(H * R)
    total, T, scale = sum(kv_lens), sum(q_lens), 0.9 * R ** -0.5
    c, q = rnd(total, R, dtype=dtype), rnd(T, H * R, dtype=dtype)
    nb, bt, rows = place(kv_lens, bs)
    cache = torch.full((nb, 1, bs, R), 37.0, dtype=dtype, device=DEV)
    cache[rows // bs, 0, rows % bs] = c
    standing_out(q, c, H, R, q_lens, kv_lens, bs)
    # from sinks that take nothing to ones that take all; gates among other columns
    sink = torch.linspace(-20.0, 12.0, H, device=DEV)[torch.randperm(H)] if H > 1 else rnd(1, dtype=F32)
    proj = rnd(T, H + 13, scale=2.0, dtype=dtype)
    gate = proj[:, 5:5 + H]
    shape = lat.LatentShape.of(H, R, dtype)
    meta = lat.build_plan(shape, q_lens, kv_lens, bt, bs, DEV)
    seq = torch.repeat_interleave(torch.arange(len(q_lens)), torch.tensor(q_lens)).int().to(DEV)
    pos = torch.cat([torch.arange(k - n, k) for n, k in zip(q_lens, kv_lens)]).to(DEV)
    for s, g in ((sink, gate), (sink, None), (None, gate), (None, None)):
        got = lat.latent_attention(q, cache, meta, shape, scale, seq, pos, s, g)
        ops.check_status()
        close(got, attention_want(q, c, s, g, H, R, q_lens, kv_lens, scale), dtype)


@pytest.mark.parametrize("H,R", [(6, 64), (16, 512), (20, 128)])
def test_sinks_and_gates_do_not_depend_on_the_split(H, R):
    torch.manual_seed(R)
    lens = [1500, 130, 1]
    nb, bt, rows = place(lens, 64)
    c, q = rnd(sum(lens), R), rnd(3, H * R)
    cache = torch.zeros(nb, 1, 64, R, dtype=BF16, device=DEV)
    cache[rows // 64, 0, rows % 64] = c
    sink, gate, scale = rnd(H, scale=3.0, dtype=F32), rnd(3, H), R ** -0.5
    want = attention_want(q, c, sink, gate, H, R, [1, 1, 1], lens, scale)
    shape = lat.LatentShape.of(H, R, BF16)
    for cap in (1, 2, 5, 16):
        plan = lat.LatentDecodePlan(shape, 3, 1, 64)
        plan.splits, plan.work_cap = cap, 400
        host = torch.zeros(plan.int32_words, dtype=torch.int32)
        dev = torch.zeros_like(host, device=DEV)
        plan.bind(host.numpy(), dev, bt)
        plan.fill([1, 1, 1], lens)
        dev.copy_(host)
        close(lat.latent_attention(q, cache, plan.meta, shape, scale, sink=sink, gate=gate), want, BF16)
    ops.check_status()


@pytest.mark.parametrize("H,dq,dv", [(4, 64, 64), (3, 128, 128), (2, 192, 128)])
def test_expanded_attention_with_sinks_and_head_gates(H, dq, dv):
    """Long chunks, with keys before them, over expanded keys and values."""
    torch.manual_seed(dq)
    q_lens, kv_lens = [200, 130], [333, 130]
    T, n, scale = sum(q_lens), sum(kv_lens), dq ** -0.5
    q, kv = rnd(T, H * dq), rnd(n, H * (dq + dv))
    k, v = kv[:, :H * dq], kv[:, H * dq:]
    o = t = 0
    for a, b in zip(q_lens, kv_lens):
        for j in range(a):
            for h in range(H):
                key = o + (0, b - a + j, (b - a + j) // 64 * 64, 1)[(h + j) % 4]
                q[t + j, h * dq:(h + 1) * dq] += k[key, h * dq:(h + 1) * dq]
        o, t = o + b, t + a
    sink, gate = torch.linspace(-3.0, 6.0, H, device=DEV), rnd(T, H, scale=2.0)
    mask = MaskSpec()
    step = lat.AttentionStep(0)
    step.exp_q_lens, step.exp_kv_lens = q_lens, kv_lens
    step.exp_plans[(H, (dq, dv), mask)] = ops.build_attention_metadata(
        q_lens, kv_lens, None, 1, H, dv, DEV, Hkv=H,
        seq_rows=np.cumsum(kv_lens) - np.asarray(kv_lens), allow_split=False, mask=mask)
    out = torch.empty(T, H * dv, dtype=BF16, device=DEV)
    lat.expanded_attention(q, k, v, step, H, (dq, dv), scale, out, mask, sink, gate)
    ops.check_status()
    o = t = 0
    for a, b in zip(q_lens, kv_lens):
        for h in range(H):
            s = torch.full((b, b), -1e9, dtype=torch.float64)
            s[b - a:] = f64(q)[t:t + a, h * dq:(h + 1) * dq] @ f64(k)[o:o + b, h * dq:(h + 1) * dq].t() * scale
            x = oracle.weights_of(s, float(sink[h]))[b - a:] @ f64(v)[o:o + b, h * dv:(h + 1) * dv]
            close(out[t:t + a, h * dv:(h + 1) * dv].cpu(), x * oracle.sigmoid(f64(gate)[t:t + a, h:h + 1]), BF16)
        o, t = o + b, t + a


# ------------------------------------------------------------------ the model
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
    u.check_schedules(cfg, path, dtype, DEV, w)
    ops.check_status()


def test_other_block_sizes_and_eager_steps(model):
    cfg, w, path = model["bfloat16"]
    for bs in (16, 128):
        u.check_schedules(cfg, path, "bfloat16", DEV, w, names=("mixed", "decode"), block_size=bs,
                          max_num_seqs=4, enforce_eager=bs == 16)


def test_captured_steps_are_used(model):
    cfg, w, path = model["bfloat16"]
    sess = u.session(path, "bfloat16", 256, DEV)
    u.run(sess, {"b": u.tokens(cfg, 20, 2)}, [[("b", 3)]] + [[("b", 1)]] * 17)
    m = sess.engine.runner.model
    assert sess.engine.runner.graph_replays == (17 if m.supports_graphs else 0)


def test_residual_stream_after_every_run(model):
    cfg, w, path = model["float32"]
    toks, want, got = u.tokens(cfg, 70, 8), [], []
    oracle.forward(cfg, w, toks, want)
    sess = u.session(path, "float32", 128, DEV)
    forward = sess.engine.runner.model.forward
    sess.engine.runner.model.forward = lambda b, kv: forward(b, kv, layers_out=got)
    sess.step([{"id": "a", "tokens": toks, "want": [0]}], ["a"])
    assert len(got) == len(want)
    for a, b in zip(got, want):
        assert float((a.cpu().double() - b).abs().max()) < 2e-4 * float(b.abs().max())


def test_long_decoding(tmp_path):
    """Several hundred tokens one by one, in captured steps, with states that remember them and keys
    that stand out of all of them."""
    cfg = u.config(64, 80, [
        (u.latent(4, 32, 32, 64), u.moe(32, 6, 2, (3, 2), 24)), (u.hgrn2(2, 32, 32), u.dense(64)),
        (u.latent(2, 32, 48, 128), None)], loop=(0, 2, 2), bigram=(61, 3, 7), mult=0.4, cap=5.0)
    for dtype in ("bfloat16", "float32"):
        w = u.weights(cfg, seed=6, peak=2.0 if dtype == "float32" else 0.5)
        w["l1.mix.f.b"] = w["l1.mix.f.b"] * 0 + 7.0
        w["l1.mix.lower"] = w["l1.mix.lower"] * 0 + 0.9
        sess = u.session(u.save(tmp_path / dtype, cfg, w), dtype, 704, DEV)
        seqs = {"a": u.tokens(cfg, 640, 1)}
        u.compare(cfg, w, u.run(sess, seqs, [[("a", 4)]] + [[("a", 1)]] * 636), seqs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(model, dtype):
    cfg, w, path = model[dtype]
    llm = LLM(model=path, device=DEV, dtype=dtype, num_gpu_blocks_override=60, block_size=16,
              max_model_len=256, max_num_batched_tokens=32)
    prompts = [u.tokens(cfg, n, 10 + n) for n in (100, 3, 17, 64, 1)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    ops.check_status()
    for p, ro in zip(prompts, outs):
        toks = ro.outputs[0].token_ids
        assert len(toks) == 12
        gap = greedy_gaps(cfg, w, p, toks)
        z = oracle.forward(cfg, w, p)
        spread = float((z - z.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        # (in 16 bits a swapped expert may move a single choice further)
        off = gap > (1e-3 if dtype == "float32" else 0.3) * spread
        assert int(off.sum()) <= (0 if dtype == "float32" else 3), gap.tolist()


def test_preemption_sampling_and_sleep(tmp_path):
    """Requests whose pages and slots are taken away, and a wake-up from level-2 sleep, change no
    token; sampled requests run beside greedy ones."""
    cfg = u.CONFIGS["mixed"]
    path = u.save(tmp_path, cfg, u.weights(cfg, seed=5))
    kw = dict(model=path, device=DEV, dtype="float32", block_size=16, max_model_len=256)
    prompts = [{"prompt_token_ids": u.tokens(cfg, n, n)} for n in (49, 57, 68)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    plain = LLM(num_gpu_blocks_override=64, **kw)
    want = [plain.generate(p, sp)[0].outputs[0].token_ids for p in prompts]
    plain.sleep(2)
    plain.wake_up()
    for llm in (plain, LLM(num_gpu_blocks_override=13, **kw), LLM(num_gpu_blocks_override=64, max_num_seqs=2, **kw)):
        assert [o.outputs[0].token_ids for o in llm.generate(prompts, sp)] == want
        kv = llm.engine.kv_manager
        assert len(kv.states.free) == kv.states.num_slots - 1
    hot = SamplingParams(temperature=1.0, top_p=0.9, max_tokens=8, ignore_eos=True, seed=3)
    a = plain.generate(prompts, [hot, sp, hot])
    assert a[1].outputs[0].token_ids == want[1] and len(a[0].outputs[0].token_ids) == 8
    ops.check_status()
