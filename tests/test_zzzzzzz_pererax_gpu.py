"""Pererax on a GPU: each kernel against the fp64 restatement, then the model through the engine's
step function, captured decode steps and scheduler."""

import numpy as np
import pytest
import torch

import pererax_oracle as oracle
import pererax_util as u
from arcticinference_b200 import LLM, SamplingParams, ops
from arcticinference_b200.config import MaskSpec
from arcticinference_b200.ops import head_ops as hd
from arcticinference_b200.ops import state_ops as states
from arcticinference_b200.ops import stream_ops as st
from test_pererax_cpu import delta_case, delta_want, greedy_gaps
from test_zzzzzz_zatirax_gpu import close, place, targets, visible_of

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32


def rnd(*shape, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, device=DEV) * scale).to(dtype)


def f64(t):
    return t.detach().double().cpu()


# ------------------------------------------------------------------ recurrences
def steps_of(lens, cuts, slots):
    """Batches of a schedule: ``cuts`` lists, per step, the tokens each sequence brings (0: left out);
    sequences lie one after the other in memory. Yields (rows to gather, step table)."""
    at, phase = [0] * len(lens), [0] * len(lens)
    base = [sum(lens[:i]) for i in range(len(lens))]
    for step in cuts:
        rows, table = [], []
        for i, n in enumerate(step):
            if n:
                table.append((len(rows), n, slots[i], at[i], phase[i]))
                rows += range(base[i] + at[i], base[i] + at[i] + n)
                at[i], phase[i] = at[i] + n, phase[i] ^ 1
        yield rows, states.StateStep.build(np.asarray(table, dtype=np.int32), DEV)
    assert at == list(lens)


# three sequences: whole; token by token; uneven portions (tiles are of 16 tokens, in groups of 4)
LENS = [53, 18, 7]
CUTS = [[[53, 18, 7]], [[1, 1, 1]] * 7 + [[1, 1, 0]] * 11 + [[1, 0, 0]] * 35,
        [[2, 0, 7], [16, 1, 0], [1, 2, 0], [31, 15, 0], [3, 0, 0]]]
SIZES = [(4, 2, 32, 48, 3), (3, 3, 64, 64, 4), (2, 1, 128, 128, 4), (6, 2, 24, 40, 2), (3, 1, 7, 11, 5),
         (1, 1, 1, 1, 1), (2, 2, 200, 72, 3), (1, 1, 256, 300, 2), (2, 1, 96, 170, 8), (8, 8, 16, 16, 1)]


def check_scan(run, want, lens, dtype):
    for cuts in CUTS:
        got = torch.empty(want.shape, dtype=torch.float64)
        for rows, step in steps_of(lens, cuts, [3, 1, 2]):
            got[rows] = f64(run(rows, step))
        ops.check_status()
        for i, n in enumerate(lens):
            a = sum(lens[:i])
            e = (got - want)[a:a + n].abs().max() / want[a:a + n].abs().max()
            assert float(e) < (0.02 if dtype == BF16 else 3e-5), (cuts[0], i, float(e))


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,G,d,dv,taps", SIZES)
def test_delta_scan(H, G, d, dv, taps, strong, dtype):
    s, proj, decay, gate, w = delta_case(H, G, d, dv, taps, LENS, seed=d)
    if strong:      # some heads erase channels within a token, others within a few
        w["a_exp"] = torch.logspace(0.3, 2.0, H) if H > 1 else torch.tensor([60.0])
        w["dt_bias"] += 1.0
    proj, decay, gate = (t.to(dtype) for t in (proj, decay, gate))
    want, a = [], 0
    for n in LENS:
        want.append(delta_want(s, proj[a:a + n], decay[a:a + n], gate[a:a + n], w, 0.01))
        a += n
    dev = lambda t: t.to(DEV)
    wd = [dev(t).contiguous() for t in w.values()]
    proj, decay, gate = dev(proj), dev(decay), dev(gate)
    state = torch.full((4, H, d, s.state_cols), float("nan"), device=DEV)
    conv = torch.full((4, 2, taps - 1, s.channels), float("nan"), dtype=dtype, device=DEV)

    def run(rows, step):
        return states.delta_scan(proj[rows], decay[rows], gate[rows], *wd, s, state, conv, step, 0.01)
    check_scan(run, torch.cat(want), LENS, dtype)
    assert bool(torch.isnan(state[0]).all())


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,d,dv,cap", [(3, 32, 48, 8.0), (2, 64, 127, 15.0), (1, 128, 128, 5.0),
                                        (5, 24, 40, 12.0), (3, 7, 11, 3.0), (1, 1, 1, 1.0),
                                        (2, 200, 170, 6.0), (1, 256, 512, 10.0), (4, 16, 64, 30.0)])
def test_memory_scan(H, d, dv, cap, dtype):
    torch.manual_seed(d)
    T, nk, nv = sum(LENS), H * d, H * dv
    s = states.MemoryShape(H, d, dv, cap, 0, nk, 2 * nk, 2 * nk + nv, 2 * nk + nv + H)
    # (columns of a wider projection, the gates scaled so that maxima jump and forgetting varies)
    proj, gate = torch.randn(T, 2 * nk + nv + 2 * H + 3), torch.randn(T, nv)
    proj[:, s.i_at:s.f_at + H] *= 3.0
    proj, gate = proj.to(dtype), gate.to(dtype)
    norm, ib, fb = torch.randn(nv), torch.randn(H) * 2, torch.randn(H) * 4 + 2
    p, want, a = f64(proj), [], 0
    for n in LENS:
        r = p[a:a + n]
        i, f = oracle.memory_gates(r[:, s.i_at:s.i_at + H] + ib, r[:, s.f_at:s.f_at + H] + fb, cap)
        o = torch.cat([oracle.rms(oracle.memory_scan(
            r[:, h * d:(h + 1) * d] * d ** -0.5, r[:, nk + h * d:nk + (h + 1) * d],
            r[:, 2 * nk + h * dv:2 * nk + (h + 1) * dv], i[:, h], f[:, h]), 0.01) for h in range(H)], 1)
        want.append(o * norm.double() * oracle.sigmoid(f64(gate[a:a + n])))
        a += n
    proj, gate, norm, ib, fb = (t.to(DEV) for t in (proj, gate, norm, ib, fb))
    state = torch.full((4, H, d, s.state_cols), float("nan"), device=DEV)
    top = torch.full((4, 2, H), float("nan"), device=DEV)

    def run(rows, step):
        return states.memory_scan(proj[rows], gate[rows], ib, fb, norm, s, state, top, step, 0.01)
    check_scan(run, torch.cat(want), LENS, dtype)


@pytest.mark.parametrize("rows", [1, 20])
def test_padding_rows_put_out_zeros(rows):
    H, G, d, dv, taps = 2, 1, 32, 200, 3
    s, proj, decay, gate, w = delta_case(H, G, d, dv, taps, [2 * rows])
    dev = lambda t: t.to(DEV)
    state = torch.ones(2, H, d, s.state_cols, device=DEV)
    conv = torch.ones(2, 2, taps - 1, s.channels, device=DEV)
    step = states.StateStep.build(np.asarray([(0, rows, 1, 0, 0), (rows, rows, 0, 0, 0)],
                                             dtype=np.int32), DEV)
    out = states.delta_scan(dev(proj), dev(decay), dev(gate), *map(dev, w.values()), s, state, conv,
                            step, 0.01)
    assert float(out[rows:].abs().max()) == 0 < float(out[:rows].abs().max())
    assert bool((state[0] == 1).all()) and bool((conv[0] == 1).all())
    ops.check_status()


def test_the_split_of_a_head_does_not_matter():
    H, G, d, dv, taps = 2, 1, 64, 128, 4
    s, proj, decay, gate, w = delta_case(H, G, d, dv, taps, [70])
    outs = []
    for blocks in (1, 1000):      # as one block per head, or as many as its columns allow
        state = torch.zeros(2, H, d, s.state_cols, device=DEV)
        conv = torch.zeros(2, 2, taps - 1, s.channels, device=DEV)
        step = states.StateStep.build(np.asarray([(0, 70, 1, 0, 0)], dtype=np.int32), DEV)
        saved, states.slices_for = states.slices_for, lambda *a: 1 if blocks == 1 else 8
        try:
            outs.append((states.delta_scan(*(t.to(DEV) for t in (proj, decay, gate, *w.values())), s,
                                           state, conv, step, 0.01), state, conv))
        finally:
            states.slices_for = saved
    for a, b in zip(*outs):
        close(a, b, F32)


# ------------------------------------------------------------------ stream, router, experts
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W", [(1, 8), (37, 101), (5, 2048), (3, 6148), (2, 9000), (4, 320)])
def test_stream_add(T, W, dtype):
    torch.manual_seed(W)
    x0, w, w1, w2 = rnd(T, W, dtype=F32), *(rnd(W, dtype=F32) for _ in range(3))
    y, y2, rows_y = rnd(T, W, dtype=dtype), rnd(T, W, dtype=dtype), rnd(3 * T, W, dtype=dtype)
    act = torch.empty(T, W, dtype=dtype, device=DEV)

    def check(want, *a, **kw):
        for copy in (act, None):
            x = x0.clone()
            st.stream_add(x, x if copy is None and dtype == F32 else act, w, 0.05, *a, **kw)
            close(x.cpu(), f64(x0) + oracle.norm(want, w, 0.05), F32)
            if copy is not None:
                assert torch.equal(act, x.to(dtype))

    check(f64(y), y)
    check(0.5 * (oracle.norm(f64(y), w1, 0.05) + oracle.norm(f64(y2), w2, 0.05)), y, pair=(y2, w1, w2))
    rows = torch.randint(-1, 3 * T, (T, 3), device=DEV, dtype=torch.int32)
    r = st.Routing(rows, torch.rand(T, 3, device=DEV), rows, 3, 4)
    k = rows.long().cpu()
    mix = sum(f64(r.weights)[:, j:j + 1] * torch.where(k[:, j:j + 1] < 0, f64(x0), f64(rows_y)[k[:, j]])
              for j in range(3))
    check(mix, rows_y, experts=r)
    check(mix + f64(y2), rows_y, experts=r, shared=y2)
    ops.check_status()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W,experts,identity,top,ff", [
    (3, 96, 5, 3, 2, 40), (300, 264, 40, 24, 6, 72), (1500, 136, 8, 4, 2, 64), (40, 77, 1, 6, 3, 9),
    (1, 64, 4, 0, 4, 16), (7, 128, 3, 2, 5, 24)])
def test_router_and_experts(T, W, experts, identity, top, ff, dtype):
    torch.manual_seed(T)
    x, n = rnd(T, W, dtype=F32), experts + identity
    act = x if dtype == F32 else x.to(dtype)
    router, corr = rnd(n, W, scale=W ** -0.5, dtype=dtype), torch.rand(n, device=DEV)
    r, rows = st.route(x, act, router, corr, top, identity, 1.4)
    ids, weights, lead = oracle.route(f64(x), router, corr, top, 1.4)
    sure = lead > 1e-4
    assert float(sure.double().mean()) > 0.8
    assert torch.equal(r.ids.cpu().long()[sure], ids[sure])
    assert float((r.weights.cpu() - weights)[sure].abs().max()) < 1e-4
    used = r.rows.cpu()
    assert torch.equal(used < 0, r.ids.cpu() >= experts)
    flat = used[used >= 0].long()
    assert flat.unique().numel() == flat.numel() == int((r.ids < experts).sum())
    token = torch.arange(T).unsqueeze(1).expand(T, top)[used >= 0]
    assert torch.equal(rows[flat.to(DEV)], act[token.to(DEV)])
    gate, up, down = rnd(experts, ff, W, scale=2 * W ** -0.5, dtype=dtype), rnd(
        experts, ff, W, scale=2 * W ** -0.5, dtype=dtype), rnd(experts, W, ff, scale=ff ** -0.5, dtype=dtype)
    k = -ff % st.GATE_BLOCK
    h = st.grouped_linear(rows, st.interleave_gate_up(gate, up), r, act=st.Gate("clamped_swish", 0.9))
    y = st.grouped_linear(h, torch.nn.functional.pad(down, (0, k)).contiguous(), r)
    for e in range(experts):
        t, j = torch.nonzero(r.ids.cpu() == e, as_tuple=True)
        if t.numel():
            xe = f64(act)[t]
            want = oracle.apply(down[e], oracle.clamped_swish(oracle.apply(gate[e], xe),
                                                              oracle.apply(up[e], xe), 0.9))
            close(y[used[t, j].long().to(DEV)].cpu(), want, dtype, 2.0)
    ops.check_status()


# ------------------------------------------------------------------ attention
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,G,dim,dims,shared", [
    (4, 2, 64, 64, True), (6, 3, 40, 16, False), (3, 1, 7, 6, True), (40, 8, 128, 32, True),
    (2, 2, 96, 2, False), (2, 1, 256, 128, True), (16, 1, 64, 32, False)])
def test_projection_norm_and_cache(H, G, dim, dims, shared, dtype):
    torch.manual_seed(dim)
    shape = hd.HeadShape.of(H, G, dim, dim, dtype)
    D, bs, T = shape.D, 16, 6
    nv = 0 if shared else G * D
    proj = torch.zeros(T, (H + G) * D + nv, dtype=dtype, device=DEV)
    x, v = rnd(T, H + G, dim, dtype=dtype), rnd(T, G, dim, dtype=dtype)
    proj[:, :(H + G) * D].view(T, H + G, D)[:, :, :dim] = x
    if not shared:
        proj[:, (H + G) * D:].unflatten(1, (G, D))[:, :, :dim] = v
    pad = lambda w, n: torch.nn.functional.pad(w.view(n, dim), (0, D - dim)).reshape(-1).contiguous()
    wq, wk = rnd(H * dim, dtype=F32), rnd(G * dim, dtype=F32)
    k, vc = (torch.zeros(3, G, bs, D, dtype=dtype, device=DEV) for _ in range(2))
    slots = torch.tensor([47, -1, 0, 17, 16, 5], device=DEV)
    pos = torch.tensor([0, 1, 300, 7, 4000, 63], device=DEV)
    rot = {"base": 500.0, "dims": dims}
    freq = torch.tensor([500.0 ** (-2.0 * i / dims) for i in range(dims // 2)]).to(DEV)
    hd.head_rope_cache(proj, shape, dim, pad(wq, H), pad(wk, G), hd.rotary_table(pos, freq), 0.02, slots,
                       k, vc, whole=True, shared_kv=shared)
    ops.check_status()
    qn = oracle.projection_norm(f64(x[:, :H].reshape(T, -1)), wq, 0.02)
    kn = oracle.projection_norm(f64(x[:, H:].reshape(T, -1)), wk, 0.02)
    scale = 1.0 if dtype == BF16 else 10.0
    for h in range(H):
        got = proj[:, h * D:(h + 1) * D]
        close(got[:, :dim].cpu(), oracle.rotate(qn[:, h * dim:(h + 1) * dim], pos.cpu(), rot), dtype, scale)
        assert float(got[:, dim:].abs().sum()) == 0
    for g in range(G):
        want = oracle.rotate(kn[:, g * dim:(g + 1) * dim], pos.cpu(), rot)
        for i, s in enumerate(slots.tolist()):
            if s >= 0:
                close(k[s // bs, g, s % bs, :dim].cpu(), want[i], dtype, scale)
                assert torch.equal(vc[s // bs, g, s % bs, :dim], x[i, H + g] if shared else v[i, g])
    assert int((vc != 0).any(-1).sum()) <= 5 * G


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("mask", [MaskSpec(), MaskSpec("window", 64), MaskSpec("window", 300)])
@pytest.mark.parametrize("cap", [1.5, 30.0])
@pytest.mark.parametrize("H,G,dim,vdim,bs,q_lens,kv_lens", [
    (4, 4, 64, 64, 64, [1, 1, 1], [1, 64, 65]),
    (8, 2, 128, 128, 64, [1] * 20, [300 + 7 * i for i in range(20)]),
    (6, 2, 40, 24, 16, [30, 1, 2], [30, 500, 129]),
    (12, 1, 64, 64, 64, [100], [900]),
    (2, 2, 128, 96, 128, [300, 1], [1200, 3000]),
    (3, 3, 64, 64, 32, [1], [4000]),
    (4, 2, 160, 144, 64, [3, 1], [60, 300])])
def test_capped_attention(H, G, dim, vdim, bs, q_lens, kv_lens, cap, mask, dtype):
    """Single keys stand out (up to the cap and beyond) at the mask's edges and page borders."""
    torch.manual_seed(H * dim)
    shape = hd.HeadShape.of(H, G, dim, vdim, dtype, mask)
    D, Dv, T, total = shape.D, shape.Dv, sum(q_lens), sum(kv_lens)
    nb, bt, rows = place(kv_lens, bs)
    k, v = rnd(total, G, dim, dtype=dtype), rnd(total, G, vdim, dtype=dtype)
    kc, vc = (torch.full((nb, G, bs, n), 37.0, dtype=dtype, device=DEV) for n in (D, Dv))
    kc[rows // bs, :, rows % bs] = torch.nn.functional.pad(k, (0, D - dim))
    vc[rows // bs, :, rows % bs] = torch.nn.functional.pad(v, (0, Dv - vdim))
    q, scale = rnd(T, H, dim, dtype=dtype), 0.9 * dim ** -0.5
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        for j in range(n):
            at = targets(mask, kl - n + j, kl)
            for h in range(H):
                q[t + j, h] = q[t + j, h] * 0.3 + k[o + at[(h + j) % 6], h // (H // G)] * 1.5
        o, t = o + kl, t + n
    sink = torch.zeros(H, device=DEV)
    seq = torch.repeat_interleave(torch.arange(len(q_lens)), torch.tensor(q_lens)).int().to(DEV)
    pos = torch.cat([torch.arange(a - n, a) for n, a in zip(q_lens, kv_lens)]).to(DEV)
    qp = torch.nn.functional.pad(q, (0, D - dim)).reshape(T, H * D)
    meta = hd.build_plan(shape, q_lens, kv_lens, bt, bs, DEV)
    for s in (sink, None):
        got = hd.head_attention(qp, kc, vc, meta, shape, scale, s, None, seq, pos, cap)
        ops.check_status()
        o = t = 0
        for n, kl in zip(q_lens, kv_lens):
            ks, vs = (x[o:o + kl].double().repeat_interleave(H // G, 1) for x in (k, v))
            sc = oracle.capped(torch.einsum("thd,khd->htk", q[t:t + n].double(), ks) * scale, cap)
            w = oracle.weights_of(sc, visible_of(mask, n, kl), s is not None)
            close(got[t:t + n].view(n, H, Dv)[..., :vdim], torch.einsum("htk,khd->thd", w, vs), dtype)
            o, t = o + kl, t + n


def test_capped_attention_does_not_depend_on_the_split():
    torch.manual_seed(1)
    lens = [1500, 130, 1]
    nb, bt, _ = place(lens, 64)
    shape = hd.HeadShape.of(6, 2, 64, 64, BF16)
    q, kc, vc = rnd(3, 6 * 64), rnd(nb, 2, 64, 64), rnd(nb, 2, 64, 64)
    outs = []
    for cap in (1, 2, 5, 16):
        plan = hd.HeadDecodePlan(shape, 3, 1, 64)
        plan.splits, plan.work_cap = cap, 400
        host = torch.zeros(plan.int32_words, dtype=torch.int32)
        dev = torch.zeros_like(host, device=DEV)
        plan.bind(host.numpy(), dev, bt)
        plan.fill([1, 1, 1], lens)
        dev.copy_(host)
        outs.append(hd.head_attention(q, kc, vc, plan.meta, shape, 0.2, torch.zeros(6, device=DEV),
                                      softcap=3.0))
        close(outs[-1], outs[0], BF16)
    ops.check_status()


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
    """Several hundred tokens one by one, in captured steps, with states that remember them."""
    cfg = u.config(64, 80, [
        (u.delta(2, 2, 32, 32, 4), u.moe(32, 3, 1, 2)),
        (u.parallel((4, 2, 32, 32, 10.0, (16, 1000.0), None), (2, 32, 48, 12.0)), None),
        (u.window(4, 2, 32, 100, (32, 500.0)), u.moe(16, 2, 2, 1)), 0])
    w = u.weights(cfg, seed=6, peak=0.4)
    for i in (0,):
        w["l%d.mix.dt_bias" % i] = w["l%d.mix.dt_bias" % i] * 0 - 6.0
    path = u.save(tmp_path, cfg, w)
    for dtype in ("bfloat16", "float32"):
        sess = u.session(path, dtype, 704, DEV)
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


def test_states_after_portions_and_after_single_tokens_agree():
    """The state of a 16-bit model's recurrences is fp32: portions (tensor cores, operands of 16 bits)
    leave what one-token steps (fp32 multiply-adds) leave."""
    n = 70
    s, proj, decay, gate, w = delta_case(2, 1, 64, 96, 4, [n], seed=5)
    args = [t.to(DEV) for t in (proj.to(BF16), decay.to(BF16), gate.to(BF16), *w.values())]
    nk, nv = 2 * 64, 2 * 96
    ms = states.MemoryShape(2, 64, 96, 8.0, 0, nk, 2 * nk, 2 * nk + nv, 2 * nk + nv + 2)
    mem = [rnd(n, 2 * nk + nv + 4), rnd(n, nv), rnd(2, dtype=F32), rnd(2, dtype=F32) + 4, rnd(nv, dtype=F32)]
    left = []
    for cuts in ([n], [1] * n):
        S, conv = torch.zeros(2, 2, 64, 96, device=DEV), torch.zeros(2, 2, 3, s.channels, dtype=BF16, device=DEV)
        Z, top = torch.zeros(2, 2, 64, ms.state_cols, device=DEV), torch.zeros(2, 2, 2, device=DEV)
        at = phase = 0
        for k in cuts:
            step = states.StateStep.build(np.asarray([(0, k, 1, at, phase)], dtype=np.int32), DEV)
            r = slice(at, at + k)
            states.delta_scan(*(t[r] for t in args[:3]), *args[3:], s, S, conv, step, 1e-6)
            states.memory_scan(*(t[r] for t in mem[:2]), *mem[2:], ms, Z, top, step, 1e-6)
            at, phase = at + k, phase ^ 1
        left.append((S[1], conv[1, phase].float(), Z[1], top[1, phase]))
    ops.check_status()
    for a, b in zip(*left):
        assert float((a - b).abs().max()) < 1e-4 * float(b.abs().max())
