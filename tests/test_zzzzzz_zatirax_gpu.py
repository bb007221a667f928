"""Zatirax on a GPU: each kernel against an fp64 restatement, then the model through the engine's
step function, captured decode steps and scheduler against the plain restatement."""

import pytest
import torch

import zatirax_oracle as oracle
import zatirax_util as u
from arcticinference_b200 import LLM, SamplingParams, ops
from arcticinference_b200.config import MaskSpec
from arcticinference_b200.ops import head_ops as hd
from arcticinference_b200.ops import latent_ops as lat
from arcticinference_b200.ops import stream_ops as st

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32


def rnd(*shape, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, device=DEV) * scale).to(dtype)


def close(got, want, dtype, scale=1.0):
    want = want.float().to(got.device)
    tol = (0.012 if dtype == BF16 else 3e-5) * scale * max(1.0, float(want.abs().max()))
    err = float((got.float() - want).abs().max())
    assert err < tol, (err, tol)


# ------------------------------------------------------------------ residual stream, feed-forward
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W", [(1, 8), (37, 101), (5, 2048), (3, 6148), (2, 9000), (4, 320)])
def test_stream_sandwich(T, W, dtype):
    torch.manual_seed(W)
    x0, y = rnd(T, W, dtype=F32), rnd(T, W, dtype=dtype)
    w1, w2, v = (rnd(W, dtype=F32) for _ in range(3))
    f = lambda t: t.double().cpu()
    branch = oracle.norm(f(y), w1, 0.05)
    for step in (None, v):
        for write in (True, False):
            x = x0.clone()
            act = torch.empty(T, W, dtype=dtype, device=DEV) if write else None
            st.stream_sandwich(x, y, w1, step, w2 if write else None, act, eps=0.05)
            want = f(x0) + branch + (0 if step is None else f(v))
            close(x.cpu(), want, F32)
            if write:
                close(act.cpu(), oracle.norm(want, w2, 0.05), dtype)
    act = torch.empty(T, W, dtype=dtype, device=DEV)
    x = x0.clone()
    st.stream_sandwich(x, None, None, None, w2, act, eps=0.05)
    assert torch.equal(x, x0)
    close(act.cpu(), oracle.norm(f(x0), w2, 0.05), dtype)
    rows = torch.tensor([T - 1, 0], device=DEV)
    out = st.stream_final_norm(x0, rows, w1, 0.05, dtype, offset=0.0)
    close(out.cpu(), oracle.norm(f(x0), w1, 0.05)[rows.cpu()], dtype)


def test_scaled_embedding():
    table, ids = rnd(50, 77), torch.tensor([3, 49, 0], device=DEV)
    x, act = st.stream_embedding(ids, table, 1.7)
    assert torch.equal(x, table[ids].float() * 1.7) and torch.equal(act, x.to(BF16))
    x, act = st.stream_embedding(ids, table, 0.3, rounded=False)
    assert act is None and torch.equal(x, table[ids].float() * torch.tensor(0.3, device=DEV))


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("limit", [0.8, 7.0])
@pytest.mark.parametrize("T,W,ff", [(3, 96, 40), (300, 264, 200), (700, 136, 16)])
def test_clamped_swish(T, W, ff, limit, dtype):
    torch.manual_seed(ff)
    x = rnd(T, W, dtype=dtype)
    gate, up = (rnd(ff, W, scale=3 * W ** -0.5, dtype=dtype) for _ in range(2))
    got = st.gated_linear(x, st.interleave_gate_up(gate, up), st.Gate("clamped_swish", limit))
    xs = x.double().cpu()
    want = oracle.clamped_swish(oracle.apply(gate, xs), oracle.apply(up, xs), limit)
    close(got[:, :ff].cpu(), want, dtype, 2.0)
    assert float(got[:, ff:].abs().sum()) == 0
    ops.check_status()


# ------------------------------------------------------------------ norms, rotation, cache writes
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,G,dim,vdim,dims,normed", [
    (4, 2, 64, 64, 64, True), (6, 3, 40, 24, 16, True), (3, 1, 7, 11, 6, True),
    (40, 8, 128, 128, 32, True), (2, 2, 96, 128, 2, False), (2, 1, 256, 64, 128, True)])
def test_head_rope_cache(H, G, dim, vdim, dims, normed, dtype):
    torch.manual_seed(dim)
    shape = hd.HeadShape.of(H, G, dim, vdim, dtype)
    D, Dv, bs, T = shape.D, shape.Dv, 16, 6
    rot = u.rotary(dims, 500.0)
    proj = torch.zeros(T, (H + G) * D + G * Dv + 8, dtype=dtype, device=DEV)
    x = rnd(T, H + G, dim, dtype=dtype)
    v = rnd(T, G, vdim, dtype=dtype)
    proj[:, :(H + G) * D].view(T, H + G, D)[:, :, :dim] = x
    proj[:, (H + G) * D:(H + G) * D + G * Dv].unflatten(1, (G, Dv))[:, :, :vdim] = v
    pad = lambda w: torch.cat([w, torch.zeros(D - dim, device=DEV)])
    wq, wk = rnd(dim, dtype=F32), rnd(dim, dtype=F32)
    k, vc = (torch.zeros(3, G, bs, n, dtype=dtype, device=DEV) for n in (D, Dv))
    slots = torch.tensor([47, -1, 0, 17, 16, 5], device=DEV)
    pos = torch.tensor([0, 1, 300, 7, 4000, 63], device=DEV)
    freq = torch.tensor(oracle.frequencies(rot)).float().to(DEV)
    hd.head_rope_cache(proj, shape, dim, pad(wq) if normed else None, pad(wk) if normed else None,
                       hd.rotary_table(pos, freq), 0.02, slots, k, vc)
    ops.check_status()
    for j in range(H + G):
        want = x[:, j].double().cpu()
        if normed:
            want = oracle.norm(want, wq if j < H else wk, 0.02)
        want = oracle.rotate(want, pos.cpu(), rot)
        if j < H:
            got = proj[:, j * D:(j + 1) * D]
            close(got[:, :dim].cpu(), want, dtype, 1.0 if dtype == BF16 else 10.0)
            assert float(got[:, dim:].abs().sum()) == 0
        else:
            for i, s in enumerate(slots.tolist()):
                if s >= 0:
                    close(k[s // bs, j - H, s % bs, :dim].cpu(), want[i], dtype,
                          1.0 if dtype == BF16 else 10.0)
                    assert torch.equal(vc[s // bs, j - H, s % bs, :vdim], v[i, j - H])
    assert int((vc != 0).any(-1).sum()) <= 5 * G        # nothing else was written


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,dim,rot,rank,extra", [(5, 24, 8, 40, 0), (3, 16, 32, 100, 64),
                                                  (2, 3, 2, 13, 0), (16, 128, 64, 512, 64)])
def test_latent_rope_cache(H, dim, rot, rank, extra, dtype):
    torch.manual_seed(rank)
    dq, T, bs = dim + rot + 8, 5, 16
    at = -(-rank // 128) * 128 if extra else rank
    W = at + max(extra, rot)
    W = -(-W // 8) * 8
    r = u.rotary(rot, 300.0)
    buf = rnd(T, H * dq + rank + rot + 6, dtype=dtype)
    start = buf.double().cpu()
    weight, cache = rnd(rank, dtype=F32), torch.zeros(2, 1, bs, W, dtype=dtype, device=DEV)
    slots = torch.tensor([31, 0, -1, 16, 9], device=DEV)
    pos = torch.tensor([0, 5000, 3, 64, 129], device=DEV)
    freq = torch.tensor(oracle.frequencies(r)).float().to(DEV)
    lat.latent_rope_cache(buf, buf[:, H * dq:], H, dq, dim, weight, rank,
                          hd.rotary_table(pos, freq), 0.02, slots, cache, at)
    ops.check_status()
    scale = 1.0 if dtype == BF16 else 10.0
    for h in range(H):
        a = slice(h * dq + dim, h * dq + dim + rot)
        close(buf[:, a].cpu(), oracle.rotate(start[:, a], pos.cpu(), r), dtype, scale)
        assert torch.equal(buf[:, h * dq:h * dq + dim].cpu().double(), start[:, h * dq:h * dq + dim])
    want = torch.zeros(2 * bs, W, dtype=torch.float64)
    c = start[:, H * dq:]
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            want[s, :rank] = oracle.norm(c[:, :rank], weight, 0.02)[i]
            want[s, at:at + rot] = oracle.rotate(c[:, rank:rank + rot], pos.cpu(), r)[i]
    close(cache.view(2 * bs, W).cpu(), want, dtype, scale)


# ------------------------------------------------------------------ attention under masks
MASKS = [MaskSpec(), MaskSpec("window", 1), MaskSpec("window", 64), MaskSpec("window", 131),
         MaskSpec("window", 1000), MaskSpec("chunk", 50), MaskSpec("chunk", 128),
         MaskSpec("chunk", 700)]


def place(lens, bs):
    """Shuffled blocks for sequences of these lengths: (number of blocks, block tables, cache row of
    every token in order)."""
    n_blk = [-(-n // bs) for n in lens]
    order = (torch.randperm(sum(n_blk) + 1) + 1).tolist()
    bt, rows = torch.zeros(len(lens), max(n_blk), dtype=torch.int32), []
    for i, n in enumerate(lens):
        for b in range(n_blk[i]):
            bt[i, b] = order.pop()
        p = torch.arange(n)
        rows.append(bt[i].long()[p // bs] * bs + p % bs)
    return sum(n_blk) + 2, bt.to(DEV), torch.cat(rows).to(DEV)


def targets(mask, pos, kl):
    """Keys to stand out for a token: at and just outside the mask's edge, itself, a block's
    border, the middle."""
    first = int(mask.first_key(pos))
    return [first, max(0, first - 1), pos, pos // 64 * 64, max(0, first - 60), (first + pos) // 2]


def visible_of(mask, n, kl):
    at = torch.arange(kl - n, kl, device=DEV).unsqueeze(1)
    j = torch.arange(kl, device=DEV)
    return (j <= at) & (j >= mask.first_key(at))


CASES = [
    (4, 4, 64, 64, 64, [1, 1, 1], [1, 64, 65]),
    (8, 2, 128, 128, 64, [1] * 20, [300 + 7 * i for i in range(20)]),
    (6, 2, 40, 24, 16, [30, 1, 2], [30, 500, 129]),
    (12, 1, 64, 64, 64, [100], [900]),
    (2, 2, 128, 96, 128, [300, 1], [1200, 3000]),
    (3, 3, 64, 64, 32, [1], [4000]),
    (1, 1, 7, 11, 64, [5, 1], [70, 200]),
    (4, 2, 160, 144, 64, [3, 1], [60, 300]),
    (40, 8, 128, 128, 64, [1] * 3, [2000, 1, 130]),
]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("mask", MASKS)
@pytest.mark.parametrize("H,G,dim,vdim,bs,q_lens,kv_lens", CASES)
def test_head_attention(H, G, dim, vdim, bs, q_lens, kv_lens, mask, dtype):
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
            want = targets(mask, kl - n + j, kl)
            for h in range(H):
                q[t + j, h] = q[t + j, h] * 0.3 + k[o + want[(h + j) % 6], h // (H // G)] * 1.5
        o, t = o + kl, t + n
    sink, gate = rnd(H, dtype=F32) * 2, rnd(T, H * Dv, dtype=dtype)
    seq = torch.repeat_interleave(torch.arange(len(q_lens)), torch.tensor(q_lens)).int().to(DEV)
    pos = torch.cat([torch.arange(a - n, a) for n, a in zip(q_lens, kv_lens)]).to(DEV)
    qp = torch.nn.functional.pad(q, (0, D - dim)).reshape(T, H * D)
    meta = hd.build_plan(shape, q_lens, kv_lens, bt, bs, DEV)
    for s, g in ((sink, gate), (None, None), (sink, None)):
        got = hd.head_attention(qp, kc, vc, meta, shape, scale, s, g, seq, pos)
        ops.check_status()
        o = t = 0
        for n, kl in zip(q_lens, kv_lens):
            ks, vs = (x[o:o + kl].double().repeat_interleave(H // G, 1) for x in (k, v))
            sc = torch.einsum("thd,khd->htk", q[t:t + n].double(), ks) * scale
            sc = sc.masked_fill(~visible_of(mask, n, kl), float("-inf"))
            if s is not None:
                sc = torch.cat([sc, s.double().view(H, 1, 1).expand(H, n, 1)], -1)
            want = torch.einsum("htk,khd->thd", sc.softmax(-1)[..., :kl], vs)
            if g is not None:
                want = want * torch.sigmoid(g[t:t + n].double().view(n, H, Dv)[..., :vdim])
            got_h = got[t:t + n].view(n, H, Dv)
            close(got_h[..., :vdim], want, dtype)
            o, t = o + kl, t + n


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("mask", MASKS)
@pytest.mark.parametrize("H,rank,extra,bs,q_lens,kv_lens", [
    (9, 64, 0, 64, [1, 1, 1], [1, 64, 65]),
    (5, 64, 0, 16, [30, 1, 2], [30, 500, 129]),
    (3, 128, 64, 64, [1, 1, 9], [700, 64, 400]),
    (16, 512, 64, 64, [1] * 4, [2000, 1, 127, 128]),
    (16, 512, 64, 64, [40, 1], [700, 3000]),
    (5, 256, 0, 32, [33, 1, 2], [33, 385, 130]),
    (60, 512, 64, 64, [3, 1], [300, 900]),
    (40, 256, 64, 128, [1, 20], [300, 150]),
    (130, 384, 64, 16, [1, 2], [200, 70]),
    (3, 100, 8, 16, [4, 1], [60, 40]),
])
def test_latent_attention(H, rank, extra, bs, q_lens, kv_lens, mask, dtype):
    torch.manual_seed(H * rank)
    total, T, W = sum(kv_lens), sum(q_lens), rank + extra
    nb, bt, rows = place(kv_lens, bs)
    c = rnd(total, W, dtype=dtype)
    cache = torch.full((nb, 1, bs, W), 37.0, dtype=dtype, device=DEV)
    cache.view(nb * bs, W)[rows] = c
    q, scale = rnd(T, H, W, dtype=dtype), 0.9 * W ** -0.5
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        for j in range(n):
            want = targets(mask, kl - n + j, kl)
            for h in range(H):
                q[t + j, h] = q[t + j, h] * 0.3 + c[o + want[(h + j) % 6]] * 0.35
        o, t = o + kl, t + n
    shape = lat.LatentShape.of(H, rank, dtype, extra, mask)
    meta = lat.build_plan(shape, q_lens, kv_lens, bt, bs, DEV)
    seq = torch.repeat_interleave(torch.arange(len(q_lens)), torch.tensor(q_lens)).int().to(DEV)
    pos = torch.cat([torch.arange(k - n, k) for n, k in zip(q_lens, kv_lens)]).to(DEV)
    got = lat.latent_attention(q.reshape(T, H * W), cache, meta, shape, scale, seq, pos)
    ops.check_status()
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        cs = c[o:o + kl].double()
        s = torch.einsum("thr,kr->htk", q[t:t + n].double(), cs) * scale
        s = s.masked_fill(~visible_of(mask, n, kl), float("-inf")).softmax(-1)
        want = torch.einsum("htk,kr->thr", s, cs[:, :rank]).reshape(n, H * rank)
        close(got[t:t + n], want, dtype)
        o, t = o + kl, t + n


@pytest.mark.parametrize("mask", MASKS)
def test_attention_does_not_depend_on_the_split(mask):
    torch.manual_seed(1)
    lens = [1500, 130, 1]
    nb, bt, _ = place(lens, 64)
    head, latent = hd.HeadShape.of(6, 2, 64, 64, BF16, mask), \
        lat.LatentShape.of(16, 512, BF16, 64, mask)
    q, kc, vc = rnd(3, 6 * 64), rnd(nb, 2, 64, 64), rnd(nb, 2, 64, 64)
    ql, cache = rnd(3, 16 * 576), rnd(nb, 1, 64, 576)
    sink, gate = rnd(6, dtype=F32), rnd(3, 6 * 64)
    outs = {}
    for cap in (1, 2, 5, 16):
        for shape, cls in ((head, hd.HeadDecodePlan), (latent, lat.LatentDecodePlan)):
            plan = cls(shape, 3, 1, 64)
            plan.splits, plan.work_cap = cap, 400
            host = torch.zeros(plan.int32_words, dtype=torch.int32)
            dev = torch.zeros_like(host, device=DEV)
            plan.bind(host.numpy(), dev, bt)
            plan.fill([1, 1, 1], lens)
            dev.copy_(host)
            out = hd.head_attention(q, kc, vc, plan.meta, shape, 0.2, sink, gate) \
                if shape is head else lat.latent_attention(ql, cache, plan.meta, shape, 0.05)
            close(out, outs.setdefault(shape, out), BF16)
    ops.check_status()


# ------------------------------------------------------------------ the model
@pytest.fixture(scope="module", params=sorted(u.CONFIGS))
def model(request, tmp_path_factory):
    cfg = u.CONFIGS[request.param]
    w = u.weights(cfg, seed=3, peak=u.PEAK[request.param])
    return cfg, w, u.save(tmp_path_factory.mktemp(request.param), cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_schedules(model, dtype):
    cfg, w, path = model
    u.check_schedules(cfg, path, dtype, DEV, w)
    ops.check_status()


def test_other_block_sizes_and_eager_steps(model):
    cfg, w, path = model
    for bs in (16, 128):
        u.check_schedules(cfg, path, "bfloat16", DEV, w, names=("mixed", "decode"), block_size=bs,
                          enforce_eager=bs == 16)


def test_captured_steps_are_used(model):
    cfg, w, path = model
    sess = u.session(path, "bfloat16", 256, DEV)
    u.run(sess, {"b": u.tokens(cfg, 20, 2)}, [[("b", 3)]] + [[("b", 1)]] * 17)
    m = sess.engine.runner.model
    assert sess.engine.runner.graph_replays == (17 if m.supports_graphs else 0)


def test_residual_stream_after_every_run(model):
    cfg, w, path = model
    toks, want, got = u.tokens(cfg, 70, 8), [], []
    oracle.forward(cfg, w, toks, want)
    sess = u.session(path, "float32", 128, DEV)
    runner = sess.engine.runner
    forward = runner.model.forward
    runner.model.forward = lambda b, kv: forward(b, kv, layers_out=got)
    sess.step([{"id": "a", "tokens": toks, "want": [0]}], ["a"])
    assert len(got) == len(want)
    for a, b in zip(got, want):
        assert float((a.cpu().double() - b).abs().max()) < 1e-4 * float(b.abs().max())


def test_expanded_form_agrees(tmp_path):
    cfg = u.EXPANDED
    w = u.weights(cfg, seed=4, peak=1.0)
    sess = u.session(u.save(tmp_path, cfg, w), "bfloat16", 64 * 12, DEV)
    m = sess.engine.runner.model
    assert {x.expand for x in m.mixers} >= {(64, 64), (128, 128), (192, 128)}
    m.expand_min_tokens = 20
    seqs = {"a": u.tokens(cfg, 400, 1), "b": u.tokens(cfg, 190, 2), "c": u.tokens(cfg, 30, 3)}
    steps = [[("a", 130), ("b", 2)], [("a", 268), ("b", 40), ("c", 3)],
             [("c", 26), ("b", 148), ("a", 1)], [("c", 1), ("a", 1)]]
    u.compare(cfg, w, u.run(sess, seqs, steps), seqs, "bfloat16")
    ops.check_status()


def test_long_decoding(tmp_path):
    """Several hundred tokens one by one over the borders of pages, windows and chunks, in captured
    steps."""
    cfg = u.config(64, 80, [(u.latent(3, 24, 8, 24, 48, 100), (48, 1.0)),
                            (u.attention(4, 2, 32, 32, 150, u.rotary(16)), (32, 2.0)),
                            (u.latent(4, 16, 16, 16, 140, 300), None),
                            (u.attention(2, 2, 24, 48, 400, u.rotary(24)), None)], loop=(0, 2, 2))
    w = u.weights(cfg, seed=6, peak=1.0)
    path = u.save(tmp_path, cfg, w)
    for dtype in ("bfloat16", "float32"):
        sess = u.session(path, dtype, 704, DEV)
        seqs = {"a": u.tokens(cfg, 640, 1)}
        u.compare(cfg, w, u.run(sess, seqs, [[("a", 4)]] + [[("a", 1)]] * 636), seqs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(model, dtype):
    cfg, w, path = model
    llm = LLM(model=path, device=DEV, dtype=dtype, num_gpu_blocks_override=60, block_size=16,
              max_model_len=256, max_num_batched_tokens=32)
    prompts = [u.tokens(cfg, n, 10 + n) for n in (100, 3, 17, 64, 1)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    ops.check_status()
    for p, ro in zip(prompts, outs):
        toks = ro.outputs[0].token_ids
        assert len(toks) == 12
        z = oracle.forward(cfg, w, (list(p) + toks)[:-1])[len(p) - 1:]
        gap = z.max(-1).values - z.gather(1, torch.tensor(toks).unsqueeze(1)).squeeze(1)
        spread = float((z - z.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        assert float(gap.max()) < (1e-4 if dtype == "float32" else 0.15) * spread


def test_speculation_and_sleep(tmp_path):
    """Suffix drafts verified in one step, and a wake-up from level-2 sleep, change no token."""
    cfg = u.CONFIGS["mixed"]
    path = u.save(tmp_path, cfg, u.weights(cfg, seed=5))
    kw = dict(model=path, device=DEV, dtype="float32", num_gpu_blocks_override=64, block_size=16,
              max_model_len=256)
    p = u.tokens(cfg, 6, 1) * 6
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    plain = LLM(**kw)
    want = plain.generate({"prompt_token_ids": p}, sp)[0].outputs[0].token_ids
    plain.sleep(2)
    plain.wake_up()
    assert plain.generate({"prompt_token_ids": p}, sp)[0].outputs[0].token_ids == want
    spec = LLM(speculative_config={"method": "suffix"}, **kw)
    for _ in range(2):
        assert spec.generate({"prompt_token_ids": p}, sp)[0].outputs[0].token_ids == want
    assert spec.engine.get_stats()["draft_tokens"] > 0
    ops.check_status()
