"""Taralix on a GPU: each kernel against an fp32 restatement, then the model through the engine's
step function, captured decode steps and scheduler against the plain restatement."""

import pytest
import torch

import taralix_oracle as oracle
import taralix_util as u
from arcticinference_b200 import LLM, SamplingParams, ops
from arcticinference_b200.ops import latent_ops as lat
from arcticinference_b200.ops import stream_ops as st

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
BF16, F32 = torch.bfloat16, torch.float32


def rnd(*shape, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, device=DEV) * scale).to(dtype)


def close(got, want, dtype, scale=1.0):
    want = want.float()
    tol = (0.012 if dtype == BF16 else 3e-5) * scale * max(1.0, float(want.abs().max()))
    err = float((got.float() - want).abs().max())
    assert err < tol, (err, tol)


# ------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W", [(1, 8), (37, 101), (5, 2048), (3, 6148), (2, 20000)])
def test_stream_norm(T, W, dtype):
    torch.manual_seed(W)
    x0, y, w = rnd(T, W, dtype=F32), rnd(T, W, dtype=dtype), rnd(W, scale=0.3, dtype=F32)
    x, act = x0.clone(), torch.empty(T, W, dtype=dtype, device=DEV)
    if dtype == F32:
        act = x
    st.stream_norm(x, act, y, w, 1.7, 0.05)
    want = oracle.zero_centred_norm(1.7 * x0.double().cpu() + y.double().cpu(), w, 0.05)
    close(x.cpu(), want, F32)
    close(act.cpu(), want, dtype)
    rows = torch.tensor([T - 1, 0, T - 1], device=DEV)
    out = st.stream_final_norm(x0, rows, w, 0.05, dtype)
    close(out.cpu(), oracle.zero_centred_norm(x0.double().cpu(), w, 0.05)[rows.cpu()], dtype)


@pytest.mark.parametrize("rank,ld", [(72, 300), (600, 800), (13, 77)])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_stream_embedding_and_latent_cache(dtype, rank, ld):
    torch.manual_seed(1)
    table, ids = rnd(50, 77, dtype=dtype), torch.tensor([3, 49, 0, 3], device=DEV)
    x, act = st.stream_embedding(ids, table)
    assert torch.equal(x, table[ids].float()) and torch.equal(act, table[ids])
    buf, w = rnd(6, ld, dtype=dtype), rnd(rank, dtype=F32)
    off, Rp = ld - rank - ld % 4, -(-rank // 128) * 128
    cache = torch.zeros(3, 1, 16, Rp, dtype=dtype, device=DEV)
    slots = torch.tensor([47, -1, 0, 17, 16, 5], device=DEV)
    lat.latent_norm_cache(buf[:, off:], w, rank, 0.02, slots, cache)
    want = torch.zeros(48, Rp)
    c = oracle.plain_norm(buf[:, off:off + rank].double().cpu(), w, 0.02).float()
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            want[s, :rank] = c[i]
    close(cache.view(48, Rp).cpu(), want, dtype)
    ops.check_status()


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("T,W,ff", [(3, 96, 40), (300, 264, 200), (700, 136, 16)])
def test_gated_linear(T, W, ff, act, dtype):
    torch.manual_seed(ff)
    x = rnd(T, W, dtype=dtype)
    gate, up = (rnd(ff, W, scale=W ** -0.5, dtype=dtype) for _ in range(2))
    w = st.interleave_gate_up(gate, up)
    got = st.gated_linear(x, w, act)
    f = oracle.silu if act == "silu" else oracle.gelu_tanh
    want = f(oracle.apply(gate, x.double().cpu())) * oracle.apply(up, x.double().cpu())
    assert got.shape[1] == -(-ff // 16) * 16
    close(got[:, :ff].cpu(), want, dtype, 2.0)
    assert float(got[:, ff:].abs().sum()) == 0
    ops.check_status()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W,ff,E,top", [(1, 64, 24, 4, 2), (5, 101, 19, 3, 3), (9, 272, 112, 33, 1),
                                          (333, 264, 200, 7, 3), (1500, 128, 48, 40, 6)])
def test_mixture_of_experts(T, W, ff, E, top, dtype):
    torch.manual_seed(E)
    x = rnd(T, W, dtype=F32)
    act = x if dtype == F32 else x.to(BF16)
    router, bias = rnd(E, W, scale=2 * W ** -0.5, dtype=dtype), rnd(E, dtype=F32)
    if E == 7:
        bias[2] = -50.0        # an expert nobody uses
        bias[5] = 50.0         # one that every token uses
    gate, up = (rnd(E, ff, W, scale=W ** -0.5, dtype=dtype) for _ in range(2))
    down = rnd(E, W, ff, scale=ff ** -0.5, dtype=dtype)
    r, rows = st.route(x, act, router, bias, top)
    ids, weights = oracle.route(x.double().cpu(), router, bias, top)
    margin = oracle.route_margin(x.double().cpu(), router, bias, top)
    sure = margin > 1e-4
    assert sure.double().mean() > 0.98
    assert torch.equal(r.ids.cpu().sort(-1).values[sure], ids.int().sort(-1).values[sure])
    close(r.weights.cpu().sum(-1), torch.ones(T), F32)
    by_id = lambda i, v: v.float().gather(1, i.long().argsort(-1))
    close(by_id(r.ids.cpu(), r.weights.cpu())[sure], by_id(ids, weights)[sure], F32)
    # every (token, choice) has a row of its own, inside its expert's range, with its activations
    flat = r.rows.flatten().long().cpu()
    assert torch.equal(flat.sort().values, torch.arange(T * top))
    assert torch.equal(rows[r.rows.flatten().long()], act.repeat_interleave(top, 0))
    n = int(r.num_tiles)
    owner = torch.full((T * top,), -1)
    for e, row0, cnt, _ in r.tiles[:n].tolist():
        assert 0 < cnt <= 128 and (owner[row0:row0 + cnt] == -1).all()
        owner[row0:row0 + cnt] = e
    assert torch.equal(owner[flat], r.ids.flatten().long().cpu())
    h = st.grouped_linear(rows, st.interleave_gate_up(gate, up), r, act="silu")
    ffp = -(-ff // 16) * 16
    dp = torch.zeros(E, W, ffp, dtype=dtype, device=DEV)
    dp[:, :, :ff] = down
    y = st.grouped_linear(h, dp, r)
    x2, a2, nw = x.clone(), torch.empty_like(act), rnd(W, scale=0.2, dtype=F32)
    if dtype == F32:
        a2 = x2
    st.stream_norm(x2, a2, y, nw, 0.8, 1e-3, experts=r)
    ops.check_status()
    w = {"router": router, "router.b": bias}
    for e in range(E):
        w.update({"e%d.gate" % e: gate[e], "e%d.up" % e: up[e], "e%d.down" % e: down[e]})
    some = torch.nonzero(sure).flatten()[:: max(1, T // 60)]
    want = oracle.mixture(act.double().cpu()[some], w, "", top)
    want = oracle.zero_centred_norm(0.8 * x.double().cpu()[some] + want, nw, 1e-3)
    # (the oracle routes the rounded activations: leave out tokens that rounding may swap)
    keep = margin[some] > (0.05 if dtype == BF16 else 1e-4)
    close(x2.cpu()[some][keep], want[keep], dtype, 2.0)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 24, 56), (70, 5, 64, 128), (130, 16, 128, 512),
                                     (9, 2, 7, 13), (300, 1, 40, 8)])
def test_head_linear(T, H, K, N, dtype):
    torch.manual_seed(N)
    buf = rnd(T, H * K + 16, dtype=dtype)
    x, w = buf[:, :H * K], rnd(H, N, K, scale=K ** -0.5, dtype=dtype)
    got = st.head_linear(x, w)
    want = torch.einsum("thk,hnk->thn", x.reshape(T, H, K).double(), w.double()).reshape(T, H * N)
    close(got, want, dtype)
    ops.check_status()


# ------------------------------------------------------------------ attention in latent space
def _paged(c, lens, bs, R):
    """Latents of each sequence in shuffled blocks of a cache; unused rows hold large values (a
    key past the end of a sequence must not be seen)."""
    n_blk = [-(-n // bs) for n in lens]
    nb = sum(n_blk) + 2
    cache = torch.full((nb, 1, bs, R), 37.0, dtype=c.dtype, device=DEV)
    order = (torch.randperm(nb - 1) + 1).tolist()
    bt = torch.zeros(len(lens), max(n_blk), dtype=torch.int32)
    o = 0
    for i, n in enumerate(lens):
        for b in range(n_blk[i]):
            bt[i, b] = order.pop()
            rows = min(bs, n - b * bs)
            cache[bt[i, b], 0, :rows] = c[o + b * bs:o + b * bs + rows]
        o += n
    return cache, bt.to(DEV)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,R,bs,q_lens,kv_lens", [
    (9, 64, 64, [1, 1, 1], [1, 64, 65]),
    (5, 64, 16, [30, 1, 2], [30, 500, 129]),
    (12, 64, 64, [100], [300]),
    (1, 128, 16, [1, 3], [257, 128]),
    (16, 512, 64, [1] * 4, [2000, 1, 127, 128]),
    (16, 512, 64, [7, 1], [700, 3000]),
    (5, 256, 64, [33, 1, 2], [33, 385, 130]),
    (20, 384, 32, [2, 1], [140, 999]),
    (40, 256, 128, [1, 1], [300, 5]),
    (130, 128, 64, [1, 2], [200, 70]),
    (64, 512, 64, [2], [1000]),
    (3, 100, 16, [4, 1], [60, 40]),
])
def test_latent_attention(H, R, bs, q_lens, kv_lens, dtype):
    torch.manual_seed(H * R)
    total = sum(kv_lens)
    c = rnd(total, R, dtype=dtype)
    cache, bt = _paged(c, kv_lens, bs, R)
    T = sum(q_lens)
    q = rnd(T, H * R, dtype=dtype)
    scale = 0.9 * R ** -0.5
    # single keys that stand out: the first one, the token itself and block borders
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        for j in range(n):
            pos = kl - n + j
            for h in range(H):
                key = (0, pos, pos // bs * bs, max(0, pos // bs * bs - 1), pos // 2)[h % 5]
                v = q[t + j].view(H, R)
                v[h] = v[h] * 0.3 + c[o + key] * 0.35
        o, t = o + kl, t + n
    shape = lat.LatentShape.of(H, R, dtype)
    meta = lat.build_plan(shape, q_lens, kv_lens, bt, bs, DEV)
    seq = torch.repeat_interleave(torch.arange(len(q_lens)), torch.tensor(q_lens)).int().to(DEV)
    pos = torch.cat([torch.arange(k - n, k) for n, k in zip(q_lens, kv_lens)]).to(DEV)
    got = lat.latent_attention(q, cache, meta, shape, scale, seq, pos)
    ops.check_status()
    o = t = 0
    for n, kl in zip(q_lens, kv_lens):
        cs = c[o:o + kl].double()
        s = torch.einsum("thr,kr->htk", q[t:t + n].reshape(n, H, R).double(), cs) * scale
        mask = torch.arange(kl, device=DEV) > torch.arange(kl - n, kl, device=DEV).unsqueeze(1)
        s = s.masked_fill(mask, float("-inf")).softmax(-1)
        want = torch.einsum("htk,kr->thr", s, cs).reshape(n, H * R)
        close(got[t:t + n], want, dtype)
        o, t = o + kl, t + n


@pytest.mark.parametrize("splits", [1, 2, 5, 16])
@pytest.mark.parametrize("H,R", [(7, 64), (16, 512), (24, 128)])
def test_latent_attention_does_not_depend_on_the_split(H, R, splits):
    torch.manual_seed(splits)
    lens = [1500, 130, 1]
    c = rnd(sum(lens), R)
    cache, bt = _paged(c, lens, 64, R)
    q = rnd(3, H * R)
    shape = lat.LatentShape.of(H, R, BF16)
    outs = []
    for cap in (1, splits):
        plan = lat.LatentDecodePlan(shape, 3, 1, 64)
        plan.splits, plan.work_cap = cap, 400
        host = torch.zeros(plan.int32_words, dtype=torch.int32)
        dev = torch.zeros_like(host, device=DEV)
        plan.bind(host.numpy(), dev, bt)
        plan.fill([1, 1, 1], lens)
        dev.copy_(host)
        outs.append(lat.latent_attention(q, cache, plan.meta, shape, R ** -0.5))
    ops.check_status()
    close(outs[1], outs[0], BF16)


# ------------------------------------------------------------------ the model
@pytest.fixture(scope="module", params=sorted(u.CONFIGS))
def model(request, tmp_path_factory):
    cfg = u.CONFIGS[request.param]
    w = u.weights(cfg, seed=3, peak=1.0)
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
    seqs = {"b": u.tokens(cfg, 20, 2)}
    u.run(sess, seqs, [[("b", 3)]] + [[("b", 1)]] * 17)
    m = sess.engine.runner.model
    assert sess.engine.runner.graph_replays == (17 if m.supports_graphs else 0)


def test_residual_stream_after_every_layer(model):
    cfg, w, path = model
    toks = u.tokens(cfg, 70, 8)
    want = []
    oracle.forward(cfg, w, toks, want)
    sess = u.session(path, "float32", 128, DEV)
    runner, got = sess.engine.runner, []
    forward = runner.model.forward
    runner.model.forward = lambda b, kv: forward(b, kv, layers_out=got)
    sess.step([{"id": "a", "tokens": toks, "want": [0]}], ["a"])
    assert len(got) == len(want)
    for a, b in zip(got, want):
        assert float((a.cpu().double() - b).abs().max()) < 1e-4 * float(b.abs().max())


def test_expanded_form_agrees(tmp_path):
    cfg = u.CONFIGS["wide_latents"]
    w = u.weights(cfg, seed=4, peak=1.0)
    sess = u.session(u.save(tmp_path, cfg, w), "bfloat16", 64 * 9, DEV)
    m = sess.engine.runner.model
    assert m.expand_min_tokens is not None
    m.expand_min_tokens = 20
    seqs = {"a": u.tokens(cfg, 200, 1), "b": u.tokens(cfg, 190, 2), "c": u.tokens(cfg, 30, 3)}
    steps = [[("a", 130), ("b", 2)], [("a", 68), ("b", 40), ("c", 3)],
             [("c", 26), ("b", 148), ("a", 1)], [("c", 1), ("a", 1)]]
    u.compare(cfg, w, u.run(sess, seqs, steps), seqs, "bfloat16")
    ops.check_status()


def test_long_decoding(tmp_path):
    """Several hundred tokens one by one over page borders, in captured steps."""
    cfg = u.config(64, 80, [(u.attention(3, 32, 24, 48), u.moe(32, 4, 2)),
                            (u.attention(2, 24, 32, 48, src=0), u.dense(48)),
                            (u.attention(4, 16, 16, 140), None)], alpha=1.6)
    w = u.weights(cfg, seed=6, peak=2.0)
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
        margins = []
        z = oracle.forward(cfg, w, (list(p) + toks)[:-1], margins=margins)[len(p) - 1:]
        gap = z.max(-1).values - z.gather(1, torch.tensor(toks).unsqueeze(1)).squeeze(1)
        spread = float((z - z.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        if dtype == "float32":
            assert float(gap.max()) < 1e-4 * spread
        else:       # the largest logit within rounding, but for close calls of a router
            assert float(gap.median()) < 0.1 * spread
            assert (gap < 0.1 * spread).double().mean() > 0.7


def test_speculation_and_sleep(tmp_path):
    """Suffix drafts verified in one step, and a wake-up from level-2 sleep, change no token."""
    cfg = u.CONFIGS["mixed"]
    w = u.weights(cfg, seed=5)
    path = u.save(tmp_path, cfg, w)
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
