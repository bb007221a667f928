"""Small Zatirax configurations with random weights, and schedules that run them through the
engine's step function for comparison with the plain restatement (``zatirax_oracle``)."""

import torch

import zatirax_oracle as oracle
from taralix_util import error, errors, portions, run, save, session, tokens  # noqa: F401


def rotary(dims, base=10000.0, scaling=None):
    """``scaling``: factor, low, high, original."""
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def attention(heads, kv_heads, dim, vdim, chunk, rot, scale=None):
    return {"type": "attention", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
        "rot": rot, "scale": dim ** -0.5 if scale is None else scale}}


def latent(heads, dim, rot_dim, vdim, rank, window, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
        "mask": {"size": window}, "rot": rotary(rot_dim, base),
        "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def config(width, vocab, layers, loop=None, embedding=1.0, eps=1e-5):
    """``layers``: (layer, (ff, limit) or None); ``loop``: start, stop, times."""
    return {"architecture": "Zatirax", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": embedding},
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "layers": [{**l, "mlp": None if f is None else
                        {"kind": "dense", "ff": f[0], "limit": f[1]}} for l, f in layers]}


# Sizes that differ from each other everywhere, that no kernel tiles by, and that are 1; windows
# and chunks shorter and longer than pages, on their borders and not.
CONFIGS = {
    "mixed": config(160, 211, [
        (attention(6, 2, 40, 24, 37, rotary(16, 500.0, (4.0, 1.0, 4.0, 64))), (136, 1.5)),
        (latent(5, 24, 8, 40, 40, 21), (72, 0.7)),                  # 48 numbers a token
        (attention(4, 4, 64, 64, 64, rotary(64, 9000.0)), None),
        (latent(3, 16, 32, 16, 100, 65, base=300.0), (24, 3.0)),    # 132 numbers a token
        (attention(10, 1, 16, 8, 130, rotary(2), scale=0.4), (40, 2.0))],
        loop=(1, 3, 2), embedding=1.7, eps=0.02),
    "wide_latents": config(128, 130, [
        (latent(20, 32, 32, 64, 200, 90), (96, 2.0)),
        (latent(9, 96, 32, 128, 256, 150), (48, 1.0)),
        (attention(3, 3, 128, 96, 100, rotary(32)), (56, 4.0)),
        (latent(52, 8, 16, 24, 512, 128), None)], embedding=0.3, eps=1e-4),
    "all_looped": config(64, 40, [
        (latent(1, 1, 2, 1, 1, 1, scale=1.0), (1, 1.0)),
        (attention(1, 1, 2, 1, 1, rotary(2), scale=1.0), None),
        (attention(2, 1, 8, 16, 5, rotary(8, 50.0, (2.0, 1.0, 3.0, 20))), (16, 0.5))],
        # (a norm over one number is its sign: eps keeps 16-bit rounding from turning it)
        loop=(0, 3, 3), eps=0.5),
    # rows that are no multiple of 16 bytes, latents and heads beyond the tensor-core kernels
    "odd": config(101, 53, [
        (attention(3, 1, 7, 11, 33, rotary(6, 80.0)), (19, 1.0)),
        (latent(3, 7, 2, 11, 13, 30), (33, 2.5)),
        (attention(4, 2, 160, 144, 70, rotary(40)), None),
        (latent(1, 5, 4, 3, 540, 48), (5, 1.0)),
        (latent(3, 100, 64, 100, 128, 77), (24, 1.0))], loop=(4, 5, 2),
        eps=0.1),
}


# windows long enough that long chunks go through expanded keys and values, and one that is not
EXPANDED = config(128, 90, [
    (latent(5, 16, 16, 24, 200, 150), (48, 1.0)),
    (latent(3, 96, 32, 128, 480, 200), None),
    (latent(4, 128, 64, 128, 500, 250), (56, 2.0)),
    (latent(2, 72, 64, 40, 300, 260), None),
    (latent(6, 40, 24, 32, 160, 30), None),
    (attention(4, 2, 64, 64, 120, rotary(32)), None)], eps=1e-3)

# how far single keys stand out (heads of a few dimensions do by themselves, in 16 bits too far)
PEAK = {"mixed": 1.0, "wide_latents": 1.0, "all_looped": 1.0, "odd": 0.0}


def weights(cfg, seed=0, peak=0.0):
    """Random checkpoint tensors. ``peak`` > 0 scales the queries, so that single keys stand out of
    hundreds and a missing or extra one shows."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, add=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (torch.randn(*shape, generator=g) * std + add).to(torch.bfloat16)

    W = cfg["width"]
    put("embed", cfg["vocab"], W, std=1.0)
    put("head", cfg["vocab"], W)
    put("final.norm", W, std=0.2, add=1.0)
    if cfg["loop"]:
        put("loop.step", cfg["loop"]["times"], W, std=0.7)
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], "l%d." % i
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            put(p + n, W, std=0.2, add=1.0)
        if l["type"] == "attention":
            put(p + "mix.q", m["heads"] * m["dim"], W)
            put(p + "mix.k", m["kv_heads"] * m["dim"], W)
            put(p + "mix.v", m["kv_heads"] * m["vdim"], W)
            put(p + "mix.q.norm", m["dim"], std=0.3, add=1.0 + peak)
            put(p + "mix.k.norm", m["dim"], std=0.3, add=1.0)
            put(p + "mix.sink", m["heads"], std=1.5)
            put(p + "mix.g", m["heads"] * m["vdim"], W)
        else:
            put(p + "mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), W, std=W ** -0.5 * (1.0 + peak))
            put(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W)
            put(p + "mix.dkv.norm", m["kv_rank"], std=0.2, add=1.0)
            put(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"])
            put(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        put(p + "mix.o", W, m["heads"] * m["vdim"])
        if f:
            put(p + "mlp.gate", f["ff"], W, std=2.0 * W ** -0.5)
            put(p + "mlp.up", f["ff"], W, std=2.0 * W ** -0.5)
            put(p + "mlp.down", W, f["ff"])
    return w


TOLERANCE = {"float32": 2e-5, "bfloat16": 0.06}


def compare(cfg, w, got, seqs, dtype):
    for i, s in seqs.items():
        e = errors(got[i], oracle.forward(cfg, w, s))
        assert float(e.max()) < TOLERANCE[dtype], (i, dtype, int(e.argmax()), float(e.max()))


def schedules(cfg):
    """(name, sequences, steps): whole prompts, token by token, portions down to two tokens (cuts
    inside and at the borders of pages, windows and chunks), and batches of unequal requests whose
    pages are used again."""
    a, b, c, d = tokens(cfg, 190, 1), tokens(cfg, 70, 2), tokens(cfg, 1, 3), tokens(cfg, 129, 4)
    yield "whole", {"a": a, "c": c}, [[("a", 190)], [("c", 1)]]
    yield "decode", {"b": b}, [[("b", 3)]] + [[("b", 1)]] * 67
    yield "portions", {"a": a}, [[("a", n)] for n in portions(190, [2, 61, 1, 2, 3, 7, 64])]
    steps = [[("a", 60), ("b", 2)], [("a", 4), ("b", 62), ("d", 128)], [("b", 1), ("a", 1), ("c", 1)],
             [("d", 1), ("a", 63), ("b", 5)], [("a", 62)], [("e", 65)], [("f", 1), ("e", 64)],
             [("f", 128)]]
    seqs = {"a": a, "b": b, "c": c, "d": d, "e": tokens(cfg, 129, 5), "f": tokens(cfg, 129, 6)}
    yield "mixed", seqs, steps


def check_schedules(cfg, path, dtype, device, w, names=None, **kw):
    for name, seqs, steps in schedules(cfg):
        if names is None or name in names:
            sess = session(path, dtype, 64 * 10, device, **dict(kw))
            compare(cfg, w, run(sess, seqs, steps), seqs, dtype)
            pool = sess.engine.kv_manager.pool
            assert pool.num_free == pool.num_blocks - 1      # everything was given back
