"""Small Pefivik configurations with random weights, and schedules that run them through the engine's
step function for comparison with the plain restatement (``pefivik_oracle``)."""

import torch

import pefivik_oracle as oracle
import pererax_util
from taralix_util import error, errors, portions, run, save, session, tokens  # noqa: F401


def latent(heads, dim, vdim, rank, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank,
        "scale": dim ** -0.5 if scale is None else scale}}


def hgrn2(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups, shared, scale=1.7):
    """``groups``: (how many, how many of them can be chosen from); ``shared``: ff or None."""
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {
        "experts": experts, "top": top, "scale": scale,
        "groups": dict(zip(("count", "keep"), groups))}}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def config(width, vocab, layers, loop, bigram, mult, cap, eps=1e-5):
    """``layers``: (mixer, feed-forward or None) each; ``loop``: (start, stop, times) or None;
    ``bigram``: (buckets, mul_prev, mul_cur)."""
    return {"architecture": "Pefivik", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
            "residual_mult": mult, "logit_softcap": cap,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "layers": [{**m, "mlp": f} for m, f in layers]}


# Sizes that differ from each other everywhere, that no kernel tiles by, and that are 1; every kind of
# layer first, last and repeated; groups of one expert, of two and of more, all of them kept or one.
CONFIGS = {
    "mixed": config(160, 211, [
        (latent(6, 24, 40, 56, 0.3), moe(40, 12, 3, (4, 2), 72)),
        (hgrn2(3, 40, 24), dense(136)),
        (latent(3, 72, 16, 72, 0.21), None),
        (hgrn2(6, 24, 56), moe(24, 6, 2, (3, 1), 40, scale=0.8)),
        (latent(10, 40, 8, 72), dense(88))], loop=(1, 4, 3), bigram=(97, 5, 12), mult=0.4, cap=3.0,
        eps=0.01),
    # latents of several hundred columns (long prompts go through expanded keys and values)
    "wide_latents": config(128, 130, [
        (latent(5, 64, 64, 200), dense(96)),
        (latent(20, 32, 64, 500), moe(48, 8, 4, (2, 2), 24)),
        (latent(3, 96, 128, 130), None)], loop=(0, 2, 2), bigram=(211, 7, 90), mult=0.7, cap=12.0,
        eps=1e-4),
    "states": config(96, 60, [
        (hgrn2(2, 64, 64), moe(32, 9, 4, (3, 2), 40)),
        (hgrn2(4, 16, 72), dense(64)),
        (hgrn2(3, 128, 128), None)], loop=None, bigram=(50, 1, 1), mult=1.0, cap=2.0, eps=1e-3),
    # rows that are no multiple of 16 bytes, sizes beyond the tensor-core kernels
    "odd": config(101, 53, [
        (hgrn2(3, 7, 11), moe(19, 5, 2, (5, 3), 33)),
        (latent(3, 7, 11, 13), dense(37)),
        (latent(1, 5, 3, 540), None),
        (hgrn2(2, 200, 170), dense(1))], loop=(1, 3, 2), bigram=(1, 3, 2), mult=0.25, cap=40.0, eps=0.05),
    "ones": config(64, 40, [
        (latent(1, 1, 1, 1, 1.0), moe(1, 1, 1, (1, 1), 1)),
        (hgrn2(1, 1, 1), dense(1))], loop=(0, 1, 1), bigram=(3, 1, 0), mult=1.0, cap=1.0, eps=0.5),
}

# how far single keys stand out (in 16 bits too far means that rounding picks another)
PEAK = {"mixed": (3.0, 0.6), "wide_latents": (3.0, 0.6), "states": (0.0, 0.0), "odd": (1.0, 0.0),
        "ones": (0.0, 0.0)}


def peak(name, dtype):
    return PEAK[name][dtype == "bfloat16"]


def weights(cfg, seed=0, peak=0.0):
    """Random checkpoint tensors. ``peak`` > 0 scales the query maps, so that single keys stand out of
    hundreds and a missing or extra one shows. Sinks run from none to more than the keys together;
    forget gates from ones that erase a channel in a token to ones that keep it for hundreds."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, add=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        w[name] = (torch.randn(shape, generator=g) * std + add).to(torch.bfloat16)

    def spread(name, lo, hi, *shape):
        w[name] = (torch.rand(shape, generator=g) * (hi - lo) + lo).to(torch.bfloat16)

    W, b = cfg["width"], cfg["embedding"]["bigram"]
    put("embed", cfg["vocab"], W, std=1.0)
    put("bigram", b["buckets"] + 1, W, std=0.8)
    put("head", cfg["vocab"], W, std=1.5 * W ** -0.5)
    spread("final.norm", 0.7, 1.4)
    if cfg["loop"] is not None:
        put("loop.step", cfg["loop"]["times"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], "l%d." % i
        for n in ("norm1",) + (("norm2",) if f else ()):
            spread(p + n, 0.7, 1.4)
        p += "mix."
        if l["type"] == "latent_attention":
            put(p + "q", m["heads"] * m["dim"], W, std=W ** -0.5 * (1.0 + peak))
            put(p + "dkv", m["kv_rank"], W)
            put(p + "dkv.norm", m["kv_rank"], std=0.2, add=1.0)
            put(p + "uk", m["heads"] * m["dim"], m["kv_rank"])
            put(p + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            spread(p + "sink", -2.0, 5.0, m["heads"])
            put(p + "g", m["heads"], W, std=1.5 * W ** -0.5)
        else:
            nk = m["heads"] * m["dim"]
            for x, n in (("q", nk), ("f", nk), ("v", m["heads"] * m["vdim"])):
                put(p + x, n, W)
            spread(p + "f.b", -4.0, 6.0, nk)
            spread(p + "lower", 0.0, 0.8, nk)
            put(p + "norm", m["vdim"], std=0.2, add=1.0)
        put(p + "o", W, m["heads"] * m["vdim"], std=1.5 * (m["heads"] * m["vdim"]) ** -0.5)
        if not f:
            continue
        p = "l%d.mlp." % i
        if f["kind"] == "dense":
            put(p + "up", f["ff"], W)
            put(p + "up.b", f["ff"], std=0.5)
            put(p + "down", W, f["ff"])
            put(p + "down.b", W, std=0.5)
            w[p + "act"] = torch.tensor([0.6, -0.5, 0.4, 0.3]).to(torch.bfloat16)
            continue
        put(p + "router", f["router"]["experts"], W, std=1.5 * W ** -0.5)
        parts = {"e%d." % e: f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f.get("shared"):
            parts["shared."] = f["shared"]["ff"]
        for q, ff in parts.items():
            put(p + q + "gate", ff, W, std=2.0 * W ** -0.5)
            put(p + q + "up", ff, W, std=2.0 * W ** -0.5)
            put(p + q + "down", W, ff)
    return w


TOLERANCE = {"float32": 5e-5, "bfloat16": 0.08}
# In 16 bits a token whose last chosen and first rejected scores (of experts or groups) nearly tie may
# take the other one; such tokens are left out, and some of those that read what they left behind may
# be off.
CLOSE_CALL = 0.01


def compare(cfg, w, got, seqs, dtype):
    for i, s in seqs.items():
        margins = []
        want = oracle.forward(cfg, w, s, margins=margins)
        keep = torch.ones(len(s), dtype=torch.bool)
        if dtype == "bfloat16" and margins:
            keep = torch.stack(margins).min(0).values > CLOSE_CALL
            assert len(s) < 8 or keep.double().mean() > 0.4
            if not keep.any():
                continue
        e = errors(got[i][keep], want[keep]).sort(descending=True).values
        swapped = dtype == "bfloat16" and not bool(keep.all())
        spared = e.numel() // 8 if swapped else 0
        assert float(e[spared]) < TOLERANCE[dtype], (i, dtype, e[:8].tolist())
        assert float(e[0]) < TOLERANCE[dtype] * (6 if swapped else 1), (i, dtype, e[:8].tolist())


schedules = pererax_util.schedules      # portions cut pages, tiles and pairs of tokens


def check_schedules(cfg, path, dtype, device, w, names=None, **kw):
    for name, seqs, steps in schedules(cfg):
        if names is None or name in names:
            sess = session(path, dtype, 64 * 10, device, **dict(kw))
            compare(cfg, w, run(sess, seqs, steps), seqs, dtype)
            kv = sess.engine.kv_manager      # everything was given back
            assert kv.pool.num_free == kv.pool.num_blocks - 1
            assert kv.states is None or len(kv.states.free) == kv.states.num_slots - 1
