"""Prefill and decode throughput of layer-list decoders (Taralix, Zatirax, Pererax, Pefivik) beside Llama
layers of equal size (random weights), with the device time of every op and the time its roofline allows.

    python bench.py --workload layers [--layer-case NAME]       (or: python benchmarks/layer_bench.py)

Cases (width, heads x (dim, vdim), kv_rank, feed-forward):

    moe-2048     2048, 16 x (128, 128), 512, 64 experts of 1408, 6 per token   (Taralix, Pererax, Pefivik)
    moe-4096     4096, 32 x (128, 128), 512, 64 experts of 2048, 6 per token   (Taralix, Pererax, Pefivik)
    dense-2560   2560, 40 x (64, 64),   256, 6400                      (Taralix, Zatirax, Pefivik)
    dense-4096   4096, 32 x (128, 128), 512, 14336                     (Taralix, Zatirax, Pefivik)
    masks-4096   dense-4096 with windows and chunks of 1024 positions          (Zatirax)

Taralix: every second layer shares the latents of the one before it. Zatirax: attention layers with
8 K/V heads (a quarter of the dimensions rotated) alternate with latent layers that add a rotated
key part of 64; windows and chunks of 4096 positions, which hold every context here, but in
masks-4096. Pererax: delta-rule layers (every head with keys of its own), attention beside a matrix
memory, and windowed attention (1024 positions), the attentions with 8 K/V heads; of the experts per
token one is the shared expert and 8 identity experts take part in the choice. Pefivik: latent layers
with sinks and head gates alternate with HGRN2 layers; of the experts per token one is the shared expert,
the others come from 4 of 8 groups; the dense feed-forwards, which have two matrices, are 3/2 as wide. The
Llama beside them has the same width, query heads, head dimension and active feed-forward width, and 8
K/V heads. Prefill: four prompts of 2048 tokens in one step. Decode: 128 sequences at 2000 tokens of
context, captured step. Both are one forward pass without the LM head, timed with CUDA events; the
weights of a pass exceed L2. The roofline of an op is the larger of its algorithmic bytes over the
measured copy bandwidth and its flops over the measured bf16 rate; only visible keys count. The
recurrences compute in fp32: three (delta rule) or two (the others) multiply-adds per state element
and token over the fp32 rate (128 per SM and cycle) are a third bound of theirs; ``of_bytes`` leaves it
out.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, REPO)

CASES = {
    "moe-2048": dict(width=2048, heads=16, dim=128, rank=512, ff=1408, experts=64, top=6),
    "dense-2560": dict(width=2560, heads=40, dim=64, rank=256, ff=6400, experts=0, top=1),
    "dense-4096": dict(width=4096, heads=32, dim=128, rank=512, ff=14336, experts=0, top=1),
    "moe-4096": dict(width=4096, heads=32, dim=128, rank=512, ff=2048, experts=64, top=6),
    "masks-4096": dict(width=4096, heads=32, dim=128, rank=512, ff=14336, experts=0, top=1,
                       mask=1024),
}
LAYERS, VOCAB, KV_HEADS, ROT = 4, 32000, 8, 64
PREFILL = [2048] * 4
DECODE, CONTEXT = 128, 2000


def taralix_config(c):
    from arcticinference_b200.config import ModelConfig
    mlp = {"kind": "dense", "ff": c["ff"]} if not c["experts"] else \
        {"kind": "moe", "expert": {"ff": c["ff"]},
         "router": {"experts": c["experts"], "top": c["top"]}}
    layers = []
    for i in range(LAYERS):
        m = {"heads": c["heads"], "dim": c["dim"], "vdim": c["dim"], "kv_rank": c["rank"],
             "scale": c["dim"] ** -0.5}
        if i % 2:
            m["kv_from"] = i - 1
        layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return ModelConfig.from_layer_list({
        "architecture": "Taralix", "width": c["width"], "vocab": VOCAB, "norm": {"eps": 1e-6},
        "postln_alpha": 1.5, "layers": layers})


def zatirax_config(c):
    from arcticinference_b200.config import ModelConfig
    H, d, size = c["heads"], c["dim"], c.get("mask", 4096)
    rot = lambda n: {"base": 10000.0, "dims": n}
    attn = {"type": "attention", "mixer": {
        "heads": H, "kv_heads": KV_HEADS, "dim": d, "vdim": d, "scale": d ** -0.5,
        "mask": {"size": size}, "rot": {**rot(d // 4), "scaling": {
            "factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    latent = {"type": "latent_attention", "mixer": {
        "heads": H, "dim": d, "rot_dim": ROT, "vdim": d, "kv_rank": c["rank"],
        "scale": (d + ROT) ** -0.5, "mask": {"size": size}, "rot": rot(ROT)}}
    mlp = {"kind": "dense", "ff": c["ff"], "limit": 7.0}
    # runs: attention, latent, attention, latent
    layers = [attn, latent, attn, latent][:LAYERS]
    return ModelConfig.from_layer_list({
        "architecture": "Zatirax", "width": c["width"], "vocab": VOCAB, "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.0}, "loop": None,
        "layers": [{**l, "mlp": mlp} for l in layers]})


def pererax_config(c):
    from arcticinference_b200.config import ModelConfig
    H, d = c["heads"], c["dim"]
    rot = {"base": 10000.0, "dims": d}
    attn = {"heads": H, "kv_heads": KV_HEADS, "dim": d, "vdim": d, "scale": d ** -0.5, "rot": rot}
    delta = {"type": "channel_delta", "mixer": {"heads": H, "kv_heads": H, "dim": d, "vdim": d, "conv": 4}}
    both = {"type": "parallel", "mixer": {
        "left": {**attn, "softcap": 30.0},
        "right": {"heads": H // 2, "dim": d // 2, "vdim": d, "gate_cap": 15.0}}}
    window = {"type": "attention", "mixer": {**attn, "mask": {"size": 1024}}}
    mlp = {"kind": "moe", "expert": {"ff": c["ff"], "limit": 7.0},
           "router": {"experts": c["experts"], "identity": 8, "top": c["top"] - 1, "scale": 2.5},
           "shared": {"ff": c["ff"], "limit": 7.0}}
    return ModelConfig.from_layer_list({
        "architecture": "Pererax", "width": c["width"], "vocab": VOCAB, "norm": {"eps": 1e-6},
        "layers": [{**l, "mlp": mlp} for l in (delta, both, window, delta)]})


def pefivik_config(c):
    from arcticinference_b200.config import ModelConfig
    H, d = c["heads"], c["dim"]
    latent = {"type": "latent_attention", "mixer": {
        "heads": H, "dim": d, "vdim": d, "kv_rank": c["rank"], "scale": d ** -0.5}}
    scan = {"type": "hgrn2", "mixer": {"heads": H, "dim": d, "vdim": d}}
    mlp = {"kind": "dense", "ff": c["ff"] * 3 // 2}
    if c["experts"]:
        mlp = {"kind": "moe", "expert": {"ff": c["ff"]}, "shared": {"ff": c["ff"]},
               "router": {"experts": c["experts"], "top": c["top"] - 1, "scale": 2.5,
                          "groups": {"count": 8, "keep": 4}}}
    return ModelConfig.from_layer_list({
        "architecture": "Pefivik", "width": c["width"], "vocab": VOCAB, "norm": {"eps": 1e-6},
        "embedding": {"bigram": {"buckets": 50021, "mul_prev": 10007, "mul_cur": 3}},
        "residual_mult": 0.5, "logit_softcap": 30.0, "loop": None,
        "layers": [{**l, "mlp": mlp} for l in (latent, scan, latent, scan)]})


def model_configs(c):
    from arcticinference_b200.config import ModelConfig
    llama = ModelConfig(hidden_size=c["width"], num_hidden_layers=LAYERS,
                        num_attention_heads=c["heads"], num_key_value_heads=KV_HEADS,
                        head_dim=c["dim"], intermediate_size=c["ff"] * c["top"], vocab_size=VOCAB,
                        max_position_embeddings=8192)
    out = {}
    if c["experts"]:
        out["pererax"] = pererax_config(c)
    else:
        out["zatirax"] = zatirax_config(c)
    if "mask" not in c:
        out["pefivik"] = pefivik_config(c)
        out["taralix"] = taralix_config(c)
        out["llama"] = llama
    return out


def peaks():
    try:
        with open(os.path.join(REPO, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "of measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "of fallback"


def visible_pairs(mask, q_lens, kv_lens):
    """(query, key) pairs that attend, and keys that any query of a sequence sees."""
    import numpy as np
    pairs = keys = 0
    for q, kl in zip(q_lens, kv_lens):
        pos = np.arange(kl - q, kl)
        pairs += int((pos + 1 - mask.first_key(pos)).sum())
        keys += kl - int(mask.first_key(kl - q))
    return pairs, keys


FP32_FMAS = 148 * 128 * 1.965e9      # per second, every SM at its highest clock


def rooflines(model, q_lens, kv_lens, fp32: bool = True):
    """op -> seconds the layers' algorithmic bytes and flops allow (2 bytes per element; ``fp32``: and
    the fp32 multiply-adds of recurrences)."""
    from arcticinference_b200.config import (AttentionSpec, DeltaRuleSpec, ForgetScanSpec, MaskSpec,
                                             ParallelSpec)
    cfg = model.cfg
    hbm, flops, _ = peaks()
    T, S = sum(q_lens), len(q_lens)
    out: dict = {}

    def add(op, nbytes, nflops=0.0, fmas=0.0):
        out[op] = out.get(op, 0.0) + max(nbytes / hbm, nflops / flops, fp32 * fmas / FP32_FMAS)

    def attention(m):
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        pairs, ctx = visible_pairs(m.mask, q_lens, kv_lens)
        add("head_rope_cache", 2.0 * T * (2 * (H + G) * d + (1 if m.values_are_keys else 2) * G * dv))
        add("attention_masked", 2.0 * (ctx * G * (d + dv) + T * H * (d + (2 if m.output_gate else 1) * dv)),
            2.0 * pairs * H * (d + dv))
        linear(W, H * dv)

    def state(H, d, dv):     # read (by sequences that have one) and written
        return 4.0 * S * H * d * dv * (2 if max(q_lens) < max(kv_lens) else 1)

    def delta(m):
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        low, n = model.layers[i].w_low.shape[2], model.layers[i].w_low.shape[1]
        linear(2 * G * d + H * dv + H + 2 * low, W)
        linear(2 * n, low, op="head_linear")
        add("delta_scan", 2.0 * T * (2 * G * d + 3 * H * dv + H * d) + state(H, d, dv),
            fmas=3.0 * T * H * d * dv)
        linear(W, H * dv)

    def forget(m):
        H, d, dv = m.heads, m.dim, m.vdim
        linear(H * (2 * d + dv), W)
        add("forget_scan", 2.0 * T * H * (2 * d + 2 * dv) + state(H, d, dv), fmas=2.0 * T * H * d * dv)
        linear(W, H * dv)

    def parallel(m):
        l, r = m.left, m.right
        linear(l.heads * l.dim + l.kv_heads * (l.dim + l.vdim) + 2 * r.heads * (r.dim + r.vdim + 1), W)
        attention(l)
        add("memory_scan", 2.0 * T * r.heads * (2 * r.dim + 3 * r.vdim) +
            state(r.heads, r.dim, r.vdim + 1), fmas=2.0 * T * r.heads * r.dim * (r.vdim + 1))
        linear(W, r.heads * r.vdim)

    def linear(n, k, rows=T, op="linear", weights=1):
        add(op, 2.0 * (weights * n * k + rows * (n + k)), 2.0 * rows * n * k)

    W = cfg.hidden_size
    decode = max(q_lens) == 1
    if cfg.layer_specs is None:
        H, Hk, D, I = cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim, cfg.intermediate_size
        pairs, ctx = visible_pairs(MaskSpec(), q_lens, kv_lens)
        for _ in range(cfg.num_hidden_layers):
            linear((H + 2 * Hk) * D, W)
            add("rope_cache", 2.0 * T * (2 * (H + Hk) + 3 * Hk) * D)
            add("attention", 2.0 * (2 * ctx * Hk * D + 2 * T * H * D), 4.0 * pairs * H * D)
            linear(W, H * D)
            linear(2 * I, W)
            add("silu_mul_blocked", 2.0 * T * 3 * I)
            linear(W, I)
            add("rmsnorm", 2 * 2.0 * T * 4 * W)
        return out
    norm = {"sandwich": "stream_sandwich", "post": "stream_norm", "output": "stream_add",
            "pre": "stream_pre"}[cfg.design.residual]
    for i, _ in cfg.layer_runs:
        l = cfg.layer_specs[i]
        m, f = l.mixer, l.mlp
        if isinstance(m, DeltaRuleSpec):
            delta(m)
        elif isinstance(m, ForgetScanSpec):
            forget(m)
        elif isinstance(m, ParallelSpec):
            parallel(m)
        elif isinstance(m, AttentionSpec):
            values = 0 if m.values_are_keys else m.kv_heads * m.vdim
            linear(m.heads * m.dim + m.kv_heads * m.dim + values +
                   (m.heads * m.vdim if m.output_gate else 0), W)
            attention(m)
        else:
            H, d, dv = m.heads, m.dim, m.vdim
            masked = m.mask.kind != "causal" or m.sink is not None or m.head_gate
            pairs, ctx = visible_pairs(m.mask, q_lens, kv_lens)
            R, rot = m.kv_rank, m.rot_dim
            own = R + rot if m.kv_from is None else 0
            dq = d + rot
            linear(H * dq + own + (H if m.head_gate else 0), W)
            if rot:
                add("latent_rope_cache", 2.0 * T * 2 * (R + rot + H * rot))
            elif own:
                add("latent_norm_cache", 2.0 * T * 2 * R)
            if decode or not model.mixers[i].expand:
                add("head_linear", 2.0 * (H * R * d + T * H * (dq + R + rot)), 2.0 * T * H * R * d)
                add("latent_attention", 2.0 * (ctx * (R + rot) + T * H * (2 * R + rot)),
                    2.0 * pairs * H * (2 * R + rot))
                add("head_linear", 2.0 * (H * R * dv + T * H * (dv + R)), 2.0 * T * H * R * dv)
            else:
                if own:
                    add("gather_rows", 2.0 * 2 * ctx * (R + rot))
                linear(H * (d + dv), R, rows=ctx)
                add("attention_masked" if masked else "attention_contiguous",
                    2.0 * (ctx + T) * H * (dq + dv), 2.0 * pairs * H * (dq + dv))
            linear(W, H * dv)
        add(norm, T * W * (14.0 if isinstance(m, ParallelSpec) else 12.0))

        def dense(ff):
            linear(2 * ff, W, op="gated_linear" if T > 256 else "linear")
            if T <= 256:
                add("gated_act", 2.0 * T * 3 * ff)
            linear(W, ff)
        if f.experts:
            outputs = f.experts + f.identity
            n = T * f.top * f.experts // outputs     # (identity experts have no rows)
            used = min(f.experts, n)
            add("route", 4.0 * T * W + 2.0 * outputs * W)
            add("_permute", 2.0 * (T + n) * W)
            linear(2 * f.ff, W, rows=n, op="grouped_linear", weights=used)
            linear(W, f.ff, rows=n, op="grouped_linear", weights=used)
            if f.shared is not None:
                dense(f.shared.ff)
            add(norm, T * W * (12.0 if f.shared is not None else 10.0) + 2.0 * n * W)
        elif f.act == "poly_norm":
            linear(f.ff, W)
            add("poly_norm", 2.0 * T * 2 * f.ff)
            linear(W, f.ff)
            add(norm, T * W * 12.0)
        else:
            dense(f.ff)
            add(norm, T * W * 12.0)
    return out


def build_runner(cfg):
    from arcticinference_b200.config import (CacheConfig, EngineConfig, ParallelConfig,
                                             SchedulerConfig)
    from arcticinference_b200.engine.model_runner import ModelRunner
    blocks = max(sum(-(-n // 64) for n in PREFILL), DECODE * (-(-(CONTEXT + 64) // 64))) + 1
    ec = EngineConfig(model=cfg, parallel=ParallelConfig(),
                      cache=CacheConfig(num_gpu_blocks=blocks, enable_prefix_caching=False),
                      scheduler=SchedulerConfig(max_model_len=CONTEXT + 64, max_num_seqs=DECODE),
                      load_format="dummy")
    ec.validate()
    r = ModelRunner(ec, "cuda")
    r.load_model()
    r.init_kv_cache(blocks)
    runs = getattr(r.kv, "runs", None)
    for c in (r.kv.k + r.kv.v if runs is None else [t for run in runs + r.kv.states for t in run]):
        c.normal_()     # a cache, and states, that hold something
    return r


def step_of(lens, new):
    """A scheduler output in which request i has ``lens[i]`` tokens, the last ``new`` of them now."""
    from arcticinference_b200.engine.request import Request
    from arcticinference_b200.engine.sampling_params import SamplingParams
    from arcticinference_b200.engine.scheduler import ScheduledRequest, SchedulerOutput
    out, blk = SchedulerOutput(), 1
    for i, n in enumerate(lens):
        r = Request("r%d" % i, [(7 * i + 13 * j) % VOCAB for j in range(n)],
                    SamplingParams(temperature=0.0))
        k = -(-n // 64)
        r.block_ids = list(range(blk, blk + k))
        r.state_slot = i + 1
        blk += k
        q = n if new is None else new
        out.scheduled.append(ScheduledRequest(r, n - q, q, 0, True))
        out.total_tokens += q
    return out


def timed(fn, warmup=5, reps=20):
    import torch
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = (torch.cuda.Event(enable_timing=True) for _ in range(2))
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def measure(name, cfg):
    import torch
    from arcticinference_b200 import ops
    from arcticinference_b200.engine.cuda_graph import DecodeGraph
    r = build_runner(cfg)
    res = {}
    with torch.inference_mode():
        for phase, lens, new in (("prefill", PREFILL, None), ("decode", [CONTEXT] * DECODE, 1)):
            out = step_of(lens, new)
            batch, _ = r.prepare(out)
            fwd = lambda: r.model.forward(batch, r.kv)
            if phase == "prefill":
                ms = timed(fwd)
            else:
                g = DecodeGraph(r, "tp", DECODE)
                g.fill(out)
                g.upload()
                torch.cuda.synchronize()
                g._body = lambda: (fwd_graph(r, g), None)
                g.capture()
                g.fill(out)     # (capturing leaves the rows without state slots)
                g.upload()
                ms = timed(g.graph.replay)
            with ops.OpTimer() as t:
                for _ in range(5):
                    fwd()
            q = [n if new is None else new for n in lens]
            ideal = rooflines(r.model, q, lens)
            by_bytes = rooflines(r.model, q, lens, fp32=False)
            table = {}
            for op, (us, cnt) in t.summary().items():
                if op == "_start":
                    continue
                row = {"us": round(us / 5, 1), "calls": cnt // 5}
                if op in ideal:
                    row["of_roofline"] = round(1e6 * ideal[op] / (us / 5), 3)
                    if by_bytes[op] < ideal[op]:
                        row["of_bytes"] = round(1e6 * by_bytes[op] / (us / 5), 3)
                table[op] = row
            tokens = sum(q)
            res[phase] = {"ms": round(ms, 4), "tokens_per_s": round(tokens / ms * 1e3),
                          "roofline_ms": round(1e3 * sum(ideal.values()), 4), "ops": table}
    ops.check_status()
    del r
    torch.cuda.empty_cache()
    return res


def fwd_graph(r, g):
    return r.model.forward(g.batch, r.kv)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--layer-case", choices=sorted(CASES), default=None)
    ap.add_argument("--model", choices=["pefivik", "pererax", "zatirax", "taralix", "llama"], default=None)
    ns = ap.parse_args(argv)
    import torch
    torch.cuda.set_device(0)
    for name, c in CASES.items():
        if ns.layer_case not in (None, name):
            continue
        line = {"workload": "layers", "case": name, "layers": LAYERS, **c,
                "peaks": peaks()[2], "prefill_tokens": sum(PREFILL), "decode_batch": DECODE,
                "context": CONTEXT, "data": "random weights and latents", "dtype": "bf16",
                "l2": "weights and cache of a pass exceed L2"}
        for kind, cfg in model_configs(c).items():
            if ns.model in (None, kind):
                line[kind] = measure(name, cfg)
        print(json.dumps(line), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
