"""Taralix: a decoder whose layers are listed one by one, with latent attention (no positions,
latents optionally shared with an earlier layer), dense or mixture-of-experts feed-forwards, and
the norm after each residual sum.

    x <- norm1(alpha * x + attention(x));   x <- norm2(alpha * x + feed_forward(x))

The residual stream ``x`` is fp32 from the embedding to the final norm; the projections read its
rounding to the model's element type, which the same kernel that normalises the stream writes
beside it. Per layer: one projection for the queries and the latent (where the layer has its
own), latent norm + cache write, attention (``ops/latent_ops.py``: in latent space, or through
expanded keys and values for long chunks of wide latents), output projection, sum + norm; then
gate / up with the activation in the product's epilogue, down, sum + norm (for experts the norm
kernel also takes the weighted sum of the chosen experts' rows). Routing stays on the device.

Sizes that the tensor-core kernels tile by are padded with zeros when the weights are packed
(head dimensions, latent width, feed-forward width, vocabulary rows), which changes no value.

Served in bfloat16 or, with every product and sum in IEEE fp32, in float32.
"""

from __future__ import annotations

import re
from typing import Iterable

import numpy as np
import torch

from .. import ops
from ..config import ModelConfig
from ..ops import latent_ops as lat
from ..ops import stream_ops as st
from .llama import ForwardBatch, ShardSpec

_NAME_RE = re.compile(r"^l(\d+)\.(.+)$")
_EXPERT_RE = re.compile(r"^mlp\.e(\d+)\.(gate|up|down)$")

# temporary keys and values of the expanded form, at most (one layer's, reused by the next)
EXPAND_LIMIT_BYTES = 2 << 30

LAYER_TENSORS = ("norm1", "norm2", "wq", "ckv_norm", "wuk_t", "wuv", "wukv", "wo", "w_gu",
                 "w_down", "router", "router_b")


def _up(n: int, m: int) -> int:
    return -(-n // m) * m


class TaralixLayer:
    """Weights and shapes of one layer."""

    __slots__ = LAYER_TENSORS + ("extra", "spec", "source", "shape", "scale", "dq", "dv", "rank", "expand",
                                 "ckv_cols")

    def __init__(self):
        for n in LAYER_TENSORS:
            setattr(self, n, None)
        self.extra = {}

    def tensors(self):
        for name in LAYER_TENSORS:
            t = getattr(self, name)
            if t is not None:
                yield name, t


def required_tensors(spec) -> list:
    """Checkpoint names (without the layer's prefix) of one layer."""
    names = ["norm1", "mix.q", "mix.uk", "mix.uv", "mix.o"]
    if spec.mixer.kv_from is None:
        names += ["mix.dkv", "mix.dkv.norm"]
    if spec.mlp is not None:
        names.append("norm2")
        if spec.mlp.experts:
            names += ["mlp.router", "mlp.router.b"]
            names += ["mlp.e%d.%s" % (e, n) for e in range(spec.mlp.experts)
                      for n in ("gate", "up", "down")]
        else:
            names += ["mlp.gate", "mlp.up", "mlp.down"]
    return names


def random_state(cfg: ModelConfig, seed: int, device, dtype) -> Iterable:
    """(name, tensor) pairs of a random checkpoint: matrices with variance 1 / fan-in, so that
    the normalised stream keeps scores and activations of order one."""
    gen = torch.Generator(device=device)
    count = 0

    def rnd(*shape, std=None):
        nonlocal count
        count += 1
        gen.manual_seed(seed * 1000003 + count)
        std = shape[-1] ** -0.5 if std is None else std
        return (torch.randn(*shape, generator=gen, device=device) * std).to(dtype)

    W = cfg.hidden_size
    yield "embed", rnd(cfg.vocab_size, W, std=1.0)
    yield "head", rnd(cfg.vocab_size, W)
    yield "final.norm", rnd(W, std=0.1)
    for i, l in enumerate(cfg.layer_specs):
        m, f, p = l.mixer, l.mlp, "l%d." % i
        yield p + "norm1", rnd(W, std=0.1)
        yield p + "mix.q", rnd(m.heads * m.dim, W)
        if m.kv_from is None:
            yield p + "mix.dkv", rnd(m.kv_rank, W)
            yield p + "mix.dkv.norm", 1.0 + rnd(m.kv_rank, std=0.1)
        yield p + "mix.uk", rnd(m.heads * m.dim, m.kv_rank)
        yield p + "mix.uv", rnd(m.heads * m.vdim, m.kv_rank)
        yield p + "mix.o", rnd(W, m.heads * m.vdim)
        if f is None:
            continue
        yield p + "norm2", rnd(W, std=0.1)
        if f.experts:
            yield p + "mlp.router", rnd(f.experts, W)
            yield p + "mlp.router.b", rnd(f.experts, std=0.1)
        for q in (["mlp.e%d." % e for e in range(f.experts)] if f.experts else ["mlp."]):
            yield p + q + "gate", rnd(f.ff, W)
            yield p + q + "up", rnd(f.ff, W)
            yield p + q + "down", rnd(W, f.ff)


class TaralixForCausalLM:
    supports_graphs = True

    def __init__(self, cfg: ModelConfig, shard: ShardSpec = None, device="cuda", dtype=None,
                 comm=None):
        if comm is not None:
            raise NotImplementedError("%s on more than one GPU" % cfg.architecture)
        self.cfg = cfg
        self.shard = shard or ShardSpec()
        self.device = torch.device(device)
        self.dtype = dtype or (torch.float32 if cfg.dtype == "float32" else torch.bfloat16)
        self.comm = self.pp = None
        self.layer_lo, self.layer_hi = 0, cfg.num_hidden_layers
        # what the engine asks of any decoder: query heads and cached heads per rank
        self.h, self.hkv = cfg.num_attention_heads, 1
        self.D = cfg.head_dim
        self.layers: list = [None] * cfg.num_hidden_layers
        self.embed = self.norm = self.lm_head = None
        self._lay_out()

    # ------------------------------------------------------------------ shapes
    def _lay_out(self) -> None:
        """Padded sizes of every layer. Layers that share latents agree on their width."""
        specs = self.cfg.layer_specs
        bf16 = self.dtype == torch.bfloat16
        self.owners = [i if l.mixer.kv_from is None else l.mixer.kv_from
                       for i, l in enumerate(specs)]
        self.ranks = []
        for o in self.owners:
            heads = max(l.mixer.heads for l, s in zip(specs, self.owners) if s == o)
            self.ranks.append(lat.padded_rank(specs[o].mixer.kv_rank, heads, self.dtype))
        self._geometry = []
        for l, rank in zip(specs, self.ranks):
            m = l.mixer
            shape = lat.LatentShape.of(m.heads, rank, self.dtype)
            d = max(m.dim, m.vdim)
            expand = None
            if bf16 and shape.kernel != "packed" and d <= 128:
                d = 64 if d <= 64 else 128
                if d <= rank:
                    expand = d
            dq = dv = expand
            if expand is None:
                dq, dv = (_up(m.dim, 8), _up(m.vdim, 8)) if bf16 else (m.dim, m.vdim)
            self._geometry.append((shape, dq, dv, expand))
        # queries per sequence from which expanding its context costs fewer multiply-adds than
        # attending in latent space: q * (rank - d) > rank * d, for the layers together
        gain = sum(2 * l.mixer.heads * (r - e) for l, r, (_, _, _, e)
                   in zip(specs, self.ranks, self._geometry) if e)
        cost = sum(2 * l.mixer.heads * r * e for l, r, (_, _, _, e)
                   in zip(specs, self.ranks, self._geometry) if e)
        expands = any(g[3] for g in self._geometry)
        self.expand_min_tokens = max(128, min(512, cost // gain if gain else 512)) if expands \
            else None
        self._expand_row_bytes = max((2 * l.mixer.heads * e * 2 for l, (_, _, _, e)
                                      in zip(specs, self._geometry) if e), default=0)
        self.shapes = list(dict.fromkeys(g[0] for g in self._geometry))
        # captured steps need a plan per shape; the "exact" kernel and 32-bit models run eagerly
        self.supports_graphs = bf16 and all(s.kernel != "exact" for s in self.shapes)

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0) -> None:
        self.load_state(random_state(self.cfg, seed, self.device, torch.bfloat16))

    def load_weights(self, path: str) -> None:
        from .loader import iter_safetensors_dir
        self.load_state(iter_safetensors_dir(path))

    def load_state(self, state: Iterable) -> None:
        """Consume (name, tensor) pairs in any order; a layer is packed once it is complete."""
        cfg = self.cfg
        pending: dict = {}
        need = [set(required_tensors(l)) for l in cfg.layer_specs]
        for name, t in state:
            if name == "embed":
                self.embed = self._put(t)
            elif name == "final.norm":
                self.norm = self._put(t, torch.float32)
            elif name == "head":
                rows = _up(t.shape[0], 8) if self.dtype == torch.bfloat16 else t.shape[0]
                self.lm_head = self._pad(self._put(t), rows)
            else:
                m = _NAME_RE.match(name)
                if m is None or int(m.group(1)) >= len(need) or \
                        m.group(2) not in need[int(m.group(1))]:
                    raise ValueError("unexpected tensor %r in a %s checkpoint"
                                     % (name, cfg.architecture))
                l = int(m.group(1))
                d = pending.setdefault(l, {})
                d[m.group(2)] = t
                if len(d) == len(need[l]):
                    self.layers[l] = self._pack(l, d)
                    del pending[l]
        missing = [n for n, t in (("embed", self.embed), ("final.norm", self.norm),
                                  ("head", self.lm_head)) if t is None]
        missing += ["l%d.%s" % (l, n) for l, lw in enumerate(self.layers) if lw is None
                    for n in sorted(need[l] - set(pending.get(l, ())))]
        if missing:
            raise ValueError("checkpoint is incomplete: %s" % missing[:8])

    def _put(self, t, dtype=None):
        return t.to(device=self.device, dtype=dtype or self.dtype).contiguous()

    @staticmethod
    def _pad(t, *sizes):
        """Zero-padded to ``sizes`` in the leading dimensions."""
        if all(a == b for a, b in zip(t.shape, sizes)):
            return t
        out = torch.zeros(*sizes, *t.shape[len(sizes):], dtype=t.dtype, device=t.device)
        out[tuple(slice(0, n) for n in t.shape)] = t
        return out

    def _expect(self, t, *shape):
        if tuple(t.shape) != shape:
            raise ValueError("tensor of shape %s, expected %s" % (tuple(t.shape), shape))
        return self._put(t)

    def _pack(self, l: int, t: dict) -> TaralixLayer:
        spec, rank = self.cfg.layer_specs[l], self.ranks[l]
        m, f, W = spec.mixer, spec.mlp, self.cfg.hidden_size
        H, R = m.heads, m.kv_rank
        lw = TaralixLayer()
        lw.spec, lw.source, lw.rank = spec, self.owners[l], rank
        lw.shape, lw.dq, lw.dv, lw.expand = self._geometry[l]
        align = 8 if self.dtype == torch.bfloat16 else 1
        q = self._pad(self._expect(t["mix.q"], H * m.dim, W).view(H, m.dim, W), H, lw.dq)
        # the attention kernels take a maximum of unscaled scores, i.e. a positive scale
        lw.scale = m.scale
        if m.scale <= 0:
            q, lw.scale = (-q, -m.scale) if m.scale < 0 else (torch.zeros_like(q), 1.0)
        rows = [q.reshape(H * lw.dq, W)]
        lw.ckv_cols = 0
        if m.kv_from is None:
            lw.ckv_cols = _up(R, align)
            rows.append(self._pad(self._expect(t["mix.dkv"], R, W), lw.ckv_cols))
            lw.ckv_norm = self._expect(t["mix.dkv.norm"], R).float()
        lw.wq = torch.cat(rows, 0).contiguous()
        uk = self._pad(self._expect(t["mix.uk"], H * m.dim, R).view(H, m.dim, R), H, lw.dq, rank)
        uv = self._pad(self._expect(t["mix.uv"], H * m.vdim, R).view(H, m.vdim, R), H, lw.dv, rank)
        lw.wuk_t = uk.transpose(1, 2).contiguous()
        lw.wuv = uv.contiguous()
        if lw.expand:
            lw.wukv = torch.cat([uk.reshape(H * lw.dq, rank), uv.reshape(H * lw.dv, rank)], 0)
        o = self._expect(t["mix.o"], W, H * m.vdim).view(W, H, m.vdim)
        lw.wo = self._pad(o, W, H, lw.dv).reshape(W, H * lw.dv).contiguous()
        lw.norm1 = self._expect(t["norm1"], W).float()
        if f is None:
            return lw
        lw.norm2 = self._expect(t["norm2"], W).float()
        if f.experts:
            lw.router = self._expect(t["mlp.router"], f.experts, W)
            lw.router_b = self._expect(t["mlp.router.b"], f.experts).float()
            stack = lambda n, *s: torch.stack(
                [self._expect(t["mlp.e%d.%s" % (e, n)], *s) for e in range(f.experts)])
            gate, up, down = stack("gate", f.ff, W), stack("up", f.ff, W), stack("down", W, f.ff)
        else:
            gate, up, down = (self._expect(t["mlp.gate"], f.ff, W),
                              self._expect(t["mlp.up"], f.ff, W),
                              self._expect(t["mlp.down"], W, f.ff))
        lw.w_gu = st.interleave_gate_up(gate, up)
        lw.w_down = self._pad(down, *down.shape[:-1], _up(f.ff, st.GATE_BLOCK)).contiguous()
        return lw

    def num_parameters(self) -> int:
        return sum(t.numel() for _, t in self.named_tensors())

    def named_tensors(self):
        yield "embed", self.embed
        yield "norm", self.norm
        yield "lm_head", self.lm_head
        for i, lw in enumerate(self.layers):
            if lw is not None:
                for name, t in lw.tensors():
                    yield "layers.%d.%s" % (i, name), t

    def vocab_shard(self, mode_ways: int, index: int):
        return 0, self.cfg.vocab_size

    # ------------------------------------------------- cache and attention planning
    def kv_bytes_per_block(self, block_size: int) -> int:
        from ..engine.kv_cache import LatentCacheTensors
        return LatentCacheTensors.bytes_per_block(self.owners, self.ranks, block_size,
                                                  self.dtype.itemsize)

    def new_kv_cache(self, num_blocks: int, block_size: int):
        from ..engine.kv_cache import LatentCacheTensors
        return LatentCacheTensors(self.owners, self.ranks, num_blocks, block_size, self.dtype,
                                  self.device)

    def _expanded(self, q_lens, kv_lens) -> list:
        """Which sequences of a step go through expanded keys and values."""
        if self.expand_min_tokens is None:
            return [False] * len(q_lens)
        out = [q >= self.expand_min_tokens for q in q_lens]
        total = sum(k for k, e in zip(kv_lens, out) if e) * self._expand_row_bytes
        # the longest contexts stay in latent space when the temporaries would grow too large
        for i in sorted((i for i, e in enumerate(out) if e), key=lambda i: -kv_lens[i]):
            if total <= EXPAND_LIMIT_BYTES:
                break
            out[i] = False
            total -= kv_lens[i] * self._expand_row_bytes
        return out

    def batch_order(self, q_lens, kv_lens):
        exp = self._expanded(q_lens, kv_lens)
        if not any(exp) or exp == sorted(exp):
            return None
        return sorted(range(len(exp)), key=lambda i: exp[i])      # stable: absorbed ones first

    def plan_attention(self, q_lens, kv_lens, block_tables, block_arrays, block_size):
        exp = self._expanded(q_lens, kv_lens)
        n = exp.index(True) if any(exp) else len(exp)
        T, n_abs = sum(q_lens), sum(q_lens[:n])
        step = lat.LatentStep(n_abs)
        step.tok_seq = ops.upload(np.repeat(np.arange(len(q_lens), dtype=np.int32), q_lens),
                                  self.device)
        dev = self.device
        for shape, _, _, expand in self._geometry:
            full = expand is None or n_abs == T
            if (shape, full) in step.absorbed or (not full and n_abs == 0):
                continue
            k = len(q_lens) if full else n
            step.absorbed[(shape, full)] = lat.build_plan(shape, q_lens[:k], kv_lens[:k],
                                                          block_tables, block_size, dev)
        if n < len(q_lens):
            step.exp_q_lens, step.exp_kv_lens = list(q_lens[n:]), list(kv_lens[n:])
            slots = []
            for kl, blocks in zip(kv_lens[n:], block_arrays[n:]):
                pos = np.arange(kl, dtype=np.int64)
                slots.append(blocks.astype(np.int64)[pos // block_size] * block_size +
                             pos % block_size)
            step.ctx_slots = ops.upload(np.concatenate(slots), dev)
            starts = np.cumsum(step.exp_kv_lens) - np.asarray(step.exp_kv_lens)
            for (shape, _, _, expand) in self._geometry:
                if expand and shape.heads not in step.exp_plans:
                    H = shape.heads
                    step.exp_plans[H] = ops.build_attention_metadata(
                        step.exp_q_lens, step.exp_kv_lens, None, 1, H, expand, dev, Hkv=H,
                        seq_rows=starts, allow_split=False)
        return step

    def decode_plans(self, bucket: int, max_q: int, block_size: int) -> list:
        return [lat.LatentDecodePlan(s, bucket, max_q, block_size) for s in self.shapes]

    def decode_attention(self, plans: list, block_tables):
        step = lat.LatentStep(plans[0].bucket)
        for p in plans:
            step.absorbed[(p.shape, True)] = p.meta
        return step

    # ------------------------------------------------------------------ forward
    def _attention(self, lw: TaralixLayer, act, batch: ForwardBatch, kv, l: int, contexts: dict):
        m, step, T = lw.spec.mixer, batch.attn_meta, act.shape[0]
        H, nq = m.heads, m.heads * lw.dq
        proj = ops.linear(act, lw.wq)
        cache = kv.k[l]
        if m.kv_from is None:
            lat.latent_norm_cache(proj[:, nq:], lw.ckv_norm, m.kv_rank, self.cfg.rms_norm_eps,
                                  batch.slots, cache)
        n = T if lw.expand is None else step.n_absorbed
        out = torch.empty(T, H * lw.dv, dtype=self.dtype, device=self.device)
        if n:
            q = st.head_linear(proj[:n, :nq], lw.wuk_t)
            o = lat.latent_attention(q, cache, step.absorbed[(lw.shape, n == T)], lw.shape,
                                     lw.scale, step.tok_seq, batch.positions)
            st.head_linear(o, lw.wuv, out=out[:n])
        if n < T:
            c = contexts.get(lw.source)
            if c is None:
                c = contexts[lw.source] = ops.gather_rows(cache.view(-1, lw.rank), step.ctx_slots)
            kvs = ops.linear(c, lw.wukv)
            lat.expanded_attention(proj[n:, :nq], kvs[:, :nq], kvs[:, nq:], step, H, lw.expand,
                                   lw.scale, out[n:])
        return ops.linear(out, lw.wo)

    def _feed_forward(self, lw: TaralixLayer, x, act):
        """(output rows, routing): with a routing the rows are the experts', still to be summed."""
        f = lw.spec.mlp
        if not f.experts:
            return ops.linear(st.gated_linear(act, lw.w_gu, f.act), lw.w_down), None
        routing, rows = st.route(x, act, lw.router, lw.router_b, f.top)
        h = st.grouped_linear(rows, lw.w_gu, routing, act=f.act)
        return st.grouped_linear(h, lw.w_down, routing), routing

    def forward(self, batch: ForwardBatch, kv, layers_out: list = None) -> torch.Tensor:
        """Final-norm states of the sampled rows [B, W]. ``layers_out`` receives a copy of the
        residual stream after every layer."""
        eps, alpha = self.cfg.rms_norm_eps, self.cfg.postln_alpha
        x, act = st.stream_embedding(batch.input_ids, self.embed)
        contexts: dict = {}
        for l, lw in enumerate(self.layers):
            y = self._attention(lw, act, batch, kv, l, contexts)
            st.stream_norm(x, act, y, lw.norm1, alpha, eps)
            if lw.spec.mlp is not None:
                y, routing = self._feed_forward(lw, x, act)
                st.stream_norm(x, act, y, lw.norm2, alpha, eps, experts=routing)
            if layers_out is not None:
                layers_out.append(x.clone())
        return st.stream_final_norm(x, batch.logits_indices, self.norm, eps, self.dtype)

    def compute_logits(self, hidden: torch.Tensor, fp32: bool = False) -> torch.Tensor:
        V = self.cfg.vocab_size
        if fp32 and self.dtype != torch.float32:
            return hidden.float() @ self.lm_head[:V].float().t()
        return ops.linear(hidden, self.lm_head)[:, :V]
