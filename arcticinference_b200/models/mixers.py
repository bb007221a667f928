"""The mixers of layer-list decoders: how each kind packs its weights, what it caches, how its
attention is planned and how it runs. A mixer object belongs to a layer and holds its shapes; its
weights lie in the layer's :class:`LayerWeights`.

* :class:`LatentMixer`: keys and values from one cached latent per token, optionally with a rotated
  key part that the heads share (``ops/latent_ops.py``);
* :class:`HeadMixer`: cached keys and values, with norms, rotation, sink and output gate as its spec
  asks (``ops/head_ops.py``).

Sizes that the tensor-core kernels tile by are padded with zeros, which changes no value.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config import AttentionSpec, LatentAttentionSpec
from ..ops import head_ops as heads
from ..ops import latent_ops as lat
from ..ops import stream_ops as st


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def padded(t, *sizes):
    """Zero-padded to ``sizes`` in the leading dimensions."""
    if all(a == b for a, b in zip(t.shape, sizes)):
        return t
    out = torch.zeros(*sizes, *t.shape[len(sizes):], dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class LayerWeights:
    """Packed weights of one layer, by attribute name."""

    def __init__(self):
        self.names: list = []
        self.extra: dict = {}

    def put(self, **tensors) -> None:
        for name, t in tensors.items():
            setattr(self, name, t)
            self.names.append(name)

    def tensors(self):
        for name in self.names:
            yield name, getattr(self, name)


class Checkpoint:
    """A layer's checkpoint tensors while it is packed."""

    def __init__(self, tensors: dict, dtype: torch.dtype, device):
        self.tensors, self.dtype, self.device = tensors, dtype, device

    def take(self, name: str, *shape, dtype=None) -> torch.Tensor:
        t = self.tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError("tensor %s of shape %s, expected %s" % (name, tuple(t.shape), shape))
        return t.to(device=self.device, dtype=dtype or self.dtype).contiguous()

    def vector(self, name: str, n: int) -> torch.Tensor:
        """A norm's weight or the like: kept in 32 bits."""
        return self.take(name, n).float()


def frequencies(rotary, device) -> torch.Tensor:
    f = rotary.frequencies() if rotary is not None else []
    return torch.tensor(f, dtype=torch.float64).float().to(device)


def angles(rotary, freq, batch, shared: dict) -> torch.Tensor:
    """The step's rotary table for these frequencies, made by the first run that needs it."""
    table = shared.get(rotary)
    if table is None:
        table = shared[rotary] = heads.rotary_table(batch.positions, freq)
    return table


class LatentMixer:
    def __init__(self, spec: LatentAttentionSpec, heads_sharing: int, dtype: torch.dtype, device):
        """``heads_sharing``: the most heads among the layers that read these latents."""
        self.spec, self.dtype = spec, dtype
        bf16 = dtype == torch.bfloat16
        self.layout = lat.LatentLayout.of(spec.kv_rank, spec.rot_dim, heads_sharing, dtype)
        self.shape = lat.LatentShape.of(spec.heads, self.layout.rank, dtype, self.layout.key_extra,
                                        spec.mask)
        self.freq = frequencies(spec.rotary if spec.rot_dim else None, device)
        self.dq0 = spec.dim + spec.rot_dim
        # expanded form of long chunks: widths of its keys and values, None where it does not pay.
        # ``gain``: multiply-adds saved per query, key and head; ``cost``: spent per row of the
        # context and head. A bounded mask spreads a row's cost over fewer queries.
        self.expand = None
        self.gain = self.cost = 0.0
        wide = lat.expanded_widths(self.dq0, spec.vdim)
        if bf16 and self.shape.kernel != "packed" and wide is not None:
            gain = self.layout.width + self.layout.rank - sum(wide)
            cost = self.layout.width * sum(wide)
            if spec.mask.kind != "causal":
                gain -= cost / spec.mask.size
            if wide[1] <= self.layout.rank and gain > 0:
                self.expand, self.gain, self.cost = wide, spec.heads * gain, spec.heads * cost
        self.dq, self.dv = self.expand or (self.dq0, spec.vdim)
        if bf16:
            self.dq, self.dv = round_up(self.dq, 8), round_up(self.dv, 8)

    @property
    def capturable(self) -> bool:
        """Whether captured decode steps can hold it."""
        return self.shape.kernel != "exact"

    @property
    def cache_rows(self) -> list:
        return [(1, self.layout.width)]

    @staticmethod
    def names(m: LatentAttentionSpec) -> list:
        own = [] if m.kv_from is not None else ["mix.dkv", "mix.dkv.norm"]
        return ["mix.q", "mix.uk", "mix.uv", "mix.o"] + own

    @staticmethod
    def random(m: LatentAttentionSpec, W: int, rnd):
        yield "mix.q", rnd(m.heads * (m.dim + m.rot_dim), W)
        if m.kv_from is None:
            yield "mix.dkv", rnd(m.kv_rank + m.rot_dim, W)
            yield "mix.dkv.norm", 1.0 + rnd(m.kv_rank, std=0.1)
        yield "mix.uk", rnd(m.heads * m.dim, m.kv_rank)
        yield "mix.uv", rnd(m.heads * m.vdim, m.kv_rank)
        yield "mix.o", rnd(W, m.heads * m.vdim)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        m, lo = self.spec, self.layout
        H, R, dq, dv = m.heads, m.kv_rank, self.dq, self.dv
        q = padded(c.take("mix.q", H * self.dq0, W).view(H, self.dq0, W), H, dq)
        # the attention kernels take a maximum of unscaled scores, i.e. a positive scale
        self.scale = m.scale
        if m.scale <= 0:
            q, self.scale = (-q, -m.scale) if m.scale < 0 else (torch.zeros_like(q), 1.0)
        rows = [q.reshape(H * dq, W)]
        if m.kv_from is None:
            n = R + m.rot_dim
            cols = round_up(n, 8) if self.dtype == torch.bfloat16 else n
            rows.append(padded(c.take("mix.dkv", n, W), cols))
            lw.put(ckv_norm=c.vector("mix.dkv.norm", R))
        lw.put(wq=torch.cat(rows, 0).contiguous())
        uk = padded(c.take("mix.uk", H * m.dim, R).view(H, m.dim, R), H, dq, lo.width)
        for i in range(m.rot_dim):      # the shared rotated part passes through
            uk[:, m.dim + i, lo.rot_at + i] = 1.0
        uv = padded(c.take("mix.uv", H * m.vdim, R).view(H, m.vdim, R), H, dv, lo.rank)
        lw.put(wuk_t=uk.transpose(1, 2).contiguous(), wuv=uv.contiguous())
        if self.expand:
            wide = padded(uv, H, dv, lo.width)
            lw.put(wukv=torch.cat([uk.reshape(H * dq, lo.width), wide.reshape(H * dv, lo.width)], 0))
        o = c.take("mix.o", W, H * m.vdim).view(W, H, m.vdim)
        lw.put(wo=padded(o, W, H, dv).reshape(W, H * dv).contiguous())

    # ---- planning
    def add_plan(self, step, q_lens, kv_lens, block_tables, block_size, device) -> None:
        n, T = step.n_absorbed, sum(q_lens)
        full = self.expand is None or n == T
        if (self.shape, full) in step.absorbed or (not full and n == 0):
            return
        k = len(q_lens) - (0 if full else len(step.exp_q_lens))
        step.absorbed[(self.shape, full)] = lat.build_plan(
            self.shape, q_lens[:k], kv_lens[:k], block_tables, block_size, device)

    def decode_plan(self, bucket: int, max_q: int, block_size: int):
        return lat.LatentDecodePlan(self.shape, bucket, max_q, block_size)

    # ---- the layer's mixer
    def run(self, act, lw: LayerWeights, batch, cache, step, shared: dict, eps: float):
        """``cache``: this run's tensors; ``shared``: what several runs of a step use, i.e. rotary
        tables and, by cache tensor and mask, gathered latents of the expanded sequences."""
        m, T = self.spec, act.shape[0]
        H, nq = m.heads, m.heads * self.dq
        proj = ops.linear(act, lw.wq)
        cache = cache[0]
        if m.rot_dim:
            lat.latent_rope_cache(proj, proj[:, nq:], H, self.dq, m.dim, lw.ckv_norm, m.kv_rank,
                                  angles(m.rotary, self.freq, batch, shared), eps, batch.slots,
                                  cache, self.layout.rot_at)
        elif m.kv_from is None:
            lat.latent_norm_cache(proj[:, nq:], lw.ckv_norm, m.kv_rank, eps, batch.slots, cache)
        n = T if self.expand is None else step.n_absorbed
        out = torch.empty(T, H * self.dv, dtype=self.dtype, device=act.device)
        if n:
            q = st.head_linear(proj[:n, :nq], lw.wuk_t)
            o = lat.latent_attention(q, cache, step.absorbed[(self.shape, n == T)], self.shape,
                                     self.scale, step.tok_seq, batch.positions)
            st.head_linear(o, lw.wuv, out=out[:n])
        if n < T:
            key = (cache.data_ptr(), m.mask)
            c = shared.get(key)
            if c is None:
                c = shared[key] = ops.gather_rows(cache.view(-1, self.layout.width),
                                                    step.ctx[m.mask][0])
            kvs = ops.linear(c, lw.wukv)
            lat.expanded_attention(proj[n:, :nq], kvs[:, :nq], kvs[:, nq:], step, H, self.expand,
                                   self.scale, out[n:], m.mask)
        return ops.linear(out, lw.wo)


class HeadMixer:
    expand, gain, cost = None, 0.0, 0.0

    def __init__(self, spec: AttentionSpec, dtype: torch.dtype, device):
        self.spec, self.dtype = spec, dtype
        self.shape = heads.HeadShape.of(spec.heads, spec.kv_heads, spec.dim, spec.vdim, dtype,
                                        spec.mask)
        self.freq = frequencies(spec.rotary, device)

    @property
    def capturable(self) -> bool:
        return self.shape.kernel != "exact"

    @property
    def cache_rows(self) -> list:
        s = self.shape
        return [(s.kv_heads, s.D), (s.kv_heads, s.Dv)]

    @staticmethod
    def names(m: AttentionSpec) -> list:
        return ["mix.q", "mix.k", "mix.v", "mix.o"] + \
            (["mix.q.norm", "mix.k.norm"] if m.qk_norm else []) + \
            (["mix.sink"] if m.sink else []) + (["mix.g"] if m.output_gate else [])

    @staticmethod
    def random(m: AttentionSpec, W: int, rnd):
        yield "mix.q", rnd(m.heads * m.dim, W)
        yield "mix.k", rnd(m.kv_heads * m.dim, W)
        yield "mix.v", rnd(m.kv_heads * m.vdim, W)
        if m.qk_norm:
            yield "mix.q.norm", 1.0 + rnd(m.dim, std=0.1)
            yield "mix.k.norm", 1.0 + rnd(m.dim, std=0.1)
        if m.sink:
            yield "mix.sink", rnd(m.heads, std=1.0)
        if m.output_gate:
            yield "mix.g", rnd(m.heads * m.vdim, W)
        yield "mix.o", rnd(W, m.heads * m.vdim)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        m, s = self.spec, self.shape
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        part = lambda name, n, k, to: padded(c.take(name, n * k, W).view(n, k, W), n, to) \
            .reshape(n * to, W)
        q = part("mix.q", H, d, s.D)
        # the attention kernels take a maximum of unscaled scores, i.e. a positive scale
        self.scale, sign = (abs(m.scale), 1.0 if m.scale > 0 else -1.0) if m.scale else (1.0, 0.0)
        if m.qk_norm:
            lw.put(q_norm=padded(c.vector("mix.q.norm", d), s.D) * sign,
                   k_norm=padded(c.vector("mix.k.norm", d), s.D))
        else:
            q = q * sign
        rows = [q, part("mix.k", G, d, s.D), part("mix.v", G, dv, s.Dv)]
        if m.output_gate:
            rows.append(part("mix.g", H, dv, s.Dv))
        lw.put(wqkv=torch.cat(rows, 0).contiguous())
        if m.sink:
            lw.put(sink=c.vector("mix.sink", H))
        o = c.take("mix.o", W, H * dv).view(W, H, dv)
        lw.put(wo=padded(o, W, H, s.Dv).reshape(W, H * s.Dv).contiguous())

    # ---- planning
    def add_plan(self, step, q_lens, kv_lens, block_tables, block_size, device) -> None:
        if self.shape not in step.heads:
            step.heads[self.shape] = heads.build_plan(self.shape, q_lens, kv_lens, block_tables,
                                                      block_size, device)

    def decode_plan(self, bucket: int, max_q: int, block_size: int):
        return heads.HeadDecodePlan(self.shape, bucket, max_q, block_size)

    # ---- the layer's mixer
    def run(self, act, lw: LayerWeights, batch, cache, step, shared: dict, eps: float):
        m, s = self.spec, self.shape
        proj = ops.linear(act, lw.wqkv)
        k, v = cache
        norm = (lw.q_norm, lw.k_norm) if m.qk_norm else (None, None)
        heads.head_rope_cache(proj, s, m.dim, *norm, angles(m.rotary, self.freq, batch, shared), eps,
                              batch.slots, k, v)
        gate = proj[:, (s.heads + s.kv_heads) * s.D + s.kv_heads * s.Dv:] if m.output_gate else None
        out = heads.head_attention(proj[:, :s.heads * s.D], k, v, step.heads[s], s, self.scale,
                                   lw.sink if m.sink else None, gate, step.tok_seq, batch.positions)
        return ops.linear(out, lw.wo)


def mixer_class(spec):
    return HeadMixer if isinstance(spec, AttentionSpec) else LatentMixer
