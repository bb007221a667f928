"""The mixers of layer-list decoders: how each kind packs its weights, what it caches, how its
attention is planned and how it runs. A mixer object belongs to a layer and holds its shapes; its
weights lie in the layer's :class:`LayerWeights`.

* :class:`LatentMixer`: keys and values from one cached latent per token, optionally with a rotated
  key part that the heads share, a sink and an output gate per head (``ops/latent_ops.py``);
* :class:`HeadMixer`: cached keys and values, with norms, rotation, soft cap, sink and output gate as
  its spec asks (``ops/head_ops.py``);
* :class:`DeltaMixer`: gated delta rule, a state per head instead of a cache (``ops/state_ops.py``);
* :class:`ForgetMixer`: linear attention whose forget gate also decides what is written, a state per
  head (``ops/state_ops.py``);
* :class:`ParallelMixer`: attention and a matrix memory (:class:`MemoryMixer`) side by side.

Sizes that the tensor-core kernels tile by are padded with zeros, which changes no value.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config import (AttentionSpec, DeltaRuleSpec, ForgetScanSpec, LatentAttentionSpec,
                      MatrixMemorySpec, ParallelSpec)
from ..ops import head_ops as heads
from ..ops import latent_ops as lat
from ..ops import state_ops as states
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
    state_rows: list = []

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
        return ["mix.q", "mix.uk", "mix.uv", "mix.o"] + own + \
            (["mix.sink"] if m.sink == "learned" else []) + (["mix.g"] if m.head_gate else [])

    @staticmethod
    def random(m: LatentAttentionSpec, W: int, rnd):
        yield "mix.q", rnd(m.heads * (m.dim + m.rot_dim), W)
        if m.kv_from is None:
            yield "mix.dkv", rnd(m.kv_rank + m.rot_dim, W)
            yield "mix.dkv.norm", 1.0 + rnd(m.kv_rank, std=0.1)
        yield "mix.uk", rnd(m.heads * m.dim, m.kv_rank)
        yield "mix.uv", rnd(m.heads * m.vdim, m.kv_rank)
        if m.sink == "learned":
            yield "mix.sink", rnd(m.heads, std=1.0)
        if m.head_gate:
            yield "mix.g", rnd(m.heads, W)
        yield "mix.o", rnd(W, m.heads * m.vdim)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        m, lo = self.spec, self.layout
        H, R, dq, dv = m.heads, m.kv_rank, self.dq, self.dv
        q = padded(c.take("mix.q", H * self.dq0, W).view(H, self.dq0, W), H, dq)
        # the attention kernels take a maximum of unscaled scores, i.e. a positive scale
        self.scale = m.scale
        if m.scale <= 0:
            q, self.scale = (-q, -m.scale) if m.scale < 0 else (torch.zeros_like(q), 1.0)
        cols = Columns(self.dtype)
        cols.add(q.reshape(H * dq, W))
        if m.kv_from is None:
            cols.add(c.take("mix.dkv", R + m.rot_dim, W))
            lw.put(ckv_norm=c.vector("mix.dkv.norm", R))
        if m.head_gate:
            self.gate_at = cols.add(c.take("mix.g", H, W))
        if m.sink == "learned":
            lw.put(sink=c.vector("mix.sink", H))
        lw.put(wq=cols.weight())
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
    def run(self, act, lw: LayerWeights, batch, cache, state, step, shared: dict, eps: float):
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
        sink = lw.sink if m.sink is not None else None
        gate = proj[:, self.gate_at:self.gate_at + H] if m.head_gate else None
        n = T if self.expand is None else step.n_absorbed
        out = torch.empty(T, H * self.dv, dtype=self.dtype, device=act.device)
        if n:
            q = st.head_linear(proj[:n, :nq], lw.wuk_t)
            o = lat.latent_attention(q, cache, step.absorbed[(self.shape, n == T)], self.shape,
                                     self.scale, step.tok_seq, batch.positions, sink,
                                     gate if gate is None else gate[:n])
            st.head_linear(o, lw.wuv, out=out[:n])
        if n < T:
            key = (cache.data_ptr(), m.mask)
            c = shared.get(key)
            if c is None:
                c = shared[key] = ops.gather_rows(cache.view(-1, self.layout.width),
                                                    step.ctx[m.mask][0])
            kvs = ops.linear(c, lw.wukv)
            lat.expanded_attention(proj[n:, :nq], kvs[:, :nq], kvs[:, nq:], step, H, self.expand,
                                   self.scale, out[n:], m.mask, sink,
                                   gate if gate is None else gate[n:])
        return ops.linear(out, lw.wo)


class HeadMixer:
    expand, gain, cost = None, 0.0, 0.0
    state_rows: list = []

    def __init__(self, spec: AttentionSpec, dtype: torch.dtype, device, at: str = ""):
        """``at``: prefix of its weights' names where a layer has several mixers."""
        self.spec, self.dtype, self.at = spec, dtype, at
        self.shape = heads.HeadShape.of(spec.heads, spec.kv_heads, spec.dim, spec.vdim, dtype,
                                        spec.mask)
        self.freq = frequencies(spec.rotary, device)
        self.whole = spec.qk_norm == "projection"

    @property
    def capturable(self) -> bool:
        return self.shape.kernel != "exact"

    @property
    def cache_rows(self) -> list:
        s = self.shape
        return [(s.kv_heads, s.D), (s.kv_heads, s.Dv)]

    @staticmethod
    def names(m: AttentionSpec, p: str = "mix.") -> list:
        return [p + n for n in ["q", "k", "o"] + ([] if m.values_are_keys else ["v"]) +
                (["q.norm", "k.norm"] if m.qk_norm else []) +
                (["sink"] if m.sink == "learned" else []) + (["g"] if m.output_gate else [])]

    @staticmethod
    def random(m: AttentionSpec, W: int, rnd, p: str = "mix."):
        yield p + "q", rnd(m.heads * m.dim, W)
        yield p + "k", rnd(m.kv_heads * m.dim, W)
        if not m.values_are_keys:
            yield p + "v", rnd(m.kv_heads * m.vdim, W)
        if m.qk_norm:
            whole = m.qk_norm == "projection"
            yield p + "q.norm", 1.0 + rnd(m.dim * (m.heads if whole else 1), std=0.1)
            yield p + "k.norm", 1.0 + rnd(m.dim * (m.kv_heads if whole else 1), std=0.1)
        if m.sink == "learned":
            yield p + "sink", rnd(m.heads, std=1.0)
        if m.output_gate:
            yield p + "g", rnd(m.heads * m.vdim, W)
        yield p + "o", rnd(W, m.heads * m.vdim)

    def _put(self, lw: LayerWeights, **tensors) -> None:
        lw.put(**{self.at + n: t for n, t in tensors.items()})

    def _norm_weight(self, c: Checkpoint, name: str, n: int):
        """Weights of the query (key) norm: one head's, or every head's one after the other."""
        d, D = self.spec.dim, self.shape.D
        if not self.whole:
            return padded(c.vector(name, d), D)
        return padded(c.vector(name, n * d).view(n, d), n, D).reshape(-1).contiguous()

    def pack_rows(self, c: Checkpoint, lw: LayerWeights, W: int, p: str = "mix.") -> list:
        """Rows of the input projection; the other weights go to ``lw``."""
        m, s = self.spec, self.shape
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        part = lambda name, n, k, to: padded(c.take(p + name, n * k, W).view(n, k, W), n, to) \
            .reshape(n * to, W)
        q = part("q", H, d, s.D)
        # the attention kernels take a maximum of unscaled scores, i.e. a positive scale
        self.scale, sign = (abs(m.scale), 1.0 if m.scale > 0 else -1.0) if m.scale else (1.0, 0.0)
        if m.qk_norm:
            self._put(lw, q_norm=self._norm_weight(c, p + "q.norm", H) * sign,
                      k_norm=self._norm_weight(c, p + "k.norm", G))
        else:
            q = q * sign
        rows = [q, part("k", G, d, s.D)]
        if not m.values_are_keys:
            rows.append(part("v", G, dv, s.Dv))
        if m.output_gate:
            rows.append(part("g", H, dv, s.Dv))
        if m.sink is not None:
            self._put(lw, sink=c.vector(p + "sink", H) if m.sink == "learned" else
                      torch.zeros(H, device=c.device))
        o = c.take(p + "o", W, H * dv).view(W, H, dv)
        self._put(lw, wo=padded(o, W, H, s.Dv).reshape(W, H * s.Dv).contiguous())
        return rows

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        lw.put(wqkv=torch.cat(self.pack_rows(c, lw, W), 0).contiguous())

    # ---- planning
    def add_plan(self, step, q_lens, kv_lens, block_tables, block_size, device) -> None:
        if self.shape not in step.heads:
            step.heads[self.shape] = heads.build_plan(self.shape, q_lens, kv_lens, block_tables,
                                                      block_size, device)

    def decode_plan(self, bucket: int, max_q: int, block_size: int):
        return heads.HeadDecodePlan(self.shape, bucket, max_q, block_size)

    # ---- the layer's mixer
    def attend(self, proj, lw: LayerWeights, batch, cache, step, shared: dict, eps: float):
        """From the columns of the input projection (this mixer's from the first on) to the output
        projection."""
        m, s = self.spec, self.shape
        get = lambda name: getattr(lw, self.at + name)
        k, v = cache
        norm = (get("q_norm"), get("k_norm")) if m.qk_norm else (None, None)
        heads.head_rope_cache(proj, s, m.dim, *norm, angles(m.rotary, self.freq, batch, shared), eps,
                              batch.slots, k, v, whole=self.whole, shared_kv=m.values_are_keys)
        gate = None
        if m.output_gate:
            gate = proj[:, (s.heads + s.kv_heads) * s.D + s.kv_heads * s.Dv:]
        out = heads.head_attention(proj[:, :s.heads * s.D], k, v, step.heads[s], s, self.scale,
                                   get("sink") if m.sink else None, gate, step.tok_seq,
                                   batch.positions, m.softcap)
        return ops.linear(out, get("wo"))

    def run(self, act, lw: LayerWeights, batch, cache, state, step, shared: dict, eps: float):
        return self.attend(ops.linear(act, lw.wqkv), lw, batch, cache, step, shared, eps)


class Columns:
    """Rows of an input projection as they are put together, with the column each part starts at
    (16-bit models: parts start at multiples of eight)."""

    def __init__(self, dtype: torch.dtype):
        self.multiple = 8 if dtype == torch.bfloat16 else 1
        self.rows: list = []
        self.width = 0

    def add(self, *rows) -> int:
        """Appends matrices; returns the column of the first."""
        at = self.width
        for r in rows:
            n = round_up(r.shape[0], self.multiple)
            self.rows.append(padded(r, n))
            self.width += n
        return at

    def weight(self) -> torch.Tensor:
        return torch.cat(self.rows, 0).contiguous()


class StatefulMixer:
    """What recurrent mixers do not need of the others: cache rows, attention plans."""
    expand, gain, cost = None, 0.0, 0.0
    capturable = True
    cache_rows: list = []
    freq = shape = None

    def add_plan(self, *a) -> None:
        pass

    def decode_plan(self, *a):
        return None


class DeltaMixer(StatefulMixer):
    def __init__(self, spec: DeltaRuleSpec, dtype: torch.dtype, device):
        self.spec, self.dtype = spec, dtype
        self.channels = 2 * spec.kv_heads * spec.dim + spec.heads * spec.vdim

    @property
    def state_rows(self) -> list:
        """(shape, element type) of what a slot holds."""
        m = self.spec
        return [((m.heads, m.dim, round_up(m.vdim, 4)), torch.float32),
                ((2, m.conv - 1, self.channels), self.dtype)]

    @staticmethod
    def names(m: DeltaRuleSpec) -> list:
        return ["mix." + n for n in ("q", "k", "v", "q.conv", "k.conv", "v.conv", "b", "A_log", "norm",
                                     "a1", "a2", "dt_bias", "g1", "g2", "o")]

    @staticmethod
    def random(m: DeltaRuleSpec, W: int, rnd):
        nk, nv, rank = m.kv_heads * m.dim, m.heads * m.vdim, max(8, m.vdim)
        for x, n in (("q", nk), ("k", nk), ("v", nv)):
            yield "mix." + x, rnd(n, W)
            yield "mix." + x + ".conv", rnd(n, m.conv)
        yield "mix.b", rnd(m.heads, W)
        yield "mix.A_log", rnd(m.heads, std=0.5)
        yield "mix.norm", 1.0 + rnd(m.vdim, std=0.1)
        yield "mix.a1", rnd(rank, W)
        yield "mix.a2", rnd(m.heads * m.dim, rank, std=0.25 * rank ** -0.5)     # slow decays
        yield "mix.dt_bias", rnd(m.heads * m.dim, std=0.5) - 4.0
        yield "mix.g1", rnd(rank, W)
        yield "mix.g2", rnd(nv, rank)
        yield "mix.o", rnd(W, nv)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        m = self.spec
        H, nk, nv = m.heads, m.kv_heads * m.dim, m.heads * m.vdim
        cols = Columns(self.dtype)
        at = [cols.add(c.take("mix." + x, n, W)) for x, n in (("q", nk), ("k", nk), ("v", nv),
                                                              ("b", H))]
        # decay and gate: two maps through a few dimensions each, run as one product per kind with
        # the second maps side by side (padded to common sizes)
        ra, rg = (c.tensors["mix." + x].shape[0] for x in ("a1", "g1"))
        rank = round_up(max(ra, rg), cols.multiple)
        self.low_at = cols.add(padded(c.take("mix.a1", ra, W), rank), padded(c.take("mix.g1", rg, W), rank))
        self.low = 2 * rank
        wide = round_up(max(H * m.dim, nv), cols.multiple)
        second = torch.stack([padded(c.take("mix.a2", H * m.dim, ra), wide, rank),
                              padded(c.take("mix.g2", nv, rg), wide, rank)])
        conv = torch.cat([c.take("mix.%s.conv" % x, n, m.conv) for x, n in
                          (("q", nk), ("k", nk), ("v", nv))]).float()
        lw.put(win=cols.weight(), w_low=second.contiguous(), conv=conv.t().contiguous(),
               a_exp=c.vector("mix.A_log", H).exp(), dt_bias=c.vector("mix.dt_bias", H * m.dim),
               norm=c.vector("mix.norm", m.vdim), wo=c.take("mix.o", W, nv))
        self.scan = states.DeltaShape(H, m.kv_heads, m.dim, m.vdim, m.conv, *at)

    def run(self, act, lw: LayerWeights, batch, cache, state, step, shared: dict, eps: float):
        proj = ops.linear(act, lw.win)
        low = st.head_linear(proj[:, self.low_at:self.low_at + self.low], lw.w_low)
        out = states.delta_scan(proj, low, low[:, lw.w_low.shape[1]:], lw.conv, lw.a_exp, lw.dt_bias,
                             lw.norm, self.scan, *state, batch.state, eps)
        return ops.linear(out, lw.wo)


class ForgetMixer(StatefulMixer):
    def __init__(self, spec: ForgetScanSpec, dtype: torch.dtype, device):
        self.spec, self.dtype = spec, dtype

    @property
    def state_rows(self) -> list:
        m = self.spec
        return [((m.heads, m.dim, round_up(m.vdim, 4)), torch.float32)]

    @staticmethod
    def names(m: ForgetScanSpec) -> list:
        return ["mix." + n for n in ("q", "f", "f.b", "lower", "v", "norm", "o")]

    @staticmethod
    def random(m: ForgetScanSpec, W: int, rnd):
        nk, nv = m.heads * m.dim, m.heads * m.vdim
        for x, n in (("q", nk), ("f", nk), ("v", nv)):
            yield "mix." + x, rnd(n, W)
        yield "mix.f.b", rnd(nk, std=0.5) + 2.0
        yield "mix.lower", torch.sigmoid(rnd(nk, std=1.0))
        yield "mix.norm", 1.0 + rnd(m.vdim, std=0.1)
        yield "mix.o", rnd(W, nv)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        m, cols = self.spec, Columns(self.dtype)
        nk, nv = m.heads * m.dim, m.heads * m.vdim
        at = [cols.add(c.take("mix." + x, n, W)) for x, n in (("q", nk), ("f", nk), ("v", nv))]
        lw.put(win=cols.weight(), f_bias=c.vector("mix.f.b", nk), lower=c.vector("mix.lower", nk),
               norm=c.vector("mix.norm", m.vdim), wo=c.take("mix.o", W, nv))
        self.scan = states.ForgetShape(m.heads, m.dim, m.vdim, *at)

    def run(self, act, lw: LayerWeights, batch, cache, state, step, shared: dict, eps: float):
        out = states.forget_scan(ops.linear(act, lw.win), lw.f_bias, lw.lower, lw.norm, self.scan,
                                 *state, batch.state, eps)
        return ops.linear(out, lw.wo)


class MemoryMixer(StatefulMixer):
    def __init__(self, spec: MatrixMemorySpec, dtype: torch.dtype, device, at: str = ""):
        self.spec, self.dtype, self.at = spec, dtype, at

    @property
    def state_rows(self) -> list:
        m = self.spec
        return [((m.heads, m.dim, round_up(m.vdim + 1, 4)), torch.float32),
                ((2, m.heads), torch.float32)]

    @staticmethod
    def names(m: MatrixMemorySpec, p: str = "mix.") -> list:
        return [p + n for n in ("q", "k", "v", "g", "o", "norm", "i", "i.b", "f", "f.b")]

    @staticmethod
    def random(m: MatrixMemorySpec, W: int, rnd, p: str = "mix."):
        H, nv = m.heads, m.heads * m.vdim
        for x, n in (("q", H * m.dim), ("k", H * m.dim), ("v", nv), ("g", nv), ("i", H), ("f", H)):
            yield p + x, rnd(n, W)
        yield p + "o", rnd(W, nv)
        yield p + "norm", 1.0 + rnd(nv, std=0.1)
        yield p + "i.b", rnd(H, std=0.5)
        yield p + "f.b", rnd(H, std=0.5) + 4.0

    def pack_rows(self, c: Checkpoint, lw: LayerWeights, W: int, cols: Columns, p: str) -> None:
        m = self.spec
        H, nk, nv = m.heads, m.heads * m.dim, m.heads * m.vdim
        at = [cols.add(c.take(p + x, n, W)) for x, n in (("q", nk), ("k", nk), ("v", nv), ("i", H),
                                                         ("f", H), ("g", nv))]
        self.scan = states.MemoryShape(H, m.dim, m.vdim, m.gate_cap, *at[:5])
        self.gate_at = at[5]
        lw.put(**{self.at + n: t for n, t in (
            ("i_bias", c.vector(p + "i.b", H)), ("f_bias", c.vector(p + "f.b", H)),
            ("norm", c.vector(p + "norm", nv)), ("wo", c.take(p + "o", W, nv)))})

    def recall(self, proj, lw: LayerWeights, batch, state, eps: float):
        get = lambda name: getattr(lw, self.at + name)
        out = states.memory_scan(proj, proj[:, self.gate_at:], get("i_bias"), get("f_bias"), get("norm"),
                              self.scan, *state, batch.state, eps)
        return ops.linear(out, get("wo"))


class ParallelMixer:
    """Attention and a matrix memory side by side, on one input projection. Returns both outputs:
    their norms and their mean are taken where the stream is updated."""
    expand, gain, cost = None, 0.0, 0.0

    def __init__(self, spec: ParallelSpec, dtype: torch.dtype, device):
        self.spec, self.dtype = spec, dtype
        self.left = HeadMixer(spec.left, dtype, device, "left_")
        self.right = MemoryMixer(spec.right, dtype, device, "right_")
        self.shape = self.left.shape
        self.add_plan, self.decode_plan = self.left.add_plan, self.left.decode_plan

    @property
    def capturable(self) -> bool:
        return self.left.capturable

    @property
    def cache_rows(self) -> list:
        return self.left.cache_rows

    @property
    def state_rows(self) -> list:
        return self.right.state_rows

    @staticmethod
    def names(m: ParallelSpec) -> list:
        return HeadMixer.names(m.left, "mix.left.") + MemoryMixer.names(m.right, "mix.right.") + \
            ["mix.left.out", "mix.right.out"]

    @staticmethod
    def random(m: ParallelSpec, W: int, rnd):
        yield from HeadMixer.random(m.left, W, rnd, "mix.left.")
        yield from MemoryMixer.random(m.right, W, rnd, "mix.right.")
        yield "mix.left.out", 1.0 + rnd(W, std=0.1)
        yield "mix.right.out", 1.0 + rnd(W, std=0.1)

    def pack(self, c: Checkpoint, lw: LayerWeights, W: int) -> None:
        cols = Columns(self.dtype)
        cols.add(*self.left.pack_rows(c, lw, W, "mix.left."))
        self.right.pack_rows(c, lw, W, cols, "mix.right.")
        lw.put(win=cols.weight(), left_out=c.vector("mix.left.out", W),
               right_out=c.vector("mix.right.out", W))

    def run(self, act, lw: LayerWeights, batch, cache, state, step, shared: dict, eps: float):
        proj = ops.linear(act, lw.win)
        left = self.left.attend(proj, lw, batch, cache, step, shared, eps)
        right = self.right.recall(proj, lw, batch, state, eps)
        return left, (right, lw.left_out, lw.right_out)


MIXERS = {LatentAttentionSpec: LatentMixer, AttentionSpec: HeadMixer, DeltaRuleSpec: DeltaMixer,
          ForgetScanSpec: ForgetMixer, ParallelSpec: ParallelMixer}


def mixer_class(spec):
    return MIXERS[type(spec)]
