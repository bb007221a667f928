"""Decoders whose config.json lists their layers one by one, each with its own mixer and
feed-forward: Taralix, Zatirax, Pererax and Pefivik. ``config.LAYER_LIST_DESIGNS`` says what each name
stands for; ``mixers.py`` has the mixers.

Taralix: norms after the residual sum.

    x <- norm1(alpha * x + mixer(x));   x <- norm2(alpha * x + feed_forward(x))

Zatirax: a norm before and after each sublayer, and layers that run several times.

    x <- x + norm1b(mixer(norm1(x)));   x <- x + norm2b(feed_forward(norm2(x)))

Pererax: a norm and a learned scale on each sublayer's output, which reads the stream itself; layers
that use other layers' weights.

    x <- x + norm1(mixer(x)) * ls1;   x <- x + norm2(feed_forward(x)) * ls2

Pefivik: a norm before each sublayer, whose output enters with a constant factor; layers that run
several times, the embedding entering again ahead of every further pass; a second embedding of token
pairs; softly capped logits.

    x <- x + m * mixer(norm1(x));   x <- x + m * feed_forward(norm2(x))

The residual stream ``x`` is fp32 from the embedding to the final norm; the projections read the
model's element type, written by the same kernel that updates the stream. Per layer: one input
projection, norms and rotation with the cache write, attention, output projection, stream update;
then gate / up with the activation in the product's epilogue, down, stream update (for experts
that kernel also takes the weighted sum of the chosen experts' rows). An activation that needs a
token's whole row (PolyNorm) is a kernel of its own, which adds the up projection's bias; the down
projection's is added by the stream update. Routing stays on the device.

A *run* is one execution of a layer: a layer inside the loop has one per pass, and a layer whose
weights others use one for each of them, each with a cache and state of its own
(``ModelConfig.layer_runs``).

Served in bfloat16 or, with every product and sum in IEEE fp32, in float32.
"""

from __future__ import annotations

import re
from typing import Iterable

import numpy as np
import torch

from .. import ops
from ..config import LatentAttentionSpec, ModelConfig
from ..ops import latent_ops as lat
from ..ops import stream_ops as st
from .llama import ForwardBatch, ShardSpec
from .mixers import Checkpoint, LatentMixer, LayerWeights, mixer_class, padded, round_up

_NAME_RE = re.compile(r"^l(\d+)\.(.+)$")

# temporary keys and values of the expanded form, at most (one layer's, reused by the next)
EXPAND_LIMIT_BYTES = 2 << 30


def norm_names(cfg: ModelConfig, spec) -> list:
    names = ["norm1"] + (["norm2"] if spec.mlp is not None else [])
    return names + [n + "b" for n in names] if cfg.design.residual == "sandwich" else names


def scale_names(cfg: ModelConfig, spec) -> list:
    if cfg.design.residual != "output":
        return []
    return ["ls1"] + (["ls2"] if spec.mlp is not None else [])


def router_vector(f) -> str:
    """The vector beside the router's matrix: a bias, a correction of the choice, or none."""
    return {"chosen": "mlp.router.b", "all": "mlp.correction", "sigmoid": None}[f.scoring]


def required_tensors(cfg: ModelConfig, spec) -> list:
    """Checkpoint names (without the layer's prefix) of one layer."""
    if spec.weights_of is not None:
        return []
    names = norm_names(cfg, spec) + scale_names(cfg, spec) + \
        mixer_class(spec.mixer).names(spec.mixer)
    f = spec.mlp
    if f is not None and f.shared is not None:
        names += ["mlp.shared." + n for n in ("gate", "up", "down")]
    if f is not None and f.experts:
        names += [n for n in ("mlp.router", router_vector(f)) if n is not None]
        names += ["mlp.e%d.%s" % (e, n) for e in range(f.experts) for n in ("gate", "up", "down")]
    elif f is not None and f.act == "poly_norm":
        names += ["mlp.up", "mlp.up.b", "mlp.down", "mlp.down.b", "mlp.act"]
    elif f is not None:
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
        return (torch.randn(shape, generator=gen, device=device) * std).to(dtype)

    W, one = cfg.hidden_size, 1.0 - cfg.design.norm_offset
    yield "embed", rnd(cfg.vocab_size, W, std=1.0)
    if not cfg.tie_word_embeddings:
        yield "head", rnd(cfg.vocab_size, W)
    gains = () if cfg.design.scalar_norms else (W,)
    yield "final.norm", one + rnd(*gains, std=0.1)
    if cfg.bigram is not None:
        yield "bigram", rnd(cfg.bigram.buckets + 1, W, std=0.5)
    if cfg.loop is not None:
        yield "loop.step", rnd(cfg.loop.times, W, std=0.1)
    for i, l in enumerate(cfg.layer_specs):
        f, p = l.mlp, "l%d." % i
        if l.weights_of is not None:
            continue
        for n in norm_names(cfg, l):
            yield p + n, one + rnd(*gains, std=0.1)
        for n in scale_names(cfg, l):
            yield p + n, 1.0 + rnd(W, std=0.1)
        for n, t in mixer_class(l.mixer).random(l.mixer, W, rnd):
            yield p + n, t
        if f is None:
            continue
        if f.experts:
            outputs = f.experts + f.identity
            yield p + "mlp.router", rnd(outputs, W)
            if router_vector(f) is not None:
                yield p + router_vector(f), rnd(outputs, std=0.1 if f.scoring == "chosen" else 0.1 / outputs)
        elif f.act == "poly_norm":
            yield p + "mlp.up", rnd(f.ff, W)
            yield p + "mlp.up.b", rnd(f.ff, std=0.1)
            yield p + "mlp.down", rnd(W, f.ff)
            yield p + "mlp.down.b", rnd(W, std=0.1)
            yield p + "mlp.act", 0.5 + rnd(4, std=0.1)
            continue
        ffs = {"mlp.e%d." % e: f.ff for e in range(f.experts)} if f.experts else {"mlp.": f.ff}
        if f.shared is not None:
            ffs["mlp.shared."] = f.shared.ff
        for q, ff in ffs.items():
            yield p + q + "gate", rnd(ff, W)
            yield p + q + "up", rnd(ff, W)
            yield p + q + "down", rnd(W, ff)


class LayerListForCausalLM:
    def __init__(self, cfg: ModelConfig, shard: ShardSpec = None, device="cuda", dtype=None,
                 comm=None):
        if comm is not None:
            raise NotImplementedError("%s on more than one GPU" % cfg.architecture)
        self.cfg, self.design = cfg, cfg.design
        self.shard = shard or ShardSpec()
        self.device = torch.device(device)
        self.dtype = dtype or (torch.float32 if cfg.dtype == "float32" else torch.bfloat16)
        self.comm = self.pp = None
        self.layer_lo, self.layer_hi = 0, cfg.num_hidden_layers
        # what the engine asks of any decoder: query heads and cached heads per rank
        self.h, self.hkv = cfg.num_attention_heads, 1
        self.D = cfg.head_dim
        self.layers: list = [None] * cfg.num_hidden_layers
        self.embed = self.norm = self.lm_head = self.bigram = None
        if cfg.loop is not None:
            self.loop_step = None
        self._lay_out()

    # ------------------------------------------------------------------ shapes
    def _lay_out(self) -> None:
        """Mixers, gates and the order of runs. Layers that share latents agree on their rows."""
        specs = self.cfg.layer_specs
        source = [getattr(l.mixer, "kv_from", None) for l in specs]
        owner = [i if s is None else s for i, s in enumerate(source)]
        self.mixers = []
        for i, l in enumerate(specs):
            if isinstance(l.mixer, LatentAttentionSpec):
                sharing = max(k.mixer.heads for k, o in zip(specs, owner) if o == owner[i])
                self.mixers.append(LatentMixer(l.mixer, sharing, self.dtype, self.device))
            else:
                self.mixers.append(mixer_class(l.mixer)(l.mixer, self.dtype, self.device))
        gate = lambda f: None if f is None or f.act == "poly_norm" else st.Gate(f.act, f.limit)
        self.gates = [gate(l.mlp) for l in specs]
        self.shared_gates = [gate(l.mlp and l.mlp.shared) for l in specs]
        self.runs = self.cfg.layer_runs
        # run whose cache a run reads (its own but for shared latents, which no loop contains)
        run_of = {l: r for r, (l, _) in enumerate(self.runs) if source[l] is None}
        self.owners = [r if source[l] is None else run_of[source[l]]
                       for r, (l, _) in enumerate(self.runs)]
        self._cache_rows = [self.mixers[l].cache_rows for l, _ in self.runs]
        self._state_rows = [self.mixers[l].state_rows for l, _ in self.runs]
        self.has_state = any(self._state_rows)
        # queries per sequence from which expanding its context costs fewer multiply-adds than
        # attending in latent space, for the layers together
        exp = [self.mixers[l] for l, _ in self.runs if self.mixers[l].expand]
        self.expand_min_tokens = None
        if exp:
            q = sum(m.cost for m in exp) / sum(m.gain for m in exp)
            self.expand_min_tokens = max(128, min(512, int(q)))
        self._expand_row_bytes = max((2 * m.spec.heads * sum(m.expand) for m in exp), default=0)
        # captured steps need a plan per shape; the "exact" kernels and 32-bit models run eagerly
        self.supports_graphs = self.dtype == torch.bfloat16 and all(m.capturable for m in self.mixers)

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0) -> None:
        self.load_state(random_state(self.cfg, seed, self.device, torch.bfloat16))

    def load_weights(self, path: str) -> None:
        from .loader import iter_safetensors_dir
        self.load_state(iter_safetensors_dir(path))

    def load_state(self, state: Iterable) -> None:
        """Consume (name, tensor) pairs in any order; a layer is packed once it is complete."""
        cfg = self.cfg
        V, W = cfg.vocab_size, cfg.hidden_size
        pending: dict = {}
        need = [set(required_tensors(cfg, l)) for l in cfg.layer_specs]
        top = {"embed": (V, W), "final.norm": () if cfg.design.scalar_norms else (W,)}
        if cfg.bigram is not None:
            top["bigram"] = (cfg.bigram.buckets + 1, W)
        if not cfg.tie_word_embeddings:
            top["head"] = (V, W)
        if cfg.loop is not None:
            top["loop.step"] = (cfg.loop.times, W)
        missing = set(top)
        for name, t in state:
            if name in top:
                t = Checkpoint({name: t}, self.dtype, self.device).take(name, *top[name])
                missing.discard(name)
                rows = round_up(V, 8) if self.dtype == torch.bfloat16 else V
                if name == "embed" and cfg.tie_word_embeddings:
                    self.embed = self.lm_head = padded(t, rows)
                elif name == "embed":
                    self.embed = t
                elif name == "final.norm":
                    self.norm = t.float().expand(W).contiguous()
                elif name == "bigram":
                    self.bigram = t
                elif name == "loop.step":
                    self.loop_step = t.float()
                else:
                    self.lm_head = padded(t, rows)
                continue
            m = _NAME_RE.match(name)
            if m is None or int(m.group(1)) >= len(need) or m.group(2) not in need[int(m.group(1))]:
                raise ValueError("unexpected tensor %r in a %s checkpoint"
                                 % (name, cfg.architecture))
            l = int(m.group(1))
            d = pending.setdefault(l, {})
            d[m.group(2)] = t
            if len(d) == len(need[l]):
                self.layers[l] = self._pack(l, d)
                del pending[l]
        missing = sorted(missing)
        missing += ["l%d.%s" % (l, n) for l, lw in enumerate(self.layers) if lw is None and need[l]
                    for n in sorted(need[l] - set(pending.get(l, ())))]
        if missing:
            raise ValueError("checkpoint is incomplete: %s" % missing[:8])

    def _pack(self, l: int, t: dict) -> LayerWeights:
        spec, W = self.cfg.layer_specs[l], self.cfg.hidden_size
        f = spec.mlp
        c, lw = Checkpoint(t, self.dtype, self.device), LayerWeights()
        self.mixers[l].pack(c, lw, W)
        scales = dict(zip(("norm1", "norm2"), scale_names(self.cfg, spec)))
        for n in norm_names(self.cfg, spec):
            if self.design.scalar_norms:
                lw.put(**{n: c.take(n).float().reshape(1)})
                continue
            v = c.vector(n, W)
            if n in scales:      # norm and layer scale are factors of the same vector
                v = v * c.vector(scales[n], W)
            lw.put(**{n: v})
        if f is None:
            return lw
        if f.shared is not None:
            ff = f.shared.ff
            gate, up = (c.take("mlp.shared." + n, ff, W) for n in ("gate", "up"))
            down = c.take("mlp.shared.down", W, ff)
            lw.put(shared_gu=st.interleave_gate_up(gate, up),
                   shared_down=padded(down, W, round_up(ff, st.GATE_BLOCK)).contiguous())
        if f.experts:
            outputs = f.experts + f.identity
            b = router_vector(f)
            lw.put(router=c.take("mlp.router", outputs, W))
            if b is not None:
                lw.put(router_b=c.vector(b, outputs))
            stack = lambda n, *s: torch.stack(
                [c.take("mlp.e%d.%s" % (e, n), *s) for e in range(f.experts)])
            gate, up, down = stack("gate", f.ff, W), stack("up", f.ff, W), stack("down", W, f.ff)
        elif f.act == "poly_norm":
            n = round_up(f.ff, 8) if self.dtype == torch.bfloat16 else f.ff
            lw.put(w_up=padded(c.take("mlp.up", f.ff, W), n).contiguous(),
                   w_down=padded(c.take("mlp.down", W, f.ff), W, n).contiguous(),
                   up_bias=padded(c.take("mlp.up.b", f.ff), n), down_bias=c.vector("mlp.down.b", W),
                   act=c.vector("mlp.act", 4))
            return lw
        else:
            gate, up, down = (c.take("mlp.gate", f.ff, W), c.take("mlp.up", f.ff, W),
                              c.take("mlp.down", W, f.ff))
        lw.put(w_gu=st.interleave_gate_up(gate, up),
               w_down=padded(down, *down.shape[:-1], round_up(f.ff, st.GATE_BLOCK)).contiguous())
        return lw

    def num_parameters(self) -> int:
        return sum(t.numel() for _, t in self.named_tensors())

    def named_tensors(self):
        yield "embed", self.embed
        yield "norm", self.norm
        yield "lm_head", self.lm_head
        if self.bigram is not None:
            yield "bigram", self.bigram
        if self.cfg.loop is not None:
            yield "loop_step", self.loop_step
        for i, lw in enumerate(self.layers):
            if lw is not None:
                for name, t in lw.tensors():
                    yield "layers.%d.%s" % (i, name), t

    def vocab_shard(self, mode_ways: int, index: int):
        return 0, self.cfg.vocab_size

    # ------------------------------------------------- cache and attention planning
    def kv_bytes_per_block(self, block_size: int) -> int:
        from ..engine.kv_cache import RunCacheTensors
        return RunCacheTensors.bytes_per_block(self.owners, self._cache_rows, block_size,
                                               self.dtype.itemsize)

    def state_bytes_per_slot(self) -> int:
        from ..engine.kv_cache import RunCacheTensors
        return RunCacheTensors.bytes_per_slot(self._state_rows)

    def new_kv_cache(self, num_blocks: int, block_size: int, num_slots: int = 0):
        from ..engine.kv_cache import RunCacheTensors
        return RunCacheTensors(self.owners, self._cache_rows, num_blocks, block_size, self.dtype,
                               self.device, self._state_rows, num_slots)

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
        dev = self.device
        step = lat.AttentionStep(sum(q_lens[:n]))
        step.exp_q_lens, step.exp_kv_lens = list(q_lens[n:]), list(kv_lens[n:])
        step.tok_seq = ops.upload(np.repeat(np.arange(len(q_lens), dtype=np.int32), q_lens), dev)
        for m in self.mixers:
            m.add_plan(step, q_lens, kv_lens, block_tables, block_size, dev)
            if n < len(q_lens) and m.expand:
                self._plan_expanded(step, m, block_arrays[n:], block_size)
        return step

    def _plan_expanded(self, step, m: LatentMixer, block_arrays, block_size) -> None:
        mask, H = m.spec.mask, m.spec.heads
        q_lens, kv_lens = step.exp_q_lens, step.exp_kv_lens
        lo = [int(mask.first_key(k - q)) for q, k in zip(q_lens, kv_lens)]
        if mask not in step.ctx:
            slots = []
            for a, b, blocks in zip(lo, kv_lens, block_arrays):
                pos = np.arange(a, b, dtype=np.int64)
                slots.append(blocks.astype(np.int64)[pos // block_size] * block_size +
                             pos % block_size)
            step.ctx[mask] = (ops.upload(np.concatenate(slots), self.device), lo)
        key = (H, m.expand, mask)
        if key not in step.exp_plans:
            rows = np.asarray(kv_lens) - np.asarray(lo)
            step.exp_plans[key] = ops.build_attention_metadata(
                q_lens, kv_lens, None, 1, H, m.expand[1], self.device, Hkv=H,
                seq_rows=np.cumsum(rows) - rows - np.asarray(lo), allow_split=False, mask=mask)

    def decode_plans(self, bucket: int, max_q: int, block_size: int) -> list:
        return [m.decode_plan(bucket, max_q, block_size)
                for m in {m.shape: m for m in self.mixers if m.shape is not None}.values()]

    def decode_attention(self, plans: list, block_tables):
        step = lat.AttentionStep(block_tables.shape[0])
        for p in plans:
            if isinstance(p, lat.LatentDecodePlan):
                step.absorbed[(p.shape, True)] = p.meta
            else:
                step.heads[p.shape] = p.meta
        return step

    # ------------------------------------------------------------------ forward
    def _feed_forward(self, l: int, x, act):
        """(output rows, routing): with a routing the rows are the experts', still to be summed, and
        with a bias on the down projection it is still to be added. ``x``: what the router reads."""
        lw, f, gate = self.layers[l], self.cfg.layer_specs[l].mlp, self.gates[l]
        if f.act == "poly_norm":
            h = st.poly_norm(ops.linear(act, lw.w_up), lw.up_bias, lw.act, f.ff, self.cfg.rms_norm_eps)
            return ops.linear(h, lw.w_down), None
        if not f.experts:
            return ops.linear(st.gated_linear(act, lw.w_gu, gate), lw.w_down), None
        routing, rows = st.route(x, act, lw.router, getattr(lw, "router_b", None), f.top, f.identity,
                                 f.router_scale if f.scoring != "chosen" else None,
                                 (f.groups, f.keep_groups) if f.scoring == "sigmoid" else None)
        h = st.grouped_linear(rows, lw.w_gu, routing, act=gate)
        return st.grouped_linear(h, lw.w_down, routing), routing

    def _shared_expert(self, l: int, act):
        """Rows of the expert that every token uses, None where there is none."""
        lw, gate = self.layers[l], self.shared_gates[l]
        if gate is None:
            return None
        return ops.linear(st.gated_linear(act, lw.shared_gu, gate), lw.shared_down)

    def forward(self, batch: ForwardBatch, kv, layers_out: list = None) -> torch.Tensor:
        """Final-norm states of the sampled rows [B, W]. ``layers_out`` receives a copy of the
        residual stream after every run."""
        shared: dict = {}
        step, eps = batch.attn_meta, self.cfg.rms_norm_eps
        mix = lambda r, l, act: self.mixers[l].run(act, self.layers[l], batch, kv.of(r),
                                                   kv.state_of(r), step, shared, eps)
        body = {"post": self._post_norm_body, "sandwich": self._sandwich_body,
                "output": self._output_norm_body, "pre": self._pre_norm_body}[self.design.residual]
        x = body(batch, mix, layers_out)
        return st.stream_final_norm(x, batch.logits_indices, self.norm, eps, self.dtype,
                                    self.design.norm_offset)

    def _post_norm_body(self, batch, mix, layers_out):
        eps, alpha = self.cfg.rms_norm_eps, self.cfg.postln_alpha
        x, act = st.stream_embedding(batch.input_ids, self.embed, self.cfg.embedding_scale)
        for r, (l, _) in enumerate(self.runs):
            lw = self.layers[l]
            st.stream_norm(x, act, mix(r, l, act), lw.norm1, alpha, eps)
            if self.cfg.layer_specs[l].mlp is not None:
                y, routing = self._feed_forward(l, x, act)
                st.stream_norm(x, act, y, lw.norm2, alpha, eps, experts=routing)
            if layers_out is not None:
                layers_out.append(x.clone())
        return x

    def _sandwich_body(self, batch, mix, layers_out):
        eps, offset = self.cfg.rms_norm_eps, self.design.norm_offset
        x, _ = st.stream_embedding(batch.input_ids, self.embed, self.cfg.embedding_scale,
                                   rounded=False)
        act = torch.empty(x.shape, dtype=self.dtype, device=self.device)
        update = lambda *a: st.stream_sandwich(x, *a, eps=eps, offset=offset)

        def enter(r, y=None, w_out=None):
            """The stream after a sublayer's output and what run ``r`` reads of it."""
            if r == len(self.runs):
                if y is not None:
                    update(y, w_out)
                return
            l, t = self.runs[r]
            update(y, w_out, None if t is None else self.loop_step[t], self.layers[l].norm1, act)

        enter(0)
        for r, (l, _) in enumerate(self.runs):
            lw = self.layers[l]
            y, w_out = mix(r, l, act), lw.norm1b
            if self.cfg.layer_specs[l].mlp is not None:
                update(y, w_out, None, lw.norm2, act)
                y, w_out = self._feed_forward(l, x, act)[0], lw.norm2b
            if layers_out is not None:
                update(y, w_out)
                layers_out.append(x.clone())
                y = w_out = None
            enter(r + 1, y, w_out)
        return x

    def _output_norm_body(self, batch, mix, layers_out):
        eps = self.cfg.rms_norm_eps
        x, act = st.stream_embedding(batch.input_ids, self.embed, self.cfg.embedding_scale)
        for r, (l, _) in enumerate(self.runs):
            lw = self.layers[l]
            y = mix(r, l, act)
            y, pair = y if isinstance(y, tuple) else (y, None)
            st.stream_add(x, act, lw.norm1, eps, y, pair=pair)
            if self.cfg.layer_specs[l].mlp is not None:
                y, routing = self._feed_forward(l, x, act)
                st.stream_add(x, act, lw.norm2, eps, y, experts=routing,
                              shared=self._shared_expert(l, act))
            if layers_out is not None:
                layers_out.append(x.clone())
        return x

    def _pre_norm_body(self, batch, mix, layers_out):
        cfg, loop = self.cfg, self.cfg.loop
        eps, mult = cfg.rms_norm_eps, cfg.residual_mult
        T, W, dev = batch.input_ids.numel(), cfg.hidden_size, self.device
        x0 = None       # the embedding, where later passes of the loop add it
        if loop is not None and loop.reenter and loop.times > 1:
            x0 = torch.empty(T, W, dtype=torch.float32, device=dev)
        pairs = None if cfg.bigram is None else (batch.prev_ids, self.bigram, cfg.bigram)
        x, _ = st.stream_embedding(batch.input_ids, self.embed, cfg.embedding_scale, rounded=False,
                                   pairs=pairs, keep=x0)
        act = torch.empty(T, W, dtype=self.dtype, device=dev)
        update = lambda **kw: st.stream_pre(x, mult, eps, **kw)

        def enter(r, out):
            """The stream after a sublayer's output and what run ``r`` reads of it."""
            if r == len(self.runs):
                if out:
                    update(**out)
                return
            l, t = self.runs[r]
            update(**out, base=x0 if t else None, step=None if t is None else self.loop_step[t],
                   w_in=self.layers[l].norm1, act=act)

        enter(0, {})
        for r, (l, _) in enumerate(self.runs):
            lw, out = self.layers[l], {"y": mix(r, l, act)}
            if cfg.layer_specs[l].mlp is not None:
                update(**out, w_in=lw.norm2, act=act)
                y, routing = self._feed_forward(l, act, act)
                out = {"y": y, "bias": getattr(lw, "down_bias", None), "experts": routing,
                       "shared": self._shared_expert(l, act)}
            if layers_out is not None:
                update(**out)
                layers_out.append(x.clone())
                out = {}
            enter(r + 1, out)
        return x

    def compute_logits(self, hidden: torch.Tensor, fp32: bool = False) -> torch.Tensor:
        V, cap = self.cfg.vocab_size, self.cfg.logit_softcap
        if fp32 and self.dtype != torch.float32:
            logits = hidden.float() @ self.lm_head[:V].float().t()
        else:
            logits = ops.linear(hidden, self.lm_head)[:, :V]
        return st.soft_cap(logits, cap) if cap else logits
