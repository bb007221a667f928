"""Configuration objects and the command-line flag system.

One set of dataclasses describes an engine; :class:`EngineArgs` is the flat,
CLI-facing view (``serve`` flags and ``LLM(...)`` keyword arguments) and
:meth:`EngineArgs.create_engine_config` validates it into an
:class:`EngineConfig`.

Parity notes (paths are the reference's): the Arctic flags and their defaults
come from arctic_inference/vllm/args.py:31-38,86-129; the parallel-size rules
from arctic_inference/vllm/config.py:30-46; the speculative-decoding fields,
defaults and batch-size caps from arctic_inference/vllm/config.py:50-170.
"""

from __future__ import annotations

import argparse
import dataclasses
import json
import logging
import math
import os
from dataclasses import dataclass, field
from typing import Any, Optional

logger = logging.getLogger(__name__)


# --------------------------------------------------------------------------------------
# model
# --------------------------------------------------------------------------------------

SHIFT_PARALLEL_THRESHOLD = 128


@dataclass(frozen=True)
class MaskSpec:
    """Which earlier keys a token at position p sees, besides itself:

    * ``causal``: all of them;
    * ``window``: the ``size`` positions that end at p;
    * ``chunk``: those with the same ``position // size``.
    """
    kind: str = "causal"
    size: int = 0

    @property
    def code(self) -> int:
        """The kernels' number of the kind (csrc/common/elem.cuh)."""
        return {"causal": 0, "window": 1, "chunk": 2}[self.kind]

    def first_key(self, pos):
        """First position that ``pos`` (a number or an array) sees."""
        if self.kind == "window":
            return (pos - self.size + 1) * (pos >= self.size)
        if self.kind == "chunk":
            return pos // self.size * self.size
        return pos * 0


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions over the leading ``dims`` dimensions of a vector, whose two halves form the
    pairs (i, i + dims / 2). ``scaling``: (factor, low, high, original), a context extension that divides the
    frequencies whose wavelength exceeds original / low, keeps those below original / high and
    interpolates between the two."""
    base: float
    dims: int
    scaling: Optional[tuple] = None

    def frequencies(self) -> list:
        out = []
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            if self.scaling is not None:
                factor, low, high, original = self.scaling
                turns = original * f / (2.0 * math.pi)      # within the original context
                if turns < low:
                    f /= factor
                elif turns <= high:
                    s = (turns - low) / (high - low)
                    f = (1.0 - s) * f / factor + s * f
            out.append(f)
        return out


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are linear maps of one latent vector per token: only the
    latent (``kv_rank`` numbers) is cached. ``kv_from``: take the latents of that earlier layer
    instead of projecting and caching some of one's own. ``rot_dim`` > 0: every head has that many
    further query dimensions, rotated by position, which meet one rotated key part that the heads
    share and that is cached beside the latent."""
    heads: int
    dim: int          # query / key dimensions per head (the unrotated ones)
    vdim: int         # value dimensions per head
    kv_rank: int
    scale: float      # factor of the scores
    kv_from: Optional[int] = None
    rot_dim: int = 0
    rotary: Optional[RotarySpec] = None
    mask: MaskSpec = MaskSpec()
    # a further term of the softmax denominator: exp of a "learned" number per head, or None
    sink: Optional[str] = None
    head_gate: bool = False     # heads' outputs times sigmoid of one projected number per head


@dataclass(frozen=True)
class AttentionSpec:
    """Attention with cached keys and values, ``heads // kv_heads`` query heads to each of them."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotarySpec] = None
    mask: MaskSpec = MaskSpec()
    # RMS norm before rotation: "head" (over dim of every query and key head), "projection" (over
    # all query, and all key, heads of a token at once) or None
    qk_norm: Optional[str] = None
    # a further term of the softmax denominator: exp of a "learned" number per head, exp(0)
    # ("zero"), or None
    sink: Optional[str] = None
    output_gate: bool = False   # heads' outputs times sigmoid of a projection of the layer's input
    softcap: float = 0.0        # scores become softcap * tanh(score / softcap); 0: they do not
    values_are_keys: bool = False   # the key projection (before norm and rotation) is the value


@dataclass(frozen=True)
class DeltaRuleSpec:
    """Gated delta rule with a decay per key channel: a [dim, vdim] state per head. ``kv_heads``
    query / key heads serve ``heads`` value heads; queries, keys and values pass a causal
    convolution of ``conv`` taps. The ranks of the decay and gate projections come from the
    tensors."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Matrix memory with exponential gates (the mLSTM of xLSTM): a [dim, vdim] state, a [dim]
    normaliser and a running maximum per head. ``gate_cap``: soft cap of both gates."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ForgetScanSpec:
    """Linear attention whose forget gate also decides what is written (HGRN2): a [dim, vdim] state
    per head, f = lower + (1 - lower) * sigmoid(projection + bias) per channel, and 1 - f in the
    place of a key."""
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same input; the result is half the sum of their normed outputs."""
    left: AttentionSpec
    right: MatrixMemorySpec


def mixer_parts(m) -> tuple:
    """The elementary mixers of a layer's mixer."""
    return (m.left, m.right) if isinstance(m, ParallelSpec) else (m,)


def has_state(m) -> bool:
    """Whether a mixer carries a state from token to token, which cannot be taken back."""
    return any(isinstance(x, (DeltaRuleSpec, MatrixMemorySpec, ForgetScanSpec))
               for x in mixer_parts(m))


@dataclass(frozen=True)
class FeedForwardSpec:
    """A gated feed-forward layer, or ``experts`` of them of which every token uses ``top``; with the
    activation ``poly_norm`` one without a gate and with biases."""
    ff: int
    act: str = "silu"     # silu | gelu_tanh | clamped_swish (ops.stream_ops.Gate) | poly_norm
    experts: int = 0      # 0: dense
    top: int = 0
    limit: float = 0.0    # clamped_swish: bound of gate (above) and up (both sides)
    # router: "chosen" (largest logits plus bias, softmax over the chosen ones) or "all" (softmax
    # over all; a correction enters the choice, not the weights; weights times ``router_scale``) or
    # "sigmoid" (of each logit; chosen among the ``keep_groups`` best of ``groups`` groups of
    # neighbours, a group's score being the sum of its two best; the chosen scores are normalised to
    # the sum ``router_scale``)
    scoring: str = "chosen"
    router_scale: float = 1.0
    groups: int = 1
    keep_groups: int = 1
    identity: int = 0     # further router outputs behind the experts' whose expert is the identity
    shared: Optional["FeedForwardSpec"] = None   # runs for every token beside the chosen ones


@dataclass(frozen=True)
class LayerSpec:
    """One decoder layer of a model that lists its layers one by one."""
    mixer: Any            # AttentionSpec | LatentAttentionSpec | DeltaRuleSpec | ForgetScanSpec | ...
    mlp: Optional[FeedForwardSpec] = None
    weights_of: Optional[int] = None    # layer whose tensors this one uses (cache and state are its own)


@dataclass(frozen=True)
class LoopSpec:
    """The slice ``[start, stop)`` of the layer list is executed ``times`` times before the layers
    behind it. Passes share weights, not caches; a learned vector per pass is added to the stream as
    the pass begins, and with ``reenter`` the embedding before it, from the second pass on."""
    start: int
    stop: int
    times: int
    reenter: bool = False


@dataclass(frozen=True)
class BigramSpec:
    """A second embedding, looked up by (previous token * mul_prev + token * mul_cur) mod buckets; a
    sequence's first token has the row behind the others."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayerListDesign:
    """What the name of a layer-list architecture stands for, beyond the numbers of config.json.

    ``residual``: where the norms are. "post": x <- norm(alpha * x + f(x)); "sandwich":
    x <- x + norm_b(f(norm_a(x))); "output": x <- x + norm(f(x)) * scale; "pre": x <- x +
    residual_mult * f(norm(x)). ``norm_offset``: added to the stored weights of the stream's norms.
    ``scalar_norms``: those weights are one number for all coordinates. ``masks``: kind of each mixer
    type's mask. ``attention``: options of :class:`AttentionSpec` or :class:`LatentAttentionSpec` by
    mixer type ("left": the attention side of a parallel mixer). ``scoring``: the router's.
    ``loop_reenters``: see :class:`LoopSpec`. ``tied``: the embedding is the output matrix."""
    residual: str
    norm_offset: float
    dense_act: str
    mixers: tuple
    feed_forwards: tuple
    masks: dict = field(default_factory=dict)
    attention: dict = field(default_factory=dict)
    expert_act: str = "silu"
    scoring: str = "chosen"
    tied: bool = False
    scalar_norms: bool = False
    loop_reenters: bool = False


LAYER_LIST_DESIGNS = {
    "Taralix": LayerListDesign(residual="post", norm_offset=1.0, dense_act="gelu_tanh",
                               mixers=("latent_attention",), feed_forwards=("dense", "moe")),
    "Zatirax": LayerListDesign(residual="sandwich", norm_offset=0.0, dense_act="clamped_swish",
                               mixers=("latent_attention", "attention"), feed_forwards=("dense",),
                               masks={"latent_attention": "window", "attention": "chunk"},
                               attention={"attention": dict(qk_norm="head", sink="learned",
                                                            output_gate=True)}),
    "Pererax": LayerListDesign(residual="output", norm_offset=0.0, dense_act="clamped_swish",
                               mixers=("channel_delta", "parallel", "attention"),
                               feed_forwards=("moe",), masks={"attention": "window"},
                               attention={"attention": dict(qk_norm="projection",
                                                            values_are_keys=True),
                                          "left": dict(qk_norm="projection", sink="zero")},
                               expert_act="clamped_swish", scoring="all", tied=True),
    "Pefivik": LayerListDesign(residual="pre", norm_offset=0.0, dense_act="poly_norm",
                               mixers=("latent_attention", "hgrn2"), feed_forwards=("dense", "moe"),
                               attention={"latent_attention": dict(sink="learned", head_gate=True)},
                               scoring="sigmoid", scalar_norms=True, loop_reenters=True),
}


def _read_rotary(d: Optional[dict]) -> Optional[RotarySpec]:
    if d is None:
        return None
    s = d.get("scaling")
    return RotarySpec(base=float(d["base"]), dims=int(d["dims"]),
                      scaling=None if s is None else tuple(float(s[k]) for k in
                                                           ("factor", "low", "high", "original")))


def _read_mixer(kind: str, m: dict, design: LayerListDesign):
    if kind == "parallel":
        r = m["right"]
        return ParallelSpec(_read_mixer("left", m["left"], design),
                            MatrixMemorySpec(heads=int(r["heads"]), dim=int(r["dim"]),
                                             vdim=int(r["vdim"]), gate_cap=float(r["gate_cap"])))
    if kind == "channel_delta":
        return DeltaRuleSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                             vdim=int(m["vdim"]), conv=int(m["conv"]))
    if kind == "hgrn2":
        return ForgetScanSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
    rotary, mask = _read_rotary(m.get("rot")), MaskSpec()
    if m.get("mask") is not None:
        mask = MaskSpec(design.masks[kind], int(m["mask"]["size"]))
    options = design.attention.get(kind, {})
    vdim = m["dim"] if options.get("values_are_keys") else m["vdim"]
    shape = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(vdim), scale=float(m["scale"]),
                 rotary=rotary, mask=mask)
    if kind in ("attention", "left"):
        return AttentionSpec(kv_heads=int(m["kv_heads"]), softcap=float(m.get("softcap") or 0.0),
                             **options, **shape)
    src = m.get("kv_from")
    return LatentAttentionSpec(kv_rank=int(m["kv_rank"]), rot_dim=int(m.get("rot_dim") or 0),
                               kv_from=None if src is None else int(src), **options, **shape)


def _read_experts(f: dict, design: LayerListDesign) -> FeedForwardSpec:
    gated = lambda d: dict(ff=int(d["ff"]), act=design.expert_act, limit=float(d.get("limit", 0.0)))
    r, shared = f["router"], f.get("shared")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return FeedForwardSpec(experts=int(r["experts"]), top=int(r["top"]), scoring=design.scoring,
                           router_scale=float(r.get("scale", 1.0)),
                           identity=int(r.get("identity") or 0),
                           groups=int(groups["count"]), keep_groups=int(groups["keep"]),
                           shared=FeedForwardSpec(**gated(shared)) if shared else None,
                           **gated(f["expert"]))


def read_layer_specs(layers: list, design: LayerListDesign) -> tuple:
    """The ``layers`` list of a layer-list checkpoint's config.json."""
    out = []
    for i, d in enumerate(layers):
        kind = d.get("type")
        if kind not in design.mixers:
            raise NotImplementedError("layer %d: mixer type %r (supported: %s)"
                                      % (i, kind, ", ".join(design.mixers)))
        mixer = _read_mixer(kind, d["mixer"], design)
        f, mlp = d.get("mlp"), None
        if f is not None:
            kind = f.get("kind")
            if kind not in design.feed_forwards:
                raise NotImplementedError("layer %d: feed-forward kind %r (supported: %s)"
                                          % (i, kind, ", ".join(design.feed_forwards)))
            if kind == "dense":
                mlp = FeedForwardSpec(ff=int(f["ff"]), act=design.dense_act,
                                      limit=float(f["limit"]) if "limit" in f else 0.0)
            else:
                mlp = _read_experts(f, design)
        src = d.get("weights_of")
        out.append(LayerSpec(mixer, mlp, None if src is None else int(src)))
    return tuple(out)


def _validate_mixer(i: int, m, specs: tuple) -> None:
    if min(m.heads, m.dim, m.vdim) < 1:
        raise ValueError("layer %d: heads, dim and vdim must be positive" % i)
    if isinstance(m, MatrixMemorySpec):
        if not m.gate_cap > 0:
            raise ValueError("layer %d: gate_cap must be positive" % i)
        return
    if isinstance(m, (AttentionSpec, DeltaRuleSpec)) and (m.kv_heads < 1 or m.heads % m.kv_heads):
        raise ValueError("layer %d: heads must be a multiple of kv_heads" % i)
    if isinstance(m, DeltaRuleSpec):
        if m.conv < 1:
            raise ValueError("layer %d: a convolution of %d taps" % (i, m.conv))
        return
    if isinstance(m, ForgetScanSpec):
        return
    if m.mask.kind != "causal" and m.mask.size < 1:
        raise ValueError("layer %d: a %s of %d positions" % (i, m.mask.kind, m.mask.size))
    if m.rotary is not None and (m.rotary.dims % 2 or m.rotary.dims < 0):
        raise ValueError("layer %d: rot.dims must be even" % i)
    if isinstance(m, AttentionSpec):
        if m.rotary is not None and m.rotary.dims > m.dim:
            raise ValueError("layer %d: rot.dims exceeds dim" % i)
        if m.softcap < 0:
            raise ValueError("layer %d: softcap must not be negative" % i)
        return
    if m.kv_rank < 1:
        raise ValueError("layer %d: kv_rank must be positive" % i)
    if m.rot_dim and (m.rotary is None or m.rotary.dims != m.rot_dim):
        raise ValueError("layer %d: rot.dims must equal rot_dim" % i)
    if m.kv_from is not None and m.rot_dim:
        raise NotImplementedError("layer %d: shared latents with a rotated key part" % i)
    if m.kv_from is not None:
        if not 0 <= m.kv_from < i:
            raise ValueError("layer %d: kv_from must name an earlier layer" % i)
        src = specs[m.kv_from].mixer
        if getattr(src, "kv_rank", None) != m.kv_rank or src.kv_from is not None or src.rot_dim:
            raise ValueError("layer %d: layer %d has no latents of this kv_rank of its own"
                             % (i, m.kv_from))


def _validate_feed_forward(i: int, f: FeedForwardSpec) -> None:
    if f.experts and not 1 <= f.top <= f.experts + f.identity:
        raise ValueError("layer %d: top must lie between 1 and the number of experts" % i)
    if f.ff < 1:
        raise ValueError("layer %d: ff must be positive" % i)
    if f.experts and (f.groups < 1 or f.experts % f.groups or not 1 <= f.keep_groups <= f.groups):
        raise ValueError("layer %d: router.groups must divide the experts, and keep some of them" % i)
    if f.experts and f.groups > 1 and f.top > f.keep_groups * (f.experts // f.groups):
        raise ValueError("layer %d: top exceeds the experts of the kept groups" % i)
    if f.identity < 0:
        raise ValueError("layer %d: router.identity must not be negative" % i)
    if f.act == "clamped_swish" and not f.limit > 0:
        raise ValueError("layer %d: the feed-forward's limit must be positive" % i)
    if f.shared is not None:
        _validate_feed_forward(i, f.shared)


def validate_layer_specs(specs: tuple, loop: Optional[LoopSpec] = None) -> None:
    for i, l in enumerate(specs):
        for m in mixer_parts(l.mixer):
            _validate_mixer(i, m, specs)
        if l.mlp is not None:
            _validate_feed_forward(i, l.mlp)
        if l.weights_of is not None:
            j = l.weights_of
            if not 0 <= j < len(specs) or j == i:
                raise ValueError("layer %d: weights_of must name another layer" % i)
            if specs[j].weights_of is not None and loops_back(specs, i):
                raise ValueError("layer %d: weights_of leads back to itself" % i)
            if specs[j].mixer != l.mixer or specs[j].mlp != l.mlp:
                raise ValueError("layer %d: layer %d, whose weights it uses, differs" % (i, j))
    if loop is not None:
        if not (0 <= loop.start < loop.stop <= len(specs) and loop.times >= 1):
            raise ValueError("loop: 0 <= start < stop <= layers and times >= 1 are needed")
        for i in range(len(specs)):
            src = getattr(specs[i].mixer, "kv_from", None)
            if src is not None and (loop.start <= src < loop.stop or loop.start <= i < loop.stop):
                raise NotImplementedError("layer %d: shared latents inside a loop" % i)


def loops_back(specs: tuple, i: int) -> bool:
    seen = set()
    while i is not None and i not in seen:
        seen.add(i)
        i = specs[i].weights_of
    return i is not None


def weights_index(specs: tuple, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while specs[i].weights_of is not None:
        i = specs[i].weights_of
    return i


@dataclass
class ModelConfig:
    """Architecture of a decoder (Llama, Mistral, Qwen2 and Qwen3 dense models, optionally
    SwiftKV for Llama; Taralix, Zatirax, Pererax and Pefivik, which list their layers one by one) or
    encoder (BERT)."""

    architecture: str = "LlamaForCausalLM"
    model_type: str = "llama"
    hidden_size: int = 4096
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 8
    head_dim: int = 128
    intermediate_size: int = 14336
    vocab_size: int = 128256
    rms_norm_eps: float = 1e-5
    rope_theta: float = 500000.0
    rope_scaling: Optional[dict] = None
    max_position_embeddings: int = 131072
    tie_word_embeddings: bool = False
    # SwiftKV: layers >= num_key_value_layers take K/V from a projection of the hidden
    # state after layer num_key_value_layers - 1 (None: plain Llama).
    num_key_value_layers: Optional[int] = None
    # Qwen3: RMSNorm over head_dim on every query and key head before RoPE
    qk_norm: bool = False
    # Qwen2: a bias on the query / key / value projections (none on o_proj or the MLP)
    qkv_bias: bool = False
    # attention window of the checkpoint (Mistral v0.1): contexts up to this length see every
    # earlier token, so they are served; longer ones are refused (no windowed attention kernel)
    sliding_window: Optional[int] = None
    # K/V heads of the checkpoint when ``num_key_value_heads`` was raised (see __post_init__)
    checkpoint_kv_heads: Optional[int] = None
    # models that list their layers (each with its own mixer and feed-forward)
    layer_specs: Optional[tuple] = None
    # factor of the residual stream in "norm after the sum" layers: x <- norm(alpha * x + f(x))
    postln_alpha: float = 1.0
    embedding_scale: float = 1.0
    bigram: Optional[BigramSpec] = None
    # factor of every sublayer's output in "pre" layers: x <- x + residual_mult * f(norm(x))
    residual_mult: float = 1.0
    logit_softcap: float = 0.0  # logits become softcap * tanh(logits / softcap); 0: they do not
    loop: Optional[LoopSpec] = None
    # encoder-only fields
    type_vocab_size: int = 2
    layer_norm_eps: float = 1e-12
    pooling: str = "cls"  # cls | mean
    normalize: bool = True
    hidden_act: str = "silu"
    # weights
    dtype: str = "bfloat16"
    quantization: Optional[str] = None  # None | "fp8"
    fp8_block_size: int = 128
    # "channel": a scale per output feature, activations per token; "block": 128 x 128 blocks
    fp8_scheme: str = "channel"
    eos_token_id: Optional[int] = None
    # further end-of-sequence ids (a list in config.json or generation_config.json, e.g. the
    # end-of-turn token of instruction-tuned Llama 3): they end a request like EOS does
    extra_eos_token_ids: tuple = ()
    bos_token_id: Optional[int] = None
    name_or_path: str = ""

    def __post_init__(self):
        """The attention kernels pack the G = heads / kv_heads query heads of a K/V head into
        128-row tiles, so G must divide 128. A checkpoint with another ratio (Qwen2.5-7B: 7,
        14B / 32B: 5, 1.5B: 6) is served with each of its K/V heads stored r times, r the
        smallest divisor of G that leaves G / r a divisor of 128: the model is the same
        function, the KV cache is r times larger. ``num_key_value_heads`` is the number of
        heads stored; ``checkpoint_kv_heads`` keeps the checkpoint's."""
        hq, hkv = self.num_attention_heads, self.num_key_value_heads
        if self.is_encoder or self.layer_specs is not None or hkv <= 0 or hq % hkv:
            return
        g = hq // hkv
        if 128 % g == 0:
            return
        r = next(r for r in range(2, g + 1) if g % r == 0 and 128 % (g // r) == 0)
        if self.checkpoint_kv_heads is None:
            self.checkpoint_kv_heads = hkv
        self.num_key_value_heads = hkv * r

    @property
    def kv_head_replication(self) -> int:
        return self.num_key_value_heads // (self.checkpoint_kv_heads or self.num_key_value_heads)

    @property
    def is_swiftkv(self) -> bool:
        return self.num_key_value_layers is not None and \
            self.num_key_value_layers < self.num_hidden_layers

    @property
    def is_encoder(self) -> bool:
        return self.model_type in ("bert",)

    @property
    def supports_float32(self) -> bool:
        """Whether the model can be served with 32-bit weights, activations and cache."""
        return self.layer_specs is not None

    @property
    def has_state(self) -> bool:
        """Whether layers carry a state from token to token beside, or instead of, a cache."""
        return self.layer_specs is not None and any(has_state(l.mixer) for l in self.layer_specs)

    def validate(self) -> None:
        if self.layer_specs is not None:
            validate_layer_specs(self.layer_specs, self.loop)
            if self.bigram is not None and self.bigram.buckets < 1:
                raise ValueError("embedding.bigram.buckets must be positive")
            if self.logit_softcap < 0:
                raise ValueError("logit_softcap must not be negative")
            if self.quantization is not None:
                raise NotImplementedError("quantization=%r for %s" % (self.quantization,
                                                                      self.architecture))
            return
        if self.num_attention_heads % self.num_key_value_heads:
            raise ValueError("num_attention_heads must be a multiple of num_key_value_heads")
        if self.head_dim not in (64, 128):
            raise ValueError("head_dim must be 64 or 128 (tensor-memory attention tiles)")
        if self.quantization not in (None, "fp8"):
            raise ValueError("quantization must be None or 'fp8'")
        if self.fp8_scheme not in ("channel", "block"):
            raise ValueError("fp8_scheme must be 'channel' or 'block'")
        if (self.qk_norm or self.qkv_bias) and self.is_swiftkv:
            raise NotImplementedError("SwiftKV with per-head query / key norms or a QKV bias")
        if self.qkv_bias and self.quantization == "fp8" and self.fp8_scheme == "block":
            raise NotImplementedError("a QKV bias with block-scaled fp8 linears: use "
                                      "fp8_scheme='channel'")

    @classmethod
    def from_hf_dict(cls, d: dict, name_or_path: str = "") -> "ModelConfig":
        archs = d.get("architectures") or ["LlamaForCausalLM"]
        mt = d.get("model_type", "llama")
        heads = d.get("num_attention_heads", 32)
        hidden = d.get("hidden_size", 4096)
        eos, extra_eos = d.get("eos_token_id"), ()
        if isinstance(eos, list):
            eos, extra_eos = (eos[0] if eos else None), tuple(int(t) for t in eos[1:])
        if mt not in DECODER_MODEL_TYPES and mt != "bert":
            raise NotImplementedError("model_type %r (supported: %s, bert)" %
                                      (mt, ", ".join(DECODER_MODEL_TYPES)))
        if d.get("attention_bias") or d.get("mlp_bias"):
            # (Llama's attention_bias also puts a bias on o_proj; Qwen2's QKV-only bias is
            # part of its architecture and has no flag)
            raise NotImplementedError("linear layers with bias (attention_bias / mlp_bias)")
        window = d.get("sliding_window") if d.get("use_sliding_window", True) else None
        # transformers >= 5 writes one ``rope_parameters`` dict (theta, type and the scaling
        # fields together); older checkpoints have ``rope_theta`` beside ``rope_scaling``
        rope = d.get("rope_parameters") or {}
        theta = d.get("rope_theta", rope.get("rope_theta", 10000.0))
        scaling = d.get("rope_scaling")
        if scaling is None and rope.get("rope_type", rope.get("type", "default")) != "default":
            scaling = {k: v for k, v in rope.items() if k != "rope_theta"}
        cfg = cls(
            architecture=archs[0], model_type=mt, hidden_size=hidden,
            num_hidden_layers=d.get("num_hidden_layers", 32), num_attention_heads=heads,
            num_key_value_heads=d.get("num_key_value_heads", heads),
            head_dim=d.get("head_dim") or hidden // heads,
            intermediate_size=d.get("intermediate_size", 4 * hidden),
            vocab_size=d.get("vocab_size", 32000),
            rms_norm_eps=d.get("rms_norm_eps", 1e-5),
            rope_theta=theta, rope_scaling=scaling,
            max_position_embeddings=d.get("max_position_embeddings", 4096),
            tie_word_embeddings=d.get("tie_word_embeddings", False),
            num_key_value_layers=d.get("num_key_value_layers"),
            qk_norm=(mt == "qwen3"), qkv_bias=(mt == "qwen2"), sliding_window=window,
            type_vocab_size=d.get("type_vocab_size", 2),
            layer_norm_eps=d.get("layer_norm_eps", 1e-12),
            hidden_act=d.get("hidden_act", "silu"),
            eos_token_id=eos, extra_eos_token_ids=extra_eos, bos_token_id=d.get("bos_token_id"),
            name_or_path=name_or_path)
        q = d.get("quantization_config")
        if q and q.get("quant_method") in ("fp8", "compressed-tensors"):
            cfg.quantization = "fp8"
            wbs = q.get("weight_block_size")
            if wbs:
                cfg.fp8_block_size = int(wbs[0])
        return cfg

    @classmethod
    def from_layer_list(cls, d: dict, name_or_path: str = "") -> "ModelConfig":
        """config.json of a layer-list model (``architecture``, ``width``, ``vocab``, ``norm`` and
        ``layers``; by design ``postln_alpha``, ``residual_mult``, ``embedding.scale``,
        ``embedding.bigram``, ``logit_softcap``, ``loop``). The head fields
        describe the cache as the engine sees it: one "head" of as many numbers as the widest
        layer keeps per token."""
        design = LAYER_LIST_DESIGNS[d["architecture"]]
        specs = read_layer_specs(d["layers"], design)
        if not specs:
            raise ValueError("a model without layers")
        parts = [m for l in specs for m in mixer_parts(l.mixer)]

        def kept(m):
            if isinstance(m, AttentionSpec):
                return m.kv_heads * (m.dim + m.vdim)
            return m.kv_rank + m.rot_dim if isinstance(m, LatentAttentionSpec) else m.dim
        eos, loop, emb = d.get("eos_token_id"), d.get("loop"), d.get("embedding") or {}
        bigram = emb.get("bigram")
        return cls(
            architecture=d["architecture"], model_type=d["architecture"].lower(),
            hidden_size=int(d["width"]), num_hidden_layers=len(specs),
            num_attention_heads=max(m.heads for m in parts), num_key_value_heads=1,
            head_dim=max(kept(m) for m in parts),
            intermediate_size=max((l.mlp.ff for l in specs if l.mlp is not None), default=0),
            vocab_size=int(d["vocab"]), rms_norm_eps=float(d["norm"]["eps"]),
            postln_alpha=float(d["postln_alpha"]) if design.residual == "post" else 1.0,
            embedding_scale=float(emb.get("scale", 1.0)),
            bigram=None if not bigram else BigramSpec(*(int(bigram[k]) for k in (
                "buckets", "mul_prev", "mul_cur"))),
            residual_mult=float(d["residual_mult"]) if design.residual == "pre" else 1.0,
            logit_softcap=float(d.get("logit_softcap") or 0.0),
            loop=None if not loop else LoopSpec(int(loop["start"]), int(loop["stop"]),
                                                int(loop["times"]), design.loop_reenters),
            layer_specs=specs, tie_word_embeddings=design.tied,
            # no table is indexed by position, so nothing bounds it
            max_position_embeddings=1 << 20, hidden_act="",
            eos_token_id=int(eos) if isinstance(eos, int) else None, name_or_path=name_or_path)

    @property
    def design(self) -> LayerListDesign:
        return LAYER_LIST_DESIGNS[self.architecture]

    @property
    def layer_runs(self) -> list:
        """(layer whose weights run, pass of the loop or None) in the order of execution of a
        layer-list model; the pass is named at its first layer only."""
        order = [weights_index(self.layer_specs, i) for i in range(len(self.layer_specs))]
        if self.loop is None:
            return [(l, None) for l in order]
        lo, hi, n = self.loop.start, self.loop.stop, self.loop.times
        body = [(l, t if k == 0 else None) for t in range(n) for k, l in enumerate(order[lo:hi])]
        return [(l, None) for l in order[:lo]] + body + [(l, None) for l in order[hi:]]

    @classmethod
    def from_pretrained(cls, path: str) -> "ModelConfig":
        if path in PRESETS:
            return dataclasses.replace(PRESETS[path], name_or_path=path)
        with open(os.path.join(path, "config.json")) as f:
            d = json.load(f)
        if d.get("architecture") in LAYER_LIST_ARCHITECTURES:
            cfg = cls.from_layer_list(d, path)
        else:
            cfg = cls.from_hf_dict(d, path)
        gen = os.path.join(path, "generation_config.json")
        if os.path.exists(gen):
            with open(gen) as f:
                ids = json.load(f).get("eos_token_id")
            ids = [] if ids is None else ([int(t) for t in ids] if isinstance(ids, list) else [int(ids)])
            if cfg.eos_token_id is None and ids:
                cfg.eos_token_id = ids[0]
            known = {cfg.eos_token_id, *cfg.extra_eos_token_ids}
            cfg.extra_eos_token_ids += tuple(t for t in dict.fromkeys(ids) if t not in known)
        return cfg


# decoder families the Llama code path serves: Mistral is Llama under another name once its
# sliding window is off; Qwen2 adds a bias on the QKV projection; Qwen3 (dense) adds the
# per-head query / key norms and a head_dim that is not hidden_size / heads
DECODER_MODEL_TYPES = ("llama", "llama_swiftkv", "mistral", "qwen2", "qwen3")

# models whose config.json lists the layers instead of giving one shape for all of them
LAYER_LIST_ARCHITECTURES = tuple(LAYER_LIST_DESIGNS)


def _taralix(width, vocab, layers, alpha, eps=1e-6) -> ModelConfig:
    """``layers``: (heads, dim, vdim, kv_rank, kv_from, feed-forward) each; the feed-forward is
    None, ff (dense) or (ff, experts, top)."""
    out = []
    for heads, dim, vdim, rank, src, f in layers:
        m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5}
        if src is not None:
            m["kv_from"] = src
        mlp = None
        if isinstance(f, int):
            mlp = {"kind": "dense", "ff": f}
        elif f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f[0]}, "router": {"experts": f[1], "top": f[2]}}
        out.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return ModelConfig.from_layer_list({"architecture": "Taralix", "width": width, "vocab": vocab,
                                        "norm": {"eps": eps}, "postln_alpha": alpha,
                                        "layers": out})


def _zatirax(width, vocab, layers, loop, scale=1.0, eps=1e-6) -> ModelConfig:
    """``layers``: (mixer, ff) each; a mixer with ``kv_heads`` is ordinary attention."""
    out = [{"type": "attention" if "kv_heads" in m else "latent_attention", "mixer": m,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": 7.0}}
           for m, ff in layers]
    return ModelConfig.from_layer_list({
        "architecture": "Zatirax", "width": width, "vocab": vocab, "norm": {"eps": eps},
        "embedding": {"scale": scale}, "layers": out,
        "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))})


def _pererax(width, vocab, layers, eps=1e-6) -> ModelConfig:
    """``layers``: (mixer, feed-forward) each, or the number of the layer whose weights are used.
    The feed-forward is None or (ff, experts, identity experts, top, ff of the shared expert)."""
    out = []
    for l in layers:
        if isinstance(l, int):
            out.append({**out[l], "weights_of": l})
            continue
        m, f = l
        kind = "parallel" if "left" in m else "channel_delta" if "conv" in m else "attention"
        out.append({"type": kind, "mixer": m, "mlp": None if f is None else {
            "kind": "moe", "expert": {"ff": f[0], "limit": 7.0},
            "router": {"experts": f[1], "identity": f[2], "top": f[3], "scale": 1.5},
            "shared": {"ff": f[4], "limit": 7.0} if f[4] else None}})
    return ModelConfig.from_layer_list({"architecture": "Pererax", "width": width, "vocab": vocab,
                                        "norm": {"eps": eps}, "layers": out})


def _pefivik(width, vocab, layers, loop, bigram, mult=0.5, cap=30.0, eps=1e-6) -> ModelConfig:
    """``layers``: (mixer, feed-forward) each; the feed-forward is None, ff (dense) or (ff, experts,
    top, (groups, kept), ff of the shared expert)."""
    out = []
    for m, f in layers:
        mlp = None
        if isinstance(f, int):
            mlp = {"kind": "dense", "ff": f}
        elif f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f[0]}, "shared": {"ff": f[4]} if f[4] else None,
                   "router": {"experts": f[1], "top": f[2], "scale": 1.5,
                              "groups": dict(zip(("count", "keep"), f[3]))}}
        out.append({"type": "latent_attention" if "kv_rank" in m else "hgrn2", "mixer": m,
                    "mlp": mlp})
    return ModelConfig.from_layer_list({
        "architecture": "Pefivik", "width": width, "vocab": vocab, "norm": {"eps": eps},
        "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
        "residual_mult": mult, "logit_softcap": cap, "layers": out,
        "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))})


def _llama(layers, hidden, heads, kv, inter, **kw) -> ModelConfig:
    return ModelConfig(hidden_size=hidden, num_hidden_layers=layers, num_attention_heads=heads,
                       num_key_value_heads=kv, head_dim=128, intermediate_size=inter, **kw)


_LLAMA3_SCALING = {"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0,
                   "high_freq_factor": 4.0, "original_max_position_embeddings": 8192}

# Synthetic (random-weight) presets for the architectures the benchmarks name.
PRESETS: dict[str, ModelConfig] = {
    "llama-3.1-8b": _llama(32, 4096, 32, 8, 14336, rope_scaling=dict(_LLAMA3_SCALING)),
    "llama-3.1-8b-swiftkv": _llama(32, 4096, 32, 8, 14336, rope_scaling=dict(_LLAMA3_SCALING),
                                   num_key_value_layers=16, model_type="llama_swiftkv",
                                   architecture="LlamaSwiftKVForCausalLM"),
    "llama-3.3-70b": _llama(80, 8192, 64, 8, 28672, rope_scaling=dict(_LLAMA3_SCALING)),
    "llama-3.3-70b-swiftkv": _llama(80, 8192, 64, 8, 28672, rope_scaling=dict(_LLAMA3_SCALING),
                                    num_key_value_layers=40, model_type="llama_swiftkv",
                                    architecture="LlamaSwiftKVForCausalLM"),
    "llama-tiny": ModelConfig(hidden_size=256, num_hidden_layers=2, num_attention_heads=4,
                              num_key_value_heads=2, head_dim=64, intermediate_size=512,
                              vocab_size=1024, max_position_embeddings=4096, rope_theta=10000.0),
    "llama-tiny-swiftkv": ModelConfig(hidden_size=256, num_hidden_layers=4, num_attention_heads=4,
                                      num_key_value_heads=2, head_dim=64, intermediate_size=512,
                                      vocab_size=1024, max_position_embeddings=4096,
                                      rope_theta=10000.0, num_key_value_layers=2,
                                      model_type="llama_swiftkv",
                                      architecture="LlamaSwiftKVForCausalLM"),
    "mistral-7b": _llama(32, 4096, 32, 8, 14336, architecture="MistralForCausalLM",
                         model_type="mistral", vocab_size=32768, rope_theta=1000000.0,
                         max_position_embeddings=32768),
    "qwen2.5-7b": _llama(28, 3584, 28, 4, 18944, architecture="Qwen2ForCausalLM",
                         model_type="qwen2", qkv_bias=True, vocab_size=152064,
                         rope_theta=1000000.0, rms_norm_eps=1e-6, max_position_embeddings=32768),
    # the reasoning model of the Dynasor examples (a Qwen2 architecture)
    "deepseek-r1-distill-qwen-1.5b": ModelConfig(
        architecture="Qwen2ForCausalLM", model_type="qwen2", qkv_bias=True, hidden_size=1536,
        num_hidden_layers=28, num_attention_heads=12, num_key_value_heads=2, head_dim=128,
        intermediate_size=8960, vocab_size=151936, rope_theta=10000.0, rms_norm_eps=1e-6,
        max_position_embeddings=131072),
    "qwen2-tiny": ModelConfig(architecture="Qwen2ForCausalLM", model_type="qwen2", qkv_bias=True,
                              hidden_size=256, num_hidden_layers=2, num_attention_heads=4,
                              num_key_value_heads=2, head_dim=64, intermediate_size=512,
                              vocab_size=1024, max_position_embeddings=4096, rope_theta=10000.0,
                              rms_norm_eps=1e-6),
    "qwen3-8b": _llama(36, 4096, 32, 8, 12288, architecture="Qwen3ForCausalLM",
                       model_type="qwen3", qk_norm=True, vocab_size=151936, rope_theta=1000000.0,
                       rms_norm_eps=1e-6, max_position_embeddings=40960),
    "qwen3-32b": _llama(64, 5120, 64, 8, 25600, architecture="Qwen3ForCausalLM",
                        model_type="qwen3", qk_norm=True, vocab_size=151936, rope_theta=1000000.0,
                        rms_norm_eps=1e-6, max_position_embeddings=40960),
    "qwen3-tiny": ModelConfig(architecture="Qwen3ForCausalLM", model_type="qwen3", qk_norm=True,
                              hidden_size=256, num_hidden_layers=2, num_attention_heads=8,
                              num_key_value_heads=2, head_dim=64, intermediate_size=512,
                              vocab_size=1024, max_position_embeddings=4096, rope_theta=10000.0,
                              rms_norm_eps=1e-6),
    "llama-small": ModelConfig(hidden_size=1024, num_hidden_layers=4, num_attention_heads=8,
                               num_key_value_heads=8, head_dim=128, intermediate_size=2816,
                               vocab_size=32000, max_position_embeddings=8192),
    "bert-base": ModelConfig(architecture="BertModel", model_type="bert", hidden_size=768,
                             num_hidden_layers=12, num_attention_heads=12, num_key_value_heads=12,
                             head_dim=64, intermediate_size=3072, vocab_size=30522,
                             max_position_embeddings=512, hidden_act="gelu"),
    "bert-tiny": ModelConfig(architecture="BertModel", model_type="bert", hidden_size=128,
                             num_hidden_layers=2, num_attention_heads=2, num_key_value_heads=2,
                             head_dim=64, intermediate_size=256, vocab_size=1000,
                             max_position_embeddings=512, hidden_act="gelu"),
    "taralix-tiny": _taralix(192, 1024, [(6, 32, 48, 96, None, 320), (4, 64, 32, 96, 0, (64, 8, 3)),
                                         (5, 40, 64, 40, None, None)], alpha=1.7),
    "zatirax-tiny": _zatirax(192, 1024, [
        ({"heads": 5, "dim": 40, "vdim": 48, "kv_rank": 72, "rot_dim": 24, "scale": 0.15,
          "mask": {"size": 90}, "rot": {"base": 10000.0, "dims": 24}}, 320),
        ({"heads": 6, "kv_heads": 2, "dim": 64, "vdim": 48, "scale": 0.125, "mask": {"size": 150},
          "rot": {"base": 10000.0, "dims": 48, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0,
                                                           "original": 512}}}, 256),
        ({"heads": 4, "dim": 32, "vdim": 32, "kv_rank": 48, "rot_dim": 16, "scale": 0.2,
          "mask": {"size": 33}, "rot": {"base": 5000.0, "dims": 16}}, None)], loop=(1, 3, 2)),
    "pererax-tiny": _pererax(160, 1024, [
        ({"heads": 4, "kv_heads": 2, "dim": 40, "vdim": 56, "conv": 3}, (64, 6, 2, 3, 96)),
        ({"left": {"heads": 4, "kv_heads": 2, "dim": 40, "vdim": 32, "scale": 0.16, "softcap": 20.0,
                   "rot": {"base": 10000.0, "dims": 24}},
          "right": {"heads": 3, "dim": 24, "vdim": 40, "gate_cap": 10.0}}, (48, 4, 1, 2, 0)),
        ({"heads": 6, "kv_heads": 3, "dim": 32, "vdim": 32, "scale": 0.18, "mask": {"size": 50},
          "rot": {"base": 10000.0, "dims": 32}}, None), 0, 1]),
    "pefivik-tiny": _pefivik(160, 1024, [
        ({"heads": 5, "dim": 40, "vdim": 24, "kv_rank": 56, "scale": 0.16}, 288),
        ({"heads": 3, "dim": 56, "vdim": 40}, (48, 10, 3, (5, 2), 72)),
        ({"heads": 4, "dim": 32, "vdim": 48, "kv_rank": 72, "scale": 0.18}, None)], loop=(1, 3, 2),
        bigram=(301, 13, 7)),
}


# --------------------------------------------------------------------------------------
# parallelism
# --------------------------------------------------------------------------------------
@dataclass
class ParallelConfig:
    tensor_parallel_size: int = 1
    ulysses_sequence_parallel_size: int = 1
    pipeline_parallel_size: int = 1
    data_parallel_size: int = 1
    enable_shift_parallel: bool = False
    # steps with at most this many tokens run tensor-parallel. The reference's default is 512;
    # here 128 (one 128-token tile per linear, the shape the decode GEMMs are built for):
    # measured on 2 GPUs, 256-token decode steps serve 5 % more tokens/s sequence-parallel
    shift_parallel_threshold: int = SHIFT_PARALLEL_THRESHOLD
    enable_expert_parallel: bool = False
    # "fused": own NVLink kernels; "nccl": library collectives (kept for A/B runs)
    comm_backend: str = "fused"

    def __post_init__(self):
        if self.enable_shift_parallel and self.ulysses_sequence_parallel_size == 1:
            raise ValueError("ulysses_sequence_parallel_size must be > 1 "
                             "when enable_shift_parallel is True.")
        for name in ("tensor_parallel_size", "ulysses_sequence_parallel_size",
                     "pipeline_parallel_size", "data_parallel_size"):
            if getattr(self, name) < 1:
                raise ValueError("%s must be >= 1" % name)
        if self.comm_backend not in ("fused", "nccl"):
            raise ValueError("comm_backend must be 'fused' or 'nccl'")

    @property
    def world_size(self) -> int:
        """Ranks of one engine replica: PP x SP x TP (data-parallel replicas are separate)."""
        return (self.pipeline_parallel_size * self.tensor_parallel_size *
                self.ulysses_sequence_parallel_size)

    @property
    def sp(self) -> int:
        return self.ulysses_sequence_parallel_size

    @property
    def tp(self) -> int:
        return self.tensor_parallel_size


# --------------------------------------------------------------------------------------
# speculative decoding
# --------------------------------------------------------------------------------------
@dataclass
class SpeculativeConfig:
    method: Optional[str] = None  # arctic | mlp_speculator | suffix
    model: Optional[str] = None
    num_speculative_tokens: Optional[int] = None
    disable_by_batch_size: Optional[int] = None
    hard_disable_by_batch_size: Optional[int] = None
    enable_suffix_decoding: bool = False
    suffix_cache_max_depth: int = 64
    suffix_speculative_tokens: int = 0
    suffix_cache_max_requests: int = 100000
    suffix_max_spec_factor: float = 1.0
    suffix_max_spec_offset: float = 0.0
    suffix_min_token_prob: float = 0.1
    draft_tensor_parallel_size: Optional[int] = None
    quantization: Optional[str] = None     # "fp8": block-scaled fp8 projections and LM heads of the drafter

    def __post_init__(self):
        if self.quantization not in (None, "fp8"):
            raise ValueError("speculator quantization must be None or 'fp8'")
        if self.method not in (None, "arctic", "mlp_speculator", "suffix"):
            raise ValueError("unknown speculative method %r" % (self.method,))
        arctic = self.method in ("arctic", "mlp_speculator")
        suffix_only = self.method == "suffix" or (self.method is None and
                                                  self.enable_suffix_decoding)
        hybrid = self.method == "arctic" and self.enable_suffix_decoding
        if (suffix_only or arctic) and self.disable_by_batch_size is None:
            self.disable_by_batch_size = 64
        if (self.hard_disable_by_batch_size is not None and
                self.disable_by_batch_size is not None and
                self.hard_disable_by_batch_size <= self.disable_by_batch_size):
            logger.warning("hard_disable_by_batch_size=%d <= disable_by_batch_size=%d: "
                           "the first-N cap never applies", self.hard_disable_by_batch_size,
                           self.disable_by_batch_size)
        if hybrid:
            self.suffix_speculative_tokens = self.suffix_cache_max_depth
        if suffix_only:
            self.method = "suffix"
            self.enable_suffix_decoding = True
            if self.suffix_speculative_tokens > 0:
                self.num_speculative_tokens = self.suffix_speculative_tokens
            elif self.num_speculative_tokens is None:
                self.num_speculative_tokens = 16
        elif arctic:
            if self.model is None:
                raise ValueError("speculative method %r needs a draft 'model'" % self.method)
            if not self.num_speculative_tokens:
                self.num_speculative_tokens = None  # filled from the draft model's n_predict
        if self.num_speculative_tokens is not None and self.num_speculative_tokens < 0:
            raise ValueError("num_speculative_tokens must be >= 0")

    @property
    def uses_arctic(self) -> bool:
        return self.method in ("arctic", "mlp_speculator")

    @property
    def uses_suffix(self) -> bool:
        return self.enable_suffix_decoding

    @property
    def max_draft_tokens(self) -> int:
        """Widest draft any request can carry into a verification step."""
        return max(self.num_speculative_tokens or 0, self.suffix_speculative_tokens or 0)

    def effective_draft_limit(self, batch_size: int) -> int:
        """How many requests of a running batch may draft this step: 0 once the batch
        reaches the hard cap, the first ``disable_by_batch_size`` above the soft cap,
        everyone otherwise."""
        if (self.hard_disable_by_batch_size is not None and
                batch_size >= self.hard_disable_by_batch_size):
            return 0
        if self.disable_by_batch_size is not None and batch_size > self.disable_by_batch_size:
            return self.disable_by_batch_size
        return batch_size

    @classmethod
    def from_json(cls, value) -> Optional["SpeculativeConfig"]:
        if value is None:
            return None
        if isinstance(value, cls):
            return value
        if isinstance(value, str):
            value = json.loads(value)
        known = {f.name for f in dataclasses.fields(cls)}
        unknown = set(value) - known
        if unknown:
            raise ValueError("unknown speculative-config keys: %s" % sorted(unknown))
        return cls(**value)


# --------------------------------------------------------------------------------------
# cache / scheduler / forest cascade attention
# --------------------------------------------------------------------------------------
# cache element types the attention kernels can read (the cache writers also produce nvfp4)
SUPPORTED_KV_CACHE_DTYPES = ("auto", "bfloat16")


@dataclass
class CacheConfig:
    block_size: int = 64
    gpu_memory_utilization: float = 0.9
    num_gpu_blocks: Optional[int] = None  # None: sized from free memory
    kv_cache_dtype: str = "auto"  # auto (= model dtype) | fp8 | nvfp4
    enable_prefix_caching: bool = True

    def __post_init__(self):
        if self.block_size not in (16, 32, 64, 128):
            raise ValueError("block_size must be 16, 32, 64 or 128")
        if self.kv_cache_dtype not in ("auto", "bfloat16", "fp8", "nvfp4"):
            raise ValueError("unsupported kv_cache_dtype %r" % self.kv_cache_dtype)


@dataclass
class SchedulerConfig:
    max_num_batched_tokens: int = 8192
    max_num_seqs: int = 256
    max_model_len: int = 8192
    enable_chunked_prefill: bool = True
    async_scheduling: bool = False


@dataclass
class ForestCascadeConfig:
    """Gates of forest cascade attention (shared-prefix grouping of decode batches);
    defaults as in arctic_inference/vllm/attention/flash_attn_forest_cascade.py:304-319."""
    enabled: bool = False
    max_query_len: int = 16
    min_batch_size: int = 8
    min_group_size: int = 2
    min_additional_prefix_blocks: int = 1
    min_non_singleton_fraction: float = 0.25
    max_non_singleton_groups: int = 256

    @classmethod
    def from_json(cls, value) -> "ForestCascadeConfig":
        if value is None:
            return cls(enabled=False)
        if isinstance(value, str):
            value = json.loads(value)
        known = {f.name for f in dataclasses.fields(cls)} - {"enabled"}
        unknown = set(value) - known
        if unknown:
            raise ValueError("unknown forest-cascade-attn keys: %s" % sorted(unknown))
        return cls(enabled=True, **value)


@dataclass
class EngineConfig:
    model: ModelConfig
    parallel: ParallelConfig
    cache: CacheConfig
    scheduler: SchedulerConfig
    speculative: Optional[SpeculativeConfig] = None
    forest_cascade: ForestCascadeConfig = field(default_factory=ForestCascadeConfig)
    fp32_lm_head: bool = False
    enforce_eager: bool = False
    enable_sleep_mode: bool = False
    seed: int = 0
    load_format: str = "auto"  # auto | dummy (random weights)
    tokenizer: Optional[str] = None
    served_model_name: Optional[str] = None

    def validate(self) -> None:
        m, p = self.model, self.parallel
        m.validate()
        ways = p.tp * p.sp
        if m.layer_specs is not None:
            self._validate_layer_list()
        if m.num_attention_heads % ways:
            raise ValueError("num_attention_heads (%d) must be divisible by TP*SP (%d)" %
                             (m.num_attention_heads, ways))
        if m.num_key_value_heads % p.tp and p.tp % m.num_key_value_heads:
            raise ValueError("num_key_value_heads and tensor_parallel_size must divide evenly")
        if m.is_swiftkv and p.pipeline_parallel_size > 1:
            raise ValueError("SwiftKV models do not support pipeline parallelism")
        if m.sliding_window is not None and self.scheduler.max_model_len > m.sliding_window:
            raise NotImplementedError(
                "sliding-window attention: this checkpoint attends to the last %d tokens only; "
                "contexts up to that length are served (max_model_len=%d asks for more)"
                % (m.sliding_window, self.scheduler.max_model_len))
        if not m.is_encoder and m.layer_specs is None:
            per_rank = (m.num_attention_heads // ways) // max(1, m.num_key_value_heads // ways)
            if per_rank < 1 or 128 % per_rank:
                raise NotImplementedError(
                    "%d query heads per K/V head on a rank (TP*SP = %d): the attention kernels "
                    "need a divisor of 128" % (per_rank, ways))
        # Options this engine parses for command-line compatibility but cannot honour are
        # refused here rather than ignored.
        if p.pipeline_parallel_size > 1:
            # whole-model stages (parallel/pipeline.py): one rank per stage, nothing sharded
            # inside a stage, no drafting (the drafter lives with the last stage's hidden states)
            if p.tp * p.sp > 1:
                raise NotImplementedError(
                    "pipeline_parallel_size > 1 together with tensor or sequence parallelism: "
                    "pipeline stages are whole-model stages here (TP = SP = 1)")
            if self.speculative is not None:
                raise NotImplementedError("speculative decoding with pipeline parallelism")
            if p.pipeline_parallel_size > m.num_hidden_layers:
                raise ValueError("more pipeline stages than decoder layers")
        if p.data_parallel_size > 1:
            raise NotImplementedError(
                "data_parallel_size > 1: replicas are separate engines here; start one server "
                "per replica, or use the replica pool (python -m arcticinference_b200.server.cli), "
                "which routes requests over them")
        if p.enable_expert_parallel:
            raise NotImplementedError("enable_expert_parallel: experts are not sharded over GPUs "
                                      "(mixture-of-experts models run on one GPU)")
        if self.cache.kv_cache_dtype not in SUPPORTED_KV_CACHE_DTYPES:
            raise NotImplementedError(
                "kv_cache_dtype=%r: the attention kernels read %s caches only" %
                (self.cache.kv_cache_dtype, " / ".join(SUPPORTED_KV_CACHE_DTYPES)))
        if self.speculative is not None and self.speculative.uses_suffix and \
                self.speculative.method not in ("arctic", "suffix"):
            raise ValueError("suffix decoding is only available with the arctic or suffix methods")
        if self.scheduler.max_num_batched_tokens < p.sp:
            raise ValueError("max_num_batched_tokens must be >= the sequence-parallel size")

    def _validate_layer_list(self) -> None:
        """What layer-list models do not run with is refused here."""
        m, p = self.model, self.parallel
        if p.world_size > 1:
            raise NotImplementedError("%s on more than one GPU (tensor, sequence or pipeline "
                                      "parallelism)" % m.architecture)
        if self.forest_cascade.enabled:
            raise NotImplementedError("forest cascade attention with %s" % m.architecture)
        if m.has_state and self.speculative is not None:
            raise NotImplementedError("speculative decoding with %s: the state of its recurrent "
                                      "layers cannot take rejected tokens back" % m.architecture)

    @property
    def kv_replication(self) -> int:
        """How many ranks hold a copy of each KV head (>1 when Hkv < TP*SP)."""
        ways = self.parallel.tp * self.parallel.sp
        return max(1, ways // self.model.num_key_value_heads)


# --------------------------------------------------------------------------------------
# flat CLI / keyword view
# --------------------------------------------------------------------------------------
def _env_flag(name: str) -> bool:
    return os.environ.get(name, "0").lower() in ("1", "true", "on", "yes")


@dataclass
class EngineArgs:
    model: str = "llama-tiny"
    tokenizer: Optional[str] = None
    served_model_name: Optional[str] = None
    dtype: str = "bfloat16"
    quantization: Optional[str] = None
    fp8_scheme: Optional[str] = None
    load_format: str = "auto"
    seed: int = 0
    max_model_len: Optional[int] = None
    tensor_parallel_size: int = 1
    pipeline_parallel_size: int = 1
    data_parallel_size: int = 1
    enable_expert_parallel: bool = False
    # Arctic flags
    ulysses_sequence_parallel_size: int = 1
    enable_shift_parallel: bool = False
    shift_parallel_threshold: int = SHIFT_PARALLEL_THRESHOLD
    forest_cascade_attn_configs: Optional[Any] = None
    fp32_lm_head: bool = False
    speculative_config: Optional[Any] = None
    # engine
    block_size: int = 64
    gpu_memory_utilization: float = 0.9
    num_gpu_blocks_override: Optional[int] = None
    kv_cache_dtype: str = "auto"
    enable_prefix_caching: bool = True
    max_num_batched_tokens: Optional[int] = None
    max_num_seqs: int = 256
    enable_chunked_prefill: bool = True
    async_scheduling: bool = True
    enforce_eager: bool = False
    enable_sleep_mode: bool = False
    comm_backend: str = "fused"
    distributed_executor_backend: Optional[str] = None
    hf_overrides: Optional[dict] = None

    def __post_init__(self):
        # Sequence parallelism always runs one process per GPU (arctic_inference/vllm/args.py:71-73).
        if self.ulysses_sequence_parallel_size > 1:
            self.distributed_executor_backend = "mp"
        if self.distributed_executor_backend not in (None, "mp", "external_launcher"):
            # one process per GPU under torch.distributed is the only executor there is
            raise NotImplementedError("distributed_executor_backend=%r (ranks are processes "
                                      "started by serve or torch.distributed.run)"
                                      % self.distributed_executor_backend)
        if _env_flag("ARCTIC_FP32_LM_HEAD"):
            self.fp32_lm_head = True

    # ---- CLI ---------------------------------------------------------------------------
    @staticmethod
    def add_cli_args(parser: argparse.ArgumentParser) -> argparse.ArgumentParser:
        g = parser.add_argument_group("model")
        g.add_argument("--tokenizer", type=str, default=None)
        g.add_argument("--served-model-name", type=str, default=None)
        g.add_argument("--dtype", type=str, default="bfloat16")
        g.add_argument("--quantization", "-q", type=str, default=None, choices=[None, "fp8"])
        g.add_argument("--fp8-scheme", type=str, default=None, choices=[None, "channel", "block"],
                       help="fp8 scale layout: one scale per output feature with per-token "
                            "activation scales (default), or 128 x 128 blocks")
        g.add_argument("--load-format", type=str, default="auto", choices=["auto", "dummy"])
        g.add_argument("--seed", type=int, default=0)
        g.add_argument("--max-model-len", type=int, default=None)
        g.add_argument("--hf-overrides", type=json.loads, default=None)
        g = parser.add_argument_group("parallelism")
        g.add_argument("--tensor-parallel-size", "-tp", type=int, default=1)
        g.add_argument("--pipeline-parallel-size", "-pp", type=int, default=1)
        g.add_argument("--data-parallel-size", "-dp", type=int, default=1)
        g.add_argument("--enable-expert-parallel", action="store_true")
        g.add_argument("--ulysses-sequence-parallel-size", type=int, default=1,
                       help="Number of Ulysses sequence parallel replicas")
        g.add_argument("--enable-shift-parallel", action="store_true",
                       help="Switch between sequence parallelism and full tensor parallelism "
                            "per step, by batch size")
        g.add_argument("--shift-parallel-threshold", type=int, default=SHIFT_PARALLEL_THRESHOLD,
                       help="Steps with at most this many tokens run in tensor-parallel mode")
        g.add_argument("--comm-backend", type=str, default="fused", choices=["fused", "nccl"])
        g.add_argument("--distributed-executor-backend", type=str, default=None)
        g = parser.add_argument_group("arctic")
        g.add_argument("--forest-cascade-attn-configs", type=str, default=None,
                       help="JSON object of forest cascade attention knobs; '{}' enables defaults")
        g.add_argument("--fp32-lm-head", action="store_true",
                       help="Compute the LM head in fp32")
        g.add_argument("--speculative-config", type=str, default=None,
                       help="JSON: method arctic|mlp_speculator|suffix, model, "
                            "num_speculative_tokens, enable_suffix_decoding, ...")
        g = parser.add_argument_group("engine")
        g.add_argument("--block-size", type=int, default=64)
        g.add_argument("--gpu-memory-utilization", type=float, default=0.9)
        g.add_argument("--num-gpu-blocks-override", type=int, default=None)
        g.add_argument("--kv-cache-dtype", type=str, default="auto")
        g.add_argument("--enable-prefix-caching", dest="enable_prefix_caching",
                       action="store_true", default=True)
        g.add_argument("--no-enable-prefix-caching", dest="enable_prefix_caching",
                       action="store_false")
        g.add_argument("--max-num-batched-tokens", type=int, default=None)
        g.add_argument("--max-num-seqs", type=int, default=256)
        g.add_argument("--enable-chunked-prefill", dest="enable_chunked_prefill",
                       action="store_true", default=True)
        g.add_argument("--no-enable-chunked-prefill", dest="enable_chunked_prefill",
                       action="store_false")
        g.add_argument("--async-scheduling", dest="async_scheduling", action="store_true", default=True,
                       help="queue the next decode step before the previous step's tokens are read")
        g.add_argument("--no-async-scheduling", dest="async_scheduling", action="store_false")
        g.add_argument("--enforce-eager", action="store_true")
        g.add_argument("--enable-sleep-mode", action="store_true")
        return parser

    @classmethod
    def from_cli_args(cls, ns: argparse.Namespace) -> "EngineArgs":
        names = {f.name for f in dataclasses.fields(cls)}
        return cls(**{k: v for k, v in vars(ns).items() if k in names})

    # ---- validation into an EngineConfig -------------------------------------------------
    def create_engine_config(self) -> EngineConfig:
        model = ModelConfig.from_pretrained(self.model)
        if self.hf_overrides:
            model = dataclasses.replace(model, **self.hf_overrides)
        if self.quantization is not None:
            model.quantization = self.quantization
        if self.fp8_scheme is not None:
            model.fp8_scheme = self.fp8_scheme
        if self.dtype in ("float32", "fp32", "float") and model.supports_float32:
            model.dtype = "float32"
        elif self.dtype in ("auto", "bfloat16", "bf16"):
            model.dtype = "bfloat16"
        else:
            raise NotImplementedError("dtype=%r: weights, activations and the KV cache of %s are "
                                      "bfloat16 (the kernels accumulate in fp32)"
                                      % (self.dtype, model.architecture))
        max_len = self.max_model_len or min(model.max_position_embeddings, 8192,
                                            model.sliding_window or 8192)
        parallel = ParallelConfig(
            tensor_parallel_size=self.tensor_parallel_size,
            ulysses_sequence_parallel_size=self.ulysses_sequence_parallel_size,
            pipeline_parallel_size=self.pipeline_parallel_size,
            data_parallel_size=self.data_parallel_size,
            enable_shift_parallel=self.enable_shift_parallel,
            shift_parallel_threshold=self.shift_parallel_threshold,
            enable_expert_parallel=self.enable_expert_parallel,
            comm_backend=self.comm_backend)
        cache = CacheConfig(block_size=self.block_size,
                            gpu_memory_utilization=self.gpu_memory_utilization,
                            num_gpu_blocks=self.num_gpu_blocks_override,
                            kv_cache_dtype=self.kv_cache_dtype,
                            # (a cached block holds no state of the recurrent layers)
                            enable_prefix_caching=self.enable_prefix_caching and not model.has_state)
        sched = SchedulerConfig(
            max_num_batched_tokens=self.max_num_batched_tokens or max(8192, 0),
            max_num_seqs=self.max_num_seqs, max_model_len=max_len,
            enable_chunked_prefill=self.enable_chunked_prefill,
            async_scheduling=self.async_scheduling)
        spec = SpeculativeConfig.from_json(self.speculative_config)
        cfg = EngineConfig(
            model=model, parallel=parallel, cache=cache, scheduler=sched, speculative=spec,
            forest_cascade=ForestCascadeConfig.from_json(self.forest_cascade_attn_configs),
            fp32_lm_head=self.fp32_lm_head, enforce_eager=self.enforce_eager,
            enable_sleep_mode=self.enable_sleep_mode, seed=self.seed,
            load_format="dummy" if self.model in PRESETS else self.load_format,
            tokenizer=self.tokenizer, served_model_name=self.served_model_name or self.model)
        cfg.validate()
        return cfg
