"""Ops of decoders with a 32-bit residual stream and of mixture-of-experts feed-forwards.

CUDA tensors run ``csrc/stream.cu``, ``csrc/moe.cu``, ``csrc/grouped_gemm.cu`` and, where the
tensor-core kernels do not apply (32-bit models, rows that are no multiple of 16 bytes),
``csrc/exact.cu``. CPU tensors run the PyTorch restatements below.

The stream is ``x`` fp32 [T, W]; ``act`` is what the projections read, in the model's element
type: the stream's rounding in decoders that normalise after the residual sum (the same tensor
for a 32-bit model), its norm in those that normalise before the sublayer.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import launch_counter

GATE_BLOCK = 16       # gate / up rows alternate in blocks of this many (csrc/common/elem.cuh)
TILE_ROWS = 128       # rows per tile of a grouped product


@dataclass(frozen=True)
class Gate:
    """How a gated feed-forward joins its gate and up projections: silu(g) * u, gelu_tanh(g) * u or
    clamped_swish: g' * sigmoid(alpha * g') * (u' + 1) with g' = min(g, limit) and u' clamped to
    -limit .. limit. Functions that take a gate also take its name alone."""
    name: str
    limit: float = 0.0
    alpha: float = 1.702

    @staticmethod
    def of(gate) -> "Gate":
        return gate if isinstance(gate, Gate) else Gate(gate)

    @property
    def code(self) -> int:
        return {"silu": 1, "gelu_tanh": 2, "clamped_swish": 3}[self.name]

    def join(self, g: torch.Tensor, u: torch.Tensor) -> torch.Tensor:
        if self.name == "clamped_swish":
            g = g.clamp(max=self.limit)
            return g * torch.sigmoid(self.alpha * g) * (u.clamp(-self.limit, self.limit) + 1.0)
        return (F.silu(g) if self.name == "silu" else F.gelu(g, approximate="tanh")) * u


def _nat():
    from . import native
    return native


def dtype_code(dt: torch.dtype) -> int:
    if dt == torch.bfloat16:
        return 0
    if dt == torch.float32:
        return 1
    raise TypeError("element type %s" % dt)


# ------------------------------------------------------------------------ residual stream
def bigram_rows(ids, prev, bigram) -> torch.Tensor:
    rows = (prev * bigram.mul_prev + ids * bigram.mul_cur) % bigram.buckets
    return torch.where(prev < 0, bigram.buckets, rows)


def stream_embedding(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0,
                     rounded: bool = True, pairs: tuple = None, keep: torch.Tensor = None):
    """(x, act) of the token embeddings times ``scale``; act is None unless ``rounded``. ``pairs``:
    (previous token of every token, negative where there is none, the table of a bigram embedding
    [buckets + 1, W], its BigramSpec), added in fp32. ``keep`` fp32 [T, W] receives a copy of x."""
    if not table.is_cuda:
        x = table[ids].float() * scale
        if pairs is not None:
            prev, second, bigram = pairs
            x = x + second[bigram_rows(ids, prev, bigram)].float()
        if keep is not None:
            keep.copy_(x)
        if not rounded:
            return x, None
        return (x, x) if table.dtype == torch.float32 else (x, x.to(table.dtype))
    nat = _nat()
    T, W = ids.numel(), table.shape[1]
    x = torch.empty(T, W, dtype=torch.float32, device=table.device)
    act = None
    if rounded:
        act = x if table.dtype == torch.float32 else torch.empty(T, W, dtype=table.dtype,
                                                                 device=table.device)
    prev, second, bigram = pairs or (None, None, None)
    assert ids.is_contiguous() and (prev is None or (
        prev.dtype == ids.dtype and prev.is_contiguous() and second.dtype == table.dtype and
        second.shape[0] == bigram.buckets + 1))
    rc = nat.lib().ab200_stream_embedding(
        ids.data_ptr(), table.data_ptr(), x.data_ptr(), None if act is x else nat.ptr(act),
        nat.ptr(keep), float(scale), T, W, table.shape[0], nat.ptr(prev), nat.ptr(second),
        *((bigram.buckets, bigram.mul_prev, bigram.mul_cur) if bigram else (0, 0, 0)),
        dtype_code(table.dtype), nat.status_buffer(table.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "stream_embedding")
    launch_counter.add(1)
    return x, act


def _scaled_norm_ref(s, weight, eps, offset=1.0):
    return s / torch.sqrt(s.pow(2).mean(-1, keepdim=True) + eps) * (offset + weight)


def stream_norm(x, act, y, weight, alpha: float, eps: float, experts: "Routing" = None) -> None:
    """In place: ``x <- norm(alpha * x + y) * (1 + weight)``, ``act`` its rounding. With
    ``experts`` (a :class:`Routing`) ``y`` holds the experts' output rows and the sublayer's
    output is each token's weighted sum of its own."""
    T, W = x.shape
    if not x.is_cuda:
        yf = y.float()
        if experts is not None:
            yf = (yf[experts.rows.long()] * experts.weights.unsqueeze(-1)).sum(1)
        x.copy_(_scaled_norm_ref(alpha * x + yf, weight, eps))
        if act is not x:
            act.copy_(x)
        return
    nat = _nat()
    assert x.is_contiguous() and act.is_contiguous() and y.stride(1) == 1
    rc = nat.lib().ab200_stream_norm(
        x.data_ptr(), None, y.data_ptr(), y.stride(0),
        experts.rows.data_ptr() if experts is not None else None,
        experts.weights.data_ptr() if experts is not None else None,
        experts.top if experts is not None else 0, weight.data_ptr(), float(alpha), float(eps),
        1.0, x.data_ptr(), None if act is x else act.data_ptr(), T, W, dtype_code(act.dtype),
        nat.stream_ptr())
    nat.check(rc, "stream_norm")
    launch_counter.add(1)


def stream_sandwich(x, y=None, w_out=None, step=None, w_in=None, act=None, eps: float = 0.0,
                    offset: float = 0.0) -> None:
    """In place, in one pass over the rows of the stream: ``x += norm(y) * (offset + w_out)`` if a
    sublayer's output ``y`` is given, ``x += step`` if a vector is; then ``act = norm(x) * (offset
    + w_in)`` if ``act`` is given: what the next sublayer reads."""
    T, W = x.shape
    if not x.is_cuda:
        if y is not None:
            x += _scaled_norm_ref(y.float(), w_out, eps, offset)
        if step is not None:
            x += step
        if act is not None:
            act.copy_(_scaled_norm_ref(x, w_in, eps, offset))
        return
    nat = _nat()
    dt = act.dtype if act is not None else y.dtype if y is not None else torch.float32
    assert x.is_contiguous() and act is not x and (act is None or act.is_contiguous())
    assert y is None or (y.stride(1) == 1 and y.dtype == dt)
    rc = nat.lib().ab200_stream_sandwich(
        x.data_ptr(), nat.ptr(y), y.stride(0) if y is not None else 0, nat.ptr(w_out),
        nat.ptr(step), nat.ptr(w_in), nat.ptr(act), float(eps), float(offset), T, W,
        dtype_code(dt), nat.stream_ptr())
    nat.check(rc, "stream_sandwich")
    launch_counter.add(1)


def stream_add(x, act, w, eps: float, y=None, pair=None, experts: "Routing" = None,
               shared=None) -> None:
    """In place: ``x += norm(f) * w``, ``act`` (where it is not x itself) its rounding. f is a
    sublayer's output ``y``; with ``pair`` = (y2, wy, wy2) half the sum of norm(y) * wy and
    norm(y2) * wy2; with ``experts`` (``y``: the experts' rows) each token's weighted sum, in which an
    identity expert contributes the token's x, plus the rows of ``shared``."""
    T, W = x.shape
    if not x.is_cuda:
        f = y.float()
        if pair is not None:
            f = 0.5 * (_scaled_norm_ref(f, pair[1], eps, 0.0) +
                       _scaled_norm_ref(pair[0].float(), pair[2], eps, 0.0))
        elif experts is not None:
            own = experts.rows < 0
            rows = torch.cat([f, torch.zeros(1, W)])[experts.rows.long()]     # (-1: the zero row)
            rows = torch.where(own.unsqueeze(-1), x.unsqueeze(1), rows)
            f = (rows * experts.weights.unsqueeze(-1)).sum(1)
            if shared is not None:
                f = f + shared.float()
        x += _scaled_norm_ref(f, w, eps, 0.0)
        if act is not x:
            act.copy_(x)
        return
    nat = _nat()
    y2, wy, wy2 = pair or (None, None, None)
    assert x.is_contiguous() and act.is_contiguous()
    assert all(t is None or (t.stride(1) == 1 and t.dtype == act.dtype) for t in (y, y2, shared))
    rc = nat.lib().ab200_stream_add(
        x.data_ptr(), None if act is x else act.data_ptr(), w.data_ptr(), y.data_ptr(), y.stride(0),
        nat.ptr(wy), nat.ptr(y2), y2.stride(0) if y2 is not None else 0, nat.ptr(wy2),
        experts.rows.data_ptr() if experts is not None else None,
        experts.weights.data_ptr() if experts is not None else None,
        experts.top if experts is not None else 0, nat.ptr(shared),
        shared.stride(0) if shared is not None else 0, float(eps), T, W, dtype_code(act.dtype),
        nat.stream_ptr())
    nat.check(rc, "stream_add")
    launch_counter.add(1)


def stream_pre(x, mult: float, eps: float, y=None, bias=None, experts: "Routing" = None, shared=None,
               base=None, step=None, w_in=None, act=None) -> None:
    """In place, in one pass over the rows of the stream: ``x += mult * f`` if a sublayer's output is
    given, ``x += base`` (fp32 [T, W]) and ``x += step`` (fp32 [W]) if they are; then ``act = norm(x) *
    w_in`` if ``act`` is given: what the next sublayer reads. f is ``y`` + ``bias`` (fp32 [W], or None)
    or, with ``experts`` (``y``: the experts' rows), each token's weighted sum plus the rows of
    ``shared``. ``w_in`` fp32: [W], or one number for all coordinates."""
    T, W = x.shape
    if not x.is_cuda:
        if y is not None:
            f = y.float()
            if experts is not None:
                f = (f[experts.rows.long()] * experts.weights.unsqueeze(-1)).sum(1)
            if shared is not None:
                f = f + shared.float()
            x += mult * (f if bias is None else f + bias)
        if base is not None:
            x += base
        if step is not None:
            x += step
        if act is not None:
            act.copy_(_scaled_norm_ref(x, w_in, eps, 0.0))
        return
    nat = _nat()
    dt = act.dtype if act is not None else y.dtype if y is not None else torch.float32
    assert x.is_contiguous() and act is not x and (act is None or act.is_contiguous())
    assert all(t is None or (t.stride(1) == 1 and t.dtype == dt) for t in (y, shared))
    assert base is None or base.is_contiguous()
    rc = nat.lib().ab200_stream_pre(
        x.data_ptr(), nat.ptr(y), y.stride(0) if y is not None else 0, nat.ptr(bias),
        experts.rows.data_ptr() if experts is not None else None,
        experts.weights.data_ptr() if experts is not None else None,
        experts.top if experts is not None else 0, nat.ptr(shared),
        shared.stride(0) if shared is not None else 0, float(mult), nat.ptr(base), nat.ptr(step),
        nat.ptr(w_in), int(w_in is not None and w_in.numel() == 1), nat.ptr(act), float(eps), T, W,
        dtype_code(dt), nat.stream_ptr())
    nat.check(rc, "stream_pre")
    launch_counter.add(1)


def soft_cap(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """fp32 [T, V]: cap * tanh(logits / cap). (In 16 bits logits near the cap would tie.)"""
    if not logits.is_cuda:
        return cap * torch.tanh(logits.float() / cap)
    nat = _nat()
    T, V = logits.shape
    assert logits.stride(1) == 1 and cap > 0
    out = torch.empty(T, V, dtype=torch.float32, device=logits.device)
    rc = nat.lib().ab200_soft_cap(logits.data_ptr(), logits.stride(0), out.data_ptr(), T, V,
                                  float(cap), dtype_code(logits.dtype), nat.stream_ptr())
    nat.check(rc, "soft_cap")
    launch_counter.add(1)
    return out


def stream_final_norm(x, rows, weight, eps: float, dtype: torch.dtype,
                      offset: float = 1.0) -> torch.Tensor:
    """norm(x[rows]) * (offset + weight), rounded to ``dtype``: the state the LM head reads."""
    R, W = rows.numel(), x.shape[1]
    if not x.is_cuda:
        return _scaled_norm_ref(x[rows], weight, eps, offset).to(dtype)
    nat = _nat()
    out = torch.empty(R, W, dtype=dtype, device=x.device)
    rc = nat.lib().ab200_stream_norm(x.data_ptr(), rows.data_ptr(), None, 0, None, None, 0,
                                     weight.data_ptr(), 1.0, float(eps), float(offset), None,
                                     out.data_ptr(), R, W, dtype_code(dtype), nat.stream_ptr())
    nat.check(rc, "stream_final_norm")
    launch_counter.add(1)
    return out


# ------------------------------------------------------------------------ gated feed-forward
def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[.., ff, W] gate and up matrices -> [.., 2 * ff', W] with rows alternating in blocks of
    GATE_BLOCK; ff is padded with zero rows to a multiple of it (they produce zeros)."""
    *lead, ff, W = gate.shape
    pad = -ff % GATE_BLOCK
    if pad:
        z = torch.zeros(*lead, pad, W, dtype=gate.dtype, device=gate.device)
        gate, up = torch.cat([gate, z], -2), torch.cat([up, z], -2)
    n = gate.shape[-2] // GATE_BLOCK
    g = gate.reshape(*lead, n, GATE_BLOCK, W)
    u = up.reshape(*lead, n, GATE_BLOCK, W)
    return torch.stack([g, u], -3).reshape(*lead, 2 * n * GATE_BLOCK, W).contiguous()


def _gated_ref(gu, act):
    T, n2 = gu.shape
    v = gu.float().reshape(T, n2 // (2 * GATE_BLOCK), 2, GATE_BLOCK)
    return Gate.of(act).join(v[:, :, 0], v[:, :, 1]).reshape(T, n2 // 2).to(gu.dtype)


def gated_act(gu: torch.Tensor, act) -> torch.Tensor:
    """``act`` (a Gate) of gate and up, from the product with an interleaved gate / up matrix."""
    act = Gate.of(act)
    if not gu.is_cuda:
        return _gated_ref(gu, act)
    nat = _nat()
    assert gu.is_contiguous()
    T, ff = gu.shape[0], gu.shape[1] // 2
    out = torch.empty(T, ff, dtype=gu.dtype, device=gu.device)
    rc = nat.lib().ab200_gated_act(gu.data_ptr(), out.data_ptr(), T, ff, act.code, act.limit,
                                   act.alpha, dtype_code(gu.dtype), nat.stream_ptr())
    nat.check(rc, "gated_act")
    launch_counter.add(1)
    return out


# ------------------------------------------------------------------------ feed-forward without a gate
def poly_norm(z: torch.Tensor, bias, coef, ff: int, eps: float) -> torch.Tensor:
    """a N(z') + b N(z'^2) + c N(z'^3) + e of z' = z + bias over the first ``ff`` columns of z [T, n],
    powers element by element, N dividing by the root mean square over the token's ff values;
    zeros in the columns beyond. ``bias`` [n] of z's element type, ``coef`` fp32 [4]: a, b, c, e."""
    T, n = z.shape
    if not z.is_cuda:
        v = z[:, :ff].float() + bias[:ff].float()
        unit = lambda t: t / torch.sqrt(t.pow(2).mean(-1, keepdim=True) + eps)
        out = torch.zeros(T, n, dtype=z.dtype)
        out[:, :ff] = coef[0] * unit(v) + coef[1] * unit(v * v) + coef[2] * unit(v * v * v) + coef[3]
        return out
    nat = _nat()
    assert z.is_contiguous() and bias.numel() == n and bias.dtype == z.dtype and coef.numel() == 4
    out = torch.empty_like(z)
    rc = nat.lib().ab200_poly_norm(z.data_ptr(), bias.data_ptr(), coef.data_ptr(), out.data_ptr(), T, n,
                                   ff, float(eps), dtype_code(z.dtype), nat.stream_ptr())
    nat.check(rc, "poly_norm")
    launch_counter.add(1)
    return out


# ------------------------------------------------------------------------ grouped products
@dataclass
class Routing:
    """Which experts each token uses and where its rows lie among the rows sorted by expert."""
    ids: torch.Tensor         # int32 [T, top]; from num_experts on: identity experts
    weights: torch.Tensor     # fp32 [T, top]
    rows: torch.Tensor        # int32 [T, top]; -1 for an identity expert
    top: int
    num_experts: int
    tiles: torch.Tensor = None        # int32 [max_tiles, 4]: expert, first row, rows
    num_tiles: torch.Tensor = None    # int32 [1]
    counts: list = None               # CPU path: rows per expert


def route_ref(x, w, b, top: int, scale=None, groups=None):
    z = x.float() @ w.float().t()
    if groups is not None:     # sigmoids, among the experts of the best groups
        s, (count, keep) = torch.sigmoid(z), groups
        best = s.view(*s.shape[:-1], count, -1).sort(-1, descending=True).values[..., :2].sum(-1)
        kept = torch.argsort(best, dim=-1, descending=True, stable=True)[:, :keep]
        open_ = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True)
        open_ = open_.repeat_interleave(s.shape[-1] // count, 1)
        order = torch.argsort(s.masked_fill(~open_, float("-inf")), dim=-1, descending=True,
                              stable=True)[:, :top]
        own = s.gather(1, order)
        return order, own / (own.sum(-1, keepdim=True) + 1e-20) * scale
    if scale is not None:      # softmax over all outputs, b: correction of the choice
        s = torch.softmax(z, -1)
        order = torch.argsort(s if b is None else s + b, dim=-1, descending=True, stable=True)[:, :top]
        return order, s.gather(1, order) * scale
    z = z + b
    order = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :top]
    return order, torch.softmax(z.gather(1, order), -1)


_route_states: dict = {}


def _route_state(E: int, device) -> torch.Tensor:
    """Counters of the router kernel (zero between launches), one set per device and number of
    experts."""
    key = (torch.device(device).index, E)
    t = _route_states.get(key)
    if t is None:
        t = _route_states[key] = torch.zeros(E + 1, dtype=torch.int32, device=device)
    return t


def route(x: torch.Tensor, act: torch.Tensor, w: torch.Tensor, b: torch.Tensor, top: int,
          identity: int = 0, scale: float = None, groups: tuple = None):
    """Router of a mixture of experts. ``x`` [T, W]: fp32 stream, or ``act``; ``act`` what the
    experts read, ``w`` [outputs, W], ``b`` fp32 [outputs] or None. The weights are the softmax over
    the chosen logits (with the bias ``b``) or, with a ``scale``, the chosen ones of the softmax over
    all outputs times it (``b`` then corrects the choice only). With ``groups`` = (count, kept) they
    are the chosen sigmoids, normalised to the sum ``scale``; only experts of the best groups are
    chosen, a group's score being the sum of its two best. The last ``identity`` outputs are
    identity experts. Returns (Routing, act rows sorted by expert)."""
    T, W = x.shape
    E = w.shape[0] - identity
    if not x.is_cuda:
        ids, weights = route_ref(x, w, b, top, scale, groups)
        order = torch.argsort(ids.reshape(-1), stable=True)
        rows = torch.empty_like(order)
        rows[order] = torch.arange(order.numel())
        counts = torch.bincount(ids.reshape(-1), minlength=E)[:E].tolist()
        rows = torch.where(ids < E, rows.reshape(T, top), -1).int()
        r = Routing(ids.int(), weights, rows, top, E, counts=counts)
        return r, act[order[:sum(counts)] // top]
    nat = _nat()
    L, dev, dc = nat.lib(), x.device, dtype_code(act.dtype)
    assert x.is_contiguous() and act.is_contiguous() and w.is_contiguous() and w.dtype == act.dtype
    i32 = torch.int32
    ids = torch.empty(T, top, dtype=i32, device=dev)
    weights = torch.empty(T, top, dtype=torch.float32, device=dev)
    max_tiles = min(T * top, T * top // TILE_ROWS + E)
    plan = torch.empty(E + 4 * max_tiles + 4 + T * top, dtype=i32, device=dev)
    tiles = plan[:4 * max_tiles].view(max_tiles, 4)
    num_tiles = plan[4 * max_tiles:4 * max_tiles + 1]
    cursor = plan[4 * max_tiles + 4:4 * max_tiles + 4 + E]
    rows = plan[4 * max_tiles + 4 + E:].view(T, top)
    assert x.dtype in (torch.float32, act.dtype) and (groups is None or (b is None and not identity))
    mode = 2 if groups is not None else int(scale is not None)
    rc = L.ab200_moe_route(x.data_ptr(), dtype_code(x.dtype), w.data_ptr(), nat.ptr(b), T, W,
                           E + identity, E, top, mode, scale or 0.0, *(groups or (1, 1)),
                           ids.data_ptr(), weights.data_ptr(),
                           _route_state(E, dev).data_ptr(), cursor.data_ptr(), tiles.data_ptr(),
                           num_tiles.data_ptr(), dc, nat.stream_ptr())
    nat.check(rc, "moe_route")
    launch_counter.add(1)
    r = Routing(ids, weights, rows, top, E, tiles, num_tiles)
    return r, _permute(act, r, cursor)


def _permute(act, r: Routing, cursor) -> torch.Tensor:
    nat = _nat()
    T, W = act.shape
    xp = torch.empty(T * r.top, W, dtype=act.dtype, device=act.device)
    rc = nat.lib().ab200_moe_permute(act.data_ptr(), r.ids.data_ptr(), cursor.data_ptr(),
                                     r.rows.data_ptr(), xp.data_ptr(), T, W, r.top, r.num_experts,
                                     dtype_code(act.dtype), nat.stream_ptr())
    nat.check(rc, "moe_permute")
    launch_counter.add(1)
    return xp


def _aligned(*ts) -> bool:
    """Rows of 16-bit elements that the tensor-map copies can fetch."""
    for t in ts:
        if t.dtype != torch.bfloat16 or t.data_ptr() % 16:
            return False
        if t.stride(-1) != 1 or any(s % 8 for s in t.stride()[:-1]):
            return False
    return True


def grouped_linear(x: torch.Tensor, w: torch.Tensor, routing: Routing, act=None):
    """Rows sorted by expert [n, K] times each row's expert matrix of ``w`` [E, N, K]. With
    ``act`` (a Gate) the matrices are interleaved gate / up ones, joined by it."""
    act = None if act is None else Gate.of(act)
    n, K = x.shape
    E, N, _ = w.shape
    if not x.is_cuda:
        out = torch.cat([xe.float() @ w[e].float().t()
                         for e, xe in enumerate(x.split(routing.counts))]).to(x.dtype)
        return _gated_ref(out, act) if act else out
    nat = _nat()
    fused = act is not None and _aligned(x, w) and K % 8 == 0
    out = torch.empty(n, N // 2 if fused else N, dtype=x.dtype, device=x.device)
    if _aligned(x, w, out) and K % 8 == 0:
        rc = nat.lib().ab200_grouped_gemm(
            x.data_ptr(), x.stride(0), 0, n, w.data_ptr(), w.stride(1), w.stride(0),
            out.data_ptr(), out.stride(0), 0, 0, N, K, E, routing.tiles.data_ptr(),
            routing.num_tiles.data_ptr(), routing.tiles.shape[0], act.code if act else 0,
            act.limit if act else 0.0, act.alpha if act else 0.0, nat.status_buffer(x.device).data_ptr(), nat.stream_ptr())
        nat.check(rc, "grouped_gemm n=%d N=%d K=%d" % (n, N, K))
        launch_counter.add(1)
        return out
    rc = nat.lib().ab200_linear_exact(
        x.data_ptr(), x.stride(0), 0, w.data_ptr(), w.stride(1), w.stride(0), out.data_ptr(),
        out.stride(0), 0, 0, N, K, E, routing.tiles.data_ptr(), routing.num_tiles.data_ptr(),
        routing.tiles.shape[0], dtype_code(x.dtype), nat.stream_ptr())
    nat.check(rc, "linear_exact (experts)")
    launch_counter.add(1)
    return gated_act(out, act) if act else out


def gated_linear(x: torch.Tensor, w: torch.Tensor, act) -> torch.Tensor:
    """Gate and up of a dense feed-forward joined by ``act`` (a Gate): ``w`` [2 * ff, W] is an
    interleaved gate / up matrix. Long inputs run one tensor-core kernel with the activation in its epilogue; short
    ones the framework's decode GEMM (split over K) and a separate activation."""
    from . import linear
    act = Gate.of(act)
    T = x.shape[0]
    if not x.is_cuda or T <= FUSED_GATE_MIN_TOKENS or not _aligned(x, w) or x.shape[1] % 8:
        return gated_act(linear(x, w), act)
    nat = _nat()
    N, K = w.shape
    out = torch.empty(T, N // 2, dtype=x.dtype, device=x.device)
    rc = nat.lib().ab200_grouped_gemm(
        x.data_ptr(), x.stride(0), 0, T, w.data_ptr(), w.stride(0), 0, out.data_ptr(),
        out.stride(0), 0, T, N, K, 1, None, None, 0, act.code, act.limit, act.alpha,
        nat.status_buffer(x.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "gated_linear M=%d N=%d K=%d" % (T, N, K))
    launch_counter.add(1)
    return out


FUSED_GATE_MIN_TOKENS = 256


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor = None) -> torch.Tensor:
    """One matrix per head: x [T, H * K] (row stride free), w [H, N, K] -> [T, H * N] with head h's
    columns ``x_h @ w[h].T``."""
    H, N, K = w.shape
    T = x.shape[0]
    if out is None:
        out = torch.empty(T, H * N, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        y = torch.einsum("thk,hnk->thn", x.reshape(T, H, K).float(), w.float())
        out.copy_(y.reshape(T, H * N))
        return out
    if T == 0:
        return out
    nat = _nat()
    if _aligned(x, w, out) and K % 8 == 0 and N % 8 == 0:
        rc = nat.lib().ab200_grouped_gemm(
            x.data_ptr(), x.stride(0), K, T, w.data_ptr(), w.stride(1), w.stride(0),
            out.data_ptr(), out.stride(0), N, T, N, K, H, None, None, 0, 0, 0.0, 0.0,
            nat.status_buffer(x.device).data_ptr(), nat.stream_ptr())
        nat.check(rc, "head_linear T=%d H=%d N=%d K=%d" % (T, H, N, K))
    else:
        rc = nat.lib().ab200_linear_exact(
            x.data_ptr(), x.stride(0), K, w.data_ptr(), w.stride(1), w.stride(0), out.data_ptr(),
            out.stride(0), N, T, N, K, H, None, None, 0, dtype_code(x.dtype), nat.stream_ptr())
        nat.check(rc, "linear_exact (heads)")
    launch_counter.add(1)
    return out
