"""Recurrent mixers: layers that carry a [dim, vdim] matrix per head from token to token.

CUDA tensors run ``csrc/recurrent.cu``; CPU tensors the token-by-token restatements below. What a
sequence carries lies in the rows of its state slot (``engine/kv_cache.py``); a
:class:`StateStep` says, for a step, which rows of the batch belong to which slot.
"""

from __future__ import annotations

from dataclasses import dataclass

import numpy as np
import torch
import torch.nn.functional as F

from . import launch_counter, upload
from .stream_ops import dtype_code

STEP_INTS = 5       # first row, rows, slot, start position, phase (csrc/recurrent.cu)
TILE_ROWS = 16      # tokens that portions are prepared by


def _nat():
    from . import native
    return native


def pack_steps(scheduled, q_lens, out: np.ndarray) -> None:
    """The table of a step's sequences: ``scheduled`` (ScheduledRequest) in batch order, row by row
    into ``out`` [>= n, STEP_INTS]."""
    t = 0
    for i, (s, n) in enumerate(zip(scheduled, q_lens)):
        out[i] = (t, n, s.request.state_slot, s.start, s.request.state_phase)
        t += n


@dataclass
class StateStep:
    """Sequences of a step with their state slots. Slot 0 stands for padding rows: they read no
    state, write none, and put out zeros."""
    table: torch.Tensor       # int32 [n, STEP_INTS]
    max_rows: int             # most rows of a sequence
    # steps with longer portions: the sequences cut into tiles of TILE_ROWS tokens
    tiles: torch.Tensor = None        # int32 [tiles, 2]: sequence, first of its tokens
    first_tile: torch.Tensor = None   # int32 [n]

    @staticmethod
    def build(table: np.ndarray, device) -> "StateStep":
        n, rows = table.shape[0], table[:, 1].astype(np.int64)
        if rows.max() == 1:
            return StateStep(upload(table, device), 1)
        count = -(-rows // TILE_ROWS)
        first = np.cumsum(count) - count
        seq = np.repeat(np.arange(n), count)
        tiles = np.stack([seq, (np.arange(seq.size) - first[seq]) * TILE_ROWS], 1)
        packed = upload(np.concatenate([table.ravel(), tiles.ravel(), first]).astype(np.int32), device)
        a, b = table.size, table.size + tiles.size
        return StateStep(packed[:a].view(n, STEP_INTS), int(rows.max()), packed[a:b].view(-1, 2),
                         packed[b:])

    @staticmethod
    def of(scheduled, q_lens, pad_rows: int, device) -> "StateStep":
        n = len(q_lens)
        t = np.zeros((n + (pad_rows > 0), STEP_INTS), dtype=np.int32)
        pack_steps(scheduled, q_lens, t)
        if pad_rows:
            t[n] = (sum(q_lens), pad_rows, 0, 0, 0)
        return StateStep.build(t, device)

    @property
    def uploaded_bytes(self) -> int:
        return 4 * sum(t.numel() for t in (self.table, self.tiles, self.first_tile) if t is not None)


class StateDecodePlan:
    """The table of a captured decode step, in which every row is a sequence of its own."""

    def __init__(self, bucket: int):
        self.bucket = bucket

    @property
    def int32_words(self) -> int:
        return self.bucket * STEP_INTS

    def bind(self, host, dev: torch.Tensor) -> None:
        self._host = host.reshape(self.bucket, STEP_INTS)
        self.step = StateStep(dev.view(self.bucket, STEP_INTS), 1)

    def fill(self, scheduled) -> None:
        h = self._host
        h[:, 0] = np.arange(self.bucket)
        h[:, 1] = 1
        h[:, 2:] = 0
        pack_steps(scheduled, [1] * len(scheduled), h)

    def detach(self) -> None:
        """Rows without a slot: a run that must not move any sequence's state on."""
        self._host[:, 2] = 0


MEMORY, DELTA, FORGET = 0, 1, 2     # recurrences (csrc/common/recurrent.cuh)


def slices_for(dim: int, ncols: int, rule: int, dtype: torch.dtype, blocks: int, long: bool) -> int:
    """Blocks that share a head's columns: as few as hold them, more where a prompt's few heads
    would leave most of the GPU idle."""
    least = _nat().lib().ab200_scan_min_slices(dim, ncols, rule, dtype_code(dtype), int(long))
    if least == 0:
        raise NotImplementedError("recurrent layers with keys of more than 256 dimensions")
    width = 16 if dim <= 128 or (long and dtype == torch.bfloat16) else 8     # of a warp
    most = -(-ncols // width)
    want = 148 // max(1, blocks) if long else 1
    n = max(least, min(most, want))
    # blocks of whole warps: as many as the columns then take
    cols = -(-(-(-ncols // n)) // width) * width
    return -(-ncols // cols)


def _scratch(s, ncols: int, rule: int, steps: StateStep, proj: torch.Tensor):
    """(slices, raw outputs or None, tile records or None) of a scan."""
    slices = slices_for(s.dim, ncols, rule, proj.dtype, steps.table.shape[0] * s.heads,
                        steps.max_rows > 1)
    f32 = dict(dtype=torch.float32, device=proj.device)
    raw = torch.empty(proj.shape[0], s.heads, ncols + (rule == MEMORY), **f32) if slices > 1 else None
    records = None
    if steps.max_rows > 1:
        size = _nat().lib().ab200_scan_record(s.dim, ncols, slices, rule, dtype_code(proj.dtype))
        records = torch.empty(steps.tiles.shape[0], s.heads, size, **f32)
    return slices, raw, records


# ------------------------------------------------------------------------------ delta rule
@dataclass(frozen=True)
class DeltaShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    # columns of the input projection
    q_at: int
    k_at: int
    v_at: int
    b_at: int

    @property
    def channels(self) -> int:
        """Of the convolution: queries, keys, values."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def state_cols(self) -> int:
        return -(-self.vdim // 4) * 4


def _head_output(o, norm, gate, eps):
    """o fp32 [n, heads, vdim] -> [n, heads * vdim]."""
    n = o.shape[0]
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps)
    o = (o * norm).reshape(n, -1)
    return o if gate is None else o * torch.sigmoid(gate.float())


def delta_scan_ref(proj, decay, gate, conv, a_exp, dt_bias, norm, s: DeltaShape, state, conv_state,
                   steps: StateStep, eps: float):
    H, G, d, dv, back = s.heads, s.kv_heads, s.dim, s.vdim, s.taps - 1
    out = torch.zeros(proj.shape[0], H * dv, dtype=proj.dtype)
    for first, n, slot, start, phase in steps.table.tolist():
        if slot <= 0:
            continue
        rows = slice(first, first + n)
        x = torch.cat([proj[rows, a:a + w] for a, w in ((s.q_at, G * d), (s.k_at, G * d),
                                                        (s.v_at, H * dv))], 1)
        old = conv_state[slot, phase].clone()
        old[:max(0, back - start)] = 0          # positions before the sequence
        x = torch.cat([old, x])
        conv_state[slot, phase ^ 1] = x[n:]
        y = F.silu(sum(x[j:j + n].float() * conv[j] for j in range(s.taps)))
        q, k, v = (y[:, :G * d].view(n, G, d), y[:, G * d:2 * G * d].view(n, G, d),
                   y[:, 2 * G * d:].view(n, H, dv))
        unit = lambda t: t / torch.sqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
        q, k = (unit(t).repeat_interleave(H // G, 1) for t in (q, k))
        q = q * d ** -0.5
        beta = torch.sigmoid(proj[rows, s.b_at:s.b_at + H].float())
        z = F.softplus(decay[rows, :H * d].float() + dt_bias, threshold=80.0)
        g = torch.exp(-a_exp.view(H, 1) * z.view(n, H, d))
        S = state[slot, :, :, :dv].clone() if start > 0 else torch.zeros(H, d, dv)
        o = torch.empty(n, H, dv)
        for t in range(n):
            S = g[t].unsqueeze(-1) * S
            u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot, :, :, :dv] = S
        out[rows] = _head_output(o, norm, gate[rows, :H * dv], eps).to(out.dtype)
    return out


def delta_scan(proj, decay, gate, conv, a_exp, dt_bias, norm, s: DeltaShape, state, conv_state,
               steps: StateStep, eps: float) -> torch.Tensor:
    """The gated delta rule of a step's sequences, from the input projection to the normed and gated
    heads [T, heads * vdim]. ``decay`` and ``gate``: [T, heads * dim] and [T, heads * vdim] (row
    strides free); ``conv`` fp32 [taps, channels]; ``a_exp`` fp32 [heads]: exp(A_log); ``dt_bias``
    fp32 [heads * dim]; ``norm`` fp32 [vdim]; ``state`` fp32 [slots, heads, dim, state_cols];
    ``conv_state`` [slots, 2, taps - 1, channels]."""
    if not proj.is_cuda:
        return delta_scan_ref(proj, decay, gate, conv, a_exp, dt_bias, norm, s, state, conv_state,
                              steps, eps)
    nat = _nat()
    T, n = proj.shape[0], steps.table.shape[0]
    out = torch.empty(T, s.heads * s.vdim, dtype=proj.dtype, device=proj.device)
    slices, raw, records = _scratch(s, s.vdim, DELTA, steps, proj)
    assert proj.stride(1) == decay.stride(1) == gate.stride(1) == 1
    assert state.is_contiguous() and conv_state.is_contiguous() and steps.table.is_contiguous()
    rc = nat.lib().ab200_delta_scan(
        proj.data_ptr(), proj.stride(0), s.q_at, s.k_at, s.v_at, s.b_at, decay.data_ptr(),
        decay.stride(0), gate.data_ptr(), gate.stride(0), conv.data_ptr(), s.taps, a_exp.data_ptr(),
        dt_bias.data_ptr(), norm.data_ptr(), state.data_ptr(), state.shape[3],
        conv_state.data_ptr(), state.shape[0], steps.table.data_ptr(), n, steps.max_rows,
        nat.ptr(steps.tiles), nat.ptr(steps.first_tile),
        steps.tiles.shape[0] if records is not None else 0, nat.ptr(records), T, s.heads, s.kv_heads, s.dim, s.vdim, slices, float(eps), nat.ptr(raw), out.data_ptr(),
        out.stride(0), dtype_code(proj.dtype), nat.status_buffer(proj.device).data_ptr(),
        nat.stream_ptr())
    nat.check(rc, "delta_scan")
    launch_counter.add(1 + (slices > 1) + (records is not None))
    return out


# ------------------------------------------------------------------------------ forget scan
@dataclass(frozen=True)
class ForgetShape:
    heads: int
    dim: int
    vdim: int
    # columns of the input projection
    q_at: int
    f_at: int
    v_at: int

    @property
    def state_cols(self) -> int:
        return -(-self.vdim // 4) * 4


def forget_scan_ref(proj, f_bias, lower, norm, s: ForgetShape, state, steps: StateStep, eps: float):
    H, d, dv = s.heads, s.dim, s.vdim
    out = torch.zeros(proj.shape[0], H * dv, dtype=proj.dtype)
    for first, n, slot, start, _ in steps.table.tolist():
        if slot <= 0:
            continue
        rows = slice(first, first + n)
        p = proj[rows].float()
        q = F.silu(p[:, s.q_at:s.q_at + H * d]).view(n, H, d)
        z = p[:, s.f_at:s.f_at + H * d] + f_bias
        k = ((1.0 - lower) * torch.sigmoid(-z)).view(n, H, d)      # 1 - f
        f = (lower + (1.0 - lower) * torch.sigmoid(z)).view(n, H, d)
        v = p[:, s.v_at:s.v_at + H * dv].view(n, H, dv)
        S = state[slot, :, :, :dv].clone() if start > 0 else torch.zeros(H, d, dv)
        o = torch.empty(n, H, dv)
        for t in range(n):
            S = f[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot, :, :, :dv] = S
        out[rows] = _head_output(o, norm, None, eps).to(out.dtype)
    return out


def forget_scan(proj, f_bias, lower, norm, s: ForgetShape, state, steps: StateStep,
                eps: float) -> torch.Tensor:
    """Linear attention with a forget gate f per channel and 1 - f in the key's place, over a step's
    sequences: from the input projection (queries before their silu, gates before bias and sigmoid,
    values) to the normed heads [T, heads * vdim]. ``f_bias`` and ``lower`` (the gates' lower bound)
    fp32 [heads * dim]; ``norm`` fp32 [vdim]; ``state`` fp32 [slots, heads, dim, state_cols]."""
    if not proj.is_cuda:
        return forget_scan_ref(proj, f_bias, lower, norm, s, state, steps, eps)
    nat = _nat()
    T, n = proj.shape[0], steps.table.shape[0]
    out = torch.empty(T, s.heads * s.vdim, dtype=proj.dtype, device=proj.device)
    slices, raw, records = _scratch(s, s.vdim, FORGET, steps, proj)
    assert proj.stride(1) == 1 and state.is_contiguous() and steps.table.is_contiguous()
    rc = nat.lib().ab200_forget_scan(
        proj.data_ptr(), proj.stride(0), s.q_at, s.f_at, s.v_at, f_bias.data_ptr(), lower.data_ptr(),
        norm.data_ptr(), state.data_ptr(), state.shape[3], state.shape[0], steps.table.data_ptr(), n,
        steps.max_rows, nat.ptr(steps.tiles), nat.ptr(steps.first_tile),
        steps.tiles.shape[0] if records is not None else 0, nat.ptr(records), T, s.heads, s.dim,
        s.vdim, slices, float(eps), nat.ptr(raw), out.data_ptr(), out.stride(0),
        dtype_code(proj.dtype), nat.status_buffer(proj.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "forget_scan")
    launch_counter.add(1 + (slices > 1) + (records is not None))
    return out


# ------------------------------------------------------------------------------ matrix memory
@dataclass(frozen=True)
class MemoryShape:
    heads: int
    dim: int
    vdim: int
    cap: float
    # columns of the input projection
    q_at: int
    k_at: int
    v_at: int
    i_at: int
    f_at: int

    @property
    def state_cols(self) -> int:
        """Value columns, the normaliser, padding."""
        return -(-(self.vdim + 1) // 4) * 4


def memory_scan_ref(proj, gate, i_bias, f_bias, norm, s: MemoryShape, state, max_state,
                    steps: StateStep, eps: float):
    H, d, dv = s.heads, s.dim, s.vdim
    out = torch.zeros(proj.shape[0], H * dv, dtype=proj.dtype)
    cap = lambda z: s.cap * torch.tanh(z / s.cap)
    for first, n, slot, start, phase in steps.table.tolist():
        if slot <= 0:
            continue
        rows = slice(first, first + n)
        p = proj[rows].float()
        q = p[:, s.q_at:s.q_at + H * d].view(n, H, d) * d ** -0.5
        k = p[:, s.k_at:s.k_at + H * d].view(n, H, d)
        v = torch.cat([p[:, s.v_at:s.v_at + H * dv].view(n, H, dv), torch.ones(n, H, 1)], -1)
        gi = cap(p[:, s.i_at:s.i_at + H] + i_bias)
        gf = F.logsigmoid(cap(p[:, s.f_at:s.f_at + H] + f_bias))
        S = state[slot, :, :, :dv + 1].clone() if start > 0 else torch.zeros(H, d, dv + 1)
        m = max_state[slot, phase].clone() if start > 0 else torch.zeros(H)
        o = torch.empty(n, H, dv)
        for t in range(n):
            new = torch.maximum(gf[t] + m, gi[t])
            keep, put = torch.exp(gf[t] + m - new), torch.exp(gi[t] - new)
            m = new
            S = keep.view(H, 1, 1) * S + (put.unsqueeze(-1) * k[t]).unsqueeze(-1) * v[t].unsqueeze(1)
            y = torch.einsum("hdv,hd->hv", S, q[t])
            o[t] = y[:, :dv] / (torch.maximum(y[:, dv].abs(), torch.exp(-m)) + 1e-6).unsqueeze(-1)
        state[slot, :, :, :dv + 1] = S
        max_state[slot, phase ^ 1] = m
        out[rows] = _head_output(o, norm.view(H, dv), gate[rows, :H * dv], eps).to(out.dtype)
    return out


def memory_scan(proj, gate, i_bias, f_bias, norm, s: MemoryShape, state, max_state,
                steps: StateStep, eps: float) -> torch.Tensor:
    """The matrix memory of a step's sequences, from the input projection to the normed and gated
    heads [T, heads * vdim]. ``gate`` [T, heads * vdim]; biases fp32 [heads]; ``norm`` fp32
    [heads * vdim]; ``state`` fp32 [slots, heads, dim, state_cols]; ``max_state`` fp32 [slots, 2,
    heads]."""
    if not proj.is_cuda:
        return memory_scan_ref(proj, gate, i_bias, f_bias, norm, s, state, max_state, steps, eps)
    nat = _nat()
    T, n = proj.shape[0], steps.table.shape[0]
    out = torch.empty(T, s.heads * s.vdim, dtype=proj.dtype, device=proj.device)
    slices, raw, records = _scratch(s, s.vdim + 1, MEMORY, steps, proj)
    gates = torch.empty(T, s.heads, 3, dtype=torch.float32, device=proj.device) \
        if records is not None else None
    assert proj.stride(1) == gate.stride(1) == 1
    assert state.is_contiguous() and max_state.is_contiguous() and steps.table.is_contiguous()
    rc = nat.lib().ab200_memory_scan(
        proj.data_ptr(), proj.stride(0), s.q_at, s.k_at, s.v_at, s.i_at, s.f_at, gate.data_ptr(),
        gate.stride(0), i_bias.data_ptr(), f_bias.data_ptr(), float(s.cap), norm.data_ptr(),
        state.data_ptr(), state.shape[3], max_state.data_ptr(), state.shape[0],
        steps.table.data_ptr(), n, steps.max_rows, nat.ptr(steps.tiles), nat.ptr(steps.first_tile),
        steps.tiles.shape[0] if records is not None else 0, nat.ptr(records), nat.ptr(gates), T,
        s.heads, s.dim, s.vdim, slices, float(eps),
        nat.ptr(raw), out.data_ptr(), out.stride(0), dtype_code(proj.dtype),
        nat.status_buffer(proj.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "memory_scan")
    launch_counter.add(1 + (slices > 1) + 2 * (records is not None))
    return out
