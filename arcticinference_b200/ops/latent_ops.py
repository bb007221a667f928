"""Latent attention: keys and values are linear maps of one cached latent vector per token.

Two ways to compute the same function:

* absorbed (decode and short chunks): the query heads are mapped into latent space
  (``q_h W_uk,h``), attend to the cached latents directly (one shared "head" that is key and
  value at once), and the result is mapped out of it (``W_uv,h``). The cache is read once for all
  heads.
* expanded (long chunks of wide latents): the latents of the context are gathered and expanded to
  per-head keys and values by one matrix product, and ordinary attention follows; per query-key
  pair that is ``dim + vdim`` instead of ``2 * kv_rank`` multiply-adds.

A rotated key part that the heads share is cached beside the latent and treated as more of it: the
maps into latent space carry an identity block for it, those out of it zeros, so that both forms
stay as they are.

CUDA tensors run ``csrc/latent_attention.cu`` (keys on the tensor core's M side),
``csrc/attention.cu`` (latents of at most 64, and the expanded form) or, for 32-bit models and
shapes outside those, ``csrc/exact.cu``. CPU tensors run the restatement below.
"""

from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np
import torch

from ..config import MaskSpec
from . import (AttentionMetadata, DecodePlan, attention, attention_contiguous, attention_masked,
               launch_counter, plan_attention_work, upload)
from .head_ops import attention_exact
from .stream_ops import dtype_code

KEY_TILE = 128
CAUSAL = MaskSpec()


def _nat():
    from . import native
    return native


@dataclass(frozen=True)
class LatentLayout:
    """Columns of a cached row: ``rank`` that are key and value at once (the latent, zero-padded to
    what the kernels tile by), then ``key_extra`` that belong to the key only. The rotated key
    part starts at ``rot_at``, in the padding where it fits."""
    rank: int
    key_extra: int
    rot_at: int

    @property
    def width(self) -> int:
        return self.rank + self.key_extra

    @staticmethod
    def of(rank: int, rot_dim: int, heads: int, dtype: torch.dtype) -> "LatentLayout":
        if dtype != torch.bfloat16:
            return LatentLayout(rank, rot_dim, rank)
        n = rank + rot_dim
        if n <= 64 and heads <= 128:
            return LatentLayout(64, 0, rank)
        up = lambda k: -(-k // 128) * 128
        if rot_dim and n > up(rank) and rot_dim <= 64 and up(rank) <= 512:
            return LatentLayout(up(rank), 64, up(rank))
        return LatentLayout(up(n), 0, rank)


@dataclass(frozen=True)
class LatentShape:
    """Heads, row layout and mask of an absorbed attention, and how its work is planned. The
    layers of a model that agree in them share one plan per step."""
    heads: int
    rank: int
    kernel: str       # "packed" | "latent" | "exact"
    key_extra: int = 0
    mask: MaskSpec = CAUSAL

    @staticmethod
    def of(heads: int, rank: int, dtype: torch.dtype, key_extra: int = 0,
           mask: MaskSpec = CAUSAL) -> "LatentShape":
        kernel = "exact"
        if dtype == torch.bfloat16 and rank == 64 and key_extra == 0 and heads <= 128:
            kernel = "packed"
        elif dtype == torch.bfloat16 and rank % 128 == 0 and rank <= 512 and key_extra in (0, 64):
            kernel = "latent"
        return LatentShape(heads, rank, kernel, key_extra, mask)

    @property
    def width(self) -> int:
        return self.rank + self.key_extra

    # ---- "packed": the 128-row attention kernel with the heads padded to a power of two
    @property
    def group(self) -> int:
        return 1 << max(0, (self.heads - 1).bit_length())

    # ---- "latent": rows (token, head) in order, this many per tile
    @property
    def tile_rows(self) -> int:
        # (shared memory: queries, a tile of latents and the key-only piece)
        most = 48 if self.key_extra and self.rank > 384 else 64
        return min(most, -(-self.heads // 16) * 16)

    def plan(self, q_lens, kv_lens, max_splits_cap: int = 16, align: int = 1):
        """(work [n, 8] int32, splits per token [T] int32, largest number of splits)."""
        if self.kernel == "packed":
            return plan_attention_work(q_lens, kv_lens, self.group, True, Hkv=1,
                                       max_splits_cap=max_splits_cap, mask=self.mask,
                                       align=align)
        return plan_latent_work(q_lens, kv_lens, self.heads, self.tile_rows,
                                max_splits_cap=max_splits_cap, mask=self.mask, align=align)

    def tile_keys(self, max_q: int, block_size: int) -> int:
        if self.kernel != "packed":
            return KEY_TILE
        return 64 if max_q * self.group <= 32 and block_size <= 64 else 128

    def decode_capacity(self, bucket: int, max_q: int, block_size: int):
        """(work items, splits) a captured decode step of ``bucket`` tokens may need."""
        tiles = 1 if self.kernel == "packed" else -(-self.heads // self.tile_rows)
        splits = int(max(1, min(16, 148 // max(1, bucket * tiles))))
        if self.kernel == "latent" and bucket * tiles > 37:
            # larger batches: cutting the sequences evens out the last wave of CTAs
            splits = max(splits, 4 if bucket * tiles <= 296 else 2)
        return bucket * (tiles + (max_q > 1)) * splits + tiles + 1, splits


def plan_latent_work(q_lens, kv_lens, heads: int, tile_rows: int, num_sms: int = 148,
                     max_splits_cap: int = 16, mask: MaskSpec = CAUSAL, align: int = 1):
    """Work list of the latent kernel. The (token, head) rows of a sequence are cut into tiles of
    ``tile_rows``, its keys (from the first one that its first token sees, rounded down to a
    multiple of ``align``) into pieces of whole 128-key tiles; the piece length is the one
    whose waves of CTAs cost least. Under a mask with a lower bound, the keys of a sequence with
    more than a few tokens are not cut: each of its tiles starts at its own first key. Item: sequence, first row, rows, position of the
    sequence's first query token minus its row's token (so that position = field 3 + row /
    heads), first key, last key + 1, piece, pieces."""
    ql = np.asarray(q_lens, dtype=np.int64)
    kl = np.asarray(kv_lens, dtype=np.int64)
    tok0 = np.cumsum(ql) - ql
    T = int(ql.sum())
    tok_splits = np.ones(max(T, 1), dtype=np.int32)
    live = np.nonzero(ql > 0)[0]
    if live.size == 0:
        return np.zeros((0, 8), np.int32), tok_splits, 1
    rows = ql[live] * heads
    n_tiles = -(-rows // tile_rows)
    first = lambda pos: mask.first_key(pos) // align * align
    lo = first(kl[live] - ql[live])
    key_tiles = -(-(kl[live] - lo) // KEY_TILE)
    whole = (ql[live] > 8) & (mask.kind != "causal")
    if whole.any():     # what one tile of rows walks, at most
        walk = mask.size + align + tile_rows // heads + KEY_TILE
        key_tiles = np.where(whole, np.minimum(key_tiles, -(-walk // KEY_TILE)), key_tiles)
    pieces = np.ones_like(key_tiles)
    if max_splits_cap > 1:
        best = None
        longest = int(key_tiles.max())
        for chunk in {max(1, -(-longest // s)) for s in range(1, max_splits_cap + 1)}:
            p = np.where(whole, 1, -(-key_tiles // chunk))
            items = int((p * n_tiles).sum())
            waves = -(-items // num_sms)
            cost = waves * (chunk + 3) + (2 if chunk < longest else 0)
            if best is None or cost < best[0] or (cost == best[0] and chunk > best[1]):
                best = (cost, chunk)
        pieces = np.where(whole, 1, -(-key_tiles // best[1]))
    per = -(-key_tiles // pieces)
    pieces = -(-key_tiles // per)
    rep = np.repeat(np.arange(live.size), n_tiles * pieces)
    item0 = np.cumsum(n_tiles * pieces) - n_tiles * pieces
    j = np.arange(rep.size) - item0[rep]
    tile, piece = j // pieces[rep], j % pieces[rep]
    r0 = tile * tile_rows
    ks = lo[rep] + piece * per[rep] * KEY_TILE
    ke = np.minimum(kl[live][rep], lo[rep] + (piece + 1) * per[rep] * KEY_TILE)
    own = first(kl[live][rep] - ql[live][rep] + r0 // heads)
    ks, ke = np.where(whole[rep], own, ks), np.where(whole[rep], kl[live][rep], ke)
    base = tok0[live][rep]
    work = np.stack([live[rep], base * heads + r0, np.minimum(tile_rows, rows[rep] - r0),
                     kl[live][rep] - ql[live][rep] - base, ks, ke, piece, pieces[rep]], 1)
    # keys a tile really sees end at its last token: heaviest first
    last = work[:, 3] + (work[:, 1] + work[:, 2] - 1) // heads
    work = work[np.argsort(-(np.minimum(ke, last + 1) - ks), kind="stable")]
    tok_splits[:T] = np.repeat(pieces, ql[live])
    return work.astype(np.int32), tok_splits, int(pieces.max())


@dataclass
class AttentionStep:
    """One step's attention, shared by all layers. In latent layers that expand long chunks, the
    rows [0, n_absorbed) of the batch attend in latent space and the rows after them (whole
    sequences) through expanded keys and values; the other layers absorb every row."""
    n_absorbed: int
    # (shape, every row?) -> plan; the second form covers only the first n_absorbed rows
    absorbed: dict = field(default_factory=dict)
    heads: dict = field(default_factory=dict)       # HeadShape -> AttentionMetadata
    tok_seq: torch.Tensor | None = None             # int32 [T]: row of the block table
    exp_q_lens: list = field(default_factory=list)
    exp_kv_lens: list = field(default_factory=list)
    # mask -> (cache rows of the keys its expanded sequences see, one sequence after the other,
    # and how many of each sequence's first keys are left out)
    ctx: dict = field(default_factory=dict)
    exp_plans: dict = field(default_factory=dict)   # (heads, widths, mask) -> AttentionMetadata

    @property
    def uploaded_bytes(self) -> int:
        plans = [*self.absorbed.values(), *self.heads.values(), *self.exp_plans.values()]
        n = sum(m.uploaded_bytes for m in {id(m): m for m in plans}.values())
        rows = [self.tok_seq] + [slots for slots, _ in self.ctx.values()]
        return n + sum(t.numel() * t.element_size() for t in rows if t is not None)


def finish_plan(shape: LatentShape, meta: AttentionMetadata, T: int, device) -> AttentionMetadata:
    """Scratch of the split keys."""
    if meta.max_splits > 1 and torch.device(device).type == "cuda":
        meta.o_part = torch.empty(meta.max_splits, T, shape.heads, shape.rank, dtype=torch.float32,
                                  device=device)
        meta.lse_part = torch.empty(meta.max_splits, T, shape.heads, dtype=torch.float32,
                                    device=device)
    return meta


def build_plan(shape: LatentShape, q_lens, kv_lens, block_tables, block_size, device):
    T = int(sum(q_lens))
    meta = AttentionMetadata(list(q_lens), list(kv_lens), T)
    if torch.device(device).type != "cuda" or shape.kernel == "exact":
        meta.block_tables = block_tables
        return meta
    work, tok_splits, max_splits = shape.plan(q_lens, kv_lens, align=block_size)
    meta.work = upload(work, device)
    meta.tok_splits = upload(tok_splits, device)
    meta.block_tables = block_tables
    meta.max_splits, meta.num_work = max_splits, work.shape[0]
    meta.tile_keys = shape.tile_keys(max(q_lens), block_size)
    return finish_plan(shape, meta, T, device)


class LatentDecodePlan(DecodePlan):
    """Work of one latent shape in a captured decode step."""

    def __init__(self, shape: LatentShape, bucket: int, max_q: int, block_size: int):
        self.shape, self.bucket, self.block_size = shape, bucket, block_size
        self.Hq, self.D = shape.heads, shape.rank
        self.work_cap, self.splits = shape.decode_capacity(bucket, max_q, block_size)
        self.tile_keys = shape.tile_keys(max_q, block_size)
        self.meta = AttentionMetadata([], [], bucket)

    def plan(self, q_lens, kv_lens):
        return self.shape.plan(q_lens, kv_lens, self.splits, align=self.block_size)


# ------------------------------------------------------------------------------ kernels
def latent_norm_cache(ckv: torch.Tensor, weight: torch.Tensor, rank: int, eps: float,
                      slots: torch.Tensor, cache: torch.Tensor) -> None:
    """RMS norm over the first ``rank`` columns of ``ckv`` [T, >= rank] and write to the rows
    ``slots`` of the cache [num_blocks, 1, block_size, padded rank]; slot < 0: no write."""
    nb, _, bs, Rp = cache.shape
    if not ckv.is_cuda:
        v = ckv[:, :rank].float()
        c = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps) * weight
        ok = slots >= 0
        cache.view(nb * bs, Rp)[slots[ok], :rank] = c[ok].to(cache.dtype)
        return
    nat = _nat()
    assert ckv.stride(1) == 1 and cache.is_contiguous() and slots.dtype == torch.int64
    rc = nat.lib().ab200_latent_norm_cache(
        ckv.data_ptr(), ckv.stride(0), weight.data_ptr(), rank, Rp, float(eps), slots.data_ptr(),
        cache.data_ptr(), nb * bs, ckv.shape[0], dtype_code(ckv.dtype),
        nat.status_buffer(ckv.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "latent_norm_cache")
    launch_counter.add(1)


def latent_rope_cache(q, ckv, heads: int, dq: int, dim: int, weight, rank: int, table, eps: float,
                      slots, cache, rot_at: int) -> None:
    """:func:`latent_norm_cache` for latents with a rotated key part: ``ckv`` [T, >= rank + rot]
    holds it behind the latent, the cache row from column ``rot_at``. ``q`` [T, >= heads * dq] (of
    the same row stride) is rotated in place: ``rot`` columns of every head from ``dim`` on.
    ``table``: head_ops.rotary_table."""
    nb, _, bs, W = cache.shape
    half = table.shape[1]
    if not ckv.is_cuda:
        from .head_ops import rotate_ref
        x = q[:, :heads * dq].unflatten(1, (heads, dq))      # (a view)
        part = rotate_ref(x[:, :, dim:dim + 2 * half].float(), table)
        x[:, :, dim:dim + 2 * half] = part.to(q.dtype)
        latent_norm_cache(ckv, weight, rank, eps, slots, cache)
        shared = rotate_ref(ckv[:, None, rank:rank + 2 * half].float(), table)[:, 0]
        ok = slots >= 0
        cache.view(nb * bs, W)[slots[ok], rot_at:rot_at + 2 * half] = shared[ok].to(cache.dtype)
        return
    nat = _nat()
    assert q.stride(0) == ckv.stride(0) and q.stride(1) == ckv.stride(1) == 1
    assert cache.is_contiguous() and slots.dtype == torch.int64 and table.is_contiguous()
    rc = nat.lib().ab200_latent_rope_cache(
        q.data_ptr(), ckv.data_ptr(), q.stride(0), table.data_ptr(), half, slots.data_ptr(),
        weight.data_ptr(), cache.data_ptr(), q.shape[0], heads, dq, dim, rank, W, rot_at, nb * bs,
        float(eps), dtype_code(q.dtype), nat.status_buffer(q.device).data_ptr(),
        nat.stream_ptr())
    nat.check(rc, "latent_rope_cache")
    launch_counter.add(1)


def sink_softmax(s, sink):
    """Softmax of scores [H, n, k] over their last dimension, with exp(sink[h]) in the denominator."""
    if sink is None:
        return torch.softmax(s, -1)
    s = torch.cat([s, sink.view(-1, 1, 1).expand(*s.shape[:2], 1)], -1)
    return torch.softmax(s, -1)[..., :-1]


def gated_heads(o, gate):
    """o [n, H, d] times the sigmoid of gate [n, H]."""
    return o if gate is None else o * torch.sigmoid(gate.float()).unsqueeze(-1)


def latent_attention_ref(q, cache, meta, shape: LatentShape, scale, sink=None, gate=None):
    nb, _, bs, W = cache.shape
    H, R = shape.heads, shape.rank
    flat = cache.view(nb * bs, W)
    out = torch.empty(q.shape[0], H * R, dtype=q.dtype)
    t = 0
    for i, (n, kl) in enumerate(zip(meta.q_lens, meta.kv_lens)):
        if n == 0:
            continue
        pos = torch.arange(kl)
        c = flat[meta.block_tables[i].long()[pos // bs] * bs + pos % bs].float()
        s = torch.einsum("thr,kr->htk", q[t:t + n].reshape(n, H, W).float(), c) * scale
        at = torch.arange(kl - n, kl).view(n, 1)
        s = s.masked_fill((pos > at) | (pos < shape.mask.first_key(at)), float("-inf"))
        o = torch.einsum("htk,kr->thr", sink_softmax(s, sink), c[:, :R])
        o = gated_heads(o, None if gate is None else gate[t:t + n])
        out[t:t + n] = o.reshape(n, H * R).to(q.dtype)
        t += n
    return out


def latent_attention(q: torch.Tensor, cache: torch.Tensor, meta: AttentionMetadata,
                     shape: LatentShape, scale: float, tok_seq=None, positions=None, sink=None,
                     gate=None):
    """q [T, H * width] in latent space; cache [num_blocks, 1, block_size, width]. Softmax over the
    keys the shape's mask shows; returns [T, H * rank]. ``sink`` fp32 [H]: a further term of the
    denominator, as its logarithm; ``gate`` [T, H] (row stride free): heads' outputs are multiplied
    by its sigmoid. ``tok_seq`` and ``positions`` (per token) are read by the "exact" kernel only."""
    H, R, W = shape.heads, shape.rank, shape.width
    bt = meta.block_tables
    if not q.is_cuda:
        return latent_attention_ref(q, cache, meta, shape, scale, sink, gate)
    nat = _nat()
    T = q.shape[0]
    assert q.is_contiguous() and cache.is_contiguous() and cache.shape[3] == W
    if shape.kernel == "packed":
        if shape.mask.kind == "causal" and sink is None and gate is None:
            return attention(q, cache, cache, meta, H, 1, R, scale)
        return attention_masked(q, cache, cache, meta, H, 1, R, scale, shape.mask, sink, gate)
    if shape.kernel == "exact":
        return attention_exact(q, cache, cache, bt, tok_seq, positions, H, 1, W, R, scale,
                               shape.mask, sink, gate)
    assert gate is None or gate.stride(1) == 1
    out = torch.empty(T, H * R, dtype=q.dtype, device=q.device)
    rc = nat.lib().ab200_latent_attention(
        q.data_ptr(), T * H, cache.data_ptr(), cache.shape[0], cache.shape[2], bt.data_ptr(),
        bt.shape[1], meta.work.data_ptr(), meta.num_work, nat.ptr(meta.tok_splits),
        meta.max_splits, T, H, R, shape.key_extra, shape.mask.code, shape.mask.size,
        shape.tile_rows, float(scale), nat.ptr(sink), nat.ptr(gate),
        gate.stride(0) if gate is not None else 0, out.data_ptr(), nat.ptr(meta.o_part), nat.ptr(meta.lse_part),
        nat.status_buffer(q.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "latent_attention")
    launch_counter.add(2 if meta.max_splits > 1 else 1)
    return out


def expanded_widths(dq: int, dv: int):
    """(columns of keys, of values) the expanded form stores per head: what the attention kernel
    has; None when it has nothing that wide."""
    if max(dq, dv) <= 64:
        return 64, 64
    if max(dq, dv) <= 128:
        return 128, 128
    return (192, 128) if dq <= 192 and dv <= 128 else None


def expanded_attention(q, k, v, step: AttentionStep, H: int, widths: tuple, scale: float, out,
                       mask: MaskSpec = CAUSAL, sink=None, gate=None) -> None:
    """Attention of the step's long chunks over expanded keys and values (rows of ``k`` and ``v``:
    the keys those sequences see, one sequence after the other, as ``step.ctx[mask]`` names them;
    ``widths``: columns of a head of each). ``sink`` and ``gate``: see latent_attention."""
    Dk, D = widths
    if q.is_cuda:
        meta = step.exp_plans[(H, widths, mask)]
        if mask.kind == "causal" and Dk == D and sink is None and gate is None:
            attention_contiguous(q, k, v, None, H, D, scale, causal=True, meta=meta, out=out)
        else:
            attention_masked(q, k, v, meta, H, H, D, scale, mask, sink, gate, out=out, paged=False,
                             Dk=Dk)
        return
    t = r = 0
    for n, kl, lo in zip(step.exp_q_lens, step.exp_kv_lens, step.ctx[mask][1]):
        qs = q[t:t + n].reshape(n, H, Dk).float()
        ks, vs = (z[r:r + kl - lo].reshape(kl - lo, H, d).float() for z, d in ((k, Dk), (v, D)))
        s = torch.einsum("thd,khd->htk", qs, ks) * scale
        at, pos = torch.arange(kl - n, kl).view(n, 1), torch.arange(lo, kl)
        s = s.masked_fill((pos > at) | (pos < mask.first_key(at)), float("-inf"))
        o = torch.einsum("htk,khd->thd", sink_softmax(s, sink), vs)
        o = gated_heads(o, None if gate is None else gate[t:t + n])
        out[t:t + n] = o.reshape(n, H * D).to(out.dtype)
        t, r = t + n, r + kl - lo
