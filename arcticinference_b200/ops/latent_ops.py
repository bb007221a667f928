"""Latent attention: keys and values are linear maps of one cached latent vector per token.

Two ways to compute the same function:

* absorbed (decode and short chunks): the query heads are mapped into latent space
  (``q_h W_uk,h``), attend to the cached latents directly (one shared "head" that is key and
  value at once), and the result is mapped out of it (``W_uv,h``). The cache is read once for all
  heads.
* expanded (long chunks of wide latents): the latents of the context are gathered and expanded to
  per-head keys and values by one matrix product, and ordinary attention follows; per query-key
  pair that is ``dim + vdim`` instead of ``2 * kv_rank`` multiply-adds.

CUDA tensors run ``csrc/latent_attention.cu`` (keys on the tensor core's M side),
``csrc/attention.cu`` (latents of at most 64, and the expanded form) or, for 32-bit models and
shapes outside those, ``csrc/exact.cu``. CPU tensors run the restatement below.
"""

from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np
import torch

from . import (AttentionMetadata, DecodePlan, attention, attention_contiguous, launch_counter,
               plan_attention_work, upload)
from .stream_ops import dtype_code

KEY_TILE = 128


def _nat():
    from . import native
    return native


def padded_rank(rank: int, heads: int, dtype: torch.dtype) -> int:
    """Columns of a cached latent row: what the tensor-core kernels tile by."""
    if dtype != torch.bfloat16:
        return rank
    if rank <= 64 and heads <= 128:
        return 64
    return -(-rank // 128) * 128


@dataclass(frozen=True)
class LatentShape:
    """Heads and padded latent width of an absorbed attention, and how its work is planned. The
    layers of a model that agree in both share one plan per step."""
    heads: int
    rank: int
    kernel: str       # "packed" | "latent" | "exact"

    @staticmethod
    def of(heads: int, rank: int, dtype: torch.dtype) -> "LatentShape":
        if dtype == torch.bfloat16 and rank == 64 and heads <= 128:
            return LatentShape(heads, rank, "packed")
        if dtype == torch.bfloat16 and rank % 128 == 0 and rank <= 512:
            return LatentShape(heads, rank, "latent")
        return LatentShape(heads, rank, "exact")

    # ---- "packed": the 128-row attention kernel with the heads padded to a power of two
    @property
    def group(self) -> int:
        return 1 << max(0, (self.heads - 1).bit_length())

    # ---- "latent": rows (token, head) in order, this many per tile
    @property
    def tile_rows(self) -> int:
        return min(64, -(-self.heads // 16) * 16)

    def plan(self, q_lens, kv_lens, max_splits_cap: int = 16):
        """(work [n, 8] int32, splits per token [T] int32, largest number of splits)."""
        if self.kernel == "packed":
            return plan_attention_work(q_lens, kv_lens, self.group, True, Hkv=1,
                                       max_splits_cap=max_splits_cap)
        return plan_latent_work(q_lens, kv_lens, self.heads, self.tile_rows,
                                max_splits_cap=max_splits_cap)

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
                     max_splits_cap: int = 16):
    """Work list of the latent kernel. The (token, head) rows of a sequence are cut into tiles of
    ``tile_rows``, its keys into pieces of whole 128-key tiles; the piece length is the one
    whose waves of CTAs cost least. Item: sequence, first row, rows, position of the
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
    key_tiles = -(-kl[live] // KEY_TILE)
    pieces = np.ones_like(key_tiles)
    if max_splits_cap > 1:
        best = None
        longest = int(key_tiles.max())
        for chunk in {max(1, -(-longest // s)) for s in range(1, max_splits_cap + 1)}:
            p = -(-key_tiles // chunk)
            items = int((p * n_tiles).sum())
            waves = -(-items // num_sms)
            cost = waves * (chunk + 3) + (2 if chunk < longest else 0)
            if best is None or cost < best[0] or (cost == best[0] and chunk > best[1]):
                best = (cost, chunk)
        pieces = -(-key_tiles // best[1])
    per = -(-key_tiles // pieces)
    pieces = -(-key_tiles // per)
    rep = np.repeat(np.arange(live.size), n_tiles * pieces)
    first = np.cumsum(n_tiles * pieces) - n_tiles * pieces
    j = np.arange(rep.size) - first[rep]
    tile, piece = j // pieces[rep], j % pieces[rep]
    r0 = tile * tile_rows
    ks = piece * per[rep] * KEY_TILE
    ke = np.minimum(kl[live][rep], (piece + 1) * per[rep] * KEY_TILE)
    base = tok0[live][rep]
    work = np.stack([live[rep], base * heads + r0, np.minimum(tile_rows, rows[rep] - r0),
                     kl[live][rep] - ql[live][rep] - base, ks, ke, piece, pieces[rep]], 1)
    # keys a tile really sees end at its last token: heaviest first
    last = work[:, 3] + (work[:, 1] + work[:, 2] - 1) // heads
    work = work[np.argsort(-(np.minimum(ke, last + 1) - ks), kind="stable")]
    tok_splits[:T] = np.repeat(pieces, ql[live])
    return work.astype(np.int32), tok_splits, int(pieces.max())


@dataclass
class LatentStep:
    """One step's attention, shared by all layers. In layers that expand long chunks, the rows
    [0, n_absorbed) of the batch attend in latent space and the rows after them (whole
    sequences) through expanded keys and values; the other layers absorb every row."""
    n_absorbed: int
    # (shape, every row?) -> plan; the second form covers only the first n_absorbed rows
    absorbed: dict = field(default_factory=dict)
    tok_seq: torch.Tensor | None = None             # int32 [T]: row of the block table
    # expanded part: cache rows of the context of its sequences, one after the other
    ctx_slots: torch.Tensor | None = None
    exp_q_lens: list = field(default_factory=list)
    exp_kv_lens: list = field(default_factory=list)
    exp_plans: dict = field(default_factory=dict)   # heads -> AttentionMetadata

    @property
    def uploaded_bytes(self) -> int:
        n = sum(m.uploaded_bytes for m in {id(m): m for m in self.absorbed.values()}.values())
        n += sum(m.uploaded_bytes for m in self.exp_plans.values())
        return n + sum(t.numel() * t.element_size() for t in (self.tok_seq, self.ctx_slots)
                       if t is not None)


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
    work, tok_splits, max_splits = shape.plan(q_lens, kv_lens)
    meta.work = upload(work, device)
    meta.tok_splits = upload(tok_splits, device)
    meta.block_tables = block_tables
    meta.max_splits, meta.num_work = max_splits, work.shape[0]
    meta.tile_keys = shape.tile_keys(max(q_lens), block_size)
    return finish_plan(shape, meta, T, device)


class LatentDecodePlan(DecodePlan):
    """Work of one latent shape in a captured decode step."""

    def __init__(self, shape: LatentShape, bucket: int, max_q: int, block_size: int):
        self.shape, self.bucket = shape, bucket
        self.Hq, self.D = shape.heads, shape.rank
        self.work_cap, self.splits = shape.decode_capacity(bucket, max_q, block_size)
        self.tile_keys = shape.tile_keys(max_q, block_size)
        self.meta = AttentionMetadata([], [], bucket)

    def plan(self, q_lens, kv_lens):
        return self.shape.plan(q_lens, kv_lens, max_splits_cap=self.splits)


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


def latent_attention_ref(q, cache, q_lens, kv_lens, block_tables, H, scale):
    nb, _, bs, R = cache.shape
    flat = cache.view(nb * bs, R)
    out = torch.empty_like(q)
    t = 0
    for i, (n, kl) in enumerate(zip(q_lens, kv_lens)):
        if n == 0:
            continue
        pos = torch.arange(kl)
        c = flat[block_tables[i].long()[pos // bs] * bs + pos % bs].float()
        s = torch.einsum("thr,kr->htk", q[t:t + n].reshape(n, H, R).float(), c) * scale
        limit = torch.arange(kl - n, kl).view(1, n, 1)
        s = s.masked_fill(pos.view(1, 1, kl) > limit, float("-inf"))
        o = torch.einsum("htk,kr->thr", torch.softmax(s, -1), c)
        out[t:t + n] = o.reshape(n, H * R).to(q.dtype)
        t += n
    return out


def latent_attention(q: torch.Tensor, cache: torch.Tensor, meta: AttentionMetadata,
                     shape: LatentShape, scale: float, tok_seq=None, positions=None):
    """q [T, H * R] in latent space; cache [num_blocks, 1, block_size, R]. Softmax over every key
    up to the token itself; returns [T, H * R]. ``tok_seq`` and ``positions`` (per token) are
    read by the "exact" kernel only."""
    H, R = shape.heads, shape.rank
    bt = meta.block_tables
    if not q.is_cuda:
        return latent_attention_ref(q, cache, meta.q_lens, meta.kv_lens, bt, H, scale)
    nat = _nat()
    T = q.shape[0]
    assert q.is_contiguous() and cache.is_contiguous() and cache.shape[3] == R
    if shape.kernel == "packed":
        return attention(q, cache, cache, meta, H, 1, R, scale)
    out = torch.empty_like(q)
    status = nat.status_buffer(q.device).data_ptr()
    if shape.kernel == "latent":
        rc = nat.lib().ab200_latent_attention(
            q.data_ptr(), T * H, cache.data_ptr(), cache.shape[0], cache.shape[2], bt.data_ptr(),
            bt.shape[1], meta.work.data_ptr(), meta.num_work, nat.ptr(meta.tok_splits),
            meta.max_splits, T, H, R, shape.tile_rows, float(scale), out.data_ptr(),
            nat.ptr(meta.o_part), nat.ptr(meta.lse_part), status, nat.stream_ptr())
        nat.check(rc, "latent_attention")
        launch_counter.add(2 if meta.max_splits > 1 else 1)
        return out
    rc = nat.lib().ab200_latent_attention_exact(
        q.data_ptr(), q.stride(0), cache.data_ptr(), cache.shape[0], cache.shape[2], bt.data_ptr(),
        bt.shape[1], tok_seq.data_ptr(), positions.data_ptr(), out.data_ptr(), out.stride(0), T, H,
        R, float(scale), dtype_code(q.dtype), status, nat.stream_ptr())
    nat.check(rc, "latent_attention_exact")
    launch_counter.add(1)
    return out


def expanded_attention(q, k, v, step: LatentStep, H: int, D: int, scale: float, out) -> None:
    """Attention of the step's long chunks over expanded keys and values (rows of ``k`` and ``v``:
    the contexts of those sequences, one after the other)."""
    if q.is_cuda:
        attention_contiguous(q, k, v, None, H, D, scale, causal=True, meta=step.exp_plans[H],
                             out=out)
        return
    t = r = 0
    for n, kl in zip(step.exp_q_lens, step.exp_kv_lens):
        qs = q[t:t + n].reshape(n, H, D).float()
        ks, vs = (z[r:r + kl].reshape(kl, H, D).float() for z in (k, v))
        s = torch.einsum("thd,khd->htk", qs, ks) * scale
        limit = torch.arange(kl - n, kl).view(1, n, 1)
        s = s.masked_fill(torch.arange(kl).view(1, 1, kl) > limit, float("-inf"))
        out[t:t + n] = torch.einsum("htk,khd->thd", torch.softmax(s, -1), vs) \
            .reshape(n, H * D).to(out.dtype)
        t, r = t + n, r + kl
