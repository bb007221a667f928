"""Attention over cached keys and values with what a layer may ask beyond the plain form: query / key
norms (per head or over the whole projection), partial rotary positions, keys that are the values too,
a mask with a lower bound (window or chunks), softly capped scores, a sink per head and an output gate.

CUDA tensors run ``csrc/rotary.cu`` and ``csrc/attention.cu`` or, for 32-bit models and heads wider
than the tensor-core kernel's, ``csrc/exact.cu``. CPU tensors run the restatements below.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..config import MaskSpec
from . import (AttentionMetadata, DecodePlan, attention_masked, build_attention_metadata,
               launch_counter)
from .stream_ops import dtype_code


def _nat():
    from . import native
    return native


@dataclass(frozen=True)
class HeadShape:
    """Heads, stored width and mask of an attention layer; layers that agree in them share one plan
    per step. ``D`` and ``Dv``: columns of a query / key and of a value head, zero-padded to what
    the kernel tiles by."""
    heads: int
    kv_heads: int
    D: int
    Dv: int
    kernel: str       # "tensor" | "exact"
    mask: MaskSpec = MaskSpec()

    @staticmethod
    def of(heads: int, kv_heads: int, dim: int, vdim: int, dtype: torch.dtype,
           mask: MaskSpec = MaskSpec()) -> "HeadShape":
        widest, group = max(dim, vdim), heads // kv_heads
        if dtype == torch.bfloat16 and widest <= 128 and group <= 128:
            D = 64 if widest <= 64 else 128
            return HeadShape(heads, kv_heads, D, D, "tensor", mask)
        up = (lambda n: -(-n // 8) * 8) if dtype == torch.bfloat16 else (lambda n: n)
        return HeadShape(heads, kv_heads, up(dim), up(vdim), "exact", mask)

    @property
    def group(self) -> int:
        """Rows per token of a tile of one key head: a power of two."""
        return 1 << max(0, (self.heads // self.kv_heads - 1).bit_length())


def build_plan(shape: HeadShape, q_lens, kv_lens, block_tables, block_size, device):
    if torch.device(device).type != "cuda" or shape.kernel == "exact":
        meta = AttentionMetadata(list(q_lens), list(kv_lens), int(sum(q_lens)))
        meta.block_tables = block_tables
        return meta
    return build_attention_metadata(q_lens, kv_lens, block_tables, shape.group, shape.heads, shape.D,
                                    device, Hkv=shape.kv_heads, mask=shape.mask, align=block_size)


class HeadDecodePlan(DecodePlan):
    """Work of one head shape in a captured decode step."""

    def __init__(self, shape: HeadShape, bucket: int, max_q: int, block_size: int):
        super().__init__(shape.group, shape.heads, shape.kv_heads, shape.D, bucket, max_q,
                         block_size, mask=shape.mask)
        self.shape = shape


# ------------------------------------------------------------------------------ kernels
def rotary_table(positions: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """fp32 [T, len(freq), 2]: cosine and sine of every token's angles, position * frequency in
    fp32. Layers with the same frequencies share it."""
    T, half = positions.numel(), freq.numel()
    if not positions.is_cuda:
        a = positions.float().unsqueeze(1) * freq
        return torch.stack([a.cos(), a.sin()], -1)
    nat = _nat()
    table = torch.empty(T, half, 2, dtype=torch.float32, device=positions.device)
    assert positions.dtype == torch.int64 and positions.is_contiguous()
    rc = nat.lib().ab200_rotary_table(positions.data_ptr(), freq.data_ptr(), table.data_ptr(), T,
                                      half, nat.stream_ptr())
    nat.check(rc, "rotary_table")
    launch_counter.add(1)
    return table


def rotate_ref(x, table):
    """x [T, heads, d] fp32, table [T, half, 2]: the first 2 * half dimensions rotated."""
    half = table.shape[1]
    u, v = x[..., :half], x[..., half:2 * half]
    c, s = table[:, None, :, 0], table[:, None, :, 1]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def head_rope_cache(proj, shape: HeadShape, dim: int, wq, wk, table, eps: float, slots, k_cache,
                    v_cache, whole: bool = False, shared_kv: bool = False) -> None:
    """``proj`` [T, ...] holds the query heads, key heads (``D`` columns each, ``dim`` in use) and
    value heads (``Dv``). RMS norm of every query and key head over its ``dim`` columns with the
    weights ``wq`` / ``wk`` (fp32 [D], or None), rotation by ``table`` (rotary_table), queries in
    place, keys and values to the rows ``slots`` of the caches; slot < 0: no write. ``whole``: the
    norm is over all query (key) heads of a token at once, weights fp32 [heads * D]. ``shared_kv``:
    there are no value heads; the keys before norm and rotation are the values."""
    H, G, D, Dv = shape.heads, shape.kv_heads, shape.D, shape.Dv
    T, bs = proj.shape[0], k_cache.shape[2]
    if not proj.is_cuda:
        x = proj[:, :(H + G) * D].reshape(T, H + G, D).float()
        raw = proj[:, H * D:(H + G) * D].clone()
        if whole:
            for a, n, w in ((0, H, wq), (H, G, wk)):
                y = x[:, a:a + n]
                ss = y.pow(2).sum((1, 2), keepdim=True) / (n * dim)
                x[:, a:a + n] = y / torch.sqrt(ss + eps) * w.view(n, D)
        elif wq is not None:
            w = torch.cat([wq.expand(H, D), wk.expand(G, D)])
            x = x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) / dim + eps) * w
        x = rotate_ref(x, table).to(proj.dtype)
        proj[:, :H * D] = x[:, :H].reshape(T, H * D)
        ok = slots >= 0
        blk, off = slots[ok] // bs, slots[ok] % bs
        k_cache[blk, :, off] = x[ok, H:]
        v = raw if shared_kv else proj[:, (H + G) * D:(H + G) * D + G * Dv]
        v_cache[blk, :, off] = v[ok].reshape(-1, G, Dv)
        return
    nat = _nat()
    assert proj.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert slots.dtype == torch.int64 and table.is_contiguous()
    rc = nat.lib().ab200_head_rope_cache(
        proj.data_ptr(), proj.stride(0), table.data_ptr(), table.shape[1], slots.data_ptr(),
        nat.ptr(wq), nat.ptr(wk), k_cache.data_ptr(), v_cache.data_ptr(), T, H, G, D, dim, Dv, bs,
        k_cache.shape[0] * bs, float(eps), int(whole), int(shared_kv), dtype_code(proj.dtype),
        nat.status_buffer(proj.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "head_rope_cache")
    launch_counter.add(1)


def attention_exact(q, k_cache, v_cache, block_tables, tok_seq, positions, H: int, Hkv: int, Dk: int,
                    Dv: int, scale: float, mask: MaskSpec, sink=None, gate=None,
                    softcap: float = 0.0) -> torch.Tensor:
    """fp32-accumulating attention without tensor cores; q [T, H * Dk], caches [num_blocks, Hkv,
    block_size, >= Dk / Dv] (they may be one tensor); ``gate`` [T, H * Dv], or [T, H]: one per head.
    Returns [T, H * Dv]."""
    nat = _nat()
    T = q.shape[0]
    assert gate is None or gate.stride(1) == 1
    out = torch.empty(T, H * Dv, dtype=q.dtype, device=q.device)
    assert q.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    rc = nat.lib().ab200_attention_exact(
        q.data_ptr(), q.stride(0), k_cache.data_ptr(), k_cache.shape[3], v_cache.data_ptr(),
        v_cache.shape[3], k_cache.shape[0], k_cache.shape[2], block_tables.data_ptr(),
        block_tables.shape[1], tok_seq.data_ptr(), positions.data_ptr(), nat.ptr(sink),
        nat.ptr(gate), gate.stride(0) if gate is not None else 0,
        int(gate is not None and gate.shape[1] == H), out.data_ptr(), out.stride(0), T, H,
        Hkv, Dk, Dv, mask.code, mask.size, float(scale), float(softcap), dtype_code(q.dtype),
        nat.status_buffer(q.device).data_ptr(), nat.stream_ptr())
    nat.check(rc, "attention_exact")
    launch_counter.add(1)
    return out


def head_attention_ref(q, k_cache, v_cache, meta, shape: HeadShape, scale, sink, gate, softcap=0.0):
    H, G, D, Dv = shape.heads, shape.kv_heads, shape.D, shape.Dv
    bs = k_cache.shape[2]
    out = torch.empty(q.shape[0], H * Dv, dtype=q.dtype)
    t = 0
    for i, (n, kl) in enumerate(zip(meta.q_lens, meta.kv_lens)):
        if n == 0:
            continue
        lo = int(shape.mask.first_key(kl - n))
        pos = torch.arange(lo, kl)
        blk = meta.block_tables[i].long()[pos // bs]
        k, v = (c[blk, :, pos % bs].float().repeat_interleave(H // G, 1)
                for c in (k_cache, v_cache))
        s = torch.einsum("thd,khd->htk", q[t:t + n].reshape(n, H, D).float(), k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        at = torch.arange(kl - n, kl).view(n, 1)
        s = s.masked_fill((pos > at) | (pos < shape.mask.first_key(at)), float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.view(H, 1, 1).expand(H, n, 1)], -1)
        p = torch.softmax(s, -1)[..., :kl - lo]
        out[t:t + n] = torch.einsum("htk,khd->thd", p, v).reshape(n, H * Dv).to(q.dtype)
        t += n
    if gate is not None:
        out = (out.float() * torch.sigmoid(gate.float())).to(q.dtype)
    return out


def head_attention(q, k_cache, v_cache, meta: AttentionMetadata, shape: HeadShape, scale: float,
                   sink=None, gate=None, tok_seq=None, positions=None,
                   softcap: float = 0.0) -> torch.Tensor:
    """q [T, heads * D] (row stride free); caches [num_blocks, kv_heads, block_size, D / Dv]; ``sink``
    fp32 [heads] and ``gate`` [T, heads * Dv] (row stride free) may be None; ``softcap`` > 0 caps the
    scores. Returns [T, heads * Dv]. ``tok_seq`` and ``positions`` (per token) are read by the "exact" kernel only."""
    if not q.is_cuda:
        return head_attention_ref(q, k_cache, v_cache, meta, shape, scale, sink, gate, softcap)
    if shape.kernel == "exact":
        return attention_exact(q, k_cache, v_cache, meta.block_tables, tok_seq, positions,
                               shape.heads, shape.kv_heads, shape.D, shape.Dv, scale, shape.mask,
                               sink, gate, softcap)
    return attention_masked(q, k_cache, v_cache, meta, shape.heads, shape.kv_heads, shape.D, scale,
                            shape.mask, sink, gate, softcap=softcap)
