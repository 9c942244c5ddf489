"""Operators of latent attention (compressed key / value cache): geometry of the padded layouts, weight packing, and the functions
that dispatch to the kernels of ``csrc/latent.cu`` / ``csrc/attention_tc.cu`` on CUDA and to plain PyTorch statements on the CPU.

A token's projection row holds ``[q of every head: unrotated | rotated] [latent] [rotated key] [gate]``. The cache keeps, per token,
the RMS-normed latent and the rotated key; per-head keys and values are linear in the latent. A layer without a down projection (``down`` False) has
queries and gate only and reads the cache of another layer with the same latent and rotated sizes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import _count, _cuda, ref, require_ext


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentShape:
    heads: int
    dim: int  # unrotated query / key columns per head
    rot_dim: int  # rotated columns, shared by the heads on the key side
    vdim: int
    kv_rank: int
    gate: bool = True
    down: bool = True  # the layer projects its own latent and rotated key

    def __post_init__(self):
        if min(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank) < 1 or self.rot_dim % 2:
            raise ValueError(f"latent attention sizes must be positive (and rot_dim even): {self}")
        if self.kv_rank > 1024:
            raise ValueError(f"latent size {self.kv_rank} is beyond the kernels' 1024")

    # padded sizes: query columns to the 64-column blocks of the tensor-core tiles, cached rows to the 16 of an mma.sync step
    dn = property(lambda s: _up(s.dim, 64))
    dk = property(lambda s: _up(s.dim, 64) + _up(s.rot_dim, 64))
    Rp = property(lambda s: _up(s.kv_rank, 16))
    drp = property(lambda s: _up(s.rot_dim, 16))
    Kp = property(lambda s: _up(s.kv_rank, 32))
    R8 = property(lambda s: _up(s.kv_rank, 8))
    dv8 = property(lambda s: _up(s.vdim, 8))
    off_c = property(lambda s: s.heads * s.dk)
    off_r = property(lambda s: s.off_c + s.R8)
    behind = property(lambda s: s.off_r + _up(s.rot_dim, 8) if s.down else s.off_c)
    off_g = property(lambda s: s.behind if s.gate else -1)
    width = property(lambda s: s.behind + (_up(s.heads * s.vdim, 8) if s.gate else 0))
    out_width = property(lambda s: s.heads * s.vdim)

    def geom(self) -> list[int]:
        return [self.heads, self.dk, self.dim, self.kv_rank, self.Rp, self.rot_dim, self.drp, self.vdim, self.Kp, self.off_c if self.down else -1,
                self.off_r if self.down else -1, self.off_g]

    def prefill_dv(self) -> int:
        """Padded value width of the tensor-core prefill kernel; 0 when these head sizes are outside it."""
        return require_ext().latent_prefill_dv(self.dk, self.vdim)


def pack_input(s: LatentShape, q, dkv, g, k_pad: int) -> torch.Tensor:
    """One projection matrix ``[width, k_pad]`` from the query, latent-down and gate projections, rows in the padded layout."""
    K = q.shape[1]
    w = torch.zeros(s.width, k_pad, dtype=q.dtype, device=q.device)
    heads = q.reshape(s.heads, s.dim + s.rot_dim, K)
    qv = w[: s.off_c].view(s.heads, s.dk, k_pad)
    qv[:, : s.dim, :K] = heads[:, : s.dim]
    qv[:, s.dn : s.dn + s.rot_dim, :K] = heads[:, s.dim :]
    if s.down:
        w[s.off_c : s.off_c + s.kv_rank, :K] = dkv[: s.kv_rank]
        w[s.off_r : s.off_r + s.rot_dim, :K] = dkv[s.kv_rank :]
    if s.gate:
        w[s.off_g : s.off_g + s.out_width, :K] = g
    return w


def pack_absorbed(s: LatentShape, uk, uv) -> tuple[torch.Tensor, torch.Tensor]:
    """Key weights turned to the query side ``[H, Rp, dn]`` and value weights ``[H, dv8, Kp]``, zero-padded."""
    wuk = torch.zeros(s.heads, s.Rp, s.dn, dtype=uk.dtype, device=uk.device)
    wuk[:, : s.kv_rank, : s.dim] = uk.reshape(s.heads, s.dim, s.kv_rank).transpose(1, 2)
    wuv = torch.zeros(s.heads, s.dv8, s.Kp, dtype=uv.dtype, device=uv.device)
    wuv[:, : s.vdim, : s.kv_rank] = uv.reshape(s.heads, s.vdim, s.kv_rank)
    return wuk.contiguous(), wuv.contiguous()


def pack_expand(s: LatentShape, uk, uv, dv: int) -> torch.Tensor:
    """``[H * dn + H * dv, R8]``: latent -> per-head keys and values in the column layout of the prefill kernel."""
    wk = torch.zeros(s.heads, s.dn, s.R8, dtype=uk.dtype, device=uk.device)
    wk[:, : s.dim, : s.kv_rank] = uk.reshape(s.heads, s.dim, s.kv_rank)
    wv = torch.zeros(s.heads, dv, s.R8, dtype=uv.dtype, device=uv.device)
    wv[:, : s.vdim, : s.kv_rank] = uv.reshape(s.heads, s.vdim, s.kv_rank)
    return torch.cat([wk.reshape(-1, s.R8), wv.reshape(-1, s.R8)]).contiguous()


# ---------------------------------------------------------------------------------------------------------- operators
def prepare(s: LatentShape, p, positions, slots, norm_w, cos, sin, c_cache, r_cache, eps: float) -> None:
    """Rotate the queries in place; RMS-norm the latent, rotate the shared key and write both to the cache rows ``slots`` (layers with a down
    projection)."""
    if _cuda(p):
        _count()
        require_ext().latent_prepare(p, positions, slots, norm_w, cos, sin, c_cache, r_cache, s.geom(), eps)
        return
    T, pos = p.shape[0], positions.long()
    q = p[:, : s.off_c].view(T, s.heads, s.dk)
    q[:, :, s.dn : s.dn + s.rot_dim] = ref.apply_rope(q[:, :, s.dn : s.dn + s.rot_dim], pos, cos, sin)
    if not s.down:
        return
    c = ref.rmsnorm(p[:, s.off_c : s.off_c + s.kv_rank], norm_w[: s.kv_rank], eps)
    r = ref.apply_rope(p[:, s.off_r : s.off_r + s.rot_dim].unsqueeze(1), pos, cos, sin).squeeze(1)
    c_cache.view(-1, s.Rp)[slots.long()] = F.pad(c, (0, s.Rp - s.kv_rank)).to(c_cache.dtype)
    r_cache.view(-1, s.drp)[slots.long()] = F.pad(r, (0, s.drp - s.rot_dim)).to(r_cache.dtype)


def rows_attention(s: LatentShape, p, row_idx, row_seq, row_ctx, wuk, wuv, c_cache, r_cache, block_tables, out, scale: float, window: int,
                   splits: int = 1, write=None, sink=None) -> None:
    """Rows of ``p`` one by one against the cache (decode, short portions), absorbed form. Row ``i`` is ``p[row_idx[i]]`` of block-table
    row ``row_seq[i]`` and sees the last ``window`` of its first ``row_ctx[i]`` keys; ``None`` index arrays mean ``i``. Writes the gated
    heads to columns ``[0, H * vdim)`` of the rows of ``out``. ``write`` = the arguments of :func:`prepare` behind ``p``, for a decode batch
    whose rows were not prepared yet (on CUDA in bf16 that work rides in the first launch). ``sink`` fp32 ``[H]``: a score per head without a value."""
    if write is not None and (not _cuda(p) or p.dtype == torch.float32):
        prepare(s, p, *write)
    if _cuda(p):
        if p.dtype == torch.float32:
            _count()
            require_ext().latent_rows_f32(p, row_idx, row_seq, row_ctx, wuk, wuv, c_cache, r_cache, block_tables, out, s.geom(), scale, window, sink)
        else:
            _count(3)
            require_ext().latent_decode(p, row_idx, row_seq, row_ctx, wuk, wuv, c_cache, r_cache, block_tables, out, s.geom(), scale, window, splits, sink,
                                        *(() if write is None else (*write[:5], write[7])))
        return
    n = row_ctx.shape[0]
    ps = c_cache.shape[2]
    for i in range(n):
        t = int(row_idx[i]) if row_idx is not None else i
        b = int(row_seq[i]) if row_seq is not None else i
        ctx = int(row_ctx[i])
        lo = max(0, ctx - window) if window > 0 else 0
        key = torch.arange(lo, ctx)
        slot = block_tables[b, key // ps].long() * ps + key % ps
        c, r = c_cache.view(-1, s.Rp)[slot].float(), r_cache.view(-1, s.drp)[slot].float()
        q = p[t, : s.off_c].view(s.heads, s.dk).float()
        ql = torch.einsum("hd,hrd->hr", q[:, : s.dn], wuk.float())
        sc = (ql @ c.t() + q[:, s.dn : s.dn + s.drp] @ r.t()) * scale
        if sink is not None:
            sc = torch.cat([sc, sink.view(-1, 1)], dim=1)
        o = torch.softmax(sc, dim=-1)[:, : c.shape[0]] @ c
        o = torch.einsum("hr,hvr->hv", o, wuv[:, : s.vdim, : s.Rp].float()).reshape(-1)
        if s.gate:
            o = o * torch.sigmoid(p[t, s.off_g : s.off_g + s.out_width].float())
        out[t, : s.out_width] = o.to(out.dtype)


def gather(s: LatentShape, c_cache, r_cache, block_tables, seq, key0, n_keys, row0, max_rows: int, total: int):
    """Cached rows of the key ranges, packed for :func:`prefill_attention` (CUDA): latents ``[total, R8]``, rotated keys ``[total, dk - dn]``."""
    _count()
    return require_ext().latent_gather(c_cache, r_cache, block_tables, seq, key0, n_keys, row0, max_rows, total, s.R8, s.dk - s.dn)


def prefill_attention(s: LatentShape, p, kv, kr, q_start, q_len, ctx, row0, tile_seq, tile_q0, out, scale: float, window: int, sink=None) -> None:
    """Prompt rows against expanded keys and values (CUDA, tcgen05): gated heads to columns ``[0, H * vdim)`` of ``out``."""
    _count()
    require_ext().latent_prefill(p, kv, kr, q_start, q_len, ctx, row0, tile_seq, tile_q0, out, s.geom(), scale, window, sink)


def prefill_tile_rows(dv: int) -> int:
    return require_ext().latent_prefill_tile_rows(dv)


def pick_splits(rows: int, s: LatentShape, span: Optional[int]) -> int:
    """Split-KV factor of :func:`rows_attention`, a power of two: the cheapest by waves of CTAs x (32-key tiles per CTA + a fixed cost), plus
    the merge of what does not fit one cluster of eight. (Clusters leave some SMs of a GPC unused: fewer CTAs are resident then.)"""
    two = s.heads > 16
    ctas = max(1, rows * ((s.heads + 31) // 32 if two else 1))
    slots = 148 * (1 if two or s.Rp > 512 else 2)
    tiles = max(1, (span + 31) // 32) if span is not None else 4096
    best, best_cost = 1, None
    for k in (1, 2, 4, 8, 16, 32, 64):
        if k > 1 and 2 * k > tiles:
            break
        resident = int(slots * (0.8 if k >= 8 else 0.9 if k > 1 else 1.0))
        outer = max(1, k // 8)
        cost = -(-ctas * k // resident) * (-(-tiles // k) + 6) + (outer * (0.5 + 0.08 * rows) if outer > 1 else 0.0)
        if best_cost is None or cost < best_cost:
            best, best_cost = k, cost
    return best
