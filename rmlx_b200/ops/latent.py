"""Attention over cached latents: absorbed decode (csrc/kernels/mla_decode.cu), and prompts whose contexts'
keys and values are expanded from their latents first (flash_prefill_tc.cu, latent form)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from .gemm import GemmStatus

_lib.register_cuda_sigs({
    "rmlx_mla_decode_paged": ("ppppp" "ppp" "pppiiiiiiifip", "i"),
    "rmlx_mla_decode_part_o_elems": ("iiii", "q"),
    "rmlx_mla_decode_part_ml_elems": ("iii", "q"),
    "rmlx_flash_prefill_latent_supported": ("iii", "i"),
    "rmlx_flash_prefill_latent": ("ppppippipiiiiiiiiifipip", "i"),
    "rmlx_latent_gather": ("pipippiiiip", "i"),
})

DECODE_WIDTHS = ((512, 64), (128, 64))       # (latent, rotated) widths of the decode kernel


def decode_splits(rows: int, heads: int, longest: int) -> int:
    """Splits of the cached tokens. Up to 16 head tiles: wide blocks (eight warps, one per SM), one wave of 148.
    More: narrow blocks (four warps, two per SM; the launcher picks them once the grid exceeds the SMs),
    one wave of 296. At least 8 pages per split."""
    tiles = rows * ((heads + 15) // 16)
    return max(1, min(64, (148 if tiles <= 16 else 296) // tiles, longest // 128))


class LatentDecodeScratch:
    """Split scratch of ``latent_decode`` for up to ``rows`` launch rows."""

    def __init__(self, rows: int, heads: int, splits: int, lat: int, device):
        lib = _lib.cuda()
        self.splits = splits
        self.part_o = self.part_ml = None
        if splits > 1:
            self.part_o = torch.empty(lib.rmlx_mla_decode_part_o_elems(rows, heads, splits, lat), dtype=torch.float32,
                                      device=device)
            self.part_ml = torch.empty(lib.rmlx_mla_decode_part_ml_elems(rows, heads, splits), dtype=torch.float32,
                                       device=device)


def latent_decode(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor, scale: float,
                  out: torch.Tensor, scratch: LatentDecodeScratch, rows: Optional[torch.Tensor] = None,
                  table_rows: Optional[torch.Tensor] = None, pdl: bool = False) -> torch.Tensor:
    """q [T, H, lat + rot] (absorbed) over ``cache`` [blocks, 1, 16, lat + rot + 8] -> out [T, H, lat]; row t sees
    keys 0 .. positions[t] of row table_rows[t] (default t) of the block table. ``rows``: the rows to run."""
    _lib.require_cuda_tensor(q, cache, block_table, positions, out, rows, table_rows)
    t, h, w = q.shape
    lat = out.shape[2]
    assert q.is_contiguous() and out.is_contiguous() and cache.dtype == q.dtype == out.dtype == torch.bfloat16
    rc = _lib.cuda().rmlx_mla_decode_paged(
        q.data_ptr(), cache.data_ptr(), block_table.data_ptr(), None, None, _lib.ptr(rows), positions.data_ptr(),
        _lib.ptr(table_rows), out.data_ptr(), _lib.ptr(scratch.part_o), _lib.ptr(scratch.part_ml),
        t if rows is None else rows.numel(), h, lat, w - lat, cache.shape[3], block_table.stride(0), scratch.splits, scale,
        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "mla_decode_paged")
    return out


def prefill_supported(dim: int, rot: int, vdim: int) -> bool:
    return bool(_lib.cuda().rmlx_flash_prefill_latent_supported(dim, rot, vdim))


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, pages: torch.Tensor, out: torch.Tensor,
                  pdl: bool = False) -> torch.Tensor:
    """out [16 n, lat] = the latents of ``pages`` int32 [n, 2] = (row of ``block_table``, page of the sequence)."""
    _lib.require_cuda_tensor(cache, block_table, pages, out)
    assert out.dtype == cache.dtype == torch.bfloat16 and out.shape[0] == pages.shape[0] * cache.shape[2]
    rc = _lib.cuda().rmlx_latent_gather(cache.data_ptr(), cache.shape[3], block_table.data_ptr(), block_table.stride(0),
                                        pages.data_ptr(), out.data_ptr(), pages.shape[0], out.shape[1], cache.shape[2],
                                        int(pdl), _lib.stream_ptr())
    _lib.check(rc, "latent_gather")
    return out


def flash_prefill_latent(q: torch.Tensor, kv: torch.Tensor, cache: torch.Tensor, c_rot: int, block_table: torch.Tensor,
                         tiles: torch.Tensor, tile_ctx: torch.Tensor, scale: float, out: torch.Tensor, dim: int,
                         lanes: int = 1, pdl: bool = False) -> torch.Tensor:
    """q [T, H, dim + rot]; kv [ctx rows, H, dim + dv] expanded keys and values, the sequence of tile i from row
    tile_ctx[i] on; the rotated key part at column ``c_rot`` of the cache's rows. ``tiles`` as flash_prefill_scored."""
    _lib.require_cuda_tensor(q, kv, cache, block_table, tiles, tile_ctx, out)
    t, h, dk = q.shape
    dv = out.shape[2]
    assert q.is_contiguous() and kv.is_contiguous() and out.is_contiguous() and kv.shape[1:] == (h, dim + dv)
    assert tiles.dtype == tile_ctx.dtype == torch.int32 and tile_ctx.numel() == tiles.shape[0] and cache.shape[2] == 16
    rc = _lib.cuda().rmlx_flash_prefill_latent(
        q.data_ptr(), kv.data_ptr(), cache.data_ptr(), block_table.data_ptr(), block_table.stride(0), tiles.data_ptr(),
        tile_ctx.data_ptr(), tiles.shape[0], out.data_ptr(), t, h, dim, dk - dim, dv, kv.shape[0], cache.shape[0],
        cache.shape[3], c_rot, scale, lanes, GemmStatus.get(q.device).data_ptr(), int(pdl), _lib.stream_ptr())
    _lib.check(rc, "flash_prefill_latent")
    return out
