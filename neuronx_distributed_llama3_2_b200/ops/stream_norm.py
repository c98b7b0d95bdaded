"""The fp32 residual stream of plain pre-norm decoders (``csrc/stream_norm.cu``): token embedding with additive sinusoidal
position vectors and a norm at the entry, and the residual add (with the sublayer's output bias) fused with the norm that
the next sublayer reads; ``stream_update_`` adds layer scales, a re-added embedding and a constant vector to the latter."""
from __future__ import annotations

import ctypes as _c
from typing import Optional, Tuple

import torch

from . import _lib

GROUP = "scored_serving"


def _code(dtype: torch.dtype) -> int:
    return {torch.bfloat16: 0, torch.float32: 1}[dtype]


def rms_ref(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def position_frequencies(width: int, base: float = 10000.0, device=None) -> torch.Tensor:
    """``base ** (-2 i / width)`` of the column pairs ``(2 i, 2 i + 1)``, float64 ``[ceil(width / 2)]``."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / width).to(device)


def position_vectors_ref(positions: torch.Tensor, freq: torch.Tensor, width: int) -> torch.Tensor:
    """``[..., width]`` fp32: ``sin(p f_i)`` at entry ``2 i``, ``cos(p f_i)`` at entry ``2 i + 1``."""
    ang = positions.to(torch.float64).unsqueeze(-1) * freq.to(positions.device)
    return torch.stack([torch.sin(ang), torch.cos(ang)], dim=-1).flatten(-2)[..., :width].float()


def embed_norm(table: torch.Tensor, ids: torch.Tensor, positions: torch.Tensor, freq: Optional[torch.Tensor],
               w_embed: torch.Tensor, eps: float, w_next: Optional[torch.Tensor] = None,
               out_dtype: Optional[torch.dtype] = None) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``x = rms_norm(table[ids] + position vector) * w_embed`` (fp32 ``[..., W]``) and, with ``w_next``,
    ``h = (rms_norm(x) * w_next).to(out_dtype)``.  ``freq``: ``position_frequencies`` or ``None`` (no position vectors)."""
    V, W = table.shape
    if table.is_cuda and table.dtype in (torch.bfloat16, torch.float32) and _lib.available(GROUP):
        ids_c, pos_c = ids.long().contiguous(), positions.long().contiguous()
        assert table.is_contiguous() and ids_c.shape == pos_c.shape
        we, wn = w_embed.float().contiguous(), (w_next.float().contiguous() if w_next is not None else None)
        x = torch.empty(ids.shape + (W,), dtype=torch.float32, device=table.device)
        h = torch.empty(ids.shape + (W,), dtype=out_dtype, device=table.device) if wn is not None else None
        L = _lib.lib(GROUP)
        rc = L.nxd_embed_norm(_c.c_int(_code(table.dtype)), _c.c_int(_code(out_dtype) if h is not None else 1),
                              _lib.ptr(table), _lib.ptr(ids_c), _lib.ptr(pos_c), _lib.ptr(freq), _lib.ptr(we), _lib.ptr(wn),
                              _lib.ptr(x), _lib.ptr(h), _c.c_longlong(ids_c.numel()), _c.c_int(W), _c.c_int(V),
                              _c.c_float(eps), _lib.stream_ptr())
        _lib.check(rc, "nxd_embed_norm", L)
        return x, h
    e = table[ids.long()].float()
    if freq is not None:
        e = e + position_vectors_ref(positions, freq, W)
    x = rms_ref(e, w_embed, eps)
    return x, (rms_ref(x, w_next, eps).to(out_dtype) if w_next is not None else None)


def residual_norm_(x: torch.Tensor, y: Optional[torch.Tensor], bias: Optional[torch.Tensor] = None,
                   w_next: Optional[torch.Tensor] = None, eps: float = 1e-6, out_dtype: Optional[torch.dtype] = None):
    """``x += y (+ bias)`` in place on the fp32 stream ``x`` (skipped without ``y``), then
    ``h = (x / sqrt(mean(x^2) + eps) * w_next).to(out_dtype)`` (skipped without ``w_next``); returns ``(x, h)``."""
    assert x.dtype == torch.float32 and (y is None or y.numel() == x.numel())
    W = x.shape[-1]
    if x.is_cuda and (y is None or y.dtype in (torch.bfloat16, torch.float32)) and _lib.available(GROUP):
        assert x.is_contiguous()
        yc = None if y is None else (y if y.is_contiguous() else y.contiguous())
        b = None if bias is None else bias.float().contiguous()
        w = None if w_next is None else w_next.float().contiguous()
        h = torch.empty(x.shape, dtype=out_dtype, device=x.device) if w is not None else None
        L = _lib.lib(GROUP)
        rc = L.nxd_residual_norm(_c.c_int(_code(yc.dtype) if yc is not None else 1),
                                 _c.c_int(_code(out_dtype) if h is not None else 1), _lib.ptr(x), _lib.ptr(yc), _lib.ptr(b),
                                 _lib.ptr(w), _lib.ptr(h), _c.c_longlong(x.numel() // W), _c.c_int(W), _c.c_float(eps),
                                 _lib.stream_ptr())
        _lib.check(rc, "nxd_residual_norm", L)
        return x, h
    if y is not None:
        x.add_(y.float().reshape(x.shape) + (bias.float() if bias is not None else 0.0))
    return x, (rms_ref(x, w_next, eps).to(out_dtype) if w_next is not None else None)


def stream_update_(x: Optional[torch.Tensor], y: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None,
                   scale: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None,
                   ids: Optional[torch.Tensor] = None, mul: float = 1.0, shift: Optional[torch.Tensor] = None,
                   w_next: Optional[torch.Tensor] = None, eps: float = 1e-6, out_dtype: Optional[torch.dtype] = None):
    """``x <- x + scale * (y + bias) + mul * table[ids] + shift`` (any of the terms; in place on the fp32 stream ``x [rows, W]``,
    which with ``x=None`` starts as the sum of the others), then ``h = (x / sqrt(mean(x^2) + eps) * w_next).to(out_dtype)``
    (skipped without ``w_next``); returns ``(x, h)``.  ``scale, bias, shift, w_next [W]`` fp32; ``table [vocab, W]``, ``ids
    [rows]``: the token embedding, at the entry of the model or once more ahead of a pass of a looped range of layers."""
    assert x is not None or table is not None
    rows, W = x.shape if x is not None else (ids.numel(), table.shape[1])
    src = x if x is not None else table
    if src.is_cuda and (y is None or y.dtype in (torch.bfloat16, torch.float32)) and _lib.available(GROUP):
        init = x is None
        if init:
            x = torch.empty(rows, W, dtype=torch.float32, device=table.device)
        assert x.dtype == torch.float32 and x.is_contiguous()
        yc = None if y is None else (y if y.is_contiguous() else y.contiguous())
        ids_c = None if table is None else ids.reshape(-1).long().contiguous()
        assert table is None or (table.is_contiguous() and ids_c.numel() == rows)
        h = torch.empty(rows, W, dtype=out_dtype, device=x.device) if w_next is not None else None
        L = _lib.lib(GROUP)
        rc = L.nxd_stream_update(_c.c_int(_code(yc.dtype) if yc is not None else 1),
                                 _c.c_int(_code(out_dtype) if h is not None else 1),
                                 _c.c_int(_code(table.dtype) if table is not None else 1), _lib.ptr(x), _lib.ptr(yc),
                                 _lib.ptr(bias), _lib.ptr(scale), _lib.ptr(table), _lib.ptr(ids_c), _c.c_float(mul),
                                 _c.c_int(table.shape[0] if table is not None else 0), _lib.ptr(shift), _c.c_int(int(init)),
                                 _lib.ptr(w_next), _lib.ptr(h), _c.c_longlong(rows), _c.c_int(W), _c.c_float(eps),
                                 _lib.stream_ptr())
        _lib.check(rc, "nxd_stream_update", L)
        return x, h
    if x is None:
        x = torch.zeros(rows, W, dtype=torch.float32, device=table.device)
    if y is not None:
        t = y.float().reshape(rows, W) + (bias.float() if bias is not None else 0.0)
        x.add_(t * scale.float() if scale is not None else t)
    if table is not None:
        x.add_(table[ids.reshape(-1).long()].float() * mul)
    if shift is not None:
        x.add_(shift.float())
    return x, (rms_ref(x, w_next, eps).to(out_dtype) if w_next is not None else None)
