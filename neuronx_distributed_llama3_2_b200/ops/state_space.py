"""State-space mixers over a per-line fp32 state (``csrc/state_space.cu``), next to the other recurrences (matrix memory,
delta rule, retention):

    selective_scan      S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c;   y * silu(z)
                        (Gu, Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces")
    state_space_heads   S <- exp(-exp(A_log_h) dt) S + dt B x^T;   y = S^T C + D_h x            S [state, vdim] per head
                        (Dao, Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State
                        Space Duality")

with ``dt = softplus(pre-activation + bias)`` and ``A = -exp(A_log)``, behind a short causal convolution per channel
(``conv_silu``: taps over time, bias, silu, zeros before the start), and the output side of the second kind (``gate_norm``:
gate first, then the RMS norm over equal groups of columns).

State per cache line: ``S`` and the last ``taps - 1`` raw inputs of the convolution, both fp32.  A row whose first position is 0
starts from zeros; any other row continues from what its line holds, so a prompt may arrive in portions and a line that is
handed to a new request needs no clearing.  Step sizes, decays and the state are fp32 whatever the activation dtype.  Every
op has a PyTorch restatement for CPU.
"""
from __future__ import annotations

import ctypes as _c
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib
from .linear import gemm_nt

GROUP = "state_space_serving"
IMPLS = {"auto": 0, "scan": 1, "chunks": 2}


def _code(dtype: torch.dtype) -> int:
    return {torch.bfloat16: 0, torch.float32: 1}[dtype]


def _use_kernel(x: torch.Tensor) -> bool:
    return x.is_cuda and x.dtype in (torch.bfloat16, torch.float32) and _lib.available(GROUP)


def _i32(t: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
    if t is None:
        return None
    return t if (t.dtype == torch.int32 and t.is_contiguous()) else t.to(torch.int32).contiguous()


def _rows(x: torch.Tensor) -> Tuple[torch.Tensor, int]:
    """``x [B, T, n]`` as rows of a (possibly wider) buffer: the tensor and the distance between rows in elements."""
    B, T, _ = x.shape
    if x.stride(2) == 1 and (B == 1 or x.stride(0) == T * x.stride(1)):
        return x, x.stride(1) if T > 1 or B == 1 else x.stride(0)
    x = x.contiguous()
    return x, x.stride(1)


def _line_and_count(b: int, T: int, n_new, seq_ids) -> Tuple[int, int]:
    return (b if seq_ids is None else int(seq_ids[b])), (T if n_new is None else min(int(n_new[b]), T))


def conv_silu(x: torch.Tensor, conv_w: torch.Tensor, bias: Optional[torch.Tensor], conv_state: torch.Tensor,
              q_start: torch.Tensor, n_new: Optional[torch.Tensor] = None, seq_ids: Optional[torch.Tensor] = None,
              out_pitch: Optional[int] = None) -> torch.Tensor:
    """``x [B, T, C]`` (may be a column range of a projection output) -> ``silu(conv(x) + bias) [B, T, C]`` in the same dtype.
    ``conv_w [taps, C]`` fp32, last row = the current token; ``conv_state [lines, taps - 1, C]`` fp32 is moved to the end
    of the step in place.  Padding rows come out as zeros.  ``out_pitch``: distance between the output's rows (>= C; the
    result is a view of a buffer that wide)."""
    B, T, C = x.shape
    taps = conv_w.shape[0]
    K = taps - 1
    pitch = out_pitch or C
    assert conv_w.shape[1] == C and conv_state.shape[1:] == (K, C), (x.shape, conv_w.shape, conv_state.shape)
    if _use_kernel(x):
        assert conv_w.is_contiguous() and conv_w.dtype == torch.float32
        x, ld = _rows(x)
        out = torch.empty(B, T, pitch, dtype=x.dtype, device=x.device)
        qs, nn_, sid = _i32(q_start), _i32(n_new), _i32(seq_ids)
        L = _lib.lib(GROUP)
        rc = L.nxd_conv_silu(_c.c_int(_code(x.dtype)), _c.c_int(_code(out.dtype)), _lib.ptr(x), _c.c_longlong(ld),
                             _lib.ptr(conv_w), _lib.ptr(bias), _lib.ptr(conv_state), _lib.ptr(out), _c.c_longlong(pitch),
                             _lib.ptr(qs), _lib.ptr(nn_), _lib.ptr(sid), _c.c_int(B), _c.c_int(T), _c.c_int(C),
                             _c.c_int(taps), _lib.stream_ptr())
        _lib.check(rc, "nxd_conv_silu", L)
        return out[..., :C]
    out = torch.zeros(B, T, pitch, dtype=x.dtype, device=x.device)
    w = conv_w.float()
    for b in range(B):
        line, n = _line_and_count(b, T, n_new, seq_ids)
        if n <= 0:
            continue
        p0 = int(q_start[b])
        past = conv_state[line].clone()
        if p0 < K:                                         # positions before the start of the sequence are zeros
            past[: K - p0] = 0.0
        seq = torch.cat([past, x[b, :n].float()], dim=0)   # [K + n, C]: position p0 - K + i
        acc = torch.zeros(n, C, dtype=torch.float32, device=x.device)
        for j in range(taps):
            acc += w[j] * seq[j: j + n]
        if bias is not None:
            acc += bias.float()
        out[b, :n, :C] = F.silu(acc).to(x.dtype)
        conv_state[line] = seq[n: n + K]
    return out[..., :C]


def selective_scan(x: torch.Tensor, dt: Optional[torch.Tensor], dt_bias: Optional[torch.Tensor], bc: torch.Tensor, b_offset: int,
                   c_offset: int, z: torch.Tensor, a_log: torch.Tensor, d: torch.Tensor, S: torch.Tensor,
                   q_start: torch.Tensor, n_new: Optional[torch.Tensor] = None,
                   seq_ids: Optional[torch.Tensor] = None, dt_w: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x, z [B, T, C]`` (``z`` may be a column range of a projection output), ``dt [B, T, C]`` fp32 pre-activations of the step
    sizes, ``bc [B, T, ld]`` fp32 with the ``N`` columns of B at ``b_offset`` and of C at ``c_offset``; ``a_log [C, N]``,
    ``d [C]`` fp32; ``S [lines, C, N]`` fp32, updated in place -> ``y * silu(z) [B, T, C]`` in the dtype of ``x``.
    ``dt_w [C, rank]`` instead of ``dt``: the pre-activations are the first ``rank`` columns of ``bc`` times its rows (fp32; of a
    step of one token per row made inside the recurrence's kernel)."""
    B, T, C = x.shape
    N = a_log.shape[1]
    assert a_log.shape == (C, N) and S.shape[1:] == (C, N) and bc.dtype == torch.float32
    if dt is None and T == 1 and n_new is None and _use_kernel(x) and dt_w.shape[1] % 8 == 0:
        assert z.dtype == x.dtype == dt_w.dtype and S.is_contiguous() and a_log.is_contiguous() and dt_w.is_contiguous()
        (x, ldx), (z, ldz), (bc, ldb) = _rows(x), _rows(z), _rows(bc)
        out = torch.empty(B, T, C, dtype=x.dtype, device=x.device)
        qs, sid = _i32(q_start), _i32(seq_ids)
        L = _lib.lib(GROUP)
        rc = L.nxd_selective_step(_c.c_int(_code(x.dtype)), _lib.ptr(x), _c.c_longlong(ldx), _lib.ptr(dt_w),
                                  _c.c_int(dt_w.shape[1]), _lib.ptr(dt_bias), _lib.ptr(bc), _c.c_longlong(ldb),
                                  _c.c_int(b_offset), _c.c_int(c_offset), _lib.ptr(z), _c.c_longlong(ldz), _lib.ptr(a_log),
                                  _lib.ptr(d), _lib.ptr(S), _lib.ptr(out), _c.c_longlong(C), _lib.ptr(qs), _lib.ptr(sid),
                                  _c.c_int(B), _c.c_int(C), _c.c_int(N), _lib.stream_ptr())
        _lib.check(rc, "nxd_selective_step", L)
        return out
    if dt is None:
        low = bc[..., : dt_w.shape[1]].reshape(B * T, -1).to(dt_w.dtype).contiguous()
        dt = gemm_nt(low, dt_w, out_dtype=torch.float32).view(B, T, C)
    assert dt.dtype == torch.float32
    if _use_kernel(x):
        assert z.dtype == x.dtype and S.is_contiguous() and a_log.is_contiguous()
        (x, ldx), (z, ldz), (dt, ldd), (bc, ldb) = _rows(x), _rows(z), _rows(dt), _rows(bc)
        out = torch.empty(B, T, C, dtype=x.dtype, device=x.device)
        qs, nn_, sid = _i32(q_start), _i32(n_new), _i32(seq_ids)
        L = _lib.lib(GROUP)
        rc = L.nxd_selective_scan(_c.c_int(_code(x.dtype)), _lib.ptr(x), _c.c_longlong(ldx), _lib.ptr(dt), _c.c_longlong(ldd),
                                  _lib.ptr(dt_bias), _lib.ptr(bc), _c.c_longlong(ldb), _c.c_int(b_offset),
                                  _c.c_int(c_offset), _lib.ptr(z), _c.c_longlong(ldz), _lib.ptr(a_log), _lib.ptr(d),
                                  _lib.ptr(S), _lib.ptr(out), _c.c_longlong(C), _lib.ptr(qs), _lib.ptr(nn_), _lib.ptr(sid),
                                  _c.c_int(B), _c.c_int(T), _c.c_int(C), _c.c_int(N), _lib.stream_ptr())
        _lib.check(rc, "nxd_selective_scan", L)
        return out
    out = torch.zeros(B, T, C, dtype=x.dtype, device=x.device)
    A = -torch.exp(a_log.float())
    step = F.softplus(dt + dt_bias.float() if dt_bias is not None else dt)
    for b in range(B):
        line, n = _line_and_count(b, T, n_new, seq_ids)
        if n <= 0:
            continue
        s = torch.zeros_like(S[line]) if int(q_start[b]) == 0 else S[line].clone()
        for t in range(n):
            xt, dv = x[b, t].float(), step[b, t]
            s = torch.exp(dv.unsqueeze(1) * A) * s + (dv * xt).unsqueeze(1) * bc[b, t, b_offset: b_offset + N]
            y = s @ bc[b, t, c_offset: c_offset + N] + d.float() * xt
            out[b, t] = (y * F.silu(z[b, t].float())).to(x.dtype)
        S[line] = s
    return out


def state_space_heads(xbc: torch.Tensor, offsets: Tuple[int, int, int], dt: Optional[torch.Tensor], dt_bias: Optional[torch.Tensor],
                      a_log: torch.Tensor, d: torch.Tensor, S: torch.Tensor, q_start: torch.Tensor, groups: int,
                      n_new: Optional[torch.Tensor] = None, seq_ids: Optional[torch.Tensor] = None,
                      out_dtype: torch.dtype = torch.float32, impl: str = "auto",
                      dt_from: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> torch.Tensor:
    """``xbc [B, T, ld]`` holds, at columns ``offsets = (x, B, C)``, the heads' inputs ``[H, P]`` and the groups' ``B, C [G, N]``
    (after the convolution); ``dt [B, T, H]`` fp32 pre-activations of the step sizes (may be a column range); ``dt_bias,
    a_log, d [H]`` fp32; ``S [lines, H, N, P]`` fp32, updated in place -> ``y [B, T, H, P]`` in ``out_dtype``.  ``impl``: ``auto`` |
    ``scan`` (token by token) | ``chunks`` (tensor cores, bf16; an error where it does not apply).  ``dt_from = (h [B * T, W],
    w [>= H, W])`` instead of ``dt``: the pre-activations are ``h w^T`` (fp32), of a step of one token per row made inside the
    recurrence's kernel."""
    B, T, _ = xbc.shape
    H, N, P = S.shape[1:]
    assert H % groups == 0 and a_log.shape == (H,)
    hin = dt_w = None
    if dt is None:
        hin, dt_w = dt_from
        if T > 1 or n_new is not None or impl != "auto" or not _use_kernel(xbc):
            dt, hin, dt_w = gemm_nt(hin, dt_w, out_dtype=torch.float32).view(B, T, -1)[..., :H], None, None
    assert dt is None or dt.dtype == torch.float32
    x_off, b_off, c_off = offsets
    if _use_kernel(xbc):
        assert S.is_contiguous() and out_dtype in (torch.float32, xbc.dtype)
        xbc, ld = _rows(xbc)
        dt, ldd = _rows(dt) if dt is not None else (None, 0)
        assert hin is None or (hin.is_contiguous() and dt_w.is_contiguous() and hin.dtype == dt_w.dtype == xbc.dtype)
        y = torch.empty(B, T, H, P, dtype=out_dtype, device=xbc.device)
        qs, nn_, sid = _i32(q_start), _i32(n_new), _i32(seq_ids)
        L = _lib.lib(GROUP)
        rc = L.nxd_state_space_heads(_c.c_int(_code(xbc.dtype)), _c.c_int(_code(out_dtype)), _lib.ptr(xbc),
                                     _c.c_longlong(ld), _c.c_int(x_off), _c.c_int(b_off), _c.c_int(c_off), _lib.ptr(dt),
                                     _c.c_longlong(ldd), _lib.ptr(dt_bias), _lib.ptr(a_log), _lib.ptr(d), _lib.ptr(S),
                                     _lib.ptr(y), _lib.ptr(qs), _lib.ptr(nn_), _lib.ptr(sid), _c.c_int(B), _c.c_int(T),
                                     _c.c_int(H), _c.c_int(groups), _c.c_int(N), _c.c_int(P), _c.c_int(IMPLS[impl]),
                                     _lib.ptr(hin), _lib.ptr(dt_w), _c.c_int(hin.shape[1] if hin is not None else 0),
                                     _lib.stream_ptr())
        _lib.check(rc, "nxd_state_space_heads", L)
        return y
    y = torch.zeros(B, T, H, P, dtype=out_dtype, device=xbc.device)
    step = F.softplus(dt + dt_bias.float() if dt_bias is not None else dt)
    decay = torch.exp(-torch.exp(a_log.float()) * step)
    rep = H // groups
    for b in range(B):
        line, n = _line_and_count(b, T, n_new, seq_ids)
        if n <= 0:
            continue
        s = torch.zeros_like(S[line]) if int(q_start[b]) == 0 else S[line].clone()          # [H, N, P]
        for t in range(n):
            row = xbc[b, t].float()
            x = row[x_off: x_off + H * P].reshape(H, P)
            Bt = row[b_off: b_off + groups * N].reshape(groups, N).repeat_interleave(rep, dim=0)
            Ct = row[c_off: c_off + groups * N].reshape(groups, N).repeat_interleave(rep, dim=0)
            s = decay[b, t].reshape(H, 1, 1) * s + Bt.unsqueeze(2) * (step[b, t].reshape(H, 1) * x).unsqueeze(1)
            y[b, t] = (torch.einsum("hnp,hn->hp", s, Ct) + d.float().reshape(H, 1) * x).to(out_dtype)
        S[line] = s
    return y


def gate_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, groups: int, eps: float, act: str = "silu",
              out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``y, z [N, n]`` (rows may be column ranges of wider buffers) -> ``v = y * act(z)`` (``silu`` or ``sigmoid``), every one of the
    ``groups`` equal parts of the columns divided by its root mean square (fp32, ``eps`` inside the root), times ``weight [n]``.
    Result in the dtype of ``z``, into ``out`` (a column range of a wider buffer) when given."""
    N, n = y.shape
    assert z.shape == (N, n) and n % groups == 0
    if out is None:
        out = torch.empty(N, n, dtype=z.dtype, device=z.device)
    assert out.shape == (N, n) and out.dtype == z.dtype
    if _use_kernel(z) and y.dtype in (torch.float32, z.dtype) and y.stride(1) == 1 and z.stride(1) == 1 and out.stride(1) == 1:
        L = _lib.lib(GROUP)
        rc = L.nxd_gate_norm(_c.c_int(_code(y.dtype)), _c.c_int(_code(z.dtype)), _lib.ptr(y), _c.c_longlong(y.stride(0)),
                             _lib.ptr(z), _c.c_longlong(z.stride(0)), _lib.ptr(weight), _lib.ptr(out),
                             _c.c_longlong(out.stride(0)), _c.c_longlong(N), _c.c_int(n), _c.c_int(groups), _c.c_float(eps),
                             _c.c_int(1 if act == "silu" else 0), _lib.stream_ptr())
        _lib.check(rc, "nxd_gate_norm", L)
        return out
    zf = z.float()
    v = (y.float() * (F.silu(zf) if act == "silu" else torch.sigmoid(zf))).reshape(N, groups, n // groups)
    v = (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(N, n) * weight.float()
    out.copy_(v.to(z.dtype))
    return out
