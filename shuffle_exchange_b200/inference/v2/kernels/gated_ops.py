"""Python entry points of ``csrc/gated_mixers.cu``: operands of decayed sums of outer products (lightning attention, gated linear
attention) and the gated linear recurrent unit.

Conventions of ``mixer_ops``: every wrapper has a PyTorch branch with identical semantics (CPU execution), CUDA tensors always
take the kernel; ``seq_info`` is int32 ``[n_seqs, 4]`` = (first row, rows, tokens seen, state slot).
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ....native import lib as _lib
from .mixer_ops import _dt, _out_rows, _rows

_lib.register({
    "sxb_silu_columns": "p" "l" "p" "ii" "i" "p",
    "sxb_decay_prepare": "p" "l" "iiii" "pppp" "iiii" "ff" "i" "p",
    "sxb_lru_gates": "pppppp" "iii" "i" "p",
    "sxb_lru_scan": "ppp" "l" "pp" "l" "pppp" "l" "iii" "f" "i" "i" "p",
})


def silu_columns(x: torch.Tensor) -> torch.Tensor:
    """fp32 ``silu(x)`` of rows ``[T, C]`` (a column slice is fine)."""
    T, C = x.shape
    if x.is_cuda:
        out = torch.empty(T, C, dtype=torch.float32, device=x.device)
        _lib.call("sxb_silu_columns", _rows(x).data_ptr(), x.stride(0), out.data_ptr(), T, C, _dt(x), _lib.stream_ptr())
        return out
    return torch.nn.functional.silu(x.float())


def decay_prepare(proj: torch.Tensor, q0: int, k0: int, v0: int, low0: int, w2: torch.Tensor, bias: torch.Tensor, Hn: int, Hv: int,
                  qscale: float, tau: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """From projection rows (q, k: ``Hn`` columns at ``q0`` / ``k0``, v: ``Hv`` at ``v0``, ``w2.shape[0]`` at ``low0``): fp32
    ``[T, 2 Hn + Hv] = q * qscale | k | v`` and the decay ``sigmoid(low w2 + bias)^(1 / tau)`` fp32 ``[T, Hn]``.  ``w2`` ``[rank,
    Hn]`` in the projection's dtype, ``bias`` fp32 ``[Hn]``; the product is 32-bit."""
    T, rank = proj.shape[0], w2.shape[0]
    if proj.is_cuda:
        if w2.dtype != proj.dtype or bias.dtype != torch.float32 or not w2.is_contiguous():
            raise ValueError("w2 is contiguous in the projection's dtype, the bias is fp32")
        buf = torch.empty(T, 2 * Hn + Hv, dtype=torch.float32, device=proj.device)
        decay = torch.empty(T, Hn, dtype=torch.float32, device=proj.device)
        _lib.call("sxb_decay_prepare", _rows(proj).data_ptr(), proj.stride(0), int(q0), int(k0), int(v0), int(low0), w2.data_ptr(),
                  bias.data_ptr(), buf.data_ptr(), decay.data_ptr(), T, Hn, Hv, rank, float(qscale), 1.0 / float(tau),
                  _dt(proj), _lib.stream_ptr())
        return buf, decay
    x = proj.float()
    z = x[:, low0: low0 + rank] @ w2.float() + bias
    buf = torch.cat([x[:, q0: q0 + Hn] * qscale, x[:, k0: k0 + Hn], x[:, v0: v0 + Hv]], dim=1)
    return buf, torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def lru_gates(u: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, rate: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Gates of the linear recurrent unit from its filtered input ``u`` fp32 ``[T, N]``.  With ``w`` ``[2, blocks, S, S]``
    (``[gate, part, in, out]``, ``blocks * S = N``), ``bias`` fp32 ``[2, N]`` and ``rate`` fp32 ``[N]`` (not positive): ``r, i =
    sigmoid(u_b w[gate][b] + bias[gate])``, returns fp32 ``(a, g)`` ``[T, N]`` with ``a = exp(rate r)``, ``g = sqrt(1 - a^2) i u``.
    Products and sums are 32-bit."""
    T, N = u.shape
    blocks, S = w.shape[1], w.shape[2]
    if u.is_cuda:
        if u.dtype != torch.float32 or not (u.is_contiguous() and w.is_contiguous() and bias.is_contiguous()):
            raise ValueError("u is contiguous fp32, weights and bias are contiguous")
        a, g = torch.empty_like(u), torch.empty_like(u)
        _lib.call("sxb_lru_gates", u.data_ptr(), w.data_ptr(), bias.data_ptr(), rate.data_ptr(), a.data_ptr(), g.data_ptr(), T, N,
                  blocks, _dt(w), _lib.stream_ptr())
        return a, g
    z = torch.einsum("tbk,gbkn->gtbn", u.view(T, blocks, S), w.float()).reshape(2, T, N) + bias[:, None, :]
    log_a = rate * torch.sigmoid(z[0])
    return torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * torch.sigmoid(z[1]) * u


def lru_scan(a: torch.Tensor, g: torch.Tensor, y: torch.Tensor, y_bias: torch.Tensor, x: torch.Tensor, state: torch.Tensor,
             conv_state: Optional[torch.Tensor], seq_info: torch.Tensor, single_rows: bool, out: Optional[torch.Tensor] = None,
             out_scale: float = 1.0) -> torch.Tensor:
    """Per sequence and channel, rows in order: ``s <- a s + g``; result ``s * gelu_tanh(y + y_bias) * out_scale`` ``[T, N]`` in
    ``y``'s dtype (into ``out``, which may be a column slice).  ``state`` fp32 ``[slots, N]`` is read (zero for a sequence that has
    seen no token) and written back; ``conv_state`` ``[slots, keep, N]`` (None: nothing is carried) is left holding each sequence's
    last ``keep`` rows of (carried rows, this batch's rows of ``x``).  ``y``, ``x``: column slices of the projection."""
    T, N = a.shape
    keep = 0 if conv_state is None else conv_state.shape[1]
    if a.is_cuda:
        out = _out_rows(out, T, N, y.dtype, a.device)
        if y.dtype != x.dtype or y_bias.dtype != y.dtype:
            raise ValueError("y, x and the bias share the activation dtype")
        _lib.call("sxb_lru_scan", a.data_ptr(), g.data_ptr(), _rows(y).data_ptr(), y.stride(0), y_bias.data_ptr(),
                  _rows(x).data_ptr(), x.stride(0), state.data_ptr(), _lib.ptr(conv_state), seq_info.data_ptr(), out.data_ptr(),
                  out.stride(0), seq_info.shape[0], N, keep, float(out_scale), int(single_rows), _dt(y), _lib.stream_ptr())
        return out
    res = torch.empty(T, N)
    for first, rows, seen, slot in seq_info.tolist():
        s = state[slot].clone() if seen > 0 else torch.zeros(N)
        for t in range(first, first + rows):
            s = a[t] * s + g[t]
            res[t] = s
        state[slot] = s
        if keep:
            hist = torch.zeros_like(conv_state[slot])
            have = min(seen, keep)
            if have:
                hist[keep - have:] = conv_state[slot, keep - have:]
            conv_state[slot] = torch.cat([hist, x[first: first + rows].to(conv_state.dtype)], dim=0)[-keep:]
    gate = torch.nn.functional.gelu(y.float() + y_bias.float(), approximate="tanh")
    return _out_rows(out, T, N, y.dtype, a.device).copy_(res * gate * out_scale)
