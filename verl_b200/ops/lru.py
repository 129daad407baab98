"""Gated linear recurrent unit over ragged batches with per-sequence state (``csrc/linear_recurrence.cu``)."""

from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _lib
from .gemm import gemm


def rglru(proj: torch.Tensor, conv_w: torch.Tensor, conv_b: torch.Tensor, gates: torch.Tensor, gates_b: torch.Tensor,
          lam: torch.Tensor, ring: torch.Tensor, state: torch.Tensor, cu_q: torch.Tensor, seq_lens: torch.Tensor,
          slots: torch.Tensor, max_q: int, power: float = 8.0, singles: int = 0, impl: str = "auto") -> torch.Tensor:
    """Mixer output before its last projection, [T, W].

    ``proj`` [T, gelu branch (W) | recurrent branch (W) (| padding)] of ragged sequences (``cu_q`` [B + 1]); ``seq_lens`` [B] =
    tokens of each sequence up to and including these; ``slots`` [B] int32 = state slot (< 0: padding row). u = causal
    convolution (``conv_w`` [W, taps], ``conv_b`` [W]) of the recurrent branch; r and i = sigmoid of the block-wise projections
    ``gates`` [2 * blocks, n, n] (decay, then input; [out, in]) with the biases ``gates_b`` [2 * blocks, n];
    a = exp(-``power`` * softplus(``lam``) * r); S becomes a * S + v with v = i * u * sqrt(1 - a * a); output S * gelu(gelu branch).
    Gates, decay and state are fp32. Updates in place ``state`` fp32 [slots, W] and ``ring`` [slots, taps, W] (convolution inputs, position p in
    row p % taps). Sequences that start at position 0 ignore what their slot held. ``max_q`` == 1: one token per sequence;
    otherwise the leading ``singles`` sequences have one.

    ``impl``: "tc" = gates on the tensor cores, fused with the recurrence (bf16, blocks in multiples of 8 up to 320),
    "split" = the gates' products as plain matrix products (bf16, blocks in multiples of 8), "simt" = CUDA cores, "auto" = "tc"
    where it applies, else "split"."""
    T, B, (W, taps) = proj.shape[0], slots.numel(), conv_w.shape
    n = gates.shape[1]
    if not proj.is_cuda:
        return _rglru_ref(proj, conv_w, conv_b, gates, gates_b, lam, ring, state, cu_q, seq_lens, slots, power)
    f32, dev = proj.dtype == torch.float32, proj.device
    mats = not f32 and n % 8 == 0 and proj.stride(0) % 8 == 0
    tc = mats and bool(_lib.fn("vb_rglru_tc_supported")(W, n))
    if (impl == "tc" and not tc) or (impl == "split" and not mats):
        raise ValueError(f"the recurrent unit has no form {impl!r} for width={W} block={n} in {proj.dtype}")
    tc = tc and impl in ("auto", "tc")
    split = not tc and mats and impl != "simt"
    out, u = (torch.empty((T, W), dtype=proj.dtype, device=dev) for _ in range(2))
    common = (cu_q.data_ptr(), seq_lens.data_ptr(), slots.data_ptr(), u.data_ptr())
    rc = _lib.fn("vb_rglru_conv")(proj.data_ptr(), proj.stride(0), conv_w.data_ptr(), conv_b.data_ptr(), ring.data_ptr(), *common,
                                  T, B, W, taps, int(f32), _lib.stream())
    _lib.check(rc, "vb_rglru_conv")
    ab = None if tc else torch.empty((2, T, W), dtype=torch.float32, device=dev)
    if split:
        for g in range(2 * W // n):  # decay blocks, then input blocks
            lo = g % (W // n) * n
            gemm(u[:, lo : lo + n], gates[g], out=ab[g * n // W, :, lo : lo + n])
    rc = _lib.fn("vb_rglru")(proj.data_ptr(), proj.stride(0), None if split else gates.data_ptr(), gates_b.data_ptr(),
                             lam.data_ptr(), ring.data_ptr(), state.data_ptr(), *common, _lib.ptr(ab), out.data_ptr(), T, B,
                             B if max_q == 1 else singles, W, n, taps, float(power), int(f32), int(tc),
                             _lib.status_word(dev).data_ptr(), _lib.stream())
    _lib.check(rc, "vb_rglru")
    return out


def _rglru_ref(proj, conv_w, conv_b, gates, gates_b, lam, ring, state, cu_q, seq_lens, slots, power):
    W, taps = conv_w.shape
    blocks, n = gates.shape[0] // 2, gates.shape[1]
    out = torch.zeros((proj.shape[0], W), dtype=proj.dtype)
    cu, lens, sl = cu_q.tolist(), seq_lens.tolist(), slots.tolist()
    for b in range(len(sl)):
        lo, hi, s = cu[b], cu[b + 1], sl[b]
        if hi == lo or s < 0:
            continue
        start = lens[b] - (hi - lo)
        y, x = proj[lo:hi, :W].float(), proj[lo:hi, W : 2 * W].float()
        past = [ring[s, p % taps].float() if p >= 0 else torch.zeros(W) for p in range(start - taps + 1, start)]
        inp = torch.cat([torch.stack(past), x]) if past else x
        u = sum(inp[j : j + hi - lo] * conv_w[:, j].float() for j in range(taps)) + conv_b.float()
        u = u.to(proj.dtype).float()
        for p in range(max(start, lens[b] - taps), lens[b]):
            ring[s, p % taps] = proj[lo + p - start, W : 2 * W]
        g = torch.einsum("tbi,cboi->tcbo", u.view(-1, blocks, n), gates.float().view(2, blocks, n, n))
        r, i = torch.sigmoid(g + gates_b.view(2, blocks, n)).flatten(2).unbind(1)
        log_a = -power * r * F.softplus(lam.float(), threshold=60.0)
        a, v = log_a.exp(), torch.sqrt(-torch.expm1(2 * log_a)) * i * u
        S = state[s] if start > 0 else torch.zeros_like(state[s])
        for t in range(hi - lo):
            S = a[t] * S + v[t]
            out[lo + t] = (S * F.gelu(y[t], approximate="tanh")).to(out.dtype)
        state[s] = S
    return out
