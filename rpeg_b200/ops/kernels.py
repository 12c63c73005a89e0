"""Thin tensor-level wrappers over the native sm_100a kernels (no autograd here).

Every wrapper validates shapes/dtypes/contiguity on the host, passes raw device pointers plus the
current CUDA stream to the C ABI in ``csrc/rpeg_kernels.h`` and raises on a non-zero return code.
Kernels with bounded waits share one per-device status word; ``check_status()`` reads it (this
synchronises) and raises ``KernelWaitTimeout`` if any wait ran out. With ``RPEG_CHECK_ARGS=1`` the wrappers also
validate the index VALUES held by tensor arguments before the launch (``ops/checked.py``).
"""
from __future__ import annotations

import ctypes
import math

import torch

from . import checked as _chk
from ._lib import check, lib

KV_PAGE = 64
MAX_PEERS = 8
_status: dict[int, torch.Tensor] = {}


class KernelWaitTimeout(RuntimeError):
    """A bounded device-side wait (mbarrier or peer flag) ran out; the kernel returned early."""


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def status_word(device: torch.device | None = None) -> torch.Tensor:
    dev = torch.cuda.current_device() if device is None else torch.device(device).index or 0
    if dev not in _status:
        _status[dev] = torch.zeros(4, dtype=torch.int32, device=f"cuda:{dev}")
    return _status[dev]


def check_status() -> None:
    """Read the status word of the current device (synchronises) and raise if a wait timed out."""
    st = status_word()
    vals = st.tolist()
    if vals[0] != 0:
        st.zero_()
        raise KernelWaitTimeout(f"device wait timed out: code={vals[0]} where={vals[1]} block={vals[2]} extra={vals[3]}")


def _req(t: torch.Tensor, dtype: torch.dtype, name: str) -> None:
    if not t.is_cuda or t.dtype != dtype:
        raise TypeError(f"{name}: expected a CUDA {dtype} tensor, got {t.dtype} on {t.device}")


# --------------------------------------------------------------------------- GEMM
GEMM_CHAIN = 0x1000     # flag in the tile-width argument of rpeg_gemm_bf16: launch as a programmatic dependent


def gemm(a: torch.Tensor, b: torch.Tensor, *, trans_a: bool = False, trans_b: bool = False,
         out: torch.Tensor | None = None, out_dtype: torch.dtype = torch.bfloat16, accumulate: bool = False,
         bn: int = 0, workspace: torch.Tensor | None = None, gate: tuple | None = None, chain: bool = False) -> torch.Tensor:
    """``C[M,N] = op(a) @ op(b).T`` on tcgen05 tensor cores with fp32 accumulation.

    ``gate = (flags uint32 tensor, min_version, timeout_s)`` holds back every operand load until all words of
    ``flags`` reached ``min_version`` (weights being pushed into ``b`` by other GPUs); the wait is bounded.

    ``a`` is ``[M,K]`` (or ``[K,M]`` with ``trans_a``); ``b`` is ``[N,K]`` — the ``[out,in]`` layout
    of a linear weight — or ``[K,N]`` with ``trans_b``. Rows may be strided (last dim contiguous).
    ``out_dtype=float32, accumulate=True`` adds into ``out`` (used for weight-gradient accumulation).
    ``workspace`` (fp32 scratch) lets skinny problems (M <= 256, e.g. decode) run split-K so every SM
    streams part of the weight matrix. ``chain``: the call is a link of a decode step whose kernels are launched as
    programmatic dependents (``b`` is a weight matrix that no kernel of the step writes): the grid may start under the
    previous kernel's tail and fetch weight tiles before that kernel has finished.
    """
    _req(a, torch.bfloat16, "a")
    _req(b, torch.bfloat16, "b")
    if a.dim() != 2 or b.dim() != 2 or a.stride(1) != 1 or b.stride(1) != 1:
        raise ValueError("gemm operands must be 2-D with a contiguous last dimension")
    M, K = (a.shape[1], a.shape[0]) if trans_a else (a.shape[0], a.shape[1])
    N, Kb = (b.shape[1], b.shape[0]) if trans_b else (b.shape[0], b.shape[1])
    if K != Kb:
        raise ValueError(f"gemm inner dimensions differ: {K} vs {Kb}")
    if out is None:
        if accumulate:
            raise ValueError("accumulate=True needs an `out` tensor")
        out = torch.empty((M, N), dtype=out_dtype, device=a.device)
    else:
        out_dtype = out.dtype
        if out.shape != (M, N) or out.stride(1) != 1:
            raise ValueError("gemm out has the wrong shape or a strided last dimension")
    if out_dtype not in (torch.bfloat16, torch.float32):
        raise TypeError("gemm output must be bf16 or fp32")
    if M == 0 or N == 0:
        return out
    if gate is not None:
        flags, min_version, timeout_s = gate
        rc = lib().rpeg_gemm_bf16_gated(a.data_ptr(), b.data_ptr(), out.data_ptr(), M, N, K, a.stride(0), b.stride(0),
                                        out.stride(0), int(trans_a), int(trans_b), int(out_dtype == torch.float32),
                                        int(accumulate), bn, _ptr(workspace), 0 if workspace is None else workspace.numel(),
                                        flags.data_ptr(), flags.numel(), int(min_version), int(timeout_s * 1e9),
                                        status_word(a.device).data_ptr(), _stream())
        check(rc, "rpeg_gemm_bf16_gated")
        return out
    rc = lib().rpeg_gemm_bf16(a.data_ptr(), b.data_ptr(), out.data_ptr(), M, N, K, a.stride(0), b.stride(0),
                              out.stride(0), int(trans_a), int(trans_b), int(out_dtype == torch.float32),
                              int(accumulate), bn | (GEMM_CHAIN if chain else 0), _ptr(workspace), 0 if workspace is None else workspace.numel(),
                              status_word(a.device).data_ptr(), _stream())
    check(rc, "rpeg_gemm_bf16")
    return out


def gemm_swiglu(x: torch.Tensor, w_gate_up: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``silu(x @ W_gate.T) * (x @ W_up.T)`` with ``w_gate_up = [W_gate; W_up]`` of shape ``[2f, K]``: the gated MLP's first
    linear with the activation applied to the fp32 accumulators in the GEMM epilogue, so the ``[M, 2f]`` pre-activation is
    never written. ``f`` must be a multiple of 128 (callers fall back to ``gemm`` + ``swiglu_fwd`` otherwise)."""
    _req(x, torch.bfloat16, "x")
    _req(w_gate_up, torch.bfloat16, "w_gate_up")
    M, Kd = x.shape
    f = w_gate_up.shape[0] // 2
    if w_gate_up.shape[1] != Kd or x.stride(1) != 1 or w_gate_up.stride(1) != 1:
        raise ValueError("gemm_swiglu: x [M, K] and w_gate_up [2f, K] must share K and be contiguous in it")
    if f % 128:
        raise ValueError("gemm_swiglu needs d_ff to be a multiple of 128")
    if out is None:
        out = torch.empty((M, f), dtype=torch.bfloat16, device=x.device)
    if M == 0:
        return out
    check(lib().rpeg_gemm_swiglu(x.data_ptr(), w_gate_up.data_ptr(), out.data_ptr(), M, f, Kd, x.stride(0), w_gate_up.stride(0),
                                 out.stride(0), status_word(x.device).data_ptr(), _stream()), "rpeg_gemm_swiglu")
    return out


def set_pdl(on: bool) -> None:
    """Programmatic dependent launches for the kernels launched from now on (a captured graph keeps its setting)."""
    lib().rpeg_set_pdl(int(bool(on)))


def publish_version(flag_ptrs, word: int, version: int) -> None:
    """After the copies queued on this stream: store ``version`` into word ``word`` of every flag array in
    ``flag_ptrs`` (device pointers, local or peer) with system-scope release."""
    arr = (ctypes.c_void_p * len(flag_ptrs))(*[int(p) for p in flag_ptrs])
    check(lib().rpeg_publish_version(arr, len(flag_ptrs), int(word), int(version), _stream()), "rpeg_publish_version")


def wait_flags(flags: torch.Tensor, min_version: int, timeout_s: float, result: torch.Tensor) -> None:
    """``result[0] = 1`` (int32) once all words of ``flags`` reached ``min_version``, ``0`` if ``timeout_s`` ran out first."""
    check(lib().rpeg_wait_flags(flags.data_ptr(), flags.numel(), int(min_version), int(timeout_s * 1e9), result.data_ptr(), _stream()),
          "rpeg_wait_flags")


# --------------------------------------------------------------------------- norm / rope / swiglu
def rmsnorm_fwd(x: torch.Tensor, w: torch.Tensor, eps: float, residual: torch.Tensor | None = None,
                want_sum: bool = False):
    """Returns ``(y, rstd, h)``: ``h = x + residual`` (only when asked for), ``y = rmsnorm(h) * w``."""
    _req(x, torch.bfloat16, "x")
    T, d = x.shape
    y = torch.empty_like(x)
    rstd = torch.empty(T, dtype=torch.float32, device=x.device)
    h = torch.empty_like(x) if (residual is not None and want_sum) else None
    check(lib().rpeg_rmsnorm_fwd(x.data_ptr(), _ptr(residual), w.data_ptr(), _ptr(h), y.data_ptr(),
                                 rstd.data_ptr(), T, d, eps, _stream()), "rpeg_rmsnorm_fwd")
    return y, rstd, h


def rmsnorm_bwd(dy: torch.Tensor, x: torch.Tensor, w: torch.Tensor, rstd: torch.Tensor, dw: torch.Tensor,
                dres_in: torch.Tensor | None = None) -> torch.Tensor:
    """``dx`` of ``y = rmsnorm(x) * w`` (+ ``dres_in`` added in); accumulates ``dw`` (fp32) in place."""
    T, d = x.shape
    dx = torch.empty_like(x)
    check(lib().rpeg_rmsnorm_bwd(dy.data_ptr(), x.data_ptr(), w.data_ptr(), rstd.data_ptr(), _ptr(dres_in),
                                 dx.data_ptr(), dw.data_ptr(), T, d, _stream()), "rpeg_rmsnorm_bwd")
    return dx


def rope_tables(max_pos: int, head_dim: int, theta: float, device, scaling_factor: float = 1.0,
                original_max_pos: int = 8192) -> tuple[torch.Tensor, torch.Tensor]:
    """cos/sin tables ``[max_pos, head_dim/2]``. ``scaling_factor > 1`` applies the llama3 frequency
    scaling (low_freq_factor 1, high_freq_factor 4): long wavelengths are divided by the factor, short
    ones kept, the band in between interpolated."""
    inv = 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=torch.float64) / head_dim))
    if scaling_factor > 1.0:
        low, high = 1.0, 4.0
        wavelen = 2 * math.pi / inv
        smooth = ((original_max_pos / wavelen) - low) / (high - low)
        mid = (1 - smooth) * inv / scaling_factor + smooth * inv
        inv = torch.where(wavelen > original_max_pos / low, inv / scaling_factor,
                          torch.where(wavelen < original_max_pos / high, inv, mid))
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * inv[None, :]
    return ang.cos().float().to(device).contiguous(), ang.sin().float().to(device).contiguous()


def rope_(buf: torch.Tensor, pos: torch.Tensor, cos_t: torch.Tensor, sin_t: torch.Tensor, col0: int, nheads: int,
          head_dim: int, backward: bool = False) -> None:
    """Rotate ``nheads`` heads starting at column ``col0`` of the 2-D ``buf`` in place."""
    _req(buf, torch.bfloat16, "buf")
    if _chk.active():
        _chk.rope("rpeg_rope", pos, buf.shape[0], cos_t)
    check(lib().rpeg_rope(buf.data_ptr(), pos.data_ptr(), cos_t.data_ptr(), sin_t.data_ptr(), buf.shape[0],
                          buf.stride(0), col0, nheads, head_dim, int(backward), _stream()), "rpeg_rope")


def headnorm_fwd_(buf: torch.Tensor, col0: int, nheads: int, head_dim: int, w: torch.Tensor, eps: float,
                  want_rstd: bool = True) -> torch.Tensor | None:
    """RMS-normalise every (row, head) slice of ``buf[:, col0 : col0 + nheads*head_dim]`` in place with the
    shared weight ``w [head_dim]`` (QK-norm). Returns ``rstd [T, nheads]`` for the backward pass."""
    _req(buf, torch.bfloat16, "buf")
    T = buf.shape[0]
    rstd = torch.empty((T, nheads), dtype=torch.float32, device=buf.device) if want_rstd else None
    check(lib().rpeg_headnorm_fwd(buf.data_ptr(), buf.stride(0), col0, nheads, head_dim, w.data_ptr(), _ptr(rstd), T, eps,
                                  _stream()), "rpeg_headnorm_fwd")
    return rstd


def headnorm_bwd_(dbuf: torch.Tensor, x_pre: torch.Tensor, col0: int, nheads: int, head_dim: int, w: torch.Tensor,
                  rstd: torch.Tensor, dw: torch.Tensor) -> None:
    """In place on ``dbuf`` (dy -> dx) for the slices normalised by ``headnorm_fwd_``; ``x_pre`` holds the
    pre-norm values in the same column layout; ``dw [head_dim]`` fp32 is accumulated."""
    check(lib().rpeg_headnorm_bwd(dbuf.data_ptr(), dbuf.stride(0), x_pre.data_ptr(), x_pre.stride(0), col0, nheads, head_dim,
                                  w.data_ptr(), rstd.data_ptr(), dw.data_ptr(), dbuf.shape[0], _stream()), "rpeg_headnorm_bwd")


def swiglu_fwd(gu: torch.Tensor) -> torch.Tensor:
    T, f2 = gu.shape
    out = torch.empty((T, f2 // 2), dtype=gu.dtype, device=gu.device)
    check(lib().rpeg_swiglu_fwd(gu.data_ptr(), out.data_ptr(), T, f2 // 2, _stream()), "rpeg_swiglu_fwd")
    return out


def swiglu_bwd(gu: torch.Tensor, dout: torch.Tensor) -> torch.Tensor:
    T, f2 = gu.shape
    dgu = torch.empty_like(gu)
    check(lib().rpeg_swiglu_bwd(gu.data_ptr(), dout.data_ptr(), dgu.data_ptr(), T, f2 // 2, _stream()),
          "rpeg_swiglu_bwd")
    return dgu


def add_bf16(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    out = torch.empty_like(a) if out is None else out
    check(lib().rpeg_add_bf16(a.data_ptr(), b.data_ptr(), out.data_ptr(), a.numel(), _stream()), "rpeg_add_bf16")
    return out


def embed_fwd(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    _req(ids, torch.int32, "ids")
    if _chk.active():
        _chk.embed("rpeg_embed_fwd", ids, table.shape[0])
    if out is None:
        out = torch.empty((ids.numel(), table.shape[1]), dtype=table.dtype, device=table.device)
    elif out.shape != (ids.numel(), table.shape[1]) or not out.is_contiguous() or out.dtype != table.dtype:
        raise ValueError("embed_fwd: `out` must be a contiguous [tokens, d] tensor of the table's dtype")
    check(lib().rpeg_embed_fwd(ids.data_ptr(), table.data_ptr(), out.data_ptr(), ids.numel(), table.shape[1],
                               _stream()), "rpeg_embed_fwd")
    return out


def embed_bwd(ids: torch.Tensor, dout: torch.Tensor, dtable: torch.Tensor) -> None:
    if _chk.active():
        _chk.embed("rpeg_embed_bwd", ids, dtable.numel() // dout.shape[1])
    check(lib().rpeg_embed_bwd(ids.data_ptr(), dout.data_ptr(), dtable.data_ptr(), ids.numel(), dout.shape[1],
                               _stream()), "rpeg_embed_bwd")


# --------------------------------------------------------------------------- losses
def token_logprob_fwd(logits: torch.Tensor, targets: torch.Tensor, temperature: float = 1.0):
    _req(logits, torch.bfloat16, "logits")
    _req(targets, torch.int32, "targets")
    T, V = logits.shape
    logp = torch.empty(T, dtype=torch.float32, device=logits.device)
    lse = torch.empty(T, dtype=torch.float32, device=logits.device)
    check(lib().rpeg_token_logprob_fwd(logits.data_ptr(), targets.data_ptr(), logp.data_ptr(), lse.data_ptr(), T, V,
                                       logits.stride(0), temperature, _stream()), "rpeg_token_logprob_fwd")
    return logp, lse


def token_logprob_bwd_(logits: torch.Tensor, targets: torch.Tensor, lse: torch.Tensor, coef: torch.Tensor,
                       temperature: float = 1.0) -> torch.Tensor:
    """Overwrite ``logits`` with ``d loss / d logits`` given ``coef = d loss / d logp`` per row."""
    T, V = logits.shape
    check(lib().rpeg_token_logprob_bwd(logits.data_ptr(), targets.data_ptr(), lse.data_ptr(), coef.data_ptr(), T, V,
                                       logits.stride(0), temperature, _stream()), "rpeg_token_logprob_bwd")
    return logits


def token_entropy(logits: torch.Tensor, lse: torch.Tensor, temperature: float = 1.0) -> torch.Tensor:
    """Entropy of every row's softmax (at ``temperature``) from the logits and the log-sum-exp ``token_logprob_fwd`` returned."""
    _req(logits, torch.bfloat16, "logits")
    T, V = logits.shape
    ent = torch.empty(T, dtype=torch.float32, device=logits.device)
    check(lib().rpeg_token_entropy(logits.data_ptr(), lse.data_ptr(), ent.data_ptr(), T, V, logits.stride(0), temperature, _stream()),
          "rpeg_token_entropy")
    return ent


def token_logprob_entropy_bwd_(logits: torch.Tensor, targets: torch.Tensor, lse: torch.Tensor, coef: torch.Tensor, ent: torch.Tensor,
                               ecoef: torch.Tensor, temperature: float = 1.0) -> torch.Tensor:
    """Overwrite ``logits`` with ``d loss / d logits`` given ``coef = d loss / d logp`` and ``ecoef = d loss / d entropy`` per row."""
    T, V = logits.shape
    check(lib().rpeg_token_logprob_entropy_bwd(logits.data_ptr(), targets.data_ptr(), lse.data_ptr(), coef.data_ptr(), ent.data_ptr(),
                                               ecoef.data_ptr(), T, V, logits.stride(0), temperature, _stream()),
          "rpeg_token_logprob_entropy_bwd")
    return logits


def policy_loss(lp, old_lp, ref_lp, adv, mask, clip_eps: float, kl_coef: float, inv_denom: float):
    """Clipped PPO/GRPO loss. Returns ``(coef, acc)``; ``acc = [loss, sum(lp-ref), n_clipped, sum(old-lp)]``."""
    coef = torch.empty_like(lp)
    acc = torch.zeros(4, dtype=torch.float32, device=lp.device)
    check(lib().rpeg_policy_loss(lp.data_ptr(), old_lp.data_ptr(), _ptr(ref_lp), adv.data_ptr(), mask.data_ptr(),
                                 coef.data_ptr(), acc.data_ptr(), lp.numel(), clip_eps, kl_coef, inv_denom,
                                 _stream()), "rpeg_policy_loss")
    return coef, acc


def masked_rowsum(x: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    B, T = x.shape
    out = torch.empty(B, dtype=torch.float32, device=x.device)
    check(lib().rpeg_masked_rowsum(x.data_ptr(), mask.data_ptr(), out.data_ptr(), B, T, _stream()),
          "rpeg_masked_rowsum")
    return out


def dpo_loss(pi_seq: torch.Tensor, ref_seq: torch.Tensor, beta: float):
    """Rows interleaved (chosen, rejected). Returns ``(seq_coef, acc)``; ``acc = [loss, n_correct, margin]``."""
    P = pi_seq.numel() // 2
    seq_coef = torch.empty_like(pi_seq)
    acc = torch.zeros(4, dtype=torch.float32, device=pi_seq.device)
    check(lib().rpeg_dpo_loss(pi_seq.data_ptr(), ref_seq.data_ptr(), seq_coef.data_ptr(), acc.data_ptr(), P, beta,
                              _stream()), "rpeg_dpo_loss")
    return seq_coef, acc


def expand_seq_coef(seq_coef: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    B, T = mask.shape
    coef = torch.empty_like(mask)
    check(lib().rpeg_expand_seq_coef(seq_coef.data_ptr(), mask.data_ptr(), coef.data_ptr(), B, T, _stream()),
          "rpeg_expand_seq_coef")
    return coef


def value_loss(v, ret, mask, inv_denom: float):
    dv = torch.empty_like(v)
    acc = torch.zeros(4, dtype=torch.float32, device=v.device)
    check(lib().rpeg_value_loss(v.data_ptr(), ret.data_ptr(), mask.data_ptr(), dv.data_ptr(), acc.data_ptr(),
                                v.numel(), inv_denom, _stream()), "rpeg_value_loss")
    return dv, acc


def gae(old_lp, ref_lp, values, mask, scores, beta: float, gamma: float, lam: float, whiten: bool):
    B, T = values.shape
    adv = torch.empty_like(values)
    ret = torch.empty_like(values)
    check(lib().rpeg_gae(old_lp.data_ptr(), _ptr(ref_lp), values.data_ptr(), mask.data_ptr(), scores.data_ptr(),
                         adv.data_ptr(), ret.data_ptr(), B, T, beta, gamma, lam, int(whiten), _stream()), "rpeg_gae")
    return adv, ret


def group_advantage(rewards: torch.Tensor, group: int) -> torch.Tensor:
    out = torch.empty_like(rewards)
    check(lib().rpeg_group_advantage(rewards.data_ptr(), out.data_ptr(), rewards.numel() // group, group, _stream()),
          "rpeg_group_advantage")
    return out


def sample(logits: torch.Tensor, temperature: float, greedy: bool, seed: int, forced: torch.Tensor | None = None,
           token_out: torch.Tensor | None = None, logp_out: torch.Tensor | None = None,
           seed_offset: torch.Tensor | None = None, top_k: int = 0, top_p: float = 1.0):
    """Gumbel-max sample (or argmax) per row with its log-prob; ``seed_offset`` is an int64 device
    scalar mixed into the seed so graph replays draw fresh noise. ``top_k`` / ``top_p`` restrict the draw to
    the k most likely tokens / the smallest set reaching mass ``top_p``; the log-prob is under the full softmax."""
    B, V = logits.shape
    tok = torch.empty(B, dtype=torch.int32, device=logits.device) if token_out is None else token_out
    lp = torch.empty(B, dtype=torch.float32, device=logits.device) if logp_out is None else logp_out
    if logits.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"sample: logits must be bf16 or fp32, got {logits.dtype}")
    f32 = logits.dtype == torch.float32
    if not greedy and (0 < top_k < V or top_p < 1.0):
        check((lib().rpeg_sample_filtered_f32 if f32 else lib().rpeg_sample_filtered)(logits.data_ptr(), B, V, logits.stride(0), temperature, int(top_k), float(top_p),
                                         seed & 0xFFFFFFFFFFFFFFFF, _ptr(seed_offset), _ptr(forced), tok.data_ptr(), lp.data_ptr(),
                                         _stream()), "rpeg_sample_filtered")
        return tok, lp
    check((lib().rpeg_sample_f32 if f32 else lib().rpeg_sample)(logits.data_ptr(), B, V, logits.stride(0), temperature, int(greedy),
                            seed & 0xFFFFFFFFFFFFFFFF, _ptr(seed_offset), _ptr(forced), tok.data_ptr(), lp.data_ptr(),
                            _stream()),
          "rpeg_sample")
    return tok, lp


def head_gemv(h: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None) -> torch.Tensor:
    T, d = h.shape
    out = torch.empty(T, dtype=torch.float32, device=h.device)
    check(lib().rpeg_head_gemv(h.data_ptr(), w.data_ptr(), _ptr(bias), out.data_ptr(), T, d, _stream()),
          "rpeg_head_gemv")
    return out


def head_gemv_bwd(h, w, dout, dw: torch.Tensor, db: torch.Tensor | None) -> torch.Tensor:
    T, d = h.shape
    dh = torch.empty_like(h)
    check(lib().rpeg_head_gemv_bwd(h.data_ptr(), w.data_ptr(), dout.data_ptr(), dh.data_ptr(), dw.data_ptr(),
                                   _ptr(db), T, d, _stream()), "rpeg_head_gemv_bwd")
    return dh


# --------------------------------------------------------------------------- optimizer
def adamw_(p32, m, v, grad, w16, *, lr, beta1=0.9, beta2=0.999, eps=1e-8, wd=0.0, step=1, grad_scale=1.0,
           sumsq: torch.Tensor | None = None, max_norm: float = 0.0) -> None:
    n = p32.numel()
    check(lib().rpeg_adamw(p32.data_ptr(), m.data_ptr(), v.data_ptr(), grad.data_ptr(), w16.data_ptr(), n, lr,
                           beta1, beta2, eps, wd, step, grad_scale, _ptr(sumsq),
                           0 if sumsq is None else sumsq.numel(), max_norm, _stream()), "rpeg_adamw")


def sumsq(x: torch.Tensor, out: torch.Tensor) -> None:
    check(lib().rpeg_sumsq(x.data_ptr(), x.numel(), out.data_ptr(), _stream()), "rpeg_sumsq")


# --------------------------------------------------------------------------- split-K partials and their consumers
class Partials:
    """fp32 split-K partial products ``[splits, M, N]`` living in a workspace: ``sum(0)`` is the GEMM result."""

    __slots__ = ("buf", "splits", "M", "N")

    def __init__(self, buf: torch.Tensor, splits: int, M: int, N: int):
        self.buf, self.splits, self.M, self.N = buf, splits, M, N

    @property
    def stride(self) -> int:
        return self.M * self.N

    def columns(self, c0: int) -> "Partials":
        """The same partials seen from column ``c0`` on (the row pitch stays ``N``)."""
        return Partials(self.buf[c0:], self.splits, self.M, self.N)

    def reduce(self) -> torch.Tensor:
        return self.buf[: self.splits * self.stride].view(self.splits, self.M, self.N).sum(0)


def gemm_partials(a: torch.Tensor, b: torch.Tensor, workspace: torch.Tensor) -> Partials:
    """``a [M,K] @ b [N,K]^T`` for skinny ``M`` (decode): returns the split-K partials in ``workspace`` instead
    of reducing them; ``rmsnorm_fwd_partials`` / ``swiglu_fwd_partials`` / ``rope_kv_append_partials_`` add them
    up while loading. The split count is fixed by the shapes, so the call is CUDA-graph friendly."""
    _req(a, torch.bfloat16, "a")
    _req(b, torch.bfloat16, "b")
    M, Kd = a.shape
    N = b.shape[0]
    splits = ctypes.c_int(1)
    check(lib().rpeg_gemm_bf16_partials(a.data_ptr(), b.data_ptr(), M, N, Kd, a.stride(0), b.stride(0), workspace.data_ptr(),
                                        workspace.numel(), ctypes.byref(splits), status_word(a.device).data_ptr(), _stream()),
          "rpeg_gemm_bf16_partials")
    return Partials(workspace, int(splits.value), M, N)


def rmsnorm_fwd_partials(parts: Partials, w: torch.Tensor, eps: float, residual: torch.Tensor | None = None,
                         want_sum: bool = False):
    """``y = rmsnorm(sum(parts) [+ residual]) * w``; with ``want_sum`` also returns the bf16 sum (the new residual stream)."""
    y = torch.empty((parts.M, parts.N), dtype=torch.bfloat16, device=w.device)
    h = torch.empty_like(y) if want_sum else None
    check(lib().rpeg_rmsnorm_fwd_partials(parts.buf.data_ptr(), parts.splits, parts.stride, _ptr(residual), w.data_ptr(), _ptr(h),
                                          y.data_ptr(), parts.M, parts.N, eps, _stream()), "rpeg_rmsnorm_fwd_partials")
    return y, h


def swiglu_fwd_partials(parts: Partials) -> torch.Tensor:
    f = parts.N // 2
    out = torch.empty((parts.M, f), dtype=torch.bfloat16, device=parts.buf.device)
    check(lib().rpeg_swiglu_fwd_partials(parts.buf.data_ptr(), parts.splits, parts.stride, out.data_ptr(), parts.M, f, _stream()),
          "rpeg_swiglu_fwd_partials")
    return out


def rope_kv_append_partials_(parts: Partials, qkv: torch.Tensor, q_col0, k_col0, v_col0, seq_id, pos, cos_t, sin_t, page_table,
                             kcache, vcache, n_heads, n_kv_heads, head_dim) -> None:
    """Sum the partials of a QKV projection, rotate q and k, store q into ``qkv`` (bf16, the attention
    kernel's query input) and k, v into the paged cache."""
    if _chk.active():
        _chk.kv_append("rpeg_rope_kv_append_partials", parts.M, seq_id, pos, page_table, kcache, n_kv_heads, head_dim, cos_t)
    check(lib().rpeg_rope_kv_append_partials(parts.buf.data_ptr(), parts.splits, parts.stride, qkv.data_ptr(), qkv.stride(0), q_col0,
                                             k_col0, v_col0, seq_id.data_ptr(), pos.data_ptr(), cos_t.data_ptr(), sin_t.data_ptr(),
                                             page_table.data_ptr(), page_table.stride(0), kcache.data_ptr(), vcache.data_ptr(),
                                             parts.M, n_heads, n_kv_heads, head_dim, _stream()), "rpeg_rope_kv_append_partials")


def scatter_rows_by_index(src: torch.Tensor, global_idx: torch.Tensor, rows_per_rank: int, dst_ptr_array, world: int) -> None:
    """Send every row of ``src [n, ...]`` to the rank owning its global index (``idx // rows_per_rank``), slot
    ``idx % rows_per_rank`` of that rank's symmetric buffer (``dst_ptr_array`` = ctypes ``void*[world]``)."""
    n = src.shape[0]
    row_bytes = src[0].numel() * src.element_size() if n else 0
    if _chk.active():
        _chk.global_rows("rpeg_scatter_rows_by_index", global_idx, rows_per_rank, world)
    check(lib().rpeg_scatter_rows_by_index(src.data_ptr(), n, row_bytes, global_idx.data_ptr(), rows_per_rank, dst_ptr_array, world,
                                           _stream()), "rpeg_scatter_rows_by_index")


# --------------------------------------------------------------------------- attention
def kv_append(qkv, k_col0, v_col0, seq_id, pos, page_table, kcache, vcache, n_kv_heads, head_dim) -> None:
    if _chk.active():
        _chk.kv_append("rpeg_kv_append", qkv.shape[0], seq_id, pos, page_table, kcache, n_kv_heads, head_dim)
    check(lib().rpeg_kv_append(qkv.data_ptr(), qkv.stride(0), k_col0, v_col0, seq_id.data_ptr(), pos.data_ptr(),
                               page_table.data_ptr(), page_table.stride(0), kcache.data_ptr(), vcache.data_ptr(),
                               qkv.shape[0], n_kv_heads, head_dim, _stream()), "rpeg_kv_append")


def rope_kv_append_(qkv, q_col0, k_col0, v_col0, seq_id, pos, cos_t, sin_t, page_table, kcache, vcache, n_heads, n_kv_heads,
                    head_dim) -> None:
    """Rotate the query and key heads of ``qkv`` in place and write the rotated keys and the values
    into the paged cache: one launch instead of two rotations and an append."""
    _req(qkv, torch.bfloat16, "qkv")
    if _chk.active():
        _chk.kv_append("rpeg_rope_kv_append", qkv.shape[0], seq_id, pos, page_table, kcache, n_kv_heads, head_dim, cos_t)
    check(lib().rpeg_rope_kv_append(qkv.data_ptr(), qkv.stride(0), q_col0, k_col0, v_col0, seq_id.data_ptr(), pos.data_ptr(),
                                    cos_t.data_ptr(), sin_t.data_ptr(), page_table.data_ptr(), page_table.stride(0),
                                    kcache.data_ptr(), vcache.data_ptr(), qkv.shape[0], n_heads, n_kv_heads, head_dim,
                                    _stream()), "rpeg_rope_kv_append")


def decode_scratch_numel(B: int, H: int, nsplit: int) -> int:
    return int(lib().rpeg_decode_attn_scratch_bytes(B, H, nsplit)) // 4


_GROUP_TC = False


def set_group_tc(on: bool) -> None:
    """Which group kernel ``paged_decode_attn(groups=...)`` uses when the caller does not say: the tcgen05 one or the
    CUDA-core one (the default)."""
    global _GROUP_TC
    _GROUP_TC = bool(on)


def paged_decode_attn(q, q_col0, kcache, vcache, page_table, seq_lens, n_heads, n_kv_heads, head_dim, scale,
                      nsplit: int = 1, scratch: torch.Tensor | None = None, out: torch.Tensor | None = None, groups=None,
                      group_tc: bool | None = None):
    """``groups = (group_rows [B, 8] int32, group_shared [B] int32, row_key0 [B] int32)``: rows that alias their first
    KV pages in groups (K samples of one prompt); the shared keys are then read once per group (``scratch`` must
    hold ``nsplit + 1`` partials per row and head). ``group_tc``: score the groups on the tensor cores (tcgen05, keys on
    the M axis) instead of the CUDA-core kernel."""
    B = q.shape[0]
    if _chk.active():
        _chk.paged_attention("rpeg_paged_decode_attn", B, seq_lens, page_table, kcache, n_kv_heads, head_dim)
    out = torch.empty((B, n_heads * head_dim), dtype=torch.bfloat16, device=q.device) if out is None else out
    if groups is not None:
        group_rows, group_shared, row_key0 = groups
        if scratch is None:
            scratch = torch.empty(decode_scratch_numel(B, n_heads, nsplit + 1), dtype=torch.float32, device=q.device)
        if _GROUP_TC if group_tc is None else group_tc:
            check(lib().rpeg_paged_decode_attn_grouped_tc(q.data_ptr(), q.stride(0), q_col0, kcache.data_ptr(), vcache.data_ptr(),
                                                          kcache.shape[0], page_table.data_ptr(), page_table.stride(0),
                                                          seq_lens.data_ptr(), out.data_ptr(), scratch.data_ptr(), B, n_heads,
                                                          n_kv_heads, head_dim, nsplit, scale, group_rows.data_ptr(),
                                                          group_shared.data_ptr(), row_key0.data_ptr(),
                                                          status_word(q.device).data_ptr(), _stream()),
                  "rpeg_paged_decode_attn_grouped_tc")
            return out
        check(lib().rpeg_paged_decode_attn_grouped(q.data_ptr(), q.stride(0), q_col0, kcache.data_ptr(), vcache.data_ptr(),
                                                   page_table.data_ptr(), page_table.stride(0), seq_lens.data_ptr(), out.data_ptr(),
                                                   scratch.data_ptr(), B, n_heads, n_kv_heads, head_dim, nsplit, scale,
                                                   group_rows.data_ptr(), group_shared.data_ptr(), row_key0.data_ptr(), _stream()),
              "rpeg_paged_decode_attn_grouped")
        return out
    if nsplit > 1 and scratch is None:
        scratch = torch.empty(decode_scratch_numel(B, n_heads, nsplit), dtype=torch.float32, device=q.device)
    check(lib().rpeg_paged_decode_attn(q.data_ptr(), q.stride(0), q_col0, kcache.data_ptr(), vcache.data_ptr(),
                                       page_table.data_ptr(), page_table.stride(0), seq_lens.data_ptr(),
                                       out.data_ptr(), _ptr(scratch), B, n_heads, n_kv_heads, head_dim, nsplit,
                                       scale, _stream()), "rpeg_paged_decode_attn")
    return out


def flash_attn_fwd(qkv, q_col0, k_col0, v_col0, cu_seqlens, max_seqlen, n_heads, n_kv_heads, head_dim, scale=None):
    """Causal attention over packed sequences. Returns ``(out [T, H*hd] bf16, lse [H, T] fp32)``."""
    _req(qkv, torch.bfloat16, "qkv")
    T = qkv.shape[0]
    if _chk.active():
        _chk.packed_sequences("rpeg_flash_attn_fwd", cu_seqlens, T, max_seqlen)
    scale = 1.0 / math.sqrt(head_dim) if scale is None else scale
    out = torch.empty((T, n_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    lse = torch.empty((n_heads, T), dtype=torch.float32, device=qkv.device)
    check(lib().rpeg_flash_attn_fwd(qkv.data_ptr(), qkv.stride(0), q_col0, k_col0, v_col0, cu_seqlens.data_ptr(),
                                    cu_seqlens.numel() - 1, max_seqlen, T, n_heads, n_kv_heads, head_dim, scale,
                                    out.data_ptr(), lse.data_ptr(), status_word(qkv.device).data_ptr(), _stream()),
          "rpeg_flash_attn_fwd")
    return out, lse


def flash_attn_bwd(qkv, q_col0, k_col0, v_col0, out, dout, lse, cu_seqlens, max_seqlen, n_heads, n_kv_heads, head_dim,
                   scale=None, dqkv: torch.Tensor | None = None) -> torch.Tensor:
    """Gradient of ``flash_attn_fwd`` w.r.t. the packed qkv buffer (same column blocks). ``dqkv``
    may be passed in to reuse a buffer; columns outside the three blocks are left untouched."""
    T = qkv.shape[0]
    if _chk.active():
        _chk.packed_sequences("rpeg_flash_attn_bwd", cu_seqlens, T, max_seqlen)
    scale = 1.0 / math.sqrt(head_dim) if scale is None else scale
    if dqkv is None:
        dqkv = torch.empty_like(qkv)
    dvec = torch.empty((n_heads, T), dtype=torch.float32, device=qkv.device)
    dq_acc = torch.empty((T, n_heads * head_dim), dtype=torch.float32, device=qkv.device)
    check(lib().rpeg_flash_attn_bwd(qkv.data_ptr(), qkv.stride(0), q_col0, k_col0, v_col0, out.data_ptr(),
                                    dout.data_ptr(), lse.data_ptr(), cu_seqlens.data_ptr(), cu_seqlens.numel() - 1,
                                    max_seqlen, T, n_heads, n_kv_heads, head_dim, scale, dvec.data_ptr(),
                                    dq_acc.data_ptr(), dqkv.data_ptr(), dqkv.stride(0),
                                    status_word(qkv.device).data_ptr(), _stream()), "rpeg_flash_attn_bwd")
    return dqkv


# --------------------------------------------------------------------------- decode bookkeeping
def decode_prepare(active, gen_count, forced_len, forced, eos: int) -> None:
    check(lib().rpeg_decode_prepare(active.data_ptr(), gen_count.data_ptr(), _ptr(forced_len), forced.data_ptr(),
                                    active.numel(), eos, _stream()), "rpeg_decode_prepare")


def decode_advance(sampled, sampled_lp, token, pos, seq_len, active, gen_count, out_tok, out_lp, eos: int,
                   n_finished, step_counter=None) -> None:
    check(lib().rpeg_decode_advance(sampled.data_ptr(), sampled_lp.data_ptr(), token.data_ptr(), pos.data_ptr(),
                                    seq_len.data_ptr(), active.data_ptr(), gen_count.data_ptr(), out_tok.data_ptr(),
                                    out_lp.data_ptr(), active.numel(), out_tok.shape[1], eos, n_finished.data_ptr(),
                                    _ptr(step_counter), _stream()), "rpeg_decode_advance")


def gather_rows(x: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
    if _chk.active():
        _chk.row_indices("rpeg_gather_rows", rows, x.shape[0])
    if x.dtype == torch.float32:                 # the kernel moves 16-bit elements: an fp32 row is a row of twice the width
        return gather_rows(x.view(torch.bfloat16), rows).view(torch.float32)
    out = torch.empty((rows.numel(), x.shape[1]), dtype=x.dtype, device=x.device)
    check(lib().rpeg_gather_rows(x.data_ptr(), rows.data_ptr(), out.data_ptr(), rows.numel(), x.shape[1], _stream()),
          "rpeg_gather_rows")
    return out


def scatter_rows_(x: torch.Tensor, rows: torch.Tensor, src: torch.Tensor, overwrite: bool = False) -> None:
    if _chk.active():
        _chk.row_indices("rpeg_scatter_rows", rows, x.shape[0])
    check(lib().rpeg_scatter_rows(x.data_ptr(), rows.data_ptr(), src.data_ptr(), rows.numel(), x.shape[1],
                                  int(overwrite), _stream()), "rpeg_scatter_rows")


# --------------------------------------------------------------------------- fp32 matrix products
def gemm_f32(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``a [M, K] @ b [N, K].T`` in true fp32 (CUDA cores, no reduced-precision matrix mode)."""
    _req(a, torch.float32, "a")
    _req(b, torch.float32, "b")
    if a.dim() != 2 or b.dim() != 2 or a.stride(1) != 1 or b.stride(1) != 1 or a.shape[1] != b.shape[1]:
        raise ValueError("gemm_f32 operands must be [M, K] and [N, K] with a contiguous last dimension")
    M, Kd = a.shape
    N = b.shape[0]
    if out is None:
        out = torch.empty((M, N), dtype=torch.float32, device=a.device)
    check(lib().rpeg_gemm_f32(a.data_ptr(), b.data_ptr(), out.data_ptr(), M, N, Kd, a.stride(0), b.stride(0), out.stride(0), _stream()),
          "rpeg_gemm_f32")
    return out


# --------------------------------------------------------------------------- norms around an fp32 residual stream
_NORM_ACT, _NORM_PARTIALS, _NORM_MOE, _NORM_EMBED, _NORM_STREAM = range(5)


class MoEOutput:
    """Expert outputs of ``T`` tokens before their sum: ``y`` rows in segment order, ``row_of`` / ``weights`` ``[T, top]`` (weights None:
    a plain sum)."""

    __slots__ = ("y", "row_of", "weights", "top", "n_shared")

    def __init__(self, y: torch.Tensor, row_of: torch.Tensor, weights: torch.Tensor | None, n_shared: int):
        self.y, self.row_of, self.weights, self.n_shared = y, row_of, weights, n_shared
        self.top = row_of.shape[1]


def residual_norm(src, w: torch.Tensor, eps: float, d: int, *, x: torch.Tensor | None = None, add: bool = True, ids: torch.Tensor | None = None,
                  w2: torch.Tensor | None = None, want_act: bool = True, zero_centered: bool = True) -> torch.Tensor | None:
    """``v = norm(src)``; with ``add`` the fp32 stream ``x [T, dp]`` becomes ``x + v``, without it ``x`` (if given) becomes
    ``v``. ``src``: an activation ``[T, >= dp]``, ``Partials``, ``MoEOutput``, an embedding table (with ``ids``) or the stream
    itself (fp32, when the weights are bf16). Norm weights (their dtype is the activation dtype) are applied as
    ``1 + w`` when ``zero_centered``; the mean runs over the first ``d`` of the padded ``dp = w.numel()`` columns.
    Returns the result in the activation dtype, or, with ``w2``, ``norm(result)`` under the weight ``w2``."""
    dp = w.numel()
    f32 = w.dtype == torch.float32
    splits, stride, idx, wts, top, n_shared, shared0 = 1, 0, None, None, 0, 0, 0
    if isinstance(src, Partials):
        kind, rows, ld, p, splits, stride = _NORM_PARTIALS, src.M, src.N, src.buf, src.splits, src.stride
    elif isinstance(src, MoEOutput):
        kind, p, ld, rows = _NORM_MOE, src.y, src.y.stride(0), src.row_of.shape[0]
        idx, wts, top, n_shared, shared0 = src.row_of, src.weights, src.top, src.n_shared, rows * src.top
    elif ids is not None:
        _req(ids, torch.int32, "ids")
        if _chk.active():
            _chk.embed("rpeg_residual_norm", ids, src.shape[0])
        kind, p, ld, rows, idx = _NORM_EMBED, src, src.stride(0), ids.numel(), ids
    else:
        kind, p, ld, rows = (_NORM_STREAM if src.dtype == torch.float32 and not f32 else _NORM_ACT), src, src.stride(0), src.shape[0]
        if src.dtype not in (torch.float32, w.dtype):
            raise TypeError(f"residual_norm: source dtype {src.dtype} does not go with weights of {w.dtype}")
    if ld < dp or (add and x is None) or (x is not None and (x.dtype != torch.float32 or x.shape != (rows, dp) or not x.is_contiguous())):
        raise ValueError("residual_norm: the stream must be a contiguous fp32 [T, dp] tensor and the source at least dp wide")
    y = torch.empty((rows, dp), dtype=w.dtype, device=w.device) if (want_act or w2 is not None) else None
    check(lib().rpeg_residual_norm(kind, p.data_ptr(), splits, stride, ld, _ptr(idx), _ptr(wts), top, n_shared, shared0, w.data_ptr(), _ptr(w2),
                                   _ptr(x), _ptr(y), rows, d, dp, eps, 1.0 if zero_centered else 0.0, int(add), int(f32), _stream()),
          "rpeg_residual_norm")
    return y


# --------------------------------------------------------------------------- chunked attention with a sink
def rotary_append(src, q_out: torch.Tensor, q_col0: int, k_col0: int, v_col0: int, slot, pos, cos_t, sin_t, page_table, kcache, vcache,
                  n_heads: int, dim: int, rot_dims: int, norm_eps: float | None) -> None:
    """Interleaved rotary embedding of the first ``rot_dims`` dimensions of the q and k heads of ``src`` (an activation or
    ``Partials``), then (``norm_eps`` not None) a weight-free RMS norm over ``dim`` per head; q goes to ``q_out``, k and the
    values (columns from ``v_col0``, as projected) to the cache ``[pages, n_kv, PAGE, dp]``. ``v_col0 == k_col0``: the values
    are the keys' projection."""
    n_kv, dp = kcache.shape[1], kcache.shape[3]
    part = isinstance(src, Partials)
    rows, ld = (src.M, src.N) if part else (src.shape[0], src.stride(0))
    f32 = kcache.dtype == torch.float32
    if part and f32:
        raise TypeError("rotary_append: split-K partials belong to the bf16 path")
    if q_out.dtype != kcache.dtype or vcache.dtype != kcache.dtype or (not part and src.dtype != kcache.dtype):
        raise TypeError("rotary_append: source, query buffer and caches must share a dtype")
    if rot_dims and (cos_t.shape[1] * 2 != rot_dims or cos_t.shape != sin_t.shape):
        raise ValueError("rotary_append: the tables do not fit rot_dims")
    if _chk.active():
        _chk.kv_append("rpeg_rotary_append", rows, slot, pos, page_table, kcache, n_kv, dp, cos_t if rot_dims else None)
    check(lib().rpeg_rotary_append((src.buf if part else src).data_ptr(), src.splits if part else 0, src.stride if part else 0, ld, q_col0, k_col0,
                                   v_col0, slot.data_ptr(), pos.data_ptr(), _ptr(cos_t), _ptr(sin_t), page_table.data_ptr(),
                                   page_table.stride(0), q_out.data_ptr(), q_out.stride(0), kcache.data_ptr(), vcache.data_ptr(), rows, n_heads,
                                   n_kv, dim, dp, rot_dims, int(norm_eps is not None), 0.0 if norm_eps is None else norm_eps, int(f32), _stream()),
          "rpeg_rotary_append")


def rows_attn_scratch(rows: int, n_heads: int, dp: int, nsplit: int) -> int:
    """fp32 elements of split scratch ``rows_attn`` needs."""
    return int(lib().rpeg_rows_attn_scratch(rows, n_heads, dp, nsplit))


def rows_attn(q: torch.Tensor, kcache, vcache, page_table, slot, pos, n_heads: int, *, window: int = 0, scale: float, lens=None,
              sink: torch.Tensor | None = None, nsplit: int = 1, scratch: torch.Tensor | None = None,
              arrive: torch.Tensor | None = None) -> torch.Tensor:
    """One query row per token over the paged cache: row ``t`` sees keys ``[floor(p / window) * window, p]`` of page-table row
    ``slot[t]`` with ``p = pos[t]`` (or ``lens[t] - 1``; ``lens[t] = 0``: nothing, the row is zero). ``sink [H]`` fp32 joins the
    softmax denominator. ``nsplit > 1`` needs ``scratch`` (see ``rows_attn_scratch``) and ``arrive`` (int32 ``rows * H``, zero)."""
    n_kv, dp = kcache.shape[1], kcache.shape[3]
    rows = q.shape[0]
    if q.dtype != kcache.dtype:
        raise TypeError("rows_attn: q and the caches must share a dtype")
    if _chk.active():
        seen = (pos + 1) if lens is None else lens
        _chk.paged_attention("rpeg_rows_attn", rows, seen, page_table[slot[:rows].long()], kcache, n_kv, dp)
    if nsplit > 1 and (scratch is None or scratch.numel() < rows_attn_scratch(rows, n_heads, dp, nsplit) or arrive is None or arrive.numel() < rows * n_heads):
        raise ValueError("rows_attn: split attention needs scratch and arrival counters")
    out = torch.empty((rows, n_heads * dp), dtype=q.dtype, device=q.device)
    check(lib().rpeg_rows_attn(q.data_ptr(), q.stride(0), kcache.data_ptr(), vcache.data_ptr(), page_table.data_ptr(), page_table.stride(0),
                               slot.data_ptr(), pos.data_ptr(), _ptr(lens), _ptr(sink), out.data_ptr(), out.stride(0), _ptr(scratch), _ptr(arrive),
                               rows, n_heads, n_kv, dp, window, nsplit, scale, int(q.dtype == torch.float32), status_word(q.device).data_ptr(),
                               _stream()), "rpeg_rows_attn")
    return out


WINDOW_PREFILL_MAX_DIM = 128     # head sizes the tensor-core prompt kernel covers


def window_prefill(q: torch.Tensor, kcache, vcache, page_table, cu, pos, slot, max_len: int, n_heads: int, *, window: int = 0, scale: float,
                   sink: torch.Tensor | None = None) -> torch.Tensor:
    """Prompt attention of packed portions (request ``b`` owns rows ``cu[b] .. cu[b + 1]`` at consecutive positions) over the
    paged cache that already holds their keys; visibility as in ``rows_attn``. bf16, head size up to 128, ``scale > 0``."""
    _req(q, torch.bfloat16, "q")
    n_kv, dp = kcache.shape[1], kcache.shape[3]
    T = q.shape[0]
    if _chk.active():
        _chk.packed_sequences("rpeg_window_prefill", cu, T, max_len)
        _chk.paged_attention("rpeg_window_prefill", T, pos + 1, page_table[slot[:T].long()], kcache, n_kv, dp)
    out = torch.empty((T, n_heads * dp), dtype=torch.bfloat16, device=q.device)
    check(lib().rpeg_window_prefill(q.data_ptr(), q.stride(0), kcache.data_ptr(), vcache.data_ptr(), kcache.shape[0], page_table.data_ptr(),
                                    page_table.stride(0), cu.data_ptr(), pos.data_ptr(), slot.data_ptr(), _ptr(sink), out.data_ptr(),
                                    out.stride(0), T, cu.numel() - 1, max_len, n_heads, n_kv, dp, window, scale,
                                    status_word(q.device).data_ptr(), _stream()), "rpeg_window_prefill")
    return out


# --------------------------------------------------------------------------- mixture of experts
class MoERouting:
    """Where the tokens of one mixture layer go: ``ids`` / ``weights`` / ``row_of`` ``[T, top]``, ``seg_off [E + 1]`` and the
    dispatched rows ``x_sorted [T * top, dp]``."""

    __slots__ = ("ids", "weights", "row_of", "seg_off", "x_sorted", "x")

    def __init__(self, ids, weights, row_of, seg_off, x_sorted, x):
        self.ids, self.weights, self.row_of, self.seg_off, self.x_sorted, self.x = ids, weights, row_of, seg_off, x_sorted, x


def moe_route(logits, n_experts: int, top: int, counts: torch.Tensor, *, n_groups: int = 1, keep_groups: int = 1, renormalize: bool = False,
              sigmoid: bool = False):
    """Softmax (or ``sigmoid``) routing of ``logits`` (fp32 ``[T, >= E]`` or ``Partials``): the ``top`` largest scores among the experts of the
    ``keep_groups`` best of ``n_groups`` equal groups. ``counts [E]`` int32 must be zero; every choice takes a ticket there.
    Returns ``(ids, weights, tickets)``, each ``[T, top]``."""
    part = isinstance(logits, Partials)
    rows, ld = (logits.M, logits.N) if part else (logits.shape[0], logits.stride(0))
    buf = logits.buf if part else logits
    _req(buf, torch.float32, "router logits")
    if counts.numel() < n_experts or ld < n_experts:
        raise ValueError("moe_route: counts and logits must cover every expert")
    i32 = dict(dtype=torch.int32, device=buf.device)
    ids, ticket = torch.empty((rows, top), **i32), torch.empty((rows, top), **i32)
    wts = torch.empty((rows, top), dtype=torch.float32, device=buf.device)
    check(lib().rpeg_moe_route(buf.data_ptr(), logits.splits if part else 1, logits.stride if part else 0, ld, rows, n_experts, n_groups, keep_groups,
                               top, int(renormalize), int(sigmoid), ids.data_ptr(), wts.data_ptr(), ticket.data_ptr(), counts.data_ptr(), _stream()),
          "rpeg_moe_route")
    return ids, wts, ticket


def moe_dispatch(x: torch.Tensor, ids, wts, ticket, counts, n_experts: int, *, weigh_inputs: bool = False) -> MoERouting:
    """Copy every token's row into the segments of its experts; ``weigh_inputs``: multiplied by the choice's weight there (the
    outputs are then summed as they are)."""
    rows, dp = x.shape
    top = ids.shape[1]
    if not x.is_contiguous():
        raise ValueError("moe_dispatch: the rows must be contiguous")
    row_of = torch.empty_like(ids)
    seg_off = torch.empty(n_experts + 1, dtype=torch.int32, device=x.device)
    xs = torch.empty((rows * top, dp), dtype=x.dtype, device=x.device)
    check(lib().rpeg_moe_dispatch(x.data_ptr(), dp, ids.data_ptr(), ticket.data_ptr(), _ptr(wts if weigh_inputs else None), counts.data_ptr(), rows, n_experts, top, xs.data_ptr(),
                                  row_of.data_ptr(), seg_off.data_ptr(), int(x.dtype == torch.float32), _stream()), "rpeg_moe_dispatch")
    return MoERouting(ids, None if weigh_inputs else wts, row_of, seg_off, xs, x)


FF_ACTS = {"none": 0, "gelu": 1, "swiglu": 2, "relu2": 3}


def moe_gemm(a: torch.Tensor, b: torch.Tensor, r: MoERouting, n_experts: int, n_shared: int, *, shared_x: torch.Tensor | None = None,
             act: str = "none", bn: int = 0) -> torch.Tensor:
    """``C[rows of segment s] = act(a[rows of s] @ b[s].T)`` over the experts' segments; ``b [E + n_shared, N, K]``. ``act``: none, gelu,
    relu2 (squared relu) or swiglu (``b [E + n_shared, 2 N, K]``, gate rows first: ``silu(gate) * up``). The always-on segments take their rows from ``shared_x [T, K]`` (tokens in order) or, without it, from ``a`` behind the routed rows."""
    T, top = r.row_of.shape
    S, N, Kd = b.shape
    code = FF_ACTS[act]
    N = N // 2 if act == "swiglu" else N
    if S != n_experts + n_shared or a.shape[1] != Kd or not b.is_contiguous() or a.stride(1) != 1:
        raise ValueError("moe_gemm: operand shapes do not fit the segments")
    need = T * top + (0 if shared_x is not None else n_shared * T)
    if a.shape[0] < need or (shared_x is not None and (shared_x.shape != (T, Kd) or shared_x.stride(1) != 1)):
        raise ValueError("moe_gemm: too few operand rows")
    c = torch.empty((T * (top + n_shared), N), dtype=a.dtype, device=a.device)
    if a.dtype == torch.float32:
        if shared_x is not None and shared_x.stride(0) != a.stride(0):
            raise ValueError("moe_gemm: both operands need one row pitch")
        check(lib().rpeg_moe_gemm_f32(a.data_ptr(), _ptr(shared_x), b.data_ptr(), c.data_ptr(), r.seg_off.data_ptr(), n_experts, n_shared, T, N, Kd,
                                      a.stride(0), Kd, c.stride(0), code, _stream()), "rpeg_moe_gemm_f32")
        return c
    _req(a, torch.bfloat16, "a")
    check(lib().rpeg_moe_gemm(a.data_ptr(), a.shape[0], _ptr(shared_x), b.data_ptr(), c.data_ptr(), r.seg_off.data_ptr(), n_experts, n_shared, T,
                              T * top, N, Kd, a.stride(0), 0 if shared_x is None else shared_x.stride(0), Kd, c.stride(0), code, bn,
                              status_word(a.device).data_ptr(), _stream()), "rpeg_moe_gemm")
    return c


_ZERO_SEGMENT: dict[torch.device, torch.Tensor] = {}


def ff_first(x: torch.Tensor, w: torch.Tensor, act: str) -> torch.Tensor:
    """``act(x @ w.T)``, the first product of a dense feed-forward with its activation in the epilogue (``act`` and the layout of ``w``
    as in ``moe_gemm``): a mixture of one always-on expert."""
    if x.device not in _ZERO_SEGMENT:
        _ZERO_SEGMENT[x.device] = torch.zeros(1, dtype=torch.int32, device=x.device)
    r = MoERouting(None, None, torch.empty((x.shape[0], 0), dtype=torch.int32, device=x.device), _ZERO_SEGMENT[x.device], x, x)
    return moe_gemm(x, w.unsqueeze(0), r, 0, 1, shared_x=x, act=act)


# --------------------------------------------------------------------------- stream of parallel sublayers
def stream_update(a, b, alpha: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, x: torch.Tensor, *, ids: torch.Tensor | None = None) -> torch.Tensor:
    """``x += a + b`` on the fp32 stream ``x [T, dp]``, returns ``tanh(alpha * x) * w + bias`` in the dtype of ``w``. ``a``: an activation
    ``[T, >= dp]``, ``Partials``, or an embedding table whose rows ``ids`` become ``x``; ``b``: None, an activation, ``Partials`` or a
    ``MoEOutput``. ``alpha``: fp32 scalar on the device."""
    dp, rows = w.numel(), x.shape[0]
    f32 = w.dtype == torch.float32
    if x.dtype != torch.float32 or x.shape != (rows, dp) or not x.is_contiguous() or bias.dtype != w.dtype or bias.numel() != dp:
        raise ValueError("stream_update: the stream must be a contiguous fp32 [T, dp] tensor, w and bias [dp]")
    _req(alpha, torch.float32, "alpha")

    def source(s):
        """(kind, tensor, splits, stride, row pitch)"""
        if s is None:
            return -1, None, 1, 0, 0
        if isinstance(s, Partials):
            n, out = s.M, (_NORM_PARTIALS, s.buf, s.splits, s.stride, s.N)
        elif isinstance(s, MoEOutput):
            n, out = s.row_of.shape[0], (_NORM_MOE, s.y, 1, 0, s.y.stride(0))
        else:
            n, out = rows if ids is not None else s.shape[0], (_NORM_EMBED if ids is not None else _NORM_ACT, s, 1, 0, s.stride(0))
        if n != rows or out[4] < dp or out[1].dtype != (torch.float32 if isinstance(s, Partials) else w.dtype):
            raise ValueError("stream_update: a source does not fit the stream or the weights' dtype")
        return out

    if ids is not None:
        _req(ids, torch.int32, "ids")
        if ids.numel() != rows:
            raise ValueError("stream_update: one id per row")
        if _chk.active():
            _chk.embed("rpeg_stream_update", ids, a.shape[0])
    ka, ta, pa, sa, la = source(a)
    kb, tb, pb, sb, lb = source(b)
    moe = isinstance(b, MoEOutput)
    y = torch.empty((rows, dp), dtype=w.dtype, device=w.device)
    check(lib().rpeg_stream_update(ka, ta.data_ptr(), pa, sa, la, _ptr(ids), kb, _ptr(tb), pb, sb, lb, _ptr(b.row_of if moe else None),
                                   _ptr(b.weights if moe else None), b.top if moe else 0, b.n_shared if moe else 0, rows * b.top if moe else 0,
                                   alpha.data_ptr(), w.data_ptr(), bias.data_ptr(), x.data_ptr(), y.data_ptr(), rows, dp, int(f32), _stream()),
          "rpeg_stream_update")
    return y


# --------------------------------------------------------------------------- latent attention
LATENT_MAX_RANK = 1024           # latent width the kernels cover


def head_gemm(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, transposed: bool = False) -> torch.Tensor:
    """``out[:, h] = a[:, h] @ w[h].T`` for every head (``transposed``: ``@ w[h]``); ``a [T, H, K]`` and ``out [T, H, N]`` may be strided
    views with contiguous last dimensions, ``w [H, N, K]`` (``[H, K, N]``) is contiguous."""
    T, H, Kd = a.shape
    N = out.shape[2]
    if w.shape != ((H, Kd, N) if transposed else (H, N, Kd)) or out.shape[:2] != (T, H) or a.stride(2) != 1 or out.stride(2) != 1 or not w.is_contiguous():
        raise ValueError("head_gemm: operand shapes do not fit")
    if not a.dtype == w.dtype == out.dtype:
        raise TypeError("head_gemm: operands must share a dtype")
    if a.dtype == torch.float32:
        check(lib().rpeg_gemm_f32_batched(a.data_ptr(), w.data_ptr(), out.data_ptr(), T, N, Kd, a.stride(0), N if transposed else Kd, out.stride(0),
                                          a.stride(1), N * Kd, out.stride(1), H, int(transposed), _stream()), "rpeg_gemm_f32_batched")
        return out
    _req(a, torch.bfloat16, "a")
    check(lib().rpeg_head_gemm(a.data_ptr(), w.data_ptr(), out.data_ptr(), T, N, Kd, H, a.stride(0), a.stride(1), out.stride(0), out.stride(1),
                               int(transposed), status_word(a.device).data_ptr(), _stream()), "rpeg_head_gemm")
    return out


def latent_rows(src, pos, slot, cos_t, sin_t, rot: int, rot_p: int, eps: float, *, q_latent=None, kv=None, queries=None, ff=None) -> None:
    """Between a projection and latent attention, any of (column numbers refer to ``src``, an activation or ``Partials``):
      q_latent  (column, true width, weight, out [T, width_p]): weighted RMS norm of a query latent
      kv        (column, true rank, weight, cache [pages, 1, PAGE, rank_p + rot_p], page_table): the normed latent and the rotated shared key
                part of every token into its cache row
      queries   (column, heads, dim_p, out or None, rotated [T, H, rot_p]): heads of ``[dim_p | rot_p]`` columns; the rotated parts go to the
                (strided) view ``rotated``, which may be their place in ``src``; the others to ``out [T, H * dim_p]``, if given
      ff        (column, out [T, ff_p]): the squared relu of ``ff_p`` columns, a feed-forward's activation."""
    part = isinstance(src, Partials)
    rows, ld = (src.M, src.N) if part else (src.shape[0], src.stride(0))
    ref = next(t for t in (q_latent and q_latent[3], kv and kv[3], queries and queries[4], ff and ff[1]) if t is not None)
    f32 = ref.dtype == torch.float32
    if (part and f32) or (not part and src.dtype != ref.dtype):
        raise TypeError("latent_rows: source and outputs must share a dtype (split-K partials belong to the bf16 path)")
    if rot and (cos_t.shape[1] * 2 != rot or cos_t.shape != sin_t.shape):
        raise ValueError("latent_rows: the tables do not fit the rotated width")
    nq = (0, 0, 0, None, None)
    if q_latent is not None:
        c0, n, w, out = q_latent
        if not out.is_contiguous() or out.shape != (rows, w.numel()):
            raise ValueError("latent_rows: the query latent's buffer must be [T, width]")
        nq = (c0, n, w.numel(), w.data_ptr(), out.data_ptr())
    lat = (0, 0, 0, None, None, None, 0)
    if kv is not None:
        c0, n, w, cache, table = kv
        if cache.shape[1] != 1 or cache.shape[3] != w.numel() + rot_p:
            raise ValueError("latent_rows: the cache does not fit the latent")
        if _chk.active():
            _chk.kv_append("rpeg_latent_rows", rows, slot, pos, table, cache, 1, cache.shape[3], cos_t if rot else None)
        lat = (c0, n, w.numel(), w.data_ptr(), cache.data_ptr(), table.data_ptr(), table.stride(0))
    qs = (0, 0, 0, None, 0, None, 0, 0)
    if queries is not None:
        c0, H, dim_p, out, rotated = queries
        if rotated.shape != (rows, H, rot_p) or (rot_p and rotated.stride(2) != 1) or (out is not None and (out.shape != (rows, H * dim_p) or not out.is_contiguous())):
            raise ValueError("latent_rows: the query buffers do not fit")
        if rot and _chk.active():
            _chk.rope("rpeg_latent_rows", pos, rows, cos_t)
        qs = (c0, H, dim_p, _ptr(out), H * dim_p, rotated.data_ptr(), rotated.stride(0), rotated.stride(1))
    act = (0, 0, None)
    if ff is not None:
        c0, out = ff
        if out.shape[0] != rows or not out.is_contiguous() or out.dtype != ref.dtype:
            raise ValueError("latent_rows: the feed-forward's buffer does not fit")
        act = (c0, out.shape[1], out.data_ptr())
    check(lib().rpeg_latent_rows((src.buf if part else src).data_ptr(), src.splits if part else 0, src.stride if part else 0, ld, rows, pos.data_ptr(),
                                 slot.data_ptr(), _ptr(cos_t), _ptr(sin_t), rot, rot_p, eps, *nq, *lat, *qs, *act, int(f32), _stream()), "rpeg_latent_rows")


def latent_gather(cache: torch.Tensor, page_table, slot, cu, off, lo, rows: int) -> torch.Tensor:
    """The cache rows packed requests see, ``[rows, W]``: rows ``off[b] .. off[b + 1]`` are the positions from ``lo[b]`` on of page-table row
    ``slot[cu[b]]``."""
    W = cache.shape[3]
    out = torch.empty((rows, W), dtype=cache.dtype, device=cache.device)
    if _chk.active():
        _chk.packed_sequences("rpeg_latent_gather", off, rows, rows)
        _chk.paged_attention("rpeg_latent_gather", lo.numel(), lo + off[1:] - off[:-1], page_table[slot[cu[:-1].long()].long()], cache, 1, W)
    check(lib().rpeg_latent_gather(cache.data_ptr(), W * cache.element_size(), page_table.data_ptr(), page_table.stride(0), slot.data_ptr(), cu.data_ptr(),
                                   off.data_ptr(), lo.data_ptr(), lo.numel(), rows, out.data_ptr(), _stream()), "rpeg_latent_gather")
    return out


def latent_attn_rows(q: torch.Tensor, cache: torch.Tensor, rank_p: int, page_table, slot, pos, *, window: int = 0, scale: float, lens=None,
                     sink: torch.Tensor | None = None) -> torch.Tensor:
    """Latent attention of single query rows ``q [T, H, W]`` over the cache rows of page-table row ``slot[t]``: row ``t`` at position ``p =
    pos[t]`` (or ``lens[t] - 1``; ``lens[t] = 0``: nothing, the row is zero) sees the last ``window`` positions up to its own (0: all). Returns
    the averaged latents ``[T, H, rank_p]``. ``sink [H]`` fp32 joins the softmax denominator. CUDA cores, bf16 or fp32."""
    T, H, W = q.shape
    if q.dtype != cache.dtype or not q.is_contiguous() or cache.shape[3] != W:
        raise TypeError("latent_attn_rows: q must be contiguous [T, H, W] in the cache's dtype")
    if _chk.active():
        _chk.paged_attention("rpeg_latent_attn_rows", T, (pos + 1) if lens is None else lens, page_table[slot[:T].long()], cache, 1, W)
    out = torch.empty((T, H, rank_p), dtype=q.dtype, device=q.device)
    check(lib().rpeg_latent_attn_rows(q.data_ptr(), cache.data_ptr(), page_table.data_ptr(), page_table.stride(0), slot.data_ptr(), pos.data_ptr(),
                                      _ptr(lens), _ptr(sink), out.data_ptr(), T, H, rank_p, W, window, scale, int(q.dtype == torch.float32), _stream()),
          "rpeg_latent_attn_rows")
    return out


def latent_decode_ctas_per_sm(rank_p: int, width: int) -> int:
    """CTAs of ``latent_decode`` an SM holds (0: sizes it does not cover)."""
    return int(lib().rpeg_latent_decode_ctas(rank_p, width))


def latent_decode_fits(rank_p: int, width: int) -> bool:
    return latent_decode_ctas_per_sm(rank_p, width) > 0


def latent_decode_scratch(rows: int, n_heads: int, rank_p: int, nsplit: int) -> int:
    """fp32 elements of split scratch ``latent_decode`` needs."""
    return int(lib().rpeg_latent_decode_scratch(rows, n_heads, rank_p, nsplit))


def latent_decode(q: torch.Tensor, cache: torch.Tensor, rank_p: int, page_table, slot, pos, *, window: int = 0, scale: float, lens=None,
                  sink: torch.Tensor | None = None, nsplit: int = 1, scratch: torch.Tensor | None = None) -> torch.Tensor:
    """``latent_attn_rows`` on the tensor cores (bf16, ``scale > 0``; sizes as ``latent_decode_fits``). The cache must hold finite numbers everywhere.
    ``nsplit > 1``: every row's pages are shared by that many CTAs (``scratch`` as ``latent_decode_scratch``)."""
    _req(q, torch.bfloat16, "q")
    _req(cache, torch.bfloat16, "cache")
    T, H, W = q.shape
    if not q.is_contiguous() or cache.shape[1:] != (1, KV_PAGE, W):
        raise ValueError("latent_decode: q must be contiguous [T, H, W], the cache [pages, 1, PAGE, W]")
    if nsplit > 1 and (scratch is None or scratch.numel() < latent_decode_scratch(T, H, rank_p, nsplit)):
        raise ValueError("latent_decode: split attention needs scratch")
    if _chk.active():
        _chk.paged_attention("rpeg_latent_decode", T, (pos + 1) if lens is None else lens, page_table[slot[:T].long()], cache, 1, W)
    out = torch.empty((T, H, rank_p), dtype=torch.bfloat16, device=q.device)
    check(lib().rpeg_latent_decode(q.data_ptr(), cache.data_ptr(), cache.shape[0], page_table.data_ptr(), page_table.stride(0), slot.data_ptr(), pos.data_ptr(),
                                   _ptr(lens), _ptr(sink), out.data_ptr(), _ptr(scratch), T, H, rank_p, W, window, nsplit, scale,
                                   status_word(q.device).data_ptr(), _stream()), "rpeg_latent_decode")
    return out


def latent_prefill_fits(dim_p: int, rot_p: int, vdim_p: int) -> bool:
    """Head sizes ``latent_prefill`` covers (padded): unrotated and rotated parts up to three runs of 64 together, values up to 128."""
    return bool(lib().rpeg_latent_prefill_fits(dim_p, rot_p, vdim_p))


def latent_prefill(q: torch.Tensor, kv: torch.Tensor, rows: torch.Tensor, dim_p: int, vdim_p: int, rank_p: int, cu, pos, off, lo, max_len: int, *,
                   window: int = 0, scale: float, sink: torch.Tensor | None = None) -> torch.Tensor:
    """Prompt attention of packed portions (request ``b`` owns query rows ``cu[b] .. cu[b + 1]`` at consecutive positions ``pos``) over formed keys
    and values: ``q [T, H, dim_p + rot_p]`` (may be strided), ``kv [n, H * dim_p + H * vdim_p]`` from the gathered cache rows ``rows [n, W]``, of
    which request ``b`` sees ``off[b] .. off[b + 1]``, positions ``lo[b]`` on. Visibility as in ``latent_attn_rows``. Returns
    ``[T, H * vdim_p]``. bf16, ``scale > 0``."""
    for t, name in ((q, "q"), (kv, "kv"), (rows, "rows")):
        _req(t, torch.bfloat16, name)
    T, H, hw = q.shape
    n, W = rows.shape
    if q.stride(2) != 1 or kv.shape != (n, H * (dim_p + vdim_p)) or not kv.is_contiguous() or not rows.is_contiguous() or hw - dim_p != W - rank_p:
        raise ValueError("latent_prefill: operand shapes do not fit")
    if _chk.active():
        _chk.packed_sequences("rpeg_latent_prefill", cu, T, max_len)
        _chk.packed_sequences("rpeg_latent_prefill", off, n, n)
    out = torch.empty((T, H * vdim_p), dtype=torch.bfloat16, device=q.device)
    check(lib().rpeg_latent_prefill(q.data_ptr(), q.stride(0), q.stride(1), kv.data_ptr(), rows.data_ptr(), n, W, rank_p, cu.data_ptr(), pos.data_ptr(),
                                    off.data_ptr(), lo.data_ptr(), _ptr(sink), out.data_ptr(), out.stride(0), T, cu.numel() - 1, max_len, H, dim_p,
                                    hw - dim_p, vdim_p, window, scale, status_word(q.device).data_ptr(), _stream()), "rpeg_latent_prefill")
    return out
