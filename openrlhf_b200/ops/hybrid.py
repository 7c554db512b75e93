"""Operators of hybrid decoder layers (``csrc/hybrid_ops.cu``, ``csrc/ssd.cu``, ``csrc/attn_window.cu``,
``csrc/gemm_f32.cu``) over one ragged step.

Activations and weights are bf16 (serving) or float32 (the all-32-bit mode); the residual stream, recurrent state and
logits are float32 in both. CPU tensors run the PyTorch restatements of ``ops/reference.py``, which exist for the
scheduler tests."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field

import torch

from . import _lib, reference
from .attention import PAGE

_i, _ll, _f = ctypes.c_int, ctypes.c_longlong, ctypes.c_float
_p = _lib.ptr


@dataclass
class StepBatch:
    """One model step: ``n`` sequences bring ``T`` tokens in a packed stream. int32 tensors on the model's device
    unless noted."""
    ids: torch.Tensor              # [T] int64
    pos: torch.Tensor              # [T] position inside the sequence
    slots: torch.Tensor            # [T] KV slot (page * PAGE + offset) the token is written to
    tok_seq: torch.Tensor          # [T] sequence of the token
    cu: torch.Tensor               # [n + 1] first token of every sequence
    start: torch.Tensor            # [n] position of the sequence's first token in this step
    row: torch.Tensor              # [n] row of the state pools
    block_table: torch.Tensor      # [n, max_pages]
    n: int
    T: int
    max_new: int                   # most tokens of one sequence in this step
    active: torch.Tensor | None = None    # [n] sequences with 0 leave every state as it is (idle rows of a decode bucket)
    lens: list | None = None       # host copy of the portions' lengths (None: single tokens)
    _tiles: dict = field(default_factory=dict)

    @property
    def single(self) -> bool:
        """Every sequence brings exactly one token."""
        return self.max_new == 1 and self.n == self.T

    def query_tiles(self, tq: int):
        """Query tiles of `tq` tokens: (sequence, first token inside the portion) of each, int32 on the device."""
        hit = self._tiles.get(tq)
        if hit is None:
            lens = self.lens if self.lens is not None else [1] * self.n
            pairs = torch.tensor([(i, q0) for i, k in enumerate(lens) for q0 in range(0, k, tq)], dtype=torch.int32)
            pairs = pairs.t().contiguous().to(self.cu.device)
            hit = self._tiles[tq] = (pairs[0], pairs[1], pairs.shape[1])
        return hit


@dataclass
class Projection:
    """Output of a fused input projection: a finished matrix, or the fp32 slabs of a split-K GEMM that its consumers sum
    on the way in."""
    mat: torch.Tensor | None       # [T, N] activation type
    ws: torch.Tensor | None        # fp32 [splits, T, N]
    splits: int
    rows: int
    cols: int
    dtype: torch.dtype

    def args(self):
        return (_p(self.mat), _p(self.ws), _i(self.splits), _ll(self.rows * self.cols), _i(self.cols))

    def dense(self) -> torch.Tensor:
        """As one float32 matrix (restatements)."""
        return self.mat.float()


def _f32(dtype) -> ctypes.c_int:
    return _i(int(dtype == torch.float32))


def embed(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """fp32 residual rows of the tokens; `table` [V, ld]."""
    if not ids.is_cuda:
        return table[ids].float()
    T, ld = ids.numel(), table.shape[1]
    x = torch.empty(T, ld, dtype=torch.float32, device=ids.device)
    _lib.check_rc(_lib.lib().b200_embed_f32(_p(ids), _p(table), _p(x), _i(T), _i(ld), _i(table.shape[0]),
                                            _f32(table.dtype), _lib.stream_ptr()), "embed_f32")
    return x


def rmsnorm(x: torch.Tensor, w: torch.Tensor, n: int, eps: float, rows: torch.Tensor | None = None,
            add: Projection | None = None) -> torch.Tensor:
    """RMS norm over the first `n` channels of fp32 rows (all of them, or the listed ones), in w's type. `add`: split-K
    slabs of a projection that are added to x (in place) first."""
    M = x.shape[0] if rows is None else rows.numel()
    if not x.is_cuda:
        return reference.rmsnorm_f32(x if rows is None else x[rows.long()], w, n, eps)
    y = torch.empty(M, x.shape[1], dtype=w.dtype, device=x.device)
    ws, splits, slab = (None, 0, 0) if add is None else (add.ws, add.splits, add.rows * add.cols)
    _lib.check_rc(_lib.lib().b200_rmsnorm_f32(_p(x), _p(ws), _i(splits), _ll(slab), _p(rows), _p(w), _p(y), _i(M), _i(n),
                                              _i(x.shape[1]), _f(eps), _f32(w.dtype), _lib.stream_ptr()), "rmsnorm_f32")
    return y


SMALL_M = 256      # up to this many tokens a projection is split along K into fp32 slabs


def project(h: torch.Tensor, w: torch.Tensor, act_col: int = 0, act_out: torch.Tensor | None = None) -> Projection:
    """h [T, K] @ w[N, K]^T for consumers that take a ``Projection``. With `act_out`, columns from `act_col` on may leave
    as relu^2 into it; the returned projection then has only `act_col` columns, otherwise its consumer does it."""
    from .gemm import gemm, gemm_relu2, gemm_to_workspace

    T, N = h.shape[0], w.shape[0]
    if not h.is_cuda:
        return Projection(reference.linear(h, w), None, 1, T, N, h.dtype)
    if h.dtype == torch.float32:
        return Projection(gemm_f32(h, w), None, 1, T, N, h.dtype)
    if T <= SMALL_M:
        ws, s = gemm_to_workspace(h, w)
        return Projection(None, ws, s, T, N, h.dtype)
    if act_out is not None and N > act_col:
        return Projection(gemm_relu2(h, w, act_col, act_out), None, 1, T, act_col, h.dtype)
    return Projection(gemm(h, w), None, 1, T, N, h.dtype)


def gemm_f32(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None, accumulate: bool = False) -> torch.Tensor:
    """a [M, K] @ w [N, K]^T in true fp32 (no TF32); optionally added to `out`."""
    M, K = a.shape
    N = w.shape[0]
    assert a.dtype == w.dtype == torch.float32 and a.stride(1) == 1 and w.stride(1) == 1 and w.shape[1] == K
    if out is None:
        out = torch.empty(M, N, dtype=torch.float32, device=a.device)
    _lib.check_rc(_lib.lib().b200_gemm_f32(_p(a), _p(w), _p(out), _i(M), _i(N), _i(K), _i(a.stride(0)), _i(w.stride(0)),
                                           _i(out.stride(0)), _i(int(accumulate)), _lib.stream_ptr()), "gemm_f32")
    return out


def add_norm(x: torch.Tensor, a: torch.Tensor, w: torch.Tensor, norm_w: torch.Tensor | None, n: int, eps: float):
    """x += a @ w^T (x fp32 [T, ld], in place), then the next sublayer's norm of x, or None when `norm_w` is None."""
    from .gemm import gemm, gemm_to_workspace

    if not x.is_cuda:
        x += a.float() @ w.float().t()
    elif a.dtype == torch.float32:
        gemm_f32(a, w, out=x, accumulate=True)
    elif a.shape[0] <= SMALL_M and norm_w is not None:
        ws, s = gemm_to_workspace(a, w)
        return rmsnorm(x, norm_w, n, eps, add=Projection(None, ws, s, x.shape[0], x.shape[1], a.dtype))
    else:
        gemm(a, w, out=x, accumulate=True)
    return None if norm_w is None else rmsnorm(x, norm_w, n, eps)


def head_logits(h: torch.Tensor, w: torch.Tensor, vocab: int, cap: float | None) -> torch.Tensor:
    """fp32 logits [M, vocab] (a view of padded rows), soft-capped when `cap` is given."""
    from .gemm import gemm

    if not h.is_cuda:
        z = h.float() @ w.float().t()
        return (z if cap is None else reference.softcap(z, cap))[:, :vocab]
    z = gemm_f32(h, w) if h.dtype == torch.float32 else gemm(h, w, out_f32=True)
    if cap is not None:
        _lib.check_rc(_lib.lib().b200_softcap(_p(z), _ll(z.numel()), _f(cap), _lib.stream_ptr()), "softcap")
    return z[:, :vocab]


# ---------------------------------------------------------------------------------------------- Mamba-2
@dataclass
class Mamba2Weights:
    conv: torch.Tensor       # [channels, taps]
    conv_bias: torch.Tensor  # [channels]
    dt_bias: torch.Tensor    # [heads]
    a_log: torch.Tensor      # [heads]
    d: torch.Tensor          # [heads]
    norm: torch.Tensor       # [inner]


CHUNK_MIN = 8      # portions of at least this many tokens take the tensor-core scan


def ssd_scan(xbc: torch.Tensor, dt: torch.Tensor, m, a_log: torch.Tensor, d: torch.Tensor, state: torch.Tensor,
             y: torch.Tensor, batch: StepBatch, chunked: bool | None = None, segments: int | None = None) -> None:
    """Recurrence over the convolved inputs xbc [T, channels] and step sizes dt fp32 [heads, T]; y [T, inner]. `chunked`
    picks the tensor-core kernel (bf16, sizes it covers) or the token-by-token one; None: by portion length. `segments`:
    how many pieces of a portion the tensor-core kernel runs side by side; None: as many as fill the GPU."""
    L = _lib.lib()
    seqs = (_p(batch.cu), _p(batch.start), _p(batch.row), _p(batch.active), _p(batch.tok_seq), _i(batch.n), _i(batch.T))
    H, P, N, G = _i(m.heads), _i(m.vdim), _i(m.state), _i(m.groups)
    fits = xbc.dtype == torch.bfloat16 and L.b200_ssd_chunk_fits(H, P, N, G) == 1
    if chunked is None:
        chunked = fits and batch.max_new >= CHUNK_MIN
    if chunked:
        assert fits, "sizes outside the tensor-core scan"
        chunks = (batch.max_new + 127) // 128
        if segments is None:
            # a segment costs a second, cheaper pass over its tokens: only when heads and sequences leave SMs idle
            ctas = m.heads * batch.n * ((m.vdim + 63) // 64)
            segments = min(2 * 148 // ctas, chunks // 4) if ctas <= 100 else 1
        per = (chunks + segments - 1) // segments if segments > 1 else 0
        nseg = (chunks + per - 1) // per if per else 1
        seg_state = seg_log2 = None
        if per:
            seg_state = torch.empty(batch.n, m.heads, nseg, m.state, m.vdim, dtype=torch.float32, device=xbc.device)
            seg_log2 = torch.empty(batch.n, m.heads, nseg, dtype=torch.float32, device=xbc.device)
        _lib.check_rc(L.b200_ssd_chunk(_p(xbc), _p(dt), *seqs, _p(a_log), _p(d), _p(state), _p(y), H, P, N, G, _i(per),
                                       _i(nseg), _p(seg_state), _p(seg_log2),
                                       _p(_lib.status_word(xbc.device)), _lib.stream_ptr()), "ssd_chunk")
    else:
        _lib.check_rc(L.b200_ssd_scan(_p(xbc), _p(dt), *seqs, _p(a_log), _p(d), _p(state), _p(y), H, P, N, G, _i(m.conv),
                                      _f32(xbc.dtype), _lib.stream_ptr()), "ssd_scan")


def mamba2(p: Projection, m, wt: Mamba2Weights, ring: torch.Tensor, state: torch.Tensor, batch: StepBatch, eps: float,
           out: torch.Tensor, out_pad: int, ff_col: int, ff: int) -> None:
    """Convolution, recurrence, gate and group norm of one layer: columns [0, inner) of `out` [T, ld]; the feed-forward
    columns of the projection go to columns [out_pad, out_pad + ff) as relu^2. `ring` [rows, taps, channels] and `state`
    [rows, heads, N, P] fp32 are updated in place. m: ``Mamba2Spec``."""
    if not out.is_cuda:
        reference.mamba2(p.dense(), m, wt, ring, state, batch, eps, out, out_pad, ff_col, ff)
        return
    L, st = _lib.lib(), _lib.stream_ptr
    f32 = _f32(p.dtype)
    T, dev = batch.T, out.device
    dims = (_i(m.heads), _i(m.vdim), _i(m.state), _i(m.groups), _i(m.conv))
    y = torch.empty(T, m.inner, dtype=p.dtype, device=dev)
    if batch.single:
        _lib.check_rc(L.b200_ssd_decode(
            *p.args(), _p(batch.start), _p(batch.row), _p(batch.active), _i(T), _p(ring), _p(wt.conv), _p(wt.conv_bias),
            _p(wt.dt_bias), _p(wt.a_log), _p(wt.d), _p(state), _p(y), *dims, f32, st()), "ssd_decode")
    else:
        seqs = (_p(batch.cu), _p(batch.start), _p(batch.row), _p(batch.active), _p(batch.tok_seq), _i(batch.n), _i(T))
        xbc = torch.empty(T, m.conv_channels, dtype=p.dtype, device=dev)
        dt = torch.empty(m.heads, T, dtype=torch.float32, device=dev)
        _lib.check_rc(L.b200_ssd_conv(*p.args(), *seqs, _p(ring), _p(wt.conv), _p(wt.conv_bias), _p(wt.dt_bias), _p(xbc),
                                      _p(dt), *dims, f32, st()), "ssd_conv")
        ssd_scan(xbc, dt, m, wt.a_log, wt.d, state, y, batch)
    _lib.check_rc(L.b200_gate_norm(_p(y), *p.args(), _p(wt.norm), _p(out), _i(out.stride(0)), _i(T), _i(m.inner),
                                   _i(m.norm_groups), _f(eps), _i(ff_col), _i(ff), _p(out[:, out_pad:]), f32, st()),
                  "gate_norm")


# ---------------------------------------------------------------------------------------------- attention
_rotary: dict = {}


def rotary_table(dims: int, base: float, factor: float, max_pos: int, device) -> torch.Tensor:
    """[max_pos, dims/2, 2] fp32 (cos, sin) of position * base^(-2i/dims) / factor, angles formed in float64."""
    key = (dims, float(base), float(factor), str(device))
    tab = _rotary.get(key)
    if tab is None or tab.shape[0] < max_pos:
        inv = float(base) ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims) / float(factor)
        ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * inv[None, :]
        tab = torch.stack([ang.cos(), ang.sin()], dim=-1).float().contiguous().to(device)
        _rotary[key] = tab
    return tab


def window_attention(p: Projection, m, table: torch.Tensor | None, k_cache: torch.Tensor, v_cache: torch.Tensor,
                     batch: StepBatch, out: torch.Tensor, out_pad: int, ff_col: int, ff: int) -> None:
    """Rotary embedding, cache write and attention of one layer into columns [0, heads * vdim) of `out`; feed-forward
    columns as in ``mamba2``. k_cache [slots, kv_heads, k_ld], v_cache [slots, kv_heads, v_ld]; with ``m.kv_from`` they
    are the earlier layer's and only read. m: ``AttentionSpec``."""
    if not out.is_cuda:
        reference.window_attention(p.dense(), m, table, k_cache, v_cache, batch, out, out_pad, ff_col, ff, PAGE)
        return
    L, st = _lib.lib(), _lib.stream_ptr
    f32 = _f32(p.dtype)
    T = batch.T
    # rows of q are padded like the cache rows; the padding is never read by a kernel that knows dim
    q = torch.empty(T, m.heads, m.k_ld, dtype=p.dtype, device=out.device)
    _lib.check_rc(L.b200_rope_write(
        *p.args(), _p(batch.pos), _p(batch.slots), _p(table), _i(1 if table is None else table.shape[0]), _p(q), _p(k_cache),
        _p(v_cache), _i(T), _i(m.heads), _i(0 if m.kv_from is not None else m.kv_heads), _i(m.dim), _i(m.vdim), _i(m.k_ld),
        _i(m.v_ld), _i(m.rot_dims), _i(ff_col), _i(ff), _p(out[:, out_pad:]), _i(out.stride(0)), f32, st()), "rope_write")
    attention(q, k_cache, v_cache, m, batch, out)


def attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, m, batch: StepBatch, out: torch.Tensor,
              impl: str | None = None) -> None:
    """Attention of rotated queries q [T, heads, k_ld] over the paged cache. `impl`: "ragged" (any size and type),
    "tiles" (tensor cores, bf16, heads up to 128 channels) or "decode" (the same for single tokens, groups of up to 16
    query heads); None picks."""
    L = _lib.lib()
    window = (1 << 30) if m.window is None else int(m.window)
    rep = m.heads // m.kv_heads
    fits = q.dtype == torch.bfloat16 and m.dim <= 128 and m.vdim <= 128 and rep <= 64
    if impl is None:
        impl = ("decode" if batch.single and rep <= 16 else "tiles") if fits else "ragged"
    if impl == "decode":
        # one CTA per (sequence, kv head, split): split the pages of the window while SMs are idle
        span = (batch.block_table.shape[1] if m.window is None else (m.window + 2 * PAGE - 2) // PAGE
                + (m.keep_first + PAGE - 1) // PAGE)
        splits = max(1, min(span, 2 * 148 // (batch.T * m.kv_heads)))
        part = None if splits == 1 else torch.empty(batch.T * m.heads * splits, 130, dtype=torch.float32, device=q.device)
        ml = None if part is None else part.view(-1)[batch.T * m.heads * splits * 128:]
        _lib.check_rc(L.b200_attn_decode_window(
            _p(q), _p(k_cache), _p(v_cache), _p(batch.block_table), _p(batch.start), _p(out), _i(out.stride(0)), _p(part),
            _p(ml), _i(batch.T), _i(m.heads), _i(m.kv_heads), _i(m.dim), _i(m.vdim), _i(m.k_ld), _i(m.v_ld),
            _i(k_cache.shape[0] // PAGE), _i(batch.block_table.stride(0)), _i(splits), _i(window), _i(m.keep_first),
            _i(int(m.sink)), _f(m.scale), _p(_lib.status_word(q.device)), _lib.stream_ptr()), "attn_decode_window")
        return
    if impl == "tiles":
        assert fits, "sizes outside the tensor-core kernel"
        ts, tq0, nt = batch.query_tiles(128 // rep)
        _lib.check_rc(L.b200_attn_window(
            _p(q), _p(k_cache), _p(v_cache), _p(batch.cu), _p(batch.start), _p(batch.block_table), _p(ts), _p(tq0), _i(nt),
            _i(batch.T), _i(batch.block_table.stride(0)), _i(k_cache.shape[0] // PAGE), _p(out), _i(out.stride(0)),
            _i(m.heads), _i(m.kv_heads), _i(m.dim), _i(m.vdim), _i(m.k_ld), _i(m.v_ld), _i(window), _i(m.keep_first),
            _i(int(m.sink)), _f(m.scale), _p(_lib.status_word(q.device)), _lib.stream_ptr()), "attn_window")
        return
    _lib.check_rc(L.b200_attn_ragged(
        _p(q), _p(k_cache), _p(v_cache), _p(batch.cu), _p(batch.start), _p(batch.tok_seq), _p(batch.block_table),
        _i(batch.n), _i(batch.T), _i(batch.block_table.stride(0)), _i(PAGE), _p(out), _i(out.stride(0)), _i(m.heads),
        _i(m.kv_heads), _i(m.dim), _i(m.vdim), _i(m.k_ld), _i(m.v_ld), _i(window), _i(m.keep_first), _i(int(m.sink)),
        _f(m.scale), _f32(q.dtype), _lib.stream_ptr()), "attn_ragged")
