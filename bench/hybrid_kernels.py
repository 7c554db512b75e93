"""Kernels of the hybrid layers, one line each (``python -m bench.kernels --kernel hybrid --model sigisun-1b``): prefill of
--m tokens in --seqs sequences, decode of --batch sequences at context --ctx. Bytes and FLOPs are the algorithm's: every
operand and result once; the scan counts each product of a 32-bit operand (two bf16 pieces) once under "useful" and twice
under "issued"; attention counts visible pairs only."""
from __future__ import annotations

import torch


def run(preset, T, n, B, ctx, timed, hbm, tf, tag):
    from openrlhf_b200.models.config import PRESETS
    from openrlhf_b200.models.hybrid_config import AttentionSpec, Mamba2Spec
    from openrlhf_b200.ops import _lib
    from openrlhf_b200.ops import hybrid as H
    from openrlhf_b200.ops.attention import PAGE

    cfg = PRESETS[preset]
    dev, bf = "cuda", torch.bfloat16
    layer_m = next(x for x in cfg.layers if isinstance(x.mixer, Mamba2Spec))
    layer_a = next(x for x in cfg.layers if isinstance(x.mixer, AttentionSpec))
    m, at = layer_m.mixer, layer_a.mixer
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)

    def line(name, t, byt=0.0, fl=0.0, issued=0.0):
        parts = [f"{name}: {t * 1e6:.1f} us"]
        if byt:
            parts.append(f"{byt / t / 1e9:.0f} GB/s ({byt / t / 1e9 / hbm:.2f} {tag} HBM)")
        if fl:
            parts.append(f"{fl / t / 1e12:.0f} TFLOP/s useful ({fl / t / 1e12 / tf:.2f} {tag} bf16)")
        if issued:
            parts.append(f"{issued / t / 1e12:.0f} issued ({issued / t / 1e12 / tf:.2f})")
        print(", ".join(parts), flush=True)

    # ---- prefill
    L = T // n
    pages = (L + PAGE - 1) // PAGE
    bt = torch.arange(n * pages, dtype=torch.int32, device=dev).view(n, pages)
    pos = torch.arange(L, dtype=torch.int32, device=dev).repeat(n)
    seq = torch.arange(n, dtype=torch.int32, device=dev).repeat_interleave(L)
    slots = bt[seq.long(), (pos // PAGE).long()] * PAGE + pos % PAGE
    batch = H.StepBatch(None, pos, slots, seq, i32([i * L for i in range(n + 1)]), i32([0] * n), i32(list(range(n))), bt, n, T,
                        L, lens=[L] * n)
    print(f"-- {preset}: prefill {n} x {L}, heads {m.heads} x {m.vdim}, state {m.state}; attention {at.heads}/{at.kv_heads} x "
          f"{at.dim}, window {at.window}")
    x = torch.randn(T, cfg.width_pad, device=dev)
    w = rnd(cfg.width_pad)
    line("rmsnorm fp32 -> bf16", timed(lambda: H.rmsnorm(x, w, cfg.hidden_size, 1e-6)), T * cfg.width_pad * 6.0)
    h, w1 = rnd(T, cfg.width_pad), rnd(layer_m.in_pad + layer_m.ff_pad, cfg.width_pad) * 0.02
    a = torch.empty(T, layer_m.out_pad + layer_m.ff_pad, device=dev, dtype=bf)
    act = a[:, layer_m.out_pad:]
    line("input projections + up, relu^2 epilogue", timed(lambda: H.project(h, w1, layer_m.in_pad, act)),
         fl=2.0 * T * w1.shape[0] * w1.shape[1])
    w2 = rnd(cfg.width_pad, a.shape[1]) * 0.02
    a.normal_()
    from openrlhf_b200.ops.gemm import gemm
    line("output + down, added to fp32", timed(lambda: gemm(a, w2, out=x, accumulate=True)),
         fl=2.0 * T * w2.shape[0] * w2.shape[1])
    p = H.Projection(rnd(T, layer_m.in_pad), None, 1, T, layer_m.in_pad, bf)
    wt = H.Mamba2Weights(rnd(m.conv_channels, m.conv), rnd(m.conv_channels), rnd(m.heads), rnd(m.heads) * 0.1, rnd(m.heads),
                         rnd(m.inner))
    ring = torch.zeros(max(n, B), m.conv, m.conv_channels, device=dev, dtype=bf)
    state = torch.zeros(max(n, B), m.heads, m.state, m.vdim, device=dev)
    xbc = torch.empty(T, m.conv_channels, dtype=bf, device=dev)
    dt = torch.rand(m.heads, T, device=dev) * 0.1
    y = torch.empty(T, m.inner, dtype=bf, device=dev)
    L_, c, pt = _lib.lib(), H._i, H._p
    seqs = (pt(batch.cu), pt(batch.start), pt(batch.row), pt(None), pt(batch.tok_seq), c(n), c(T))
    dims = (c(m.heads), c(m.vdim), c(m.state), c(m.groups), c(m.conv))
    dt2 = torch.empty_like(dt)
    line("convolution + silu, step sizes, ring", timed(lambda: L_.b200_ssd_conv(
        *p.args(), *seqs, pt(ring), pt(wt.conv), pt(wt.conv_bias), pt(wt.dt_bias), pt(xbc), pt(dt2), *dims, c(0),
        _lib.stream_ptr())), T * (m.conv_channels * 4.0 + m.heads * 6.0))
    xbc.normal_()
    Q, N, P = 128, m.state, m.vdim
    pair, one = T * m.heads * 2.0 * Q * N, T * m.heads * 2.0
    useful = pair + one * (Q * P + 2 * N * P)
    issued = pair + 2 * one * (Q * P + 2 * N * P)
    line("scan (chunks of 128)", timed(lambda: H.ssd_scan(xbc, dt, m, wt.a_log, wt.d, state, y, batch, chunked=True)),
         T * (m.conv_channels * 2.0 + m.inner * 2.0 + m.heads * 4.0), useful, issued)
    line("gate + group norm", timed(lambda: L_.b200_gate_norm(
        pt(y), *p.args(), pt(wt.norm), pt(a), c(a.stride(0)), c(T), c(m.inner), c(m.norm_groups), H._f(1e-6), c(0), c(0),
        pt(act), c(0), _lib.stream_ptr())), T * m.inner * 6.0)
    pa = H.Projection(rnd(T, layer_a.in_pad), None, 1, T, layer_a.in_pad, bf)
    kc = rnd(n * pages * PAGE, at.kv_heads, at.k_ld)
    vc = rnd(n * pages * PAGE, at.kv_heads, at.v_ld)
    q = rnd(T, at.heads, at.k_ld)
    oa = torch.empty(T, layer_a.out_pad + layer_a.ff_pad, device=dev, dtype=bf)
    table = H.rotary_table(at.rot_dims, at.rot_base, at.rot_factor, max(L, ctx + 1), dev)

    def rope():
        return L_.b200_rope_write(
            *pa.args(), pt(pos), pt(slots), pt(table), c(table.shape[0]), pt(q), pt(kc), pt(vc), c(T), c(at.heads),
            c(at.kv_heads), c(at.dim), c(at.vdim), c(at.k_ld), c(at.v_ld), c(at.rot_dims), c(0), c(0), pt(oa), c(oa.stride(0)),
            c(0), _lib.stream_ptr())
    line("rotation + cache write", timed(rope), T * at.in_rows * 4.0)
    k_vis = torch.arange(L, dtype=torch.float64).add(1).clamp_max(at.window + at.keep_first).sum().item() * n
    line("windowed attention", timed(lambda: H.attention(q, kc, vc, at, batch, oa)),
         fl=2.0 * k_vis * at.heads * (at.dim + at.vdim))
    del x, h, a, xbc, y, p, pa, kc, vc, q, oa
    torch.cuda.empty_cache()
    # ---- decode
    print(f"-- {preset}: decode of {B} sequences at context {ctx}")
    pages = ctx // PAGE + 1
    bt = torch.arange(B * pages, dtype=torch.int32, device=dev).view(B, pages)
    ids = torch.arange(B + 1, dtype=torch.int32, device=dev)
    pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
    batch = H.StepBatch(None, pos, pos, ids[:B], ids, pos, ids[:B], bt, B, B, 1)
    cols = layer_m.in_pad + layer_m.ff_pad
    p = H.Projection(None, torch.randn(2, B, cols, device=dev), 2, B, cols, bf)
    y = torch.empty(B, m.inner, dtype=bf, device=dev)
    line("convolution + state update + read-out", timed(lambda: L_.b200_ssd_decode(
        *p.args(), pt(pos), pt(ids), pt(None), c(B), pt(ring), pt(wt.conv), pt(wt.conv_bias), pt(wt.dt_bias), pt(wt.a_log),
        pt(wt.d), pt(state), pt(y), *dims, c(0), _lib.stream_ptr())), B * m.heads * N * P * 8.0)
    kc = rnd(B * pages * PAGE, at.kv_heads, at.k_ld)
    vc = rnd(B * pages * PAGE, at.kv_heads, at.v_ld)
    q = rnd(B, at.heads, at.k_ld)
    oa = torch.empty(B, layer_a.out_pad + layer_a.ff_pad, device=dev, dtype=bf)
    seen = min(ctx, at.window + at.keep_first)
    line("windowed decode attention", timed(lambda: H.attention(q, kc, vc, at, batch, oa)),
         B * seen * at.kv_heads * (at.dim + at.vdim) * 2.0)
    _lib.check_status()
