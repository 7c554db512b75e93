"""Sigisun on the GPU: every kernel against the plain restatement, then whole sequences through the engine in float32
and bf16, in portions, in mixed batches, with rows and pages used again, and generation with CUDA graphs."""
import pytest
import torch

import sigisun_oracle as O
from sigisun_helpers import CONFIGS, config, attn, feed, make_engine, mamba, rel_rms, tokens, write_checkpoint

pytestmark = pytest.mark.gpu
DEV = "cuda"
TYPES = [torch.float32, torch.bfloat16]


def _ids(t):
    return "f32" if t == torch.float32 else "bf16"


def close(got, want, dtype, tol32=2e-5, tol16=1.2e-2):
    """Largest difference over the largest magnitude."""
    got, want = got.double().cpu(), want.double()
    tol = tol32 if dtype == torch.float32 else tol16
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-9))
    assert err < tol, err


def step_batch(lens, starts, rows=None, pages=None, active=None, page_ids=None):
    """StepBatch of sequences with the given portions; page_ids: per sequence the list of its cache pages."""
    from openrlhf_b200.ops.hybrid import StepBatch

    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    n, T = len(lens), sum(lens)
    cu = [0]
    for k in lens:
        cu.append(cu[-1] + k)
    seq = [i for i, k in enumerate(lens) for _ in range(k)]
    pos = [s + o for s, k in zip(starts, lens) for o in range(k)]
    page_ids = page_ids or [[0] for _ in lens]
    width = max(len(p) for p in page_ids)
    slots = [page_ids[i][p // 128] * 128 + p % 128 if p // 128 < len(page_ids[i]) else 0 for i, p in zip(seq, pos)]
    return StepBatch(torch.zeros(T, dtype=torch.int64, device=DEV), i32(pos), i32(slots), i32(seq), i32(cu), i32(starts),
                     i32(rows if rows is not None else list(range(n))), i32([p + [0] * (width - len(p)) for p in page_ids]),
                     n, T, max(lens), active=None if active is None else i32(active), lens=list(lens))


def as_projection(mat, dtype, slabs):
    """A Projection of `mat` (double, CPU): a finished matrix, or three fp32 slabs that sum to it."""
    from openrlhf_b200.ops.hybrid import Projection

    T, N = mat.shape
    if slabs:
        g = torch.Generator().manual_seed(1)
        parts = torch.randn(3, T, N, generator=g)
        parts[2] = mat.float() - parts[0] - parts[1]
        return Projection(None, parts.to(DEV).contiguous(), 3, T, N, dtype)
    return Projection(mat.to(dtype).to(DEV), None, 1, T, N, dtype)


def rnd(*shape, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g).to(dtype)


# ---------------------------------------------------------------------------------------------- single mechanisms
@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
@pytest.mark.parametrize("n,ld", [(72, 72), (37, 40), (1000, 1000), (2048, 2048)])
def test_norm_of_the_fp32_residual(dtype, n, ld):
    from openrlhf_b200.ops import hybrid as H

    x = torch.zeros(9, ld)
    x[:, :n] = rnd(9, n, seed=1, dtype=torch.float32) * 3
    w = torch.zeros(ld).bfloat16()
    w[:n] = rnd(n, seed=2)
    got = H.rmsnorm(x.to(DEV), w.to(dtype).to(DEV), n, 1e-3)
    close(got[:, :n], O.rms_norm(x[:, :n].double(), w[:n].double(), 1e-3), dtype)
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
    assert torch.equal(H.rmsnorm(x.to(DEV), w.to(dtype).to(DEV), n, 1e-3, rows=rows), got[rows.long()])
    # residual add: slabs of a split-K product first
    xs = x.to(DEV)
    add = rnd(9, ld, seed=3, dtype=torch.float32)
    add[:, n:] = 0
    y = H.rmsnorm(xs, w.to(dtype).to(DEV), n, 1e-3, add=as_projection(add.double(), dtype, True))
    close(xs, (x + add).double(), torch.float32)
    close(y[:, :n], O.rms_norm((x + add)[:, :n].double(), w[:n].double(), 1e-3), dtype)


def test_softcap_embedding_and_fp32_product():
    from openrlhf_b200.ops import hybrid as H

    h, w = rnd(70, 100, seed=1, dtype=torch.float32), rnd(204, 100, seed=2, dtype=torch.float32)
    want = h.double() @ w.double().T
    close(H.gemm_f32(h.to(DEV), w.to(DEV)), want, torch.float32, tol32=2e-6)
    acc = torch.ones(70, 204, device=DEV)
    H.gemm_f32(h.to(DEV), w.to(DEV), out=acc, accumulate=True)
    close(acc, want + 1, torch.float32, tol32=2e-6)
    close(H.head_logits(h.to(DEV), w.to(DEV), 201, 5.0), O.softcap(want, 5.0)[:, :201], torch.float32, tol32=3e-6)
    tab = rnd(11, 40)
    ids = torch.tensor([3, 10, 0], device=DEV)
    assert torch.equal(H.embed(ids, tab.to(DEV)).cpu(), tab[ids.cpu()].float())


@pytest.mark.parametrize("M,N,K,col0", [(300, 352, 72, 224), (2048, 4352, 512, 2304), (1500, 8224, 264, 32)])
def test_input_projection_with_squared_relu_epilogue(M, N, K, col0):
    """The single-CTA and the CTA-pair GEMM: columns before col0 as they are, the rest as relu^2 into wider rows."""
    from openrlhf_b200.ops.gemm import gemm_relu2

    x, w = rnd(M, K, seed=1), rnd(N, K, seed=2)
    act = torch.full((M, N - col0 + 64), 5.0, dtype=torch.bfloat16, device=DEV)
    got = gemm_relu2(x.to(DEV), w.to(DEV), col0, act[:, 32:32 + N - col0])
    want = x.double() @ w.double().T
    close(got, want[:, :col0], torch.bfloat16)
    close(act[:, 32:32 + N - col0], torch.relu(want[:, col0:]) ** 2, torch.bfloat16)
    assert (act[:, :32] == 5).all() and (act[:, 32 + N - col0:] == 5).all()


MAMBAS = [mamba(4, 64, 128, 2, 4, 2), mamba(5, 7, 11, 5, 1, 5), mamba(3, 48, 16, 1, 3, 1), mamba(2, 128, 64, 1, 2, 4),
          mamba(6, 24, 96, 3, 5, 3), mamba(2, 40, 144, 2, 4, 1)]


def _mamba_case(m, dtype, T, seed=0):
    """Spec, weights (double and device) and an input projection of T tokens plus feed-forward columns."""
    from openrlhf_b200.models.hybrid_config import Mamba2Spec
    from openrlhf_b200.ops.hybrid import Mamba2Weights

    spec = Mamba2Spec(**m["mixer"])
    cfg = config([m], width=spec.inner)
    w = {k[len("l0.mix."):]: v for k, v in O.random_weights(cfg, seed).items() if k.startswith("l0.mix.")}
    dev = {k: v.to(dtype).to(DEV) for k, v in w.items()}
    wt = Mamba2Weights(dev["conv"], dev["conv.b"], dev["dt_bias"], dev["A_log"], dev["D"], dev["norm"])
    pad = (spec.in_rows + 31) // 32 * 32
    proj = torch.zeros(T, pad + 32, dtype=torch.float64)
    proj[:, :spec.in_rows] = rnd(T, spec.in_rows, seed=seed + 1).double()
    proj[:, pad:] = rnd(T, 32, seed=seed + 2).double()
    return spec, {k: v.double() for k, v in w.items()}, wt, proj, pad


def _mamba_oracle(spec, w, proj, eps):
    """Gated, normed mixer rows of one sequence from its projection, and the last recurrent state."""
    inner, gn = spec.inner, spec.groups * spec.state
    xbc = O.silu(O.causal_conv(proj[:, inner:inner + spec.conv_channels], w["conv"], w["conv.b"]))
    dt = O.softplus(proj[:, spec.in_rows - spec.heads:spec.in_rows] + w["dt_bias"])
    y, s = O.ssd_recurrence(xbc[:, :inner].reshape(-1, spec.heads, spec.vdim),
                            xbc[:, inner:inner + gn].reshape(-1, spec.groups, spec.state),
                            xbc[:, inner + gn:].reshape(-1, spec.groups, spec.state), dt, w["A_log"], w["D"])
    return O.group_rms_norm(y.reshape(-1, inner) * O.silu(proj[:, :inner]), w["norm"], spec.norm_groups, eps), s


@pytest.mark.parametrize("slabs", [False, True], ids=["matrix", "slabs"])
@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
@pytest.mark.parametrize("m", MAMBAS, ids=lambda m: "-".join(str(v) for v in m["mixer"].values()))
def test_mamba2_in_portions_of_a_mixed_batch(m, dtype, slabs):
    """Two sequences with different cuts (whole chunks, two tokens, single tokens), state rows in any order, an idle row."""
    from openrlhf_b200.ops import hybrid as H

    lens = (293, 70)
    cases = [_mamba_case(m, dtype, n, seed=7 * i) for i, n in enumerate(lens)]
    spec, w, wt, _, pad = cases[0]
    w1 = [_mamba_oracle(spec, w, c[3], 1e-4) for c in cases]          # the first case's weights for both
    rows = [3, 1]
    ring = torch.full((5, spec.conv, spec.conv_channels), 7.0, dtype=dtype, device=DEV)     # stale: must not be seen
    state = torch.full((5, spec.heads, spec.state, spec.vdim), 7.0, device=DEV)
    idle = (ring[0].clone(), state[0].clone())
    got = [[], []]
    at = [0, 0]
    for a, b in ((130, 2), (2, 40), (1, 1), (1, 1), (128, 1), (31, 25)):
        parts = [(0, a)] + ([(1, b)] if b else [])
        mat = torch.cat([cases[i][3][at[i]:at[i] + n] for i, n in parts])
        batch = step_batch([n for _, n in parts], [at[i] for i, _ in parts], [rows[i] for i, _ in parts])
        out_pad = (spec.inner + 31) // 32 * 32
        out = torch.zeros(batch.T, out_pad + 32, dtype=dtype, device=DEV)
        H.mamba2(as_projection(mat, dtype, slabs), spec, wt, ring, state, batch, 1e-4, out, out_pad, pad, 32)
        close(out[:, out_pad:], torch.relu(mat[:, pad:]) ** 2, dtype)
        o = 0
        for i, n in parts:
            got[i].append(out[o:o + n, :spec.inner])
            o += n
            at[i] += n
    assert at == list(lens)
    for i in range(2):
        close(torch.cat(got[i]), w1[i][0], dtype, tol32=1e-4, tol16=4e-2)
        close(state[rows[i]], w1[i][1], dtype, tol32=2e-5, tol16=2e-2)
    assert torch.equal(ring[0], idle[0]) and torch.equal(state[0], idle[1])


@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
def test_idle_rows_of_a_decode_batch_keep_their_state(dtype):
    from openrlhf_b200.ops import hybrid as H

    spec, w, wt, proj, pad = _mamba_case(MAMBAS[2], dtype, 3)
    ring = rnd(3, spec.conv, spec.conv_channels, seed=4, dtype=dtype).to(DEV)
    state = rnd(3, spec.heads, spec.state, spec.vdim, seed=5, dtype=torch.float32).to(DEV)
    r0, s0 = ring.clone(), state.clone()
    batch = step_batch([1, 1, 1], [9, 9, 9], active=[1, 0, 1])
    out = torch.zeros(3, (spec.inner + 31) // 32 * 32 + 32, dtype=dtype, device=DEV)
    H.mamba2(as_projection(proj, dtype, True), spec, wt, ring, state, batch, 1e-4, out, out.shape[1] - 32, pad, 32)
    assert torch.equal(ring[1], r0[1]) and torch.equal(state[1], s0[1]) and torch.isfinite(out).all()
    assert not torch.equal(state[0], s0[0]) and not torch.equal(ring[2], r0[2])


def test_tensor_core_scan_keeps_32_bit_state():
    """The chunked scan against the token-by-token fp32 kernel on the same bf16 inputs: the state to fp32 accuracy, fast
    and slow decays, portions that end inside a chunk."""
    from openrlhf_b200.models.hybrid_config import Mamba2Spec
    from openrlhf_b200.ops import hybrid as H

    for spec, lens, starts in ((Mamba2Spec(4, 64, 128, 2), [300, 1, 128, 77], [0, 5, 128, 0]),
                               (Mamba2Spec(6, 48, 32, 3), [9, 257], [3, 0]), (Mamba2Spec(2, 136, 80), [150], [1])):
        batch = step_batch(lens, starts, rows=[len(lens) - i for i in range(len(lens))])
        T = batch.T
        g = torch.Generator(device=DEV).manual_seed(0)
        xbc = torch.randn(T, spec.conv_channels, device=DEV, generator=g).bfloat16()
        dt = torch.rand(spec.heads, T, device=DEV, generator=g) ** 4 * 2
        a_log = torch.linspace(-4, 3, spec.heads, device=DEV).bfloat16()
        d = torch.randn(spec.heads, device=DEV, generator=g).bfloat16()
        s0 = torch.randn(len(lens) + 1, spec.heads, spec.state, spec.vdim, device=DEV, generator=g)
        s32, s16, s_seg = s0.clone(), s0.clone(), s0.clone()
        y32 = torch.empty(T, spec.inner, device=DEV)
        y16 = torch.empty(T, spec.inner, device=DEV, dtype=torch.bfloat16)
        H.ssd_scan(xbc.float(), dt, spec, a_log.float(), d.float(), s32, y32, batch, chunked=False)
        H.ssd_scan(xbc, dt, spec, a_log, d, s16, y16, batch, chunked=True)
        close(s16, s32.double().cpu(), torch.float32, tol32=2.0 ** -17)      # two bf16 pieces of every 32-bit operand
        close(y16, y32.double().cpu(), torch.bfloat16, tol16=4e-3)
        for segments in (2, 3):                    # pieces of a portion side by side
            s_seg.copy_(s0)
            y16.zero_()
            H.ssd_scan(xbc, dt, spec, a_log, d, s_seg, y16, batch, chunked=True, segments=segments)
            close(s_seg, s32.double().cpu(), torch.float32, tol32=2.0 ** -16)
            close(y16, y32.double().cpu(), torch.bfloat16, tol16=4e-3)


ATTN = [attn(6, 2, 64, 64, 0.2, 96 + 5, 3, 32), attn(3, 1, 22, 13, 0.3, 5, 1, 6), attn(4, 4, 128, 96, 0.1, 128, 0),
        attn(8, 1, 48, 128, 0.15, 1, 130, 8), attn(16, 1, 96, 40, 0.1, 300, 129), attn(20, 1, 16, 16, 0.4, 33, 2),
        attn(2, 2, 160, 136, 0.1, 50, 4)]


def _impls(spec, dtype):
    fits = dtype == torch.bfloat16 and spec.dim <= 128 and spec.vdim <= 128
    return ["ragged"] + (["tiles"] + (["decode"] if spec.heads // spec.kv_heads <= 16 else []) if fits else [])


@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
@pytest.mark.parametrize("m", ATTN, ids=lambda m: f"h{m['mixer']['heads']}-{m['mixer']['kv_heads']}-d{m['mixer']['dim']}"
                                                  f"-{m['mixer']['vdim']}-w{m['mixer']['mask']['size']}"
                                                  f"k{m['mixer']['mask']['keep_first']}")
def test_attention_window_edges_kept_tokens_and_pages(m, dtype):
    """Every kernel on a context of 420 tokens in scattered pages. Chosen queries have one key that outweighs everything:
    just inside and just outside the window, the last kept and the first not kept token, page borders."""
    from openrlhf_b200.models.hybrid_config import _sigisun_mixer
    from openrlhf_b200.ops import hybrid as H

    spec = _sigisun_mixer("attention", m["mixer"])
    L, win, keep = 420, spec.window, spec.keep_first
    q = rnd(L, spec.heads, spec.dim, seed=1).double()
    k = rnd(L, spec.kv_heads, spec.dim, seed=2).double() * 0.3
    v = rnd(L, spec.kv_heads, spec.vdim, seed=3).double()
    loud = set()
    for i, j in ((400, 400 - win + 1), (401, 401 - win), (419, keep - 1), (410, keep), (300, 256), (385, 384), (383, 255),
                 (260, 128), (259, 127), (150, 0), (200, 200)):
        if 0 <= j <= i and j not in loud:
            loud.add(j)
            k[j] = (q[i].view(spec.kv_heads, -1, spec.dim).mean(1) * 6).bfloat16().double()
    want = O.windowed_attention(q, k, v, spec.scale, win, keep).reshape(L, -1)
    pages = [[5, 2, 7, 3]]
    kc = torch.zeros(8 * 128, spec.kv_heads, spec.k_ld, dtype=dtype, device=DEV)
    vc = torch.zeros(8 * 128, spec.kv_heads, spec.v_ld, dtype=dtype, device=DEV)
    kc.uniform_(-4, 4), vc.uniform_(-4, 4)                      # pages hold other contexts' leftovers
    at = torch.tensor([pages[0][p // 128] * 128 + p % 128 for p in range(L)], device=DEV)
    kc[at, :, :spec.dim], vc[at, :, :spec.vdim] = k.to(dtype).to(DEV), v.to(dtype).to(DEV)
    ld = (spec.out_cols + 31) // 32 * 32 + 32
    for impl in _impls(spec, dtype):
        if impl == "decode":
            pos = sorted({0, 1, 127, 128, 129, 255, 256, 300, 383, 384, 385, 400, 401, 410, 419} |
                         {min(419, keep + win - 1), min(419, keep + win)})
            portions = [(pos, [1] * len(pos))]
        else:
            portions = [([0], [420]), ([0, 37], [37, 383]), ([128, 399], [2, 21]), (list(range(0, 420, 21)), [21] * 20)]
        for starts, lens in portions:
            batch = step_batch(lens, starts, page_ids=pages * len(lens))
            qq = torch.zeros(batch.T, spec.heads, spec.k_ld, dtype=dtype, device=DEV)
            qq[:, :, :spec.dim] = q[batch.pos.cpu().long()].to(dtype).to(DEV)
            out = torch.full((batch.T, ld), 9.0, dtype=dtype, device=DEV)
            H.attention(qq, kc, vc, spec, batch, out, impl=impl)
            close(out[:, :spec.out_cols], want[batch.pos.cpu().long()], dtype, tol16=2e-2)
            assert (out[:, spec.out_cols:] == 9).all()


@pytest.mark.parametrize("slabs", [False, True], ids=["matrix", "slabs"])
@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
@pytest.mark.parametrize("m", [ATTN[0], ATTN[1], ATTN[3]], ids=["a", "b", "c"])
def test_partial_rotation_and_cache_write(m, dtype, slabs):
    from openrlhf_b200.models.hybrid_config import _sigisun_mixer
    from openrlhf_b200.ops import hybrid as H

    spec = _sigisun_mixer("attention", m["mixer"])
    starts, lens = [0, 700], [5, 40]
    batch = step_batch(lens, starts, page_ids=[[1, 0, 0, 0, 0, 0], [6, 6, 6, 6, 6, 2]])
    T, pad = batch.T, (spec.in_rows + 31) // 32 * 32
    proj = rnd(T, pad + 64, seed=3).double()
    kc = torch.zeros(7 * 128, spec.kv_heads, spec.k_ld, dtype=dtype, device=DEV)
    vc = torch.zeros(7 * 128, spec.kv_heads, spec.v_ld, dtype=dtype, device=DEV)
    out = torch.zeros(T, (spec.out_cols + 31) // 32 * 32 + 64, dtype=dtype, device=DEV)
    table = H.rotary_table(spec.rot_dims, spec.rot_base, spec.rot_factor, 1024, DEV)
    H.window_attention(as_projection(proj, dtype, slabs), spec, table, kc, vc, batch, out, out.shape[1] - 64, pad, 64)
    nq, nk = spec.heads * spec.dim, spec.kv_heads * spec.dim
    turn = lambda x: O.rotary(x, batch.pos.cpu(), spec.rot_dims, spec.rot_base, spec.rot_factor)
    s = batch.slots.long()
    close(kc[s, :, :spec.dim], turn(proj[:, nq:nq + nk].reshape(T, spec.kv_heads, spec.dim)), dtype)
    close(vc[s, :, :spec.vdim], proj[:, nq + nk:spec.in_rows].reshape(T, spec.kv_heads, spec.vdim), dtype)
    close(out[:, -64:], torch.relu(proj[:, pad:]) ** 2, dtype)
    assert (kc[:, :, spec.dim:] == 0).all()
    untouched = torch.ones(kc.shape[0], dtype=torch.bool, device=DEV)
    untouched[s] = False
    assert (kc[untouched] == 0).all() and (vc[untouched] == 0).all()


# ---------------------------------------------------------------------------------------------- whole model
TOL = {torch.float32: 5e-5, torch.bfloat16: 0.05}
QUANTILE = {torch.float32: 1.0, torch.bfloat16: 0.95}


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def case(request, tmp_path_factory):
    cfg = CONFIGS[request.param]
    path = tmp_path_factory.mktemp(request.param)
    w = write_checkpoint(path, cfg, seed=len(request.param))
    seqs = {f"q{i}": tokens(cfg, n, i) for i, n in enumerate((300, 41, 7, 133, 1, 2))}
    return cfg, path, seqs, {k: O.forward(cfg, w, t) for k, t in seqs.items()}


@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
def test_prompts_portions_and_token_by_token(case, dtype):
    cfg, path, seqs, want = case
    eng = make_engine(path, DEV, dtype)
    toks = seqs["q0"]
    for cuts in ([300], [1], [2], [128, 1, 1, 60, 2], [129, 40, 3, 1], [5]):
        assert rel_rms(feed(eng, toks, cuts), want["q0"], QUANTILE[dtype]) < TOL[dtype], cuts
    for k in seqs:
        assert rel_rms(feed(eng, seqs[k], [len(seqs[k])]), want[k], QUANTILE[dtype]) < TOL[dtype], k


@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
def test_mixed_batches_reuse_rows_and_pages(case, dtype):
    cfg, path, seqs, want = case
    eng = make_engine(path, DEV, dtype, rows=3, pages=9)
    g = torch.Generator().manual_seed(9)
    draw = lambda a, b: int(torch.randint(a, b, (1,), generator=g))
    at, live, todo, errs = {}, [], list(seqs) + [k + "#2" for k in seqs], []
    while todo or live:
        while todo and len(live) < 3:
            live.append(todo.pop(0))
        entries = []
        for k in live:
            if draw(0, 5) == 0:
                continue
            t = seqs[k.split("#")[0]]
            part = t[at.get(k, 0):at.get(k, 0) + (draw(1, 90) if draw(0, 2) else 1)]
            entries.append((k, part, list(range(len(part)))))
        if not entries:
            continue
        lg, o = eng.extend(entries).cpu(), 0
        for k, part, _ in entries:
            a, base = at.get(k, 0), k.split("#")[0]
            d = lg[o:o + len(part)].double() - want[base][a:a + len(part)]
            errs.append((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want[base].std())
            o += len(part)
            at[k] = a + len(part)
            if at[k] == len(seqs[base]):
                eng.finish(k)
                live.remove(k)
    assert float(torch.cat(errs).quantile(QUANTILE[dtype])) < TOL[dtype]
    assert eng.blocks.num_free() == eng.num_pages - 1


def test_alone_and_in_a_batch_agree(case):
    """What else is in the batch changes rounding at most (bf16, the same portion sizes)."""
    cfg, path, seqs, _ = case
    eng = make_engine(path, DEV, torch.bfloat16)
    alone = feed(eng, seqs["q3"], [100, 1])
    eng.extend([("a", seqs["q0"][:200], []), ("b", seqs["q1"][:3], [])])
    both = [eng.extend([("a", seqs["q0"][200:230], []), ("c", seqs["q3"][:100], list(range(100))), ("b", seqs["q1"][3:4], [])])]
    for i in range(100, len(seqs["q3"])):
        both.append(eng.extend([("b", [seqs["q1"][(i % 30) + 4]], []), ("c", [seqs["q3"][i]], [0]),
                                ("a", [seqs["q0"][i]], [])]))
    for k in "abc":
        eng.finish(k)
    assert rel_rms(torch.cat(both).cpu(), alone, 0.95) < 0.03


def _by_extend(eng, prompt, n):
    toks, lg = list(prompt), eng.extend([("g", prompt, [len(prompt) - 1])])
    out = []
    for _ in range(n):
        out.append(int(lg[0].argmax()))
        lg = eng.extend([("g", [out[-1]], [0])])
    eng.finish("g")
    return out


@pytest.mark.parametrize("dtype", TYPES, ids=_ids)
def test_greedy_generation_with_graphs_and_continuous_batching(tmp_path, dtype):
    from openrlhf_b200.rollout.engine import SamplingParams

    cfg = CONFIGS["mix"]
    w = write_checkpoint(tmp_path, cfg, seed=11)
    prompts = [tokens(cfg, n, i) for i, n in enumerate((5, 200, 127, 2, 64, 129))]
    eng = make_engine(tmp_path, DEV, dtype, rows=4, check_interval=4)
    sp = SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True)
    outs = eng.generate(prompts, sp)
    again = make_engine(tmp_path, DEV, dtype, rows=8, max_prefill_tokens=128, check_interval=4, use_cuda_graph=False,
                        ).generate(prompts, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True, n=2))
    for i, (p, o, o2) in enumerate(zip(prompts, outs, again)):
        toks = o.outputs[0].token_ids
        assert len(toks) == 40
        ref = O.forward(cfg, w, p + toks)
        lp = torch.log_softmax(ref, -1)
        for k, t in enumerate(toks):                 # greedy up to rounding, and the log-probs are the model's
            row = ref[len(p) - 1 + k]
            slack = 1e-3 if dtype == torch.float32 else 0.6
            assert float(row.max() - row[t]) < slack, (i, k)
            assert abs(o.outputs[0].logprob_values[k] - float(lp[len(p) - 1 + k, t])) < slack
        if dtype == torch.float32:
            assert toks == o2.outputs[0].token_ids == o2.outputs[1].token_ids == _by_extend(eng, p, 40)


def test_long_decoding_keeps_to_the_restatement(tmp_path):
    """600 decoded tokens (several pages, windows passing over decoded tokens, a long recurrence) in float32."""
    cfg = config([mamba(2, 16, 16, 1, 4, 1, 32), attn(4, 2, 16, 16, 0.5, 70, 2, 8, ff=32),
                  attn(4, 2, 16, 16, 0.5, 400, 0, 8, kv_from=1)], width=40, vocab=64)
    w = write_checkpoint(tmp_path, cfg, seed=2)
    toks = tokens(cfg, 620)
    eng = make_engine(tmp_path, DEV, torch.float32)
    assert rel_rms(feed(eng, toks, [20, 1]), O.forward(cfg, w, toks)) < 5e-5


def test_sleep_and_wake_with_captured_graphs(tmp_path):
    from openrlhf_b200.rollout.engine import SamplingParams

    cfg = CONFIGS["attn"]
    write_checkpoint(tmp_path, cfg, seed=1)
    eng = make_engine(tmp_path, DEV, torch.bfloat16)
    sp = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True)
    p = [tokens(cfg, 150), tokens(cfg, 3, 1)]
    first = [o.outputs[0].token_ids for o in eng.generate(p, sp)]
    eng.sleep()
    eng.wake_up()
    assert [o.outputs[0].token_ids for o in eng.generate(p, sp)] == first
