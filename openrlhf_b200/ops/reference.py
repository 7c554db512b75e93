"""Plain PyTorch restatements of every operator (fp32 math where the kernels use fp32). Used on CPU by the oracle and
as the comparison target of the kernel tests; never on the GPU production path."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def linear(x, w, bias=None, residual=None):
    y = (x.float() @ w.float().t())
    if bias is not None:
        y = y + bias.float()
    if residual is not None:
        y = y + residual.float()
    return y.to(x.dtype)


def rmsnorm(x, w, eps):
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (y.to(x.dtype).float() * w.float()).to(x.dtype)


def rope(qkv, pos, table, n_heads, head_dim):
    """table [max_pos, head_dim/2, 2]; rotate-half layout on the first n_heads heads of each row."""
    T = qkv.shape[0]
    half = head_dim // 2
    cs = table[pos.long().clamp(0, table.shape[0] - 1)]  # [T, half, 2]
    cos, sin = cs[..., 0][:, None, :], cs[..., 1][:, None, :]
    x = qkv[:, : n_heads * head_dim].reshape(T, n_heads, head_dim).float()
    lo, hi = x[..., :half], x[..., half:]
    out = torch.cat([lo * cos - hi * sin, hi * cos + lo * sin], dim=-1).to(qkv.dtype)
    return torch.cat([out.reshape(T, n_heads * head_dim), qkv[:, n_heads * head_dim:]], dim=1)


def swiglu(gu):
    Fh = gu.shape[1] // 2
    g, u = gu[:, :Fh].float(), gu[:, Fh:].float()
    return (F.silu(g) * u).to(gu.dtype)


def embedding(ids, table):
    return table[ids.long()]


def attention_varlen(q, k, v, cu_seqlens, scale):
    """Causal attention per document of a packed stream. q [T,Hq,D], k/v [T,Hkv,D]."""
    T, Hq, D = q.shape
    Hkv = k.shape[1]
    rep = Hq // Hkv
    out = torch.empty_like(q)
    cu = cu_seqlens.tolist()
    for s, e in zip(cu[:-1], cu[1:]):
        if e <= s:
            continue
        qs = q[s:e].float().transpose(0, 1)                      # [Hq, L, D]
        ks = k[s:e].float().transpose(0, 1).repeat_interleave(rep, 0)
        vs = v[s:e].float().transpose(0, 1).repeat_interleave(rep, 0)
        att = (qs @ ks.transpose(1, 2)) * scale
        L = e - s
        mask = torch.ones(L, L, dtype=torch.bool, device=q.device).tril()
        att = att.masked_fill(~mask, float("-inf")).softmax(-1)
        out[s:e] = (att @ vs).transpose(0, 1).to(q.dtype)
    return out


def fused_logprob(h, w, labels, temperature=1.0, want_entropy=False):
    logits = h.float() @ w.float().t()
    ent = None
    if want_entropy:
        lse0 = torch.logsumexp(logits, -1)
        p = torch.softmax(logits, -1)
        ent = lse0 - (p * logits).sum(-1)
    z = logits / temperature
    logp = z.gather(-1, labels.long()[:, None]).squeeze(-1) - torch.logsumexp(z, -1)
    return logp, ent


def paged_decode_attention(q, k_cache, v_cache, block_table, seq_lens, scale, page=128):
    """q [B,Hq,D]; caches [num_pages*page, Hkv, D]."""
    B, Hq, D = q.shape
    Hkv = k_cache.shape[1]
    rep = Hq // Hkv
    out = torch.empty_like(q)
    for b in range(B):
        L = int(seq_lens[b])
        n = (L + page - 1) // page
        idx = torch.cat([torch.arange(page, device=q.device) + int(block_table[b, i]) * page for i in range(n)])[:L]
        ks = k_cache[idx].float().transpose(0, 1).repeat_interleave(rep, 0)  # [Hq, L, D]
        vs = v_cache[idx].float().transpose(0, 1).repeat_interleave(rep, 0)
        att = torch.einsum("hd,hld->hl", q[b].float(), ks) * scale
        out[b] = torch.einsum("hl,hld->hd", att.softmax(-1), vs).to(q.dtype)
    return out


# ---------------------------------------------------------------------------------------------- hybrid layers
def rmsnorm_f32(x, w, n, eps):
    y = x * torch.rsqrt(x[:, :n].pow(2).mean(-1, keepdim=True) + eps)
    return (y * w.float()).to(w.dtype)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def mamba2(p, m, wt, ring, state, batch, eps, out, out_pad, ff_col, ff):
    """p fp32 [T, N]; see ``ops.hybrid.mamba2``."""
    inner, cc, gn = m.inner, m.conv_channels, m.groups * m.state
    rep = m.heads // m.groups
    a = -wt.a_log.float().exp()
    for i in range(batch.n):
        t0, t1, start, row = int(batch.cu[i]), int(batch.cu[i + 1]), int(batch.start[i]), int(batch.row[i])
        idle = batch.active is not None and int(batch.active[i]) == 0
        u = p[t0:t1, inner:inner + cc]
        past = [ring[row, (start - k) % m.conv].float() if start - k >= 0 else torch.zeros(cc)
                for k in range(m.conv - 1, 0, -1)]
        ext = torch.cat([torch.stack(past), u]) if past else u
        conv = F.conv1d(ext.t()[None], wt.conv.float()[:, None], wt.conv_bias.float(), groups=cc)[0].t()
        xbc = F.silu(conv).to(out.dtype).float()
        dt = F.softplus(p[t0:t1, inner + cc:inner + cc + m.heads] + wt.dt_bias.float(), threshold=30.0)
        s = torch.zeros_like(state[row]) if start == 0 else state[row].clone()
        x = xbc[:, :inner].view(-1, m.heads, m.vdim)
        b = xbc[:, inner:inner + gn].view(-1, m.groups, m.state).repeat_interleave(rep, 1)
        c = xbc[:, inner + gn:].view(-1, m.groups, m.state).repeat_interleave(rep, 1)
        for t in range(t1 - t0):
            s = (a * dt[t]).exp()[:, None, None] * s + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
            y = torch.einsum("hnp,hn->hp", s, c[t]) + wt.d.float()[:, None] * x[t]
            y = (y.reshape(-1).to(out.dtype).float() * F.silu(p[t0 + t, :inner])).view(m.norm_groups, -1)
            y = (y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps)).reshape(-1)
            out[t0 + t, :inner] = (y * wt.norm.float()).to(out.dtype)
        if not idle:
            state[row] = s
            for o in range(max(0, t1 - t0 - (m.conv - 1)), t1 - t0):
                ring[row, (start + o) % m.conv] = u[o].to(ring.dtype)
    out[:, out_pad:out_pad + ff] = F.relu(p[:, ff_col:ff_col + ff]).square().to(out.dtype)


def window_attention(p, m, table, k_cache, v_cache, batch, out, out_pad, ff_col, ff, page):
    """p fp32 [T, N]; see ``ops.hybrid.window_attention``."""
    T, half = p.shape[0], m.rot_dims // 2

    def turn(x):
        if half == 0:
            return x
        cs = table[batch.pos.long()]
        cos, sin = cs[:, None, :, 0], cs[:, None, :, 1]
        u, v = x[..., :half], x[..., half:2 * half]
        return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], -1)

    nq, nk = m.heads * m.dim, m.kv_heads * m.dim
    q = turn(p[:, :nq].view(T, m.heads, m.dim)).to(out.dtype).float()
    slots = batch.slots.long()
    if m.kv_from is None:
        k_cache[slots, :, :m.dim] = turn(p[:, nq:nq + nk].view(T, m.kv_heads, m.dim)).to(k_cache.dtype)
        v_cache[slots, :, :m.vdim] = p[:, nq + nk:nq + nk + m.kv_heads * m.vdim].view(T, m.kv_heads, m.vdim).to(v_cache.dtype)
    rep = m.heads // m.kv_heads
    for i in range(batch.n):
        t0, t1, start = int(batch.cu[i]), int(batch.cu[i + 1]), int(batch.start[i])
        last = start + t1 - t0
        j = torch.arange(last)
        at = batch.block_table[i].long()[j // page] * page + j % page
        k = k_cache[at, :, :m.dim].float().repeat_interleave(rep, 1)
        v = v_cache[at, :, :m.vdim].float().repeat_interleave(rep, 1)
        s = torch.einsum("thd,jhd->htj", q[t0:t1], k) * m.scale
        ii = torch.arange(start, last)[:, None]
        seen = j[None] <= ii
        if m.window is not None:
            seen &= (ii - j[None] < m.window) | (j[None] < m.keep_first)
        s = s.masked_fill(~seen, float("-inf"))
        if m.sink:
            s = torch.cat([s, torch.zeros(*s.shape[:2], 1)], -1)
        w = s.softmax(-1)[..., :last]
        out[t0:t1, :m.out_cols] = torch.einsum("htj,jhd->thd", w, v).reshape(t1 - t0, -1).to(out.dtype)
    out[:, out_pad:out_pad + ff] = F.relu(p[:, ff_col:ff_col + ff]).square().to(out.dtype)
