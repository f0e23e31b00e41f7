"""Plain-PyTorch statements of the ops in `mixers.py` (CPU tensors: plumbing tests without a GPU).  fp32 math, loops over sequences."""
from __future__ import annotations

import torch


def _sequences(meta, T: int):
    """(row b, first new token, end) of every sequence of a ragged batch; a decode step has one token per row."""
    rg = meta.ragged
    if rg.cu_q is None:
        return [(b, b, b + 1) for b in range(T)]
    cu = rg.cu_q.tolist()
    return [(b, cu[b], cu[b + 1]) for b in range(len(cu) - 1)]


def bigram_embedding(tokens, prev, embed, table, spec):
    x = embed[tokens.long()].float()
    if table is not None:
        buckets, mp, mc = spec
        row = (prev.long() * mp + tokens.long() * mc) % buckets
        x = x + table[torch.where(prev < 0, torch.full_like(row, buckets), row)].float()
    return x, x.to(embed.dtype)


def output_norm_residual(x, y, nw, ls, eps, final_w=None):
    yf = y.float()
    x.add_(yf * torch.rsqrt(yf.square().mean(-1, keepdim=True) + eps) * nw.float() * ls.float())
    if final_w is None:
        return x, x.to(y.dtype)
    return x, (x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * final_w.float()).to(y.dtype)


def clamped_glu(h, limit, alpha):
    g, u = h.float().chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + 1)).to(h.dtype)


def rotate_pairs(x, positions, freq, magnitude):
    """x [T, ..., 2·len(freq)], interleaved pairs."""
    ang = positions.double()[:, None] * freq.double()[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freq.numel(),)
    c, s = (ang.cos() * magnitude).float().view(shape), (ang.sin() * magnitude).float().view(shape)
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2).to(x.dtype)


def latent_attention(proj, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps):
    T, H = proj.shape[0], lay.heads
    q = proj[:, :lay.q_rows].view(T, H, lay.dim + lay.rot)
    qn, qr = q[..., :lay.dim].float(), rotate_pairs(q[..., lay.dim:], meta.positions, freq, magnitude).float()
    flat = cache.view(-1, lay.pitch)
    if kv_norm is not None:
        kv = proj[:, lay.q_rows:].float()
        c = kv[:, :lay.rank]
        c = c * torch.rsqrt(c.square().mean(-1, keepdim=True) + eps) * kv_norm.float()
        ok = meta.slot_mapping >= 0
        rows = torch.zeros(T, lay.pitch, dtype=cache.dtype)
        rows[:, :lay.rank] = c.to(cache.dtype)
        rows[:, lay.rank_p:lay.rank_p + lay.rot] = rotate_pairs(kv[:, lay.rank:], meta.positions, freq, magnitude).to(cache.dtype)
        flat[meta.slot_mapping[ok].long()] = rows[ok]
    bs = cache.shape[1]
    wk, wv = w_ukv[: H * lay.dim].float().view(H, lay.dim, -1), w_ukv[H * lay.dim:].float().view(H, lay.vdim, -1)
    out = torch.zeros(T, H, lay.vdim)
    for b, s0, s1 in _sequences(meta, T):
        if s1 == s0 or int(meta.slot_mapping[s0]) < 0:
            continue
        pos = meta.positions[s0:s1].long()
        lo = max(0, int(pos[0]) - window + 1) if window else 0
        keys = torch.arange(lo, int(pos[-1]) + 1)
        rows = flat[meta.block_table[b, keys // bs].long() * bs + keys % bs].float()
        c, kr = rows[:, :lay.rank], rows[:, lay.rank_p:lay.rank_p + lay.rot]
        k = torch.einsum("sr,hdr->shd", c, wk)
        v = torch.einsum("sr,hdr->shd", c, wv)
        sc = (torch.einsum("thd,shd->hts", qn[s0:s1], k) + torch.einsum("thd,sd->hts", qr[s0:s1], kr)) * scale
        seen = keys[None] <= pos[:, None]
        if window:
            seen &= pos[:, None] - keys[None] < window
        sc = sc.masked_fill(~seen[None], float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.float()[:, None, None].expand(H, s1 - s0, 1)], -1)
        p = torch.softmax(sc, -1)[..., : keys.numel()]
        out[s0:s1] = torch.einsum("hts,shd->thd", p, v)
    return out.reshape(T, H * lay.vdim).to(proj.dtype)


def linear_state(proj, H, dk, dv, decay, state, meta):
    T = proj.shape[0]
    a = torch.nn.functional.silu(proj[:, : H * (2 * dk + dv)].float())
    q, k, v = a.split([H * dk, H * dk, H * dv], -1)
    q, k, v = q.view(T, H, dk), k.view(T, H, dk), v.view(T, H, dv)
    out = torch.zeros(T, H, dv)
    for b, s0, s1 in _sequences(meta, T):
        slot = int(meta.state_slots[b])
        if slot < 0 or s1 == s0:
            continue
        S = state[slot].clone() if int(meta.positions[s0]) > 0 else torch.zeros_like(state[slot])
        for t in range(s0, s1):
            S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, q[t])
        state[slot] = S
    return out.reshape(T, H * dv).to(proj.dtype)


def gated_norm(o, w, gate, eps):
    of = o.float()
    return (of * torch.rsqrt(of.square().mean(-1, keepdim=True) + eps) * w.float() * torch.sigmoid(gate.float())).to(o.dtype)


def sum_norm(x, to, addends, extra, nw, eps):
    s = x.clone()
    for a in addends:
        s += a.y.float()
    if extra is not None:
        s += extra
    if to is not None:
        to.copy_(s)
    if nw is None:
        return None
    return (s * torch.rsqrt(s.square().mean(-1, keepdim=True) + eps) * nw.float()).to(nw.dtype)


def projections(h, w, w2=None, b2=None):
    logits = None
    if w2 is not None:
        logits = h.float() @ w2.float().T + b2.float()
    return h @ w.T, logits


def topk_softmax(logits, k):
    top = logits.float().topk(k, -1)
    return torch.softmax(top.values, -1), top.indices.int()


def routed_experts(h, w13, w2, weights, index, limit, alpha):
    out = torch.zeros(h.shape, dtype=torch.float32)
    for e in range(w13.shape[0]):
        t, j = torch.where(index == e)
        if t.numel():
            y = clamped_glu(h[t] @ w13[e].T, limit, alpha) @ w2[e].T
            out.index_add_(0, t, y.float() * weights[t, j][:, None])
    return out.to(h.dtype)


def windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps):
    T, H, G = proj.shape[0], lay.heads, lay.kv_heads
    q, k, v = proj[:, : lay.rows].split([H * lay.dim, G * lay.dim, G * lay.vdim], -1)

    def prepared(x, w, heads):
        x = x.float()
        if w is not None:
            x = x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * w.float()
        x = x.view(T, heads, lay.dim)
        if lay.rot:
            x = torch.cat([rotate_pairs(x[..., : lay.rot], meta.positions, freq, magnitude), x[..., lay.rot:]], -1)
        return x.to(proj.dtype)

    q, k = prepared(q, q_norm, H), prepared(k, k_norm, G)
    ok = meta.slot_mapping >= 0
    at = meta.slot_mapping[ok].long()
    kc.view(-1, G, lay.dim)[at] = k[ok].to(kc.dtype)
    vc.view(-1, G, lay.vdim)[at] = v.reshape(T, G, lay.vdim)[ok].to(vc.dtype)
    bs = kc.shape[1]
    out.zero_()
    for b, s0, s1 in _sequences(meta, T):
        if s1 == s0 or int(meta.slot_mapping[s0]) < 0:
            continue
        pos = meta.positions[s0:s1].long()
        keys = torch.arange(int(pos[-1]) + 1)
        slot = meta.block_table[b, keys // bs].long() * bs + keys % bs
        kk = kc.view(-1, G, lay.dim)[slot].float().repeat_interleave(H // G, 1)
        vv = vc.view(-1, G, lay.vdim)[slot].float().repeat_interleave(H // G, 1)
        sc = torch.einsum("thd,shd->hts", q[s0:s1].float(), kk) * scale
        seen = keys[None] <= pos[:, None]
        if lay.window:
            seen &= (pos[:, None] - keys[None] < lay.window) | (keys[None] < lay.keep)
        sc = sc.masked_fill(~seen[None], float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.float()[:, None, None].expand(H, s1 - s0, 1)], -1)
        p = torch.softmax(sc, -1)[..., : keys.numel()]
        out[s0:s1] = torch.einsum("hts,shd->thd", p, vv).reshape(s1 - s0, -1).to(out.dtype)
    return out
