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


def bigram_embedding(tokens, prev, embed, table, spec, positions=None, freq=None):
    x = embed[tokens.long()].float()
    if table is not None:
        buckets, mp, mc = spec
        row = (prev.long() * mp + tokens.long() * mc) % buckets
        x = x + table[torch.where(prev < 0, torch.full_like(row, buckets), row)].float()
    if freq is not None:
        ang = positions.double()[:, None] * freq[None]
        x = x + torch.stack([ang.sin(), ang.cos()], -1).flatten(1)[:, : x.shape[1]].float()
    return x, x.to(embed.dtype)


def output_norm_residual(x, y, nw, ls, eps, final_w=None):
    yf = y.float()
    x.add_(yf * torch.rsqrt(yf.square().mean(-1, keepdim=True) + eps) * nw.float() * ls.float())
    if final_w is None:
        return x, x.to(y.dtype)
    return x, (x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * final_w.float()).to(y.dtype)


def clamped_glu(h, limit, alpha, shift=1.0):
    g, u = h.float().chunk(2, -1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + shift)).to(h.dtype)


def aside(a):
    if a is None:
        return
    if a.logits is not None:
        a.weights, a.index = topk_softmax(a.logits, a.top) if a.routing is None else topk_grouped(a.logits, a.correction, a.top, a.routing)
    if a.glu_in is not None:
        a.glu_out.copy_(clamped_glu(a.glu_in[:, : 2 * a.glu_out.shape[1]], a.limit, a.alpha, a.shift))


def rotate_pairs(x, positions, freq, magnitude):
    """x [T, ..., 2·len(freq)], interleaved pairs."""
    ang = positions.double()[:, None] * freq.double()[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freq.numel(),)
    c, s = (ang.cos() * magnitude).float().view(shape), (ang.sin() * magnitude).float().view(shape)
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2).to(x.dtype)


def gated(o, gate):
    return o if gate is None else o * torch.sigmoid(gate.float())


def latent_attention(q, kv, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps, gate=None):
    T, H, dtype = q.shape[0], lay.heads, q.dtype
    q = q.reshape(T, H, lay.dim + lay.rot)
    qn, qr = q[..., :lay.dim].float(), rotate_pairs(q[..., lay.dim:], meta.positions, freq, magnitude).float()
    flat = cache.view(-1, lay.pitch)
    if kv_norm is not None:
        kv = kv[:, : lay.rank + lay.rot].float()
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
    return gated(out.reshape(T, H * lay.vdim), gate).to(dtype)


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


def sum_norm(x, to, addends, extra, nw, eps, shift=0.0, gain=1.0, nw2=None):
    s = x.clone()
    for a in addends:
        s += a.y.float() if a.scale is None else a.y.float() * a.scale.float()
    if extra is not None:
        s += extra
    if to is not None:
        to.copy_(s)
    n = s * torch.rsqrt(s.square().mean(-1, keepdim=True) + eps)
    return tuple(None if w is None else (n * (w.float() + shift) * gain).to(w.dtype) for w in (nw, nw2))


def projections(h, w, w2=None, b2=None):
    logits = None
    if w2 is not None:
        logits = h.float() @ w2.float().T + b2.float()
    return h @ w.T, logits


def topk_softmax(logits, k):
    top = logits.float().topk(k, -1)
    return torch.softmax(top.values, -1), top.indices.int()


def topk_grouped(logits, correction, k, r):
    s = torch.sigmoid(logits.float())
    c = s if correction is None else s + correction.float()
    T, E = c.shape
    by_group = c.view(T, r.groups, -1)
    worth = by_group.topk(min(2, by_group.shape[-1]), -1).values.sum(-1)
    closed = torch.ones(T, r.groups, dtype=torch.bool).scatter(1, worth.topk(r.keep, -1).indices, False)
    idx = by_group.masked_fill(closed[..., None], float("-inf")).view(T, E).topk(k, -1).indices
    w = s.gather(1, idx)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * r.scale, idx.int()


def routed_experts(h, w13, w2, weights, index, limit=0.0, alpha=0.0, shift=1.0, ungated=False):
    out = torch.zeros(h.shape, dtype=torch.float32)
    for e in range(w13.shape[0]):
        t, j = torch.where(index == e)
        if t.numel():
            up = h[t] @ w13[e].T
            y = (up.float().relu().square().to(h.dtype) if ungated else clamped_glu(up, limit, alpha, shift)) @ w2[e].T
            out.index_add_(0, t, y.float() * weights[t, j][:, None])
    return out.to(h.dtype)


def windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps, bias=None, gate=None):
    T, H, G = proj.shape[0], lay.heads, lay.kv_heads
    q = proj[:, : H * lay.dim]

    def prepared(x, w, heads):
        x = x.float()
        if w is not None:
            x = x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * w.float()
        x = x.view(T, heads, lay.dim)
        if lay.rot:
            x = torch.cat([rotate_pairs(x[..., : lay.rot], meta.positions, freq, magnitude), x[..., lay.rot:]], -1)
        return x.to(proj.dtype)

    q = prepared(q, q_norm, H)
    if lay.writes:
        k, v = proj[:, H * lay.dim: lay.rows].split([G * lay.dim, G * lay.vdim], -1)
        v = v.reshape(T, G, lay.vdim)
        if lay.value_norm:
            v = v.float() * torch.rsqrt(v.float().square().mean(-1, keepdim=True) + eps)
        ok = meta.slot_mapping >= 0
        at = meta.slot_mapping[ok].long()
        kc.view(-1, G, lay.dim)[at] = prepared(k, k_norm, G)[ok].to(kc.dtype)
        vc.view(-1, G, lay.vdim)[at] = v[ok].to(vc.dtype)
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
        if lay.chunk:
            seen &= pos[:, None] // lay.chunk == keys[None] // lay.chunk
        if bias is not None:
            r1, r2 = (r.float()[:, None, None] for r in bias)
            sc = sc - r1 * torch.log1p(r2 * (pos[:, None] - keys[None]).clamp(min=0).float())
        sc = sc.masked_fill(~seen[None], float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.float()[:, None, None].expand(H, s1 - s0, 1)], -1)
        p = torch.softmax(sc, -1)[..., : keys.numel()]
        o = torch.einsum("hts,shd->thd", p, vv).reshape(s1 - s0, -1)
        out[s0:s1] = gated(o, gate[s0:s1] if gate is not None else None).to(out.dtype)
    return out


def differential_attention(proj, lay, kc, vc, meta, scale, diff, temperature, lvec, q_norm, k_norm, eps):
    T, H, G, d = proj.shape[0], lay.heads, lay.kv_heads, lay.dim

    def normed(rows, heads, w):
        x = rows.float().reshape(T, heads, 2, d)
        return x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * w.float()

    q = normed(proj[:, : lay.q_rows], H, q_norm)
    if temperature is not None:
        coef, every = temperature
        q = q * (1 + coef * torch.log(torch.floor((meta.positions.double() + 1) / every) + 1)).float()[:, None, None, None]
    q = q.to(proj.dtype).float()
    bs = kc.shape[1]
    if k_norm is not None:
        k, v = proj[:, lay.q_rows: lay.gate_at].split([G * 2 * d, G * lay.vdim], -1)
        ok = meta.slot_mapping >= 0
        at = meta.slot_mapping[ok].long()
        kc.view(-1, G, 2 * d)[at] = normed(k, G, k_norm).flatten(2)[ok].to(kc.dtype)
        vc.view(-1, G, lay.vdim)[at] = v.reshape(T, G, lay.vdim)[ok].to(vc.dtype)
    l = lvec.float()
    lam = torch.exp((l[0] * l[1]).sum()) - torch.exp((l[2] * l[3]).sum()) + diff
    out = torch.zeros(T, H, lay.vdim)
    for b, s0, s1 in _sequences(meta, T):
        if s1 == s0 or int(meta.slot_mapping[s0]) < 0:
            continue
        pos = meta.positions[s0:s1].long()
        keys = torch.arange(int(pos[-1]) + 1)
        slot = meta.block_table[b, keys // bs].long() * bs + keys % bs
        kk = kc.view(-1, G, 2, d)[slot].float().repeat_interleave(H // G, 1)
        vv = vc.view(-1, G, lay.vdim)[slot].float().repeat_interleave(H // G, 1)
        sc = torch.einsum("thmd,shmd->mhts", q[s0:s1], kk) * scale
        p = torch.softmax(sc.masked_fill(keys[None] > pos[:, None], float("-inf")), -1)
        out[s0:s1] = torch.einsum("hts,shd->thd", p[0] - lam * p[1], vv)
    out = out * torch.rsqrt(out.square().mean(-1, keepdim=True) + eps) * (1 - diff)
    gate = proj[:, lay.gate_at: lay.gate_at + H].float()
    return (out * torch.sigmoid(gate)[..., None]).reshape(T, H * lay.vdim).to(proj.dtype)


def short_conv(x, w, b, ring, slot, p0):
    """silu of the causal convolution of a piece's rows that starts at position p0, from and to the ring of its last inputs (rounded to
    the rows' dtype, as floats)."""
    taps, n = w.shape[1], x.shape[0]
    before = [ring[slot, p % taps] if p >= 0 else torch.zeros(x.shape[1]) for p in range(p0 - taps + 1, p0)]
    rows = torch.cat([torch.stack(before), x.float()]) if before else x.float()
    act = sum(rows[k: k + n] * w[:, k].float() for k in range(taps))
    if ring is not None:
        for t in range(max(0, n - taps + 1), n):
            ring[slot, (p0 + t) % taps] = x[t].float()
    return torch.nn.functional.silu(act if b is None else act + b.float()).to(x.dtype).float()


def delta_rule(proj, lay, conv, w_a, w_g, A_log, dt_bias, norm_w, state, ring, meta, eps):
    T, H, G, K, V = proj.shape[0], lay.heads, lay.kv_heads, lay.dim, lay.vdim
    raw = proj[:, lay.channels: lay.gate_at] @ w_a.T
    logg = -torch.exp(A_log.float())[:, None] * torch.nn.functional.softplus((raw.float() + dt_bias.float()).view(T, H, K), threshold=1e9)
    gate = proj[:, lay.gate_at: lay.beta_at] @ w_g.T
    beta = torch.sigmoid(proj[:, lay.beta_at: lay.beta_at + H].float())
    out = torch.zeros(T, H, V)
    for b, s0, s1 in _sequences(meta, T):
        slot = int(meta.state_slots[b])
        if slot < 0 or s1 == s0:
            continue
        p0 = int(meta.positions[s0])
        q, k, v = short_conv(proj[s0:s1, : lay.channels], conv, None, ring, slot, p0).split([G * K, G * K, H * V], -1)
        q, k = (x.reshape(-1, G, K) * torch.rsqrt(x.reshape(-1, G, K).square().sum(-1, keepdim=True) + 1e-6) for x in (q, k))
        q, k = (x.repeat_interleave(H // G, 1) for x in (q * K ** -0.5, k))
        v = v.reshape(-1, H, V)
        S = state[slot].clone() if p0 > 0 else torch.zeros_like(state[slot])
        for i, t in enumerate(range(s0, s1)):
            S = S * torch.exp(logg[t])[:, :, None]
            u = beta[t][:, None] * (v[i] - torch.einsum("hkv,hk->hv", S, k[i]))
            S = S + k[i][:, :, None] * u[:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, q[i])
        state[slot] = S
    out = out.to(proj.dtype).float()
    out = out * torch.rsqrt(out.square().mean(-1, keepdim=True) + eps) * norm_w.float()
    return (out.reshape(T, H * V) * torch.sigmoid(gate.float())).to(proj.dtype)


def residual_norm(x, y, yn, mult, nw, eps, dtype, gain=1.0):
    if y is not None:
        yf = y.float()
        x.add_(mult * (yf if yn is None else yf * torch.rsqrt(yf.square().mean(-1, keepdim=True) + eps) * yn.float()))
    return (x if nw is None else x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * nw.float() * gain).to(dtype)


def xielu(z, act):
    f = z.float()
    a, b = torch.nn.functional.softplus(act.float(), threshold=1e9)
    neg = f.clamp(max=0)
    return (0.5 * f + torch.where(f > 0, a * f * f, (0.5 + b) * (torch.expm1(neg) - neg))).to(z.dtype)


def gelu_times_rows(z, tokens, table, col):
    e = table[tokens.long(), col: col + z.shape[1]].float()
    return (torch.nn.functional.gelu(z.float(), approximate="tanh") * e).to(z.dtype)


def softcap_(logits, cap, exact=False):
    return logits.div_(cap).tanh_().mul_(cap)


def state_space(proj, lay, conv, conv_b, dt_bias, A_log, D, state, ring, meta):
    T, H, V, N, G, taps = proj.shape[0], lay.heads, lay.vdim, lay.state, lay.groups, lay.taps
    z, xbc, dt = proj[:, : lay.inner + lay.channels + H].split([lay.inner, lay.channels, H], -1)
    dt = torch.nn.functional.softplus(dt.float() + dt_bias.float(), threshold=1e9)
    decay = torch.exp(-torch.exp(A_log.float()) * dt)
    out = torch.zeros(T, H, V)
    for b, s0, s1 in _sequences(meta, T):
        slot = int(meta.state_slots[b])
        if slot < 0 or s1 == s0:
            continue
        p0 = int(meta.positions[s0])
        x, B, C = short_conv(xbc[s0:s1], conv, conv_b, ring, slot, p0).split([lay.inner, G * N, G * N], -1)
        x = x.view(-1, H, V)
        B, C = (y.reshape(-1, G, N).repeat_interleave(H // G, 1) for y in (B, C))
        S = state[slot].clone() if p0 > 0 else torch.zeros_like(state[slot])
        for i, t in enumerate(range(s0, s1)):
            S = S * decay[t][:, None, None] + (dt[t][:, None] * B[i])[:, :, None] * x[i][:, None, :]
            out[t] = torch.einsum("hnv,hn->hv", S, C[i]) + D.float()[:, None] * x[i]
        state[slot] = S
    return (out.reshape(T, lay.inner) * torch.nn.functional.silu(z.float())).to(proj.dtype)


def part_norm(x, w, parts, eps):
    p = x.float().unflatten(-1, (parts, -1))
    return ((p * torch.rsqrt(p.square().mean(-1, keepdim=True) + eps)).flatten(-2) * w.float()).to(x.dtype)
