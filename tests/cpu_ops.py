"""A CPU stand-in for the kernel library, for tests only.

The engine has no CPU path.  To check its host logic (batch building, block tables, page
reuse, the run order of layers, the scheduler) on a machine without a GPU, the tests hand
the model this object in place of ``KernelOps``.  It offers the same operations on CPU
tensors with torch arithmetic in float32; it is not bit-exact with the CUDA kernels and is
never imported by the package.
"""
from __future__ import annotations

import math

import torch


class CpuOps:
    def __init__(self, dtype="float32"):
        self.dtype = dtype
        self.act_dtype = torch.float32 if dtype == "float32" else torch.bfloat16
        self.kind = "f32" if dtype == "float32" else "bf16"
        self.launches = 0

    def embed_rows(self, table, tokens, out, scale=1.0):
        out.copy_(table[tokens.long()].float() * scale)

    def rmsnorm_residual(self, d, weight, eps, x, next_weight=None, next_eps=0.0, next_out=None):
        x += (d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps)) * weight
        if next_out is not None and next_weight is None:
            next_out.copy_(x.to(next_out.dtype))
        elif next_out is not None:
            self.rmsnorm(x, next_weight, next_eps, next_out)

    # -- scored attention and the linear recurrence (stand-ins shaped like the kernels' interface) --
    def scored_attention_tile_heights(self, group, dim, vdim):
        return [max(1, 32 // group)]

    def qkv_prepare(self, u, conv_w, conv_state, q_norm, k_norm, eps, cos, sin, ctx, block_table, kcache, vcache, q_out,
                    heads, write_kv_heads, dim, vdim, conv_wt=None, bias=None, vmix_src=None, vmix_lambda=None, v_keep=None,
                    half_layout=False, v_heads=None):
        n, cols = u.shape
        page = kcache.shape[2]
        if bias is not None:
            u = u + bias
            if conv_state is not None:
                conv_state = conv_state + bias
        y = u.clone()
        if conv_w is not None:
            taps = conv_w.shape[1]
            y.zero_()
            for r in range(n):
                s = int(ctx.row_seq[r])
                row0, pos0, slot = int(ctx.seq_row0[s]), int(ctx.seq_pos0[s]), int(ctx.seq_slot[s])
                for j in range(taps):
                    back = taps - 1 - j
                    if int(ctx.pos[r]) - back < 0:
                        continue
                    src = u[r - back] if r - back >= row0 else conv_state[slot, taps - 1 - (row0 - (r - back))]
                    y[r] += conv_w[:, j] * src
        p = ctx.pos.long()

        def finish(t, size, w):
            t = t.reshape(n, -1, size)
            if w is not None:
                t = t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
            if cos is not None and half_layout:
                t = self._turn(t, p, cos, sin, True)
            elif cos is not None:
                pairs = cos.shape[1]
                c, sn = cos[p][:, None, :], sin[p][:, None, :]
                a, b = t[..., 0:2 * pairs:2].clone(), t[..., 1:2 * pairs:2].clone()
                t = t.clone()
                t[..., 0:2 * pairs:2] = a * c - b * sn
                t[..., 1:2 * pairs:2] = b * c + a * sn
            return t

        q_out.copy_(finish(y[:, :heads * dim], dim, q_norm).reshape(n, -1).to(q_out.dtype))
        if not write_kv_heads:
            return
        g = write_kv_heads
        k = finish(y[:, heads * dim:(heads + g) * dim], dim, k_norm)
        v = y[:, (heads + g) * dim:].reshape(n, v_heads or g, vdim) if vcache is not None else None
        if vmix_src is not None:
            lam = float(vmix_lambda[0])
            v = (1.0 - lam) * v + lam * vmix_src.reshape(n, g, vdim)
        if v_keep is not None:
            v_keep.copy_(v.reshape(n, -1))
        for r in range(n):
            blk = int(block_table[int(ctx.row_seq[r]), int(p[r]) // page])
            kcache[blk, :, int(p[r]) % page, :] = k[r].to(kcache.dtype)
            if v is not None:
                vcache[blk, :, int(p[r]) % page, :] = v[r].to(vcache.dtype)

    def conv_state_update(self, u, state, ctx, taps, tiles):
        t_seq, t_row0, t_rows, count = tiles
        for i in range(count):
            s, row0, cnt = int(t_seq[i]), int(t_row0[i]), int(t_rows[i])
            slot, pos0 = int(ctx.seq_slot[s]), int(ctx.seq_pos0[s])
            old = state[slot].clone()
            for j in range(taps - 1):
                pos = pos0 + cnt - (taps - 1) + j
                if pos < 0:
                    state[slot, j] = 0
                elif pos >= pos0:
                    state[slot, j] = u[row0 + pos - pos0]
                else:
                    state[slot, j] = old[pos - pos0 + taps - 1]

    def scored_attention(self, q, kcache, vcache, block_table, out, heads, kv_heads, dim, vdim, scale, softcap, sink,
                         slopes, window, ctx, dist_a=None, dist_b=None, sinks=None, keep_first=0, chunk=0, difference=None):
        n = q.shape[0]
        if difference is not None:
            lam, keep, eps, gate, gate_group = difference
            maps = []
            for m in range(2):
                o = torch.zeros(n, heads // 2 * vdim)
                self.scored_attention(q.reshape(n, heads, dim)[:, m::2].reshape(n, -1), kcache[:, m::2], vcache, block_table, o, heads // 2,
                                      kv_heads // 2, dim, vdim, scale, softcap, sink, slopes, window, ctx, keep_first=keep_first, chunk=chunk)
                maps.append(o.view(n, heads // 2, vdim))
            o = maps[0] - float(lam) * maps[1]
            o = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * keep).reshape(n, -1)
            if gate is not None:
                o = o * torch.sigmoid(gate).repeat_interleave(gate_group, 1)
            out.copy_(o.to(out.dtype))
            return
        page = kcache.shape[2]
        grp = heads // kv_heads
        for r in range(n):
            p = int(ctx.pos[r])
            lo = max(0, p - window + 1) if window else p // chunk * chunk if chunk else 0
            idx = torch.arange(lo, p + 1)
            if window and keep_first and lo > 0:
                idx = torch.cat([torch.arange(0, min(keep_first, lo)), idx])
            blocks = block_table[int(ctx.row_seq[r])][(idx // page).long()].long()
            slots = (idx % page).long()
            k = kcache[blocks, :, slots, :].float().repeat_interleave(grp, dim=1)
            v = k if vcache is None else vcache[blocks, :, slots, :].float().repeat_interleave(grp, dim=1)
            s = torch.einsum("hd,khd->hk", q[r].float().view(heads, dim), k) * scale
            if softcap:
                s = softcap * torch.tanh(s / softcap)
            if slopes is not None:
                s = s - slopes[:, None] * (p - idx).float()[None, :]
            if dist_a is not None:
                s = s - dist_a[:, None] * torch.log1p(dist_b[:, None] * (p - idx).float()[None, :])
            m = s.max(-1, keepdim=True).values
            e = torch.exp(s - m)
            extra = torch.exp((sinks[:, None] if sinks is not None else 0.0) - m) if sink else 0.0
            den = e.sum(-1, keepdim=True) + extra
            out[r] = torch.einsum("hk,khd->hd", e / den, v).reshape(-1).to(out.dtype)

    # -- kernels on the stream, the second embedding table and the routed feed-forward (stand-ins) --
    def embed_pair(self, table, pair_table, ctx, last_token, out, scale, buckets, mul_prev, mul_cur):
        for r in range(out.shape[0]):
            s, tok = int(ctx.row_seq[r]), int(ctx.tokens[r])
            row = buckets
            if int(ctx.pos[r]) > 0:
                prev = int(ctx.tokens[r - 1]) if r > int(ctx.seq_row0[s]) else int(last_token[int(ctx.seq_slot[s])])
                row = (prev * mul_prev + tok * mul_cur) % buckets
            out[r] = table[tok].float() * scale + pair_table[row].float()

    def last_token_update(self, ctx, last_token, tiles):
        t_seq, t_row0, t_rows, count = tiles
        for i in range(count):
            last_token[int(ctx.seq_slot[int(t_seq[i])])] = int(ctx.tokens[int(t_row0[i]) + int(t_rows[i]) - 1])

    def norm_conv(self, x, weight, eps, taps_t, state, state_col0, ctx, out, normed, normed_col0):
        n, width = out.shape
        taps = taps_t.shape[0]
        h = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight
        normed[:, normed_col0:normed_col0 + width] = h
        for r in range(n):
            s = int(ctx.row_seq[r])
            row0, slot = int(ctx.seq_row0[s]), int(ctx.seq_slot[s])
            acc = torch.zeros(width)
            for j in range(taps):
                back = taps - 1 - j
                if int(ctx.pos[r]) - back < 0:
                    continue
                src = h[r - back] if r - back >= row0 else state[slot, taps - 1 - (row0 - (r - back)), state_col0:state_col0 + width]
                acc += taps_t[j] * src
            out[r] = (h[r] + acc).to(out.dtype)

    def scaled_add(self, x, scale, d, rounded=None):
        if scale is not None:
            x += scale * d
        if rounded is not None:
            rounded.copy_(x.to(rounded.dtype))

    def token_gate(self, t, table, col0, tokens, out):
        e = table[tokens.long()][:, col0:col0 + t.shape[1]].float()
        out.copy_((torch.nn.functional.gelu(t, approximate="tanh") * e).to(out.dtype))

    def normed_add_mix(self, x, y, weight, eps, mult, history, index, mix):
        if y is not None:
            x += mult * (y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps) * weight)
        if history is not None:
            width = x.shape[1]
            history[:, index * width:(index + 1) * width] = x
            x.copy_(sum(mix[j] * history[:, j * width:(j + 1) * width] for j in range(index + 1)))

    def copy_history(self, x, history):
        history[:, :x.shape[1]] = x

    def glu_clamped(self, gate_up, out, limit, alpha):
        inter = out.shape[1]
        g = gate_up[:, :inter].float().clamp(max=limit)
        u = gate_up[:, inter:].float().clamp(-limit, limit)
        out.copy_((g * torch.sigmoid(alpha * g) * (u + 1.0)).to(out.dtype))

    def route(self, logits, correction, groups, keep, top, weight_scale, chosen, weights, softmax_top=False, scoring=None,
              group_max=False, sum_eps=None, lists=None):
        if lists is not None:
            self.route(logits, correction, groups, keep, top, weight_scale, chosen, weights, softmax_top, scoring, group_max, sum_eps)
            self.group_rows(chosen, logits.shape[1], *lists)
            return
        if scoring == "softmax":
            if correction is not None or not group_max:
                raise NotImplementedError("the stand-in keeps groups by their largest score")
            s = torch.softmax(logits, -1)
            n, experts = s.shape
            best = torch.sort(s.view(n, groups, -1).max(-1).values, dim=-1, descending=True, stable=True).indices[:, :keep]
            allowed = torch.zeros(n, groups).scatter_(1, best, 1.0).repeat_interleave(experts // groups, 1) > 0
            order = torch.sort(s.masked_fill(~allowed, -1.0), dim=-1, descending=True, stable=True).indices[:, :top]
            w = torch.gather(s, 1, order)
            chosen.copy_(order.to(torch.int32))
            weights.copy_((w if sum_eps is None else w / (w.sum(-1, keepdim=True) + sum_eps)) * weight_scale)
            return
        if groups != 1 or not softmax_top:
            raise NotImplementedError("the stand-in routes by the largest logits only")
        z = logits if correction is None else logits + correction
        order = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
        chosen.copy_(order.to(torch.int32))
        weights.copy_(torch.softmax(torch.gather(logits, 1, order), -1) * weight_scale)

    def group_rows(self, chosen, experts, group_off, tile_prefix, order, place):
        pairs = chosen.numel()
        self._entry_expert = chosen.reshape(-1).long().clone()
        order.reshape(-1)[:pairs] = torch.arange(pairs, dtype=torch.int32)
        place.reshape(-1)[:pairs] = torch.arange(pairs, dtype=torch.int32)

    def grouped_linear(self, x, w, out, rows, x_group_cols=0, o_group_cols=0, lists=None, order_div=1, gather=True,
                       sorted_x=None, activation=None, max_rows=0):
        if lists is None:
            # one product per group over the same rows: group g reads the columns g * x_group_cols .. + k of x
            # and writes the columns g * o_group_cols .. + n of out (w: [groups, n, k])
            groups, n_out, k = w.shape
            for g in range(groups):
                src = x[:rows, g * x_group_cols:g * x_group_cols + k].float()
                out[:rows, g * o_group_cols:g * o_group_cols + n_out] = (src @ w[g].float().t()).to(out.dtype)
            return
        order = lists[2].reshape(-1)
        for i in range(rows):
            src = x[int(order[i]) // order_div] if gather else x[i]
            out[i] = self._activated(w[int(self._entry_expert[i])].float() @ src.float(), activation).to(out.dtype)

    def combine(self, x, d, y, place, weights, top, scale=None, d_gate=None, then=None):
        n = x.shape[0]
        add = (weights[:, :, None] * y[place.reshape(-1).long()[:n * top]].view(n, top, -1)).sum(1)
        if d is not None:
            add = add + (d if d_gate is None else d * torch.sigmoid(d_gate))
        x += add if scale is None else scale * add
        if then is not None:
            self.tanh_norm(x, *then)

    def gla_scan(self, u, z, bias, tau, state, norm_w, eps, out, heads, dim, vdim, q_scale, ctx, tiles, scratch=None):
        t_seq, t_row0, t_rows, count = tiles
        hd, hv = heads * dim, heads * vdim
        for i in range(count):
            s, row0, cnt = int(t_seq[i]), int(t_row0[i]), int(t_rows[i])
            slot = int(ctx.seq_slot[s])
            S = state[slot]
            if int(ctx.seq_pos0[s]) == 0:
                S.zero_()
            for r in range(row0, row0 + cnt):
                qv = u[r, :hd].view(heads, dim) * q_scale
                kv = u[r, hd:2 * hd].view(heads, dim)
                vv = u[r, 2 * hd:2 * hd + hv].view(heads, vdim)
                gate = u[r, 2 * hd + hv:]
                decay = torch.exp(torch.nn.functional.logsigmoid(z[r] + bias) / tau).view(heads, dim)
                S.mul_(decay[:, :, None]).add_(kv[:, :, None] * vv[:, None, :])
                o = torch.einsum("hd,hde->he", qv, S)
                o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w
                out[r] = (o.reshape(-1) * gate * torch.sigmoid(gate)).to(out.dtype)

    def rmsnorm(self, x, weight, eps, out, rows=None):
        src = x if rows is None else x[rows.long()]
        inv = torch.rsqrt(src.pow(2).mean(-1, keepdim=True) + eps)
        out.copy_(((src * inv) * weight).to(out.dtype))

    def linear(self, x, w, out, residual=None, activation=None, then=None):
        y = x.float() @ w.float().t()
        if activation is not None:
            y = self._activated(y, activation)
        if residual is not None:
            y = residual + y
        out.copy_(y.to(out.dtype))
        if then is not None:
            self.tanh_norm(out, *then)

    # -- recurrences over a matrix of state per head, the token shift, two mixers side by side ------------
    @staticmethod
    def _activated(y, activation):
        return {None: lambda t: t, "relu2": lambda t: torch.relu(t) ** 2, "tanh": torch.tanh}[activation](y)

    def activate_rows(self, x, out, activation=None):
        out.copy_(self._activated(x, activation).to(out.dtype))

    def shift_mix(self, x, mu, last, out, ctx, keep=False):
        n, width = x.shape
        for r in range(n):
            s = int(ctx.row_seq[r])
            slot = last[int(ctx.seq_slot[s])].view(-1)
            if r > int(ctx.seq_row0[s]):
                before = x[r - 1]
            else:
                before = slot.clone() if int(ctx.pos[r]) > 0 else torch.zeros(width)
            out.view(-1, n, width)[:, r] = (x[r] + (before - x[r]) * mu).to(out.dtype)
            if keep:
                slot.copy_(x[r])

    def delta_prepare(self, u, beta_col, conv_t, conv_state, z, dt_bias, a_log, out, ctx, heads, kv_heads, dim, vdim, q_scale,
                      keep=False):
        n, (taps, channels) = u.shape[0], conv_t.shape
        y = torch.zeros(n, channels)
        for r in range(n):
            s = int(ctx.row_seq[r])
            row0, slot = int(ctx.seq_row0[s]), int(ctx.seq_slot[s])
            for j in range(taps):
                back = taps - 1 - j
                if int(ctx.pos[r]) - back < 0:
                    continue
                src = u[r - back, :channels] if r - back >= row0 else conv_state[slot, taps - 1 - (row0 - (r - back))]
                y[r] += conv_t[j] * src
            if keep and conv_state is not None:
                old = conv_state[slot].clone() if int(ctx.pos[r]) > 0 else torch.zeros(taps - 1, channels)
                if 0 < int(ctx.pos[r]) < taps - 1:
                    old[:taps - 1 - int(ctx.pos[r])] = 0
                conv_state[slot] = torch.cat([old[1:], u[r:r + 1, :channels]], 0)
        y = y * torch.sigmoid(y)
        qk = y[:, :2 * kv_heads * dim].reshape(n, 2 * kv_heads, dim)
        qk = qk / torch.sqrt(qk.pow(2).sum(-1, keepdim=True) + 1e-6)
        qk[:, :kv_heads] *= q_scale
        out[:, :2 * kv_heads * dim] = qk.reshape(n, -1)
        out[:, 2 * kv_heads * dim:channels] = y[:, 2 * kv_heads * dim:]
        out[:, channels:channels + heads] = torch.sigmoid(u[:, beta_col:beta_col + heads])
        out[:, channels + heads:channels + heads + kv_heads] = (qk[:, :kv_heads] * qk[:, kv_heads:]).sum(-1)
        soft = torch.nn.functional.softplus(z + dt_bias).view(n, heads, dim)
        z.copy_(torch.exp(-torch.exp(a_log).view(1, -1, 1) * soft).reshape(n, -1))

    def space_prepare(self, u, conv0, step0, conv_t, conv_b, conv_state, dt_bias, rate, out, out_step, ctx, keep=False):
        n, (taps, channels), heads = u.shape[0], conv_t.shape, rate.shape[0]
        x = u[:, conv0:conv0 + channels]
        for r in range(n):
            s = int(ctx.row_seq[r])
            row0, slot, pos = int(ctx.seq_row0[s]), int(ctx.seq_slot[s]), int(ctx.pos[r])
            inputs = torch.zeros(taps, channels)
            for j in range(taps):
                back = taps - 1 - j
                if pos - back >= 0:
                    inputs[j] = x[r - back] if r - back >= row0 else conv_state[slot, taps - 1 - (row0 - (r - back))]
            y = conv_b + (conv_t * inputs).sum(0)
            out[r, :channels] = y * torch.sigmoid(y)
            if keep and conv_state is not None:
                conv_state[slot] = inputs[1:]
        t = torch.nn.functional.softplus(u[:, step0:step0 + heads] + dt_bias)
        out[:, out_step:out_step + heads] = t
        out[:, out_step + heads:out_step + 2 * heads] = torch.exp(-rate * t)

    def gated_group_norm(self, o, gate, weight, eps, out, groups):
        n, width = o.shape
        y = (o * gate * torch.sigmoid(gate)).view(n, groups, -1)
        y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps)
        out.copy_((y.reshape(n, width) * weight).to(out.dtype))

    def tanh_norm(self, x, alpha, weight, bias, out, rows=None, d=None):
        if d is not None:
            x += d
        src = x if rows is None else x[rows.long()]
        out.copy_((torch.tanh(alpha * src) * weight + bias).to(out.dtype))

    def state_scan(self, mode, q, k, v, state, o, ctx, tiles, heads, dim, vdim, decay=None, decay_bias=None, bonus=None,
                   beta=None, qk=None, forget=None, inp=None, forget_bias=None, inp_bias=None, cap=0.0, aux=None, step=None, skip=None):
        n = q.shape[0]
        rep = heads // (q.shape[1] // dim)
        qh = q.reshape(n, -1, dim).repeat_interleave(rep, 1)
        kh = k.reshape(n, -1, dim).repeat_interleave(rep, 1)
        vh = v.reshape(n, heads, vdim)
        t_seq, t_row0, t_rows, count = tiles
        for i in range(count):
            s, row0, cnt = int(t_seq[i]), int(t_row0[i]), int(t_rows[i])
            st = state[int(ctx.seq_slot[s])]
            if int(ctx.seq_pos0[s]) == 0:
                st.zero_()
            S = st[:, :vdim, :dim]                                    # [heads, value column, key row]
            for r in range(row0, row0 + cnt):
                kv = vh[r][:, :, None] * kh[r][:, None, :]
                if mode == "delta":
                    S.mul_(decay[r].view(heads, 1, dim))
                    w = beta[r][:, None] * (vh[r] - torch.einsum("hvd,hd->hv", S, kh[r]))
                    S.add_(w[:, :, None] * kh[r][:, None, :])
                    out = torch.einsum("hvd,hd->hv", S, qh[r])
                    assert torch.allclose((q.reshape(n, -1, dim)[r] * k.reshape(n, -1, dim)[r]).sum(-1), qk[r], atol=1e-5)
                elif mode == "space":
                    S.mul_(decay[r][:, None, None]).add_(step[r][:, None, None] * kv)
                    out = torch.einsum("hvd,hd->hv", S, qh[r]) + skip[:, None] * vh[r]
                elif mode == "bonus":
                    out = torch.einsum("hvd,hd->hv", S + bonus.view(heads, 1, dim) * kv, qh[r])
                    w = torch.exp(-torch.exp(decay[r] + decay_bias)).view(heads, 1, dim)
                    S.mul_(w).add_(kv)
                else:
                    f = torch.nn.functional.logsigmoid(cap * torch.tanh((forget[r] + forget_bias) / cap))
                    g = cap * torch.tanh((inp[r] + inp_bias) / cap)
                    m = st[:, 0, dim].clone()
                    new = torch.maximum(f + m, g)
                    keep, add = torch.exp(f + m - new), torch.exp(g - new)
                    S.mul_(keep[:, None, None]).add_(add[:, None, None] * kv)
                    st[:, vdim, :dim] = keep[:, None] * st[:, vdim, :dim] + add[:, None] * kh[r]
                    st[:, :, dim] = new[:, None]
                    aux.view(n, heads, 2)[r, :, 0] = (st[:, vdim, :dim] * qh[r]).sum(-1)
                    aux.view(n, heads, 2)[r, :, 1] = new
                    out = torch.einsum("hvd,hd->hv", S, qh[r])
                o[r] = out.reshape(-1)

    def scan_finish(self, o, weight, gate, eps, out, heads, vdim, gate_kind="sigmoid", aux=None, q_scale=1.0):
        n = o.shape[0]
        y = o.view(n, heads, vdim)
        if aux is not None:
            a = aux.view(n, heads, 2)
            y = y * q_scale / (torch.maximum((a[..., 0] * q_scale).abs(), torch.exp(-a[..., 1])) + 1e-6)[..., None]
        y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps) * weight.view(-1, vdim)
        g = torch.sigmoid(gate) * (gate if gate_kind == "silu" else 1.0)
        out.copy_((y.reshape(n, -1) * g).to(out.dtype))

    def pair_mean(self, a, wa, b, wb, eps, y=None, norm_weight=None, norm_eps=0.0, x=None, rounded=None):
        unit = lambda t: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)
        mean = 0.5 * (unit(a) * wa + unit(b) * wb)
        if y is not None:
            y.copy_(mean)
            return
        x += self._layer_normed(mean, norm_eps) * norm_weight
        if rounded is not None:
            rounded.copy_(x.to(rounded.dtype))

    def add_rows(self, x, d):
        x += d

    def fuses_swiglu(self, width, intermediate, activation="silu"):
        return False

    # -- layer norm, latent attention and the element-wise steps of gated designs ---------------------
    @staticmethod
    def _layer_normed(t, eps):
        c = t - t.mean(-1, keepdim=True)
        return c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps)

    def layernorm(self, x, weight, eps, out, rows=None, weight2=None, out2=None):
        src = x if rows is None else x[rows.long()]
        n = self._layer_normed(src.float(), eps)
        out.copy_((n * weight).to(out.dtype))
        if out2 is not None:
            out2.copy_((n * weight2).to(out2.dtype))

    def layernorm_residual(self, d, weight, eps, x, next_weight=None, next_eps=0.0, next_out=None):
        x += self._layer_normed(d, eps) * weight
        if next_out is not None and next_weight is None:
            next_out.copy_(x.to(next_out.dtype))
        elif next_out is not None:
            self.layernorm(x, next_weight, next_eps, next_out)

    @staticmethod
    def _turn(t, p, cos, sin, half_layout):
        """t: [n, ..., size]; the first 2 * pairs entries turn by the tables' rows p."""
        if cos is None:
            return t
        pairs = cos.shape[1]
        shape = (t.shape[0],) + (1,) * (t.dim() - 2) + (pairs,)
        c, s = cos[p].reshape(shape), sin[p].reshape(shape)
        out = t.clone()
        if half_layout:
            a, b = t[..., :pairs], t[..., pairs:2 * pairs]
            out[..., :pairs], out[..., pairs:2 * pairs] = a * c - b * s, b * c + a * s
        else:
            a, b = t[..., 0:2 * pairs:2], t[..., 1:2 * pairs:2]
            out[..., 0:2 * pairs:2], out[..., 1:2 * pairs:2] = a * c - b * s, b * c + a * s
        return out

    def latent_store(self, d, weight, eps, pos, row_seq, cos, sin, block_table, cache, rank, rot_dim, half_layout=False,
                     q_latent=None):
        page = cache.shape[1]
        if q_latent is not None:
            q_w, q_out = q_latent
            cq = d[:, rank + rot_dim:rank + rot_dim + q_w.shape[0]]
            q_out.copy_((cq * torch.rsqrt(cq.pow(2).mean(-1, keepdim=True) + eps) * q_w).to(q_out.dtype))
        p = pos.long()
        c = d[:, :rank]
        c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * weight
        kr = self._turn(d[:, rank:rank + rot_dim], p, cos, sin, half_layout)
        for r in range(d.shape[0]):
            blk = int(block_table[int(row_seq[r]), int(p[r]) // page])
            cache[blk, int(p[r]) % page] = torch.cat([c[r], kr[r]]).to(cache.dtype)

    def rotate_heads(self, q, heads, head_stride, offset, rot_dim, out, out_head_stride, out_offset, pos, cos, sin,
                     half_layout=False):
        n = q.shape[0]
        src = q.float().reshape(n, -1)[:, :heads * head_stride].reshape(n, heads, head_stride)[..., offset:offset + rot_dim]
        turned = self._turn(src, pos.long(), cos, sin, half_layout)
        dst = out.reshape(n, -1)[:, :heads * out_head_stride].reshape(n, heads, out_head_stride)
        dst[..., out_offset:out_offset + rot_dim] = turned.to(out.dtype)

    def latent_attention_tile_heights(self, heads, rank, rot_dim):
        return [max(1, 32 // heads)]

    def latent_attention(self, q, cache, block_table, out, heads, rank, rot_dim, scale, ctx, window=0, sinks=None):
        page = cache.shape[1]
        dk = rank + rot_dim
        for r in range(q.shape[0]):
            p = int(ctx.pos[r])
            idx = torch.arange(max(0, p - window + 1) if window else 0, p + 1)
            keys = cache[block_table[int(ctx.row_seq[r])][(idx // page).long()].long(), (idx % page).long()].float()
            s = (q[r].float().view(heads, dk) @ keys.t()) * scale
            m = s.max(-1, keepdim=True).values
            if sinks is not None:
                m = torch.maximum(m, sinks.view(-1, 1))
            e = torch.exp(s - m)
            den = e.sum(-1, keepdim=True) + (torch.exp(sinks.view(-1, 1) - m) if sinks is not None else 0.0)
            out[r] = ((e / den) @ keys[:, :rank]).reshape(-1).to(out.dtype)

    def sigmoid_gate(self, v, g, group=1):
        v.copy_((v.float() * torch.sigmoid(g.float()).repeat_interleave(group, dim=1)).to(v.dtype))

    def glu_gelu(self, gate_up, out):
        inter = out.shape[1]
        g, u = gate_up[:, :inter].float(), gate_up[:, inter:].float()
        gelu = 0.5 * g * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (g + 0.044715 * g ** 3)))
        out.copy_((gelu * u).to(out.dtype))

    def softcap_rows(self, z, cap):
        z.copy_(cap * torch.tanh(z / cap))

    def rope_cache(self, qkv, pos, row_seq, cos, sin, block_table, kcache, vcache, heads, kv_heads, head_dim,
                   write_kv=True):
        n = qkv.shape[0]
        page = kcache.shape[2]
        half = head_dim // 2
        q = qkv[:, :heads * head_dim].view(n, heads, head_dim).float()
        k = qkv[:, heads * head_dim:(heads + kv_heads) * head_dim].view(n, kv_heads, head_dim).float()
        v = qkv[:, (heads + kv_heads) * head_dim:].view(n, kv_heads, head_dim)
        if cos is not None:
            c = cos[pos.long()][:, None, :]
            s = sin[pos.long()][:, None, :]

            def rot(t):
                x1, x2 = t[..., :half], t[..., half:]
                return torch.cat([x1 * c - x2 * s, x2 * c + x1 * s], -1)

            q, k = rot(q), rot(k)
        qkv[:, :heads * head_dim] = q.reshape(n, -1).to(qkv.dtype)
        if not write_kv:
            return
        for r in range(n):
            p = int(pos[r])
            blk = int(block_table[int(row_seq[r]), p // page])
            kcache[blk, :, p % page, :] = k[r].to(kcache.dtype)
            vcache[blk, :, p % page, :] = v[r]

    def attention(self, qkv, kcache, vcache, block_table, row_seq, pos, out, heads, kv_heads, head_dim, window,
                  max_keys, scale, batch=None):
        n = qkv.shape[0]
        page = kcache.shape[2]
        grp = heads // kv_heads
        for r in range(n):
            p = int(pos[r])
            lo = max(0, p - window + 1) if window and window > 0 else 0
            table = block_table[int(row_seq[r])]
            idx = torch.arange(lo, p + 1)
            blocks = table[(idx // page).long()].long()
            slots = (idx % page).long()
            k = kcache[blocks, :, slots, :].float()  # [keys, kv_heads, hd]
            v = vcache[blocks, :, slots, :].float()
            q = qkv[r, :heads * head_dim].view(heads, head_dim).float()
            kk = k.repeat_interleave(grp, dim=1)
            vv = v.repeat_interleave(grp, dim=1)
            s = torch.einsum("hd,khd->hk", q, kk) * scale
            w = torch.softmax(s, dim=-1)
            out[r] = torch.einsum("hk,khd->hd", w, vv).reshape(-1).to(out.dtype)

    def swiglu(self, gate_up, out):
        inter = out.shape[1]
        g = gate_up[:, :inter].float()
        u = gate_up[:, inter:].float()
        out.copy_((g * torch.sigmoid(g) * u).to(out.dtype))

    def sample_rows(self, logits, temperature, uniform, out_tokens):
        for r in range(logits.shape[0]):
            t = float(temperature[r])
            row = logits[r]
            if t <= 0:
                out_tokens[r] = int(torch.argmax(row))  # torch returns the first maximum on CPU
                mx = row.max()
                out_tokens[r] = int((row == mx).nonzero()[0])
            else:
                w = torch.exp((row - row.max()) / t).double()
                cum = torch.cumsum(w, 0)
                target = float(uniform[r]) * float(cum[-1])
                hit = (cum > target).nonzero()
                out_tokens[r] = int(hit[0]) if len(hit) else int((w > 0).nonzero()[-1])

    def fingerprint_rows(self, logits, slot, state):
        import struct
        mask = (1 << 64) - 1

        def mix64(z):
            z = ((z ^ (z >> 30)) * 0xBF58476D1CE4E5B9) & mask
            z = ((z ^ (z >> 27)) * 0x94D049BB133111EB) & mask
            return z ^ (z >> 31)

        for r in range(logits.shape[0]):
            s = int(slot[r])
            h = int(state[s]) & mask
            data = logits[r].contiguous().numpy().tobytes()
            i = 0
            while i + 8 <= len(data):
                (wd,) = struct.unpack_from("<Q", data, i)
                h = ((h ^ wd) * 1099511628211) & mask
                i += 8
            while i < len(data):
                h = ((h ^ data[i]) * 1099511628211) & mask
                i += 1
            h = mix64(h)
            state[s] = h - (1 << 64) if h >= (1 << 63) else h
