"""The oracle op set: composes :mod:`blaze_b200.ops.ref` functions behind the model's op interface."""
from __future__ import annotations

from typing import Optional

import torch

from . import ref
from ..linear import Linear, QuantAct


class RefOps:
    is_cuda = False
    name = "ref"

    # -------------------------------------------------------------- basics
    def embed(self, table: torch.Tensor, tokens: torch.Tensor) -> torch.Tensor:
        return table[tokens.long()]

    def norm(self, x, residual, w, eps, zero_centered=False, quant_for: Optional[Linear] = None):
        return ref.rmsnorm(x, w, eps, residual, zero_centered)

    def linear(self, lin: Linear, x, out_dtype=None):
        return lin.ref(x, out_dtype)

    def silu_mul(self, gu, quant_for: Optional[Linear] = None):
        return ref.silu_mul(gu)

    def linear_swiglu(self, lin: Linear, x, quant_for: Optional[Linear] = None):
        return ref.silu_mul(self.linear(lin, x))

    def mul_sigmoid(self, x, gate):
        return (x.float() * torch.sigmoid(gate.float())).to(x.dtype)

    def add(self, a, b):
        return (a.float() + b.float()).to(a.dtype)

    def add_sigmoid_scaled(self, a, b, gate_logit):
        """a + b * sigmoid(gate_logit) with the sigmoid rounded to the activation dtype (``ops_basic.cu:175``)."""
        s = torch.sigmoid(gate_logit.float()).to(a.dtype).float()
        return (a.float() + b.float() * s).to(a.dtype)

    def all_reduce(self, x, group=None):
        if group is None or group.world == 1:
            return x
        return group.all_reduce(x)

    # -------------------------------------------------------------- attention
    def rope_tables(self, model, batch):
        inv = model.inv_freq
        pos = batch.positions3 if getattr(batch, "positions3", None) is not None else batch.positions
        return ref.rope_cos_sin(pos, inv, model.rope_scale, model.cfg.rope.mrope_section)

    def attn_prep_store(self, qkv, attn, model, batch, kv, layer_idx, rope):
        cfg = model.cfg
        cos, sin = rope
        q, k, v, gate = ref.attn_prep(qkv, attn.heads, attn.kv_heads, cfg.head_dim, attn.q_norm, attn.k_norm,
                                      cfg.rms_norm_eps, cos, sin, gated=cfg.attn_output_gate,
                                      zero_centered=cfg.zero_centered_norm, rotate=getattr(model, "kv_rotate", False))
        valid = batch.slot_mapping >= 0
        if kv.kv_dtype in ("nvfp4", "nvfp4_4over6"):
            kv.write_fp4(layer_idx, k[valid], v[valid], batch.slot_mapping[valid])
        elif kv.layout == "umma":
            kl, vl = kv.logical_kv(layer_idx)
            ref.kv_write(kl, vl, k[valid], v[valid], batch.slot_mapping[valid])
            # write back in kernel layout
            D = cfg.head_dim
            P, H = kl.shape[0], kl.shape[1]
            kb = kl.view(torch.uint8).view(P, H, 2, 8, D // 16, 16).permute(0, 1, 2, 4, 3, 5).reshape(P, H, -1)
            vb = vl.view(torch.uint8).transpose(2, 3).reshape(P, H, -1)
            kv.kv[layer_idx][:, :, 0] = kb
            kv.kv[layer_idx][:, :, 1] = vb
        else:
            ref.kv_write(kv.k[layer_idx], kv.v[layer_idx], k[valid], v[valid], batch.slot_mapping[valid])
        return q, gate

    def attention(self, q, model, batch, kv, layer_idx, scale, allowed=None):
        """``allowed``: per sequence a bool ``[q_len, ctx_len]`` of the keys its rows may see (None: all), a sparse selection."""
        kl, vl = kv.logical_kv(layer_idx)
        o = ref.paged_attention(q, kl, vl, kv.block_table, batch.h_slots, batch.h_q_start, batch.h_ctx_len, scale,
                                tree_mask=getattr(batch, "tree_mask", None), allowed=allowed)
        return o.reshape(q.shape[0], -1)

    # -------------------------------------------------------------- clamped GLU, static streams, differential attention
    def linear_glu(self, lin: Linear, x, limit: float):
        return ref.clamped_glu(self.linear(lin, x, torch.float32), limit).to(x.dtype)

    def streams_begin(self, table, tokens, scale: float, n: int):
        return (table[tokens.long()].float() * scale)[:, None].repeat(1, n, 1)

    def streams_step(self, src, y, prev, nxt, norm_w, eps):
        if y is not None:
            src = ref.streams_write(src, prev.mix, prev.out, y)
        u = torch.einsum("s,tsw->tw", nxt.read, src)
        return src, self.norm_rows(u, None, norm_w, eps, nxt.dtype)

    def streams_sum(self, src, y, prev):
        return (ref.streams_write(src, prev.mix, prev.out, y) if y is not None else src).sum(1)

    def norm_rows(self, x, rows, w, eps, dtype, centre: bool = False):
        """RMS norm (``centre``: layer norm) of fp32 rows, those named by ``rows``, to ``dtype``."""
        x = x if rows is None else x[rows.long()]
        if centre:
            x = x - x.mean(-1, keepdim=True)
        return (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w).to(dtype)

    def diff_attention(self, qkv, A, batch, kv, layer_idx, eps):
        a = A.spec
        T = qkv.shape[0]
        nq, nk = a.heads * 2 * a.dim, a.kv_heads * 2 * a.dim
        valid = batch.slot_mapping >= 0
        ref.kv_write(kv.k[layer_idx], kv.v[layer_idx], qkv[valid, nq:nq + nk].reshape(-1, 2 * a.kv_heads, a.dim),
                     qkv[valid, nq + nk:].reshape(-1, a.kv_heads, a.vdim), batch.slot_mapping[valid])
        o = ref.diff_attention(qkv[:, :nq].reshape(T, a.heads, 2, a.dim), kv.k[layer_idx], kv.v[layer_idx], kv.block_table, batch.h_slots,
                               batch.h_q_start, batch.h_ctx_len, a.scale, a.window, A.lam, 1.0 - a.diff, eps)
        return o.reshape(T, -1).to(qkv.dtype)

    # -------------------------------------------------------------- post-norm residual, gated softmax attention, recurrences
    def residual_norm(self, x, alpha: float, y, w, eps):
        """(fp32 ``norm(alpha * x + y)``, the same in y's type)."""
        x = self.norm_rows(alpha * x.float() + y.float(), None, w, eps, torch.float32)
        return x, x.to(y.dtype)

    def soft_attention(self, proj, M, batch, kv, layer_idx, eps, out):
        A, a, T = M.attn, M.attn.spec, proj.shape[0]
        q = proj[:, M.cols["q"]:][:, :a.heads * a.dim].reshape(T, a.heads, a.dim)
        k = proj[:, M.cols["k"]:][:, :a.kv_heads * a.dim].reshape(T, a.kv_heads, a.dim)
        v = proj[:, M.cols["v"]:][:, :a.kv_heads * a.vdim].reshape(T, a.kv_heads, a.vdim)
        if a.rot is not None:
            q, k = [ref.rotate_heads(x, batch.positions, A.freq.double().sum(0), a.rot.interleaved) for x in (q, k)]
        if a.unit_rms:
            q, k = [x.float() * torch.rsqrt(x.float().pow(2).mean(-1, keepdim=True) + eps) for x in (q, k)]
        q, valid = q.to(proj.dtype), batch.slot_mapping >= 0
        ref.kv_write(kv.k[layer_idx], kv.v[layer_idx], k[valid], v[valid], batch.slot_mapping[valid])
        o = ref.paged_attention(q.float(), kv.k[layer_idx], kv.v[layer_idx], kv.block_table, batch.h_slots, batch.h_q_start, batch.h_ctx_len,
                                a.scale, window=a.window, sink=A.sink).reshape(T, -1)
        if a.gate:
            o = o * torch.sigmoid(proj[:, M.cols["gate"]:][:, :o.shape[1]].float())
        out.copy_(o * a.out_scale)

    def recurrence(self, proj, low, M, batch, kv, layer_idx, eps, out, state_only: bool = False):
        """The recurrent mixer of a layer, one sequence at a time.  Sequences flagged in ``batch.h_gdn_defer`` leave their state
        untouched; ``state_only`` advances the states and writes nothing."""
        R, r = M.rec, M.rec.spec
        conv_state, rec_state, defer = kv.conv_state.get(layer_idx), kv.rec_state[layer_idx], getattr(batch, "h_gdn_defer", None)
        gated, plain = R.kind == "gated", R.kind in ("gated", "mingru")
        dt, H, dv = proj.dtype, r.heads, r.vdim
        for b, slot in enumerate(batch.h_slots):
            r0, r1 = batch.h_q_start[b], batch.h_q_start[b + 1]
            n = r1 - r0
            if n <= 0:
                continue
            if batch.h_ctx_len[b] == n:
                if not plain:
                    conv_state[slot].zero_()
                rec_state[slot].zero_()
            if not plain:
                y, cs = ref.gdn_conv(proj[r0:r1, M.cols["conv"]:][:, :r.conv_dim], conv_state[slot], R.conv_w, R.conv_b, round_sum=False)
            z = None
            if gated:
                cols = {c: proj[r0:r1, M.cols[c]:][:, :H * d].reshape(n, H, d) for c, d in (("q", r.dim), ("f", r.dim), ("v", dv))}
                o, S = ref.gated_linear(cols["q"], cols["f"], cols["v"], R.A, R.dt_bias, rec_state[slot])
            elif R.kind == "mingru":
                zg, u, g = [proj[r0:r1, M.cols[c]:][:, :r.width] for c in ("zg", "u", "g")]
                o, S = ref.min_gru(zg, u, rec_state[slot].view(-1))
                S = S.view(1, 1, -1)
                if not state_only:
                    out[r0:r1] = (o * torch.nn.functional.silu(g.float())).to(dt)
            elif R.kind == "delta" and r.head_decay:
                nk = r.kv_heads * r.dim
                a, b_ = [proj[r0:r1, M.cols[c]:][:, :H] for c in ("decay", "beta")]
                o, S = ref.delta_rule(y[:, :nk].view(n, -1, r.dim), y[:, nk:2 * nk].view(n, -1, r.dim), y[:, 2 * nk:].view(n, H, dv),
                                      a.reshape(n, H, 1), b_, R.A, R.dt_bias, rec_state[slot])
                z = proj[r0:r1, M.cols["z"]:][:, :H * dv]
            elif R.kind == "delta":
                nk, hd = r.kv_heads * r.dim, H * r.dim
                o, S = ref.delta_rule(y[:, :nk].view(n, -1, r.dim), y[:, nk:2 * nk].view(n, -1, r.dim), y[:, 2 * nk:].view(n, H, dv),
                                      low[r0:r1, :hd].reshape(n, H, r.dim), proj[r0:r1, M.cols["beta"]:][:, :H], R.A, R.dt_bias, rec_state[slot])
                z = low[r0:r1, hd:]
            else:
                ng = r.groups * r.state
                o, S = ref.state_space(y[:, :r.inner].view(n, H, dv), y[:, r.inner:r.inner + ng].view(n, -1, r.state),
                                       y[:, r.inner + ng:].view(n, -1, r.state), proj[r0:r1, M.cols["dt"]:][:, :H], R.A, R.dt_bias, R.D,
                                       rec_state[slot])
                z = proj[r0:r1, M.cols["z"]:][:, :r.inner]
            if not (defer is not None and defer[b]):
                if not plain:
                    conv_state[slot].copy_(cs)
                rec_state[slot].copy_(S)
            if not state_only and R.kind != "mingru":
                delta = R.kind == "delta"
                out[r0:r1] = ref.group_norm(o.reshape(n, -1), z, R.norm_w, R.norm_groups, eps, delta and r.gate == "sigmoid", not delta,
                                            r.out_scale).to(dt)

    # -------------------------------------------------------------- residual with normed branches, input convolution, latent attention
    def embed_norm(self, table, tokens, w, eps):
        """Layer-normed embedding rows, fp32."""
        return self.norm_rows(table[tokens.long()].float(), None, w, eps, torch.float32, centre=True)

    def branch_norm(self, x, y, w, eps, copy: bool = True):
        """(fp32 ``x + layer_norm(y)``, the same in y's type or None)."""
        x = x + self.norm_rows(y.float(), None, w, eps, torch.float32, centre=True)
        return x, x.to(y.dtype) if copy else None

    def input_conv(self, x, w, batch, kv, layer_idx, dtype, state_only: bool = False):
        """``x + conv(x)`` of fp32 rows in ``dtype``, with the inputs before each sequence's rows from its state row, which advances
        (not for sequences flagged in ``batch.h_gdn_defer``)."""
        out, state = torch.empty(x.shape, dtype=dtype, device=x.device), kv.input_state.get(layer_idx)
        defer = getattr(batch, "h_gdn_defer", None)
        for b, slot in enumerate(batch.h_slots):
            r0, r1 = batch.h_q_start[b], batch.h_q_start[b + 1]
            if r1 <= r0:
                continue
            fresh = batch.h_ctx_len[b] == r1 - r0
            before = x.new_zeros(w.shape[0] - 1, x.shape[1]) if state is None or fresh else state[slot]
            y, after = ref.input_conv(x[r0:r1], before, w)
            out[r0:r1] = y.to(dtype)
            if state is not None and not (defer is not None and defer[b]):
                state[slot].copy_(after)
        return None if state_only else out

    def linear_relu2(self, lin: Linear, x):
        return ref.relu2(self.linear(lin, x))

    def poly_norm(self, z, act, eps):
        return ref.poly_norm(z, act, eps).to(z.dtype)

    def latent_attention(self, proj, M, batch, kv, layer_idx, eps, out):
        """Latent attention of a mixer: its own latents go to their pages, heads' outputs (before the output projection) to ``out``."""
        A, a, T, dt = M.attn, M.attn.spec, proj.shape[0], proj.dtype
        turn = lambda x: x.float() if A.freq is None else ref.rotate_heads(x, batch.positions, A.freq.double().sum(0), False)   # noqa: E731
        if a.kv_from is None:
            c = self.norm_rows(proj[:, M.cols["kv"]:][:, :a.kv_rank].float(), None, A.c_norm, eps, dt)
            kr = turn(proj[:, M.cols["kv"] + a.kv_rank:][:, :a.rot_dim].reshape(T, 1, -1))
            valid = batch.slot_mapping >= 0
            ref.kv_write(kv.k[layer_idx], kv.v[layer_idx], c[valid][:, None], kr[valid], batch.slot_mapping[valid])
        q = self.linear(A.uq, self.norm_rows(proj[:, M.cols["q"]:][:, :a.q_rank].float(), None, A.q_norm, eps, dt)).view(T, a.heads, -1)
        # keys and values by head: the score of a latent is (uk^T q) . c, the output uv (sum of weighted latents)
        ql = torch.einsum("thd,hdr->thr", q[..., :a.dim].float(), A.uk.float())
        q = torch.cat([ql, turn(q[..., a.dim:])], -1)
        keys = torch.cat([kv.k[layer_idx], kv.v[layer_idx]], -1)
        o = ref.paged_attention(q, keys, kv.k[layer_idx], kv.block_table, batch.h_slots, batch.h_q_start, batch.h_ctx_len, a.scale,
                                window=a.window, sink=A.sink)
        out.copy_(torch.einsum("thr,her->the", o.float(), A.uv.float()).reshape(T, -1))

    def moe_rows(self, x, topk_w, topk_id, experts, shared=None, gate=None):
        """``gate``: logits ``[T]``, the shared expert's rows are multiplied by their sigmoid."""
        y = self.moe(x, topk_w, topk_id, experts)
        if shared is not None and gate is not None:
            shared = shared.float() * torch.sigmoid(gate.float()).unsqueeze(-1)
            return (y.float() + shared).to(y.dtype)
        return y if shared is None else self.add(y, shared)

    # -------------------------------------------------------------- parallel branches, position vectors, sigmoid attention
    def embed_positions(self, table, tokens, positions, scale: float, freq, copy=None):
        """Scaled embedding rows plus their position's vector, fp32; ``copy`` gets them in its own type."""
        x = table[tokens.long()].float() * scale + ref.position_vectors(positions, freq.double().sum(0), table.shape[1])
        if copy is not None:
            copy.copy_(x)
        return x

    def branch_step(self, x, br, eps, dtype, w1=None, w2=None, copy=None):
        """Add a layer's branches (None: nothing) to the fp32 rows ``x``; then their RMS norms with the weights ``w1`` and ``w2`` (None: no
        such norm) in ``dtype``.  ``copy`` gets the rows in its own type.  (rows, norm 1, norm 2)"""
        if br is not None:
            if br.norms is not None:
                y = sum(self.norm_rows(r.float(), None, w, eps, torch.float32) for r, w in zip(br.rows, br.norms)) / len(br.norms)
            else:
                y = br.rows.float()
            if br.ffn is not None:
                y = y + br.ffn.float()
            x = x + br.mult * y
        if copy is not None:
            copy.copy_(x)
        return (x,) + tuple(None if w is None else self.norm_rows(x, None, w, eps, dtype) for w in (w1, w2))

    def sigmoid_attention(self, proj, M, batch, kv, layer_idx, eps, out, state_only: bool = False):
        """Sigmoid attention of a mixer (convolution, norm and page write included) into ``out``.  Sequences flagged in
        ``batch.h_gdn_defer`` leave their convolution's inputs untouched; ``state_only`` advances those and does nothing else."""
        A, a, T, dt = M.attn, M.attn.spec, proj.shape[0], proj.dtype
        nq, nk, nv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        u = torch.cat([proj[:, M.cols[c]:][:, :n] for c, n in (("q", nq), ("k", nk), ("v", nv))], 1)
        y, defer = u.float(), getattr(batch, "h_gdn_defer", None)
        if a.conv:
            y, state = torch.empty(u.shape, device=u.device), kv.qkv_state.get(layer_idx)
            for b, slot in enumerate(batch.h_slots):
                r0, r1 = batch.h_q_start[b], batch.h_q_start[b + 1]
                if r1 <= r0:
                    continue
                fresh = state is None or batch.h_ctx_len[b] == r1 - r0
                y[r0:r1], after = ref.causal_conv(u[r0:r1], u.new_zeros(a.conv - 1, u.shape[1]) if fresh else state[slot], A.conv_w)
                if state is not None and not (defer is not None and defer[b]):
                    state[slot].copy_(after)
        if state_only:
            return
        q, k, v = y[:, :nq].view(T, -1, a.dim), y[:, nq:nq + nk].view(T, -1, a.dim), y[:, nq + nk:].view(T, -1, a.vdim)
        if a.temp_coef:
            q = q * ref.query_temperature(batch.positions, a.temp_coef, a.temp_every).view(T, 1, 1)
        if a.unit_v:
            v = v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)
        valid = batch.slot_mapping >= 0
        ref.kv_write(kv.k[layer_idx], kv.v[layer_idx], k[valid], v[valid], batch.slot_mapping[valid])
        o = ref.sigmoid_attention(q.to(dt), kv.k[layer_idx], kv.v[layer_idx], kv.block_table, batch.h_slots, batch.h_q_start,
                                  batch.h_ctx_len, a.scale, A.bias, A.PAD, a.window)
        out.copy_(o.reshape(T, -1) * a.out_scale)

    # -------------------------------------------------------------- MoE
    def router_topk(self, logits, k, renorm=True, sigmoid=False, n_exp=None):
        """``n_exp``: the experts' logits are the first ``n_exp`` columns."""
        return ref.router_topk(logits if n_exp is None else logits[:, :n_exp], k, renorm, sigmoid)

    def moe(self, x, topk_w, topk_id, experts):
        """experts: an object with ``num_experts`` and ``forward_one(e, x)``."""
        return ref.moe_forward(x, topk_w, topk_id, experts.forward_one, experts.num_experts, experts.weigh_input)

    # -------------------------------------------------------------- GDN
    def gdn(self, mixed_qkv, z, b, a, gdn, model, batch, kv, layer_idx, state_only: bool = False):
        """Causal conv + gates + delta-rule recurrence + gated norm, one sequence at a time.  Sequences flagged in
        ``batch.h_gdn_defer`` leave their state untouched; ``state_only`` advances the states and returns nothing."""
        cfg = model.cfg
        dk, dv = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        hk, hv = gdn.k_heads, gdn.v_heads
        T = mixed_qkv.shape[0]
        out = torch.empty(T, hv * dv, dtype=mixed_qkv.dtype, device=mixed_qkv.device)
        conv_state, rec_state = kv.conv_state[layer_idx], kv.rec_state[layer_idx]
        defer = getattr(batch, "h_gdn_defer", None)
        for bidx, slot in enumerate(batch.h_slots):
            r0, r1 = batch.h_q_start[bidx], batch.h_q_start[bidx + 1]
            if r1 == r0:
                continue
            fresh = batch.h_ctx_len[bidx] - (r1 - r0) == 0
            keep = not (defer is not None and defer[bidx])
            if fresh:
                conv_state[slot].zero_()
                rec_state[slot].zero_()
            y, cs = ref.gdn_conv(mixed_qkv[r0:r1], conv_state[slot], gdn.conv_w)
            if keep:
                conv_state[slot].copy_(cs)
            q = y[:, :hk * dk].view(-1, hk, dk)
            k = y[:, hk * dk:2 * hk * dk].view(-1, hk, dk)
            v = y[:, 2 * hk * dk:].view(-1, hv, dv)
            g, beta = ref.gdn_gates(a[r0:r1], b[r0:r1], gdn.A_log, gdn.dt_bias)
            if model.gdn_chunked and (r1 - r0) > 1:
                o, S = ref.gdn_chunked(q, k, v, g, beta, rec_state[slot])
            else:
                o, S = ref.gdn_recurrent(q, k, v, g, beta, rec_state[slot])
            if keep:
                rec_state[slot].copy_(S)
            if state_only:
                continue
            zz = z[r0:r1].view(-1, hv, dv)
            on = ref.gated_rmsnorm(o, zz, gdn.norm_w, cfg.rms_norm_eps, zero_centered=False, gate=cfg.gdn_output_gate)
            out[r0:r1] = on.reshape(r1 - r0, hv * dv)
        return None if state_only else out

    # -------------------------------------------------------------- head
    def argmax(self, logits):
        return ref.argmax_lowest(logits.float())
