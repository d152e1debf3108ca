"""Operators of post-norm latent-attention blocks for the decoder's program (the op names of the lowering, csrc/core/emit.hpp).

    x (fp32) -> [input convolution] -> one stacked projection (queries or their latent | cache row | gate)
             -> append (norms, rotation, paged write) -> attention -> o_proj
             -> [alpha x + . , norm1 (+ router and scatter)]                     one kernel for decode steps
             -> experts (clamped gate/up -> down) or up -> polynomial activation -> down
             -> [alpha x + . , norm2 + the next layer's convolution]              one kernel for decode steps

Attention runs in one of two forms of the same product. Decode steps and short portions apply the key expansion to the queries
and attend over the cached latents themselves (one row per token, all heads share it); longer prefill chunks expand keys and
values per head once for the whole context of the chunk and run the tensor-core kernel over them, which costs a third of the
multiplications per (query, key) pair.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import latent as lat
from ..ops import reference as ref
from .layered import GLU_SLOPE, RoutedFFSpec

EXPAND_MIN_ROWS = 33      # a chunk of at least this many rows expands keys and values


class LayeredOps:
    def _init_layered(self, num_pages: int, state_slots: int) -> None:
        cfg, w, dev = self.cfg, self.w, self.device
        if self.layout.world != 1:
            raise ValueError(f"{cfg.architecture} runs on one device (tp = pp = ep = 1)")
        if cfg.is_parallel:
            return self._init_parallel(num_pages, state_slots)
        if cfg.is_prenorm:
            return self._init_prenorm(num_pages, state_slots)
        self.act_dtype = w.embed.dtype
        tables = {}
        for sp in cfg.layers:
            key = (sp.mixer.rot_dim, sp.mixer.rope_base)
            if key not in tables:
                tables[key] = ref.rope_cos_sin_table(self.max_pos, key[0], key[1], dev)
        self.rope_tables = [tables[(sp.mixer.rot_dim, sp.mixer.rope_base)] for sp in cfg.layers]
        R = cfg.conv_tail_rows(self.page_size)
        new = lambda *shape: torch.zeros(*shape, dtype=self.act_dtype, device=dev)      # noqa: E731
        self.kv = [new(num_pages, self.page_size, sp.mixer.cache_width) for sp in cfg.layers] if num_pages else []
        # the input convolution's last inputs live with the pages of the cache (csrc/kernels/postnorm.cu)
        self.conv_tail = [new(num_pages, R, cfg.hidden_size) if R else None for _ in cfg.layers] if num_pages else []

    def _conv(self, li) -> lat.ConvState:
        return lat.ConvState(self.w.layers[li].conv, self.conv_tail[li], self.page_size)

    @staticmethod
    def _decode_rows(inp) -> bool:
        """Every row is the next token of its own sequence (a decode step)."""
        return not inp.is_prefill and inp.seq_of_token is None

    def _expanded(self, inp, m) -> bool:
        return (inp.is_prefill and inp.max_q_len >= EXPAND_MIN_ROWS
                and lat.expanded_ok(self.act_dtype, m.dim, m.rot_dim, m.vdim, m.kv_rank, self.device))

    def _context_layout(self, st):
        """(first dense row of every sequence, total rows, longest cached prefix) of this chunk's context."""
        inp = st.inp
        if inp.kv_start is None:
            kv, q = inp.seq_lens.tolist(), inp.q_len.tolist()
            starts = [0]
            for n in kv:
                starts.append(starts[-1] + n)
            inp.kv_start = torch.tensor(starts[:-1], dtype=torch.int32, device=self.device)
            inp.kv_total, inp.max_cached = starts[-1], max(a - b for a, b in zip(kv, q))
        return inp.kv_start, inp.kv_total, inp.max_cached

    # ---- mixer ----------------------------------------------------------------------------------------------
    def _latent_parts(self, st, li):
        """(weights, first column of the cache row, queries or None when they have a latent, gate or None) of a latent mixer, in the
        output of its input projection."""
        m, lw = self.cfg.layers[li].mixer, self.w.layers[li]
        if self.cfg.is_prenorm:
            col = self.layouts[li].parts[0].col
            return lw.latent, col["dkv"], st.qkv[:, col["q"]:col["q"] + m.q_width], None
        mw = lw.mixer
        gate = st.qkv[:, mw.off_gate:mw.off_gate + m.heads * m.vdim] if m.gated else None
        return mw, mw.off_kv, None if m.q_rank else st.qkv[:, :m.q_width], gate

    def _op_input_conv(self, st, li):
        if st.normed is not None:
            return              # decode: produced by the kernel that normed the previous layer
        inp = st.inp
        st.normed = lat.conv_input(st.residual, self._conv(li), inp.positions, inp.block_table, inp.seq_of_token,
                                   None if self._decode_rows(inp) else inp.q_start, self.act_dtype, write_tail=self._decode_rows(inp))

    def _op_latent_proj(self, st, li):
        st.qkv = ops.linear(st.normed, self.w.layers[li].mixer.w_in)
        st.normed = None

    def _op_latent_append(self, st, li):
        inp, m = st.inp, self.cfg.layers[li].mixer
        mw, off_kv, _, _ = self._latent_parts(st, li)
        st.dense = None
        kv_start = None
        if self._expanded(inp, m):
            kv_start, total, cached = self._context_layout(st)
            st.dense = torch.empty(total, m.cache_width, dtype=self.act_dtype, device=self.device)
            if cached > 0:
                lat.latent_gather(self.kv[li], inp.block_table, inp.seq_lens, inp.q_len, kv_start, st.dense, cached)
        tail, x = None, None
        if self.conv_tail:
            tail, x = self.conv_tail[li], None if self._decode_rows(inp) else st.residual
        st.attn = lat.latent_append(st.qkv, off_kv, mw.q_norm, mw.kv_norm, m.rot_dim, self.rope_tables[li], inp.positions, inp.seq_of_token,
                                    inp.block_table, self.kv[li], self.cfg.rms_norm_eps, x, tail, inp.seq_lens, max(self.cfg.conv_taps, 1), st.dense,
                                    kv_start)

    def _op_latent_q_up(self, st, li):
        st.attn = ops.linear(st.attn, self.w.layers[li].mixer.w_uq)     # the normed query latent -> queries

    def _op_latent_attention(self, st, li):
        inp, m = st.inp, self.cfg.layers[li].mixer
        mw, _, q, gate = self._latent_parts(st, li)
        q = st.attn if q is None else q
        if st.dense is not None:
            lat.rope_rows(q, m.heads, m.dim, m.rot_dim, self.rope_tables[li], inp.positions)
            kv = ops.linear(st.dense, mw.w_ukv)
            st.attn = lat.latent_attn_prefill(q, m.heads, m.dim, m.rot_dim, m.vdim, m.scale, st.dense, kv, inp.q_start, inp.q_len, inp.seq_lens,
                                              inp.kv_start, inp.max_q_len, gate, mw.sinks)
        else:
            q_abs = lat.head_linear(q, m.dim + m.rot_dim, mw.w_uk_t)
            o = lat.latent_attn_rows(q_abs, q, m.heads, m.dim, m.rot_dim, m.scale, self.rope_tables[li], inp.positions, inp.seq_of_token,
                                     inp.block_table, self.kv[li], inp.ctx_hint, sinks=mw.sinks)
            w_uv = mw.w_ukv[m.heads * m.dim:].view(m.heads, m.vdim, m.kv_rank)
            if self.cfg.is_prenorm:      # straight into the row that the product back reads
                lat.head_linear(o, m.kv_rank, w_uv, gate, out=st.qkv[:, :m.out_width])
                st.attn = st.dense = None
                return
            st.attn = lat.head_linear(o, m.kv_rank, w_uv, gate)
        st.dense = None
        if not self.cfg.is_prenorm:
            st.qkv = None

    def _op_latent_o_proj(self, st, li):
        st.pending, st.attn = ops.linear(st.attn, self.w.layers[li].mixer.wo), None
        st.row_idx = st.row_w = None

    # ---- norms ------------------------------------------------------------------------------------------------
    def _end_layer(self, st, li, gain):
        """The last norm of a layer. A decode step gets the next layer's convolved input from the same kernel, the last layer the
        final norm."""
        cfg, inp = self.cfg, st.inp
        last = li + 1 == len(cfg.layers)
        conv = self._conv(li + 1) if (not last and self._decode_rows(inp)) else None
        st.residual, st.normed = lat.post_norm(st.residual, st.pending, cfg.post_alpha, gain, cfg.rms_norm_eps, st.row_idx, st.row_w, self.act_dtype,
                                               want_act=False, conv=conv, positions=inp.positions, block_table=inp.block_table,
                                               final_gain=self.w.final_norm if last else None)
        st.pending = st.row_idx = st.row_w = None
        if self.capture_hidden is not None:
            self.capture_hidden.append(st.residual.detach().float().cpu())

    def _op_post_norm1(self, st, li):
        cfg, sp, lw = self.cfg, self.cfg.layers[li], self.w.layers[li]
        st.routed = None
        if sp.mlp is None:
            return self._end_layer(st, li, lw.norm1)
        T, C = st.residual.shape
        if (isinstance(sp.mlp, RoutedFFSpec) and st.residual.is_cuda and self._decode_rows(st.inp)
                and lat.can_fuse_group_route(T, C, sp.mlp.experts, sp.mlp.top, self.act_dtype, self.device)):
            out = lat.post_norm_route(st.residual, st.pending, cfg.post_alpha, lw.norm1, cfg.rms_norm_eps, lw.router, sp.mlp.top, sp.mlp.groups,
                                      sp.mlp.keep)
            st.residual, st.routed = out[0], out[1:]
        else:
            st.residual, st.normed = lat.post_norm(st.residual, st.pending, cfg.post_alpha, lw.norm1, cfg.rms_norm_eps, dtype=self.act_dtype)
        st.pending = None

    def _op_post_norm2(self, st, li):
        self._end_layer(st, li, self.w.layers[li].norm2)

    def _op_final_scalar_norm(self, st, _):
        pass                    # produced with the last layer's norm

    # ---- feed-forward -----------------------------------------------------------------------------------------
    def _op_ff_up(self, st, li):
        st.h, st.normed = ops.linear(st.normed, self.w.layers[li].w_up), None

    def _op_poly_norm(self, st, li):
        st.h = lat.poly_norm(st.h, self.w.layers[li].act, self.cfg.rms_norm_eps)

    def _op_ff_down(self, st, li):
        st.pending, st.h = ops.linear(st.h, self.w.layers[li].w2), None

    def _op_group_router(self, st, li):
        if st.routed is None:
            mlp = self.cfg.layers[li].mlp
            st.routed = lat.route_grouped(st.normed, self.w.layers[li].router, mlp.top, mlp.groups, mlp.keep)
        st.normed = None

    def _op_glu_gate_up(self, st, li):
        mlp = self.cfg.layers[li].mlp
        _, _, counts, offsets, _, _, xs = st.routed
        st.normed = None
        st.h = ops.grouped_linear(xs, self.w.layers[li].w13, counts, offsets, swiglu=True, glu=None if mlp.limit is None else (mlp.limit, GLU_SLOPE))

    def _op_glu_down(self, st, li):
        ids, wts, counts, offsets, row_of, _, _ = st.routed
        st.pending = ops.grouped_linear(st.h, self.w.layers[li].w2, counts, offsets)
        st.row_idx, st.row_w = row_of.view(ids.shape), wts
        st.h = st.routed = None
        if self.cfg.is_prenorm:
            self._layer_done(st)
