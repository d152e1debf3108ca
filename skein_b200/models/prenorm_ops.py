"""Operators of pre-norm layers for the decoder's program (the op names of the lowering, csrc/core/emit.hpp).

    x (fp32) -> [x += weighted expert rows of the layer before (+ the pass's vector), norm1]        one kernel
             -> one product: every projection of the mixer
             -> attention: rotation (+ unit heads) + append, attention (+ difference of the maps, head norm, gate)
             -> scan: convolution + silu, two products (B, C, step sizes), state and gate
             -> one product back, added to x in its epilogue
             -> [norm2 (+ router and scatter in decode steps)]                                       one kernel
             -> the expert of every token: gate / up pair, down, added to x in its epilogue
             -> experts: gate / up pairs, down; their weighted sum rides in the next norm's kernel

Shifted layers (models/prenorm_layers.py) keep the embedding output and every layer's result in one buffer, [layers + 1, rows, width]: a layer
adds to the slot its input was averaged into, which so becomes its result.

    X_0 .. X_i -> [x = sum_j w_j X_j into slot i + 1, norm in groups, token shift]                  one kernel
             -> one product: every projection of the mixer
             -> the attention above (bias, head norm, value mixing in the append), latent attention (models/layered_ops.py), or two products
                behind bottlenecks and the recurrence (models/parallel_ops.py)
             -> one product back, added to x in its epilogue
             -> [norm in groups], clamped gate / up pair, down, added to x in its epilogue

Where everything sits in the row between a mixer's two products: models/parallel_layers.py, LayerLayout.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import parallel as par
from ..ops import prenorm as pre
from ..ops import reference as ref
from ..ops import selective as sel
from ..ops import recurrent as rec
from .layered import GLU_SLOPE, LatentMixerSpec
from .parallel_layers import LayerLayout, RecurrentSpec, SelectiveSpec, attention_of


class PrenormOps:
    def _init_prenorm(self, num_pages: int, state_slots: int) -> None:
        cfg, dev = self.cfg, self.device
        self.act_dtype = self.w.embed.dtype
        self.layouts = [LayerLayout(sp, ff=False) for sp in cfg.layers]
        tables, self.rope_tables = {}, []
        for sp in cfg.layers:
            a, m = attention_of(sp.mixer), sp.mixer
            key = (a.rot_dims, a.rope_base, a.rope_factor) if a is not None else (m.rot_dim, m.rope_base, 1.0) if isinstance(m, LatentMixerSpec) else None
            if key is not None and key not in tables and (key[0] or not cfg.is_shifted):
                tables[key] = ref.rope_cos_sin_table(self.max_pos, key[0], key[1], dev, {"rope_type": "linear", "factor": key[2]})
            self.rope_tables.append(tables.get(key))
        self.num_state_slots = state_slots if cfg.has_state else 0
        self.kv, self.rec_state, self.conv_tail = [], [], []
        if not num_pages:
            return
        # a sequence's last normed rows (shifted layers)
        self.shift_state = torch.zeros(len(cfg.layers), state_slots, cfg.hidden_size, dtype=torch.float32, device=dev) if cfg.is_shifted else None
        for sp in cfg.layers:
            a, m = attention_of(sp.mixer), sp.mixer
            if isinstance(m, LatentMixerSpec):
                self.kv.append(torch.zeros(num_pages, self.page_size, m.cache_width, dtype=self.act_dtype, device=dev))
            else:
                self.kv.append(par.window_cache(num_pages, self.page_size, a.kv_heads, a.key_width, a.vdim, self.act_dtype, dev) if a is not None else None)
            pool = sel.ScanState if isinstance(m, SelectiveSpec) else rec.RecState if isinstance(m, RecurrentSpec) else None
            self.rec_state.append(pool.make(m, state_slots, self.act_dtype, dev) if pool is not None else None)

    # ---- the stream ---------------------------------------------------------------------------------------------
    def _take_experts(self, st):
        """(rows, their places, their weights) of the experts' outputs that are not part of the stream yet."""
        y, idx, w = st.pending, st.row_idx, st.row_w
        st.pending = st.row_idx = st.row_w = None
        return y, idx, w

    def _layer_done(self, st):
        """The stream as it stands behind a layer, where somebody records it."""
        if self.capture_hidden is None or self.cfg.is_shifted:      # (averaged over depth by the next norm's kernel)
            return
        if st.pending is not None:
            st.residual, _ = pre.add_norm(st.residual, *self._take_experts(st), dtype=self.act_dtype)
        self.capture_hidden.append(st.residual.detach().clone().cpu())

    def _op_loop_step(self, st, li):
        # in front of the next norm, whose kernel adds it
        st.h = self.w.loop.step[self.cfg.layers[li].loop_pass]

    def _op_pre_norm1(self, st, li):
        step, st.h = st.h, None
        st.residual, st.normed = pre.add_norm(st.residual, *self._take_experts(st), step=step, gain=self.w.layers[li].norm1,
                                              eps=self.cfg.rms_norm_eps, dtype=self.act_dtype)

    def _op_pre_norm2(self, st, li):
        f, lw, x = self.cfg.layers[li].mlp, self.w.layers[li], st.residual
        st.routed = None
        if x.is_cuda and self._decode_rows(st.inp) and pre.can_fuse_route(x, f, self.act_dtype):
            out = pre.norm_route(x, lw.norm2, self.cfg.rms_norm_eps, lw.router, f)
            st.normed, st.routed = out[0], out[1:]
        else:
            _, st.normed = pre.add_norm(x, gain=lw.norm2, eps=self.cfg.rms_norm_eps, dtype=self.act_dtype)

    def _op_final_rms_norm(self, st, _):
        st.residual, st.normed = pre.add_norm(st.residual, *self._take_experts(st), gain=self.w.final_norm, eps=self.cfg.rms_norm_eps,
                                              dtype=self.act_dtype)

    # ---- shifted layers ---------------------------------------------------------------------------------------------
    def _embed_shifted(self, st):
        T, C = st.inp.token_ids.shape[0], self.cfg.hidden_size
        st.hist = torch.empty(len(self.cfg.layers) + 1, T, C, dtype=torch.float32, device=self.device)
        ops.latent.embed_f32(st.inp.token_ids, self.w.embed, out=st.hist[0])
        st.residual = st.hist[0]

    def _averaged(self, st, n, gain, x_out, shift=None):
        """Average of the first n of the embedding output and the layers' results, norm, shift."""
        cfg = self.cfg
        st.normed = pre.depth_norm(st.hist[:n], self.w.layers[n - 2].depth if n > 1 else None, gain, cfg.norm_groups, cfg.rms_norm_eps, self.act_dtype,
                                   x_out, shift, st.inp, self._slots(st.inp), self._decode_rows(st.inp))
        if n > 1 and self.capture_hidden is not None:
            self.capture_hidden.append(x_out.detach().clone().cpu())

    def _op_depth_shift_norm(self, st, li):
        lw = self.w.layers[li]
        st.residual = st.hist[li + 1]
        self._averaged(st, li + 1, lw.norm1, st.residual, pre.TokenShift(lw.shift, self.shift_state[li]))

    def _op_group_norm2(self, st, li):
        st.normed = pre.depth_norm(st.residual[None], None, self.w.layers[li].norm2, self.cfg.norm_groups, self.cfg.rms_norm_eps, self.act_dtype)

    def _op_final_depth_norm(self, st, _):
        n = len(self.cfg.layers) + 1
        self._averaged(st, n, self.w.final_norm, None if self.capture_hidden is None else torch.empty_like(st.residual))

    def _op_clamped_gate_up(self, st, li):
        st.h = ops.swiglu_linear(st.normed, self.w.layers[li].dense13, glu=(self.cfg.layers[li].mlp.limit, GLU_SLOPE))

    def _op_clamped_down(self, st, li):
        st.residual = ops.linear(st.h, self.w.layers[li].dense2, out=st.residual, residual=st.residual, out_f32=True)
        st.h = None

    def _op_recurrence_inputs(self, st, li):
        # both products behind a bottleneck: inputs of the decays and of the output's gate
        sec, w = self.layouts[li].parts[0], self.w.layers[li].rec
        a, g = sec.col["a1"], sec.col["g1"]
        st.dense = ops.linear(st.qkv[:, a:a + w.w_decay.shape[1]], w.w_decay, out_f32=True)
        st.cat = ops.linear(st.qkv[:, g:g + w.w_gate.shape[1]], w.w_gate)

    # ---- mixers (window_append and window_attention: ParallelOps) --------------------------------------------------------
    def _op_mixer_in(self, st, li):
        lay, T = self.layouts[li], st.residual.shape[0]
        new = torch.zeros if lay.zero_fill else torch.empty
        st.qkv = new(T, lay.width, dtype=self.act_dtype, device=self.device)
        ops.linear(st.normed, self.w.layers[li].w_in, out=st.qkv[:, lay.in_first:])
        st.normed = None

    def _op_mixer_out(self, st, li):
        y = st.qkv[:, :self.layouts[li].out_cols] if st.attn is None else st.attn      # (latent attention over long portions has its own rows)
        st.residual = ops.linear(y, self.w.layers[li].w_out, out=st.residual, residual=st.residual, out_f32=True)
        st.qkv = st.attn = None
        if self.cfg.layers[li].mlp is None:
            self._layer_done(st)

    def _scan_section(self, st, li):
        sec = self.layouts[li].parts[0]
        m = sec.spec
        x, z = (st.qkv[:, sec.col[n]:sec.col[n] + m.inner] for n in ("x", "z"))
        return m, x, z, st.qkv[:, sec.out:sec.out + m.inner]

    def _op_short_conv(self, st, li):
        m, x, _, _ = self._scan_section(st, li)
        st.attn = sel.short_conv(x, m, self.w.layers[li].scan, self.rec_state[li], st.inp, self._slots(st.inp), self._decode_rows(st.inp))

    def _op_scan_inputs(self, st, li):
        m, w = self.cfg.layers[li].mixer, self.w.layers[li].scan
        st.dense = ops.linear(st.attn, w.w_x)                                        # bottleneck | B | C
        st.cat = ops.linear(st.dense[:, :w.w_dt.shape[1]], w.w_dt, out_f32=True)     # step sizes before bias and softplus

    def _op_selective_scan(self, st, li):
        m, x, z, out = self._scan_section(st, li)
        sel.scan(st.attn, st.dense, st.cat, x, z, out, m, self.w.layers[li].scan, self.rec_state[li], st.inp, self._slots(st.inp),
                 self._decode_rows(st.inp))
        st.attn = st.dense = st.cat = None

    # ---- feed-forward (glu_gate_up: LayeredOps) ------------------------------------------------------------------------
    def _op_score_router(self, st, li):
        if st.routed is None:
            st.routed = pre.route(st.normed, self.w.layers[li].router, self.cfg.layers[li].mlp)

    def _op_shared_gate_up(self, st, li):
        st.h = ops.swiglu_linear(st.normed, self.w.layers[li].shared13)

    def _op_shared_down(self, st, li):
        st.residual = ops.linear(st.h, self.w.layers[li].shared2, out=st.residual, residual=st.residual, out_f32=True)
        st.h = None
