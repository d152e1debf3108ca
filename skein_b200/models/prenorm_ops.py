"""Operators of pre-norm layers for the decoder's program (the op names of the lowering, csrc/core/emit.hpp).

    x (fp32) -> [x += weighted expert rows of the layer before (+ the pass's vector), norm1]        one kernel
             -> one product: every projection of the mixer
             -> attention: rotation (+ unit heads) + append, attention (+ difference of the maps, head norm, gate)
             -> scan: convolution + silu, two products (B, C, step sizes), state and gate
             -> one product back, added to x in its epilogue
             -> [norm2 (+ router and scatter in decode steps)]                                       one kernel
             -> the expert of every token: gate / up pair, down, added to x in its epilogue
             -> experts: gate / up pairs, down; their weighted sum rides in the next norm's kernel

Where everything sits in the row between a mixer's two products: models/parallel_layers.py, LayerLayout.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import parallel as par
from ..ops import prenorm as pre
from ..ops import reference as ref
from ..ops import selective as sel
from .parallel_layers import LayerLayout, SelectiveSpec, attention_of


class PrenormOps:
    def _init_prenorm(self, num_pages: int, state_slots: int) -> None:
        cfg, dev = self.cfg, self.device
        self.act_dtype = self.w.embed.dtype
        self.layouts = [LayerLayout(sp, ff=False) for sp in cfg.layers]
        tables, self.rope_tables = {}, []
        for sp in cfg.layers:
            a = attention_of(sp.mixer)
            key = a and (a.rot_dims, a.rope_base, a.rope_factor)
            if a is not None and key not in tables:
                tables[key] = ref.rope_cos_sin_table(self.max_pos, a.rot_dims, a.rope_base, dev, {"rope_type": "linear", "factor": a.rope_factor})
            self.rope_tables.append(tables.get(key))
        self.num_state_slots = state_slots if cfg.has_state else 0
        self.kv, self.rec_state = [], []
        if not num_pages:
            return
        for sp in cfg.layers:
            a, m = attention_of(sp.mixer), sp.mixer
            self.kv.append(par.window_cache(num_pages, self.page_size, a.kv_heads, a.key_width, a.vdim, self.act_dtype, dev) if a is not None else None)
            self.rec_state.append(sel.ScanState.make(m, state_slots, self.act_dtype, dev) if isinstance(m, SelectiveSpec) else None)

    # ---- the stream ---------------------------------------------------------------------------------------------
    def _take_experts(self, st):
        """(rows, their places, their weights) of the experts' outputs that are not part of the stream yet."""
        y, idx, w = st.pending, st.row_idx, st.row_w
        st.pending = st.row_idx = st.row_w = None
        return y, idx, w

    def _layer_done(self, st):
        """The stream as it stands behind a layer, where somebody records it."""
        if self.capture_hidden is None:
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

    # ---- mixers (window_append and window_attention: ParallelOps) --------------------------------------------------------
    def _op_mixer_in(self, st, li):
        lay, T = self.layouts[li], st.residual.shape[0]
        new = torch.zeros if lay.zero_fill else torch.empty
        st.qkv = new(T, lay.width, dtype=self.act_dtype, device=self.device)
        ops.linear(st.normed, self.w.layers[li].w_in, out=st.qkv[:, lay.in_first:])
        st.normed = None

    def _op_mixer_out(self, st, li):
        st.residual = ops.linear(st.qkv[:, :self.layouts[li].out_cols], self.w.layers[li].w_out, out=st.residual, residual=st.residual, out_f32=True)
        st.qkv = None
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
