"""Operators of parallel layers for the decoder's program (the op names of the lowering, csrc/core/emit.hpp).

    x (fp32) -> [h = tanh(alpha x) w + b]
             -> one product from h: the feed-forward's up projection (squared relu in the epilogue) and every projection of the mixer
             -> window attention: norm + rotation + append, attention
             -> recurrence: convolution, gates, state (one kernel for decode steps), gated norm
             -> one product back, added to x in its epilogue: the mixers' output projections and the down projection side by side

Where everything sits in the row between the two products: models/parallel_layers.py, LayerLayout. Before a pass of the loop,
x <- W [x; x0] + step with x0 the embedding output.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import parallel as par
from ..ops import recurrent as rec
from ..ops import reference as ref
from .parallel_layers import LayerLayout, RecurrentSpec, WindowAttnSpec, attention_of, recurrence_of


class ParallelOps:
    def _init_parallel(self, num_pages: int, state_slots: int) -> None:
        cfg, dev = self.cfg, self.device
        self.act_dtype = self.w.embed.dtype
        self.layouts = [LayerLayout(sp) for sp in cfg.layers]
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
            a, r = attention_of(sp.mixer), recurrence_of(sp.mixer)
            self.kv.append(par.window_cache(num_pages, self.page_size, a.kv_heads, a.dim, a.vdim, self.act_dtype, dev) if a is not None else None)
            self.rec_state.append(rec.RecState.make(r, state_slots, self.act_dtype, dev) if r is not None else None)

    def _slots(self, inp):
        """State slots of the step's sequences. Without any given (a single whole-sequence forward), sequence s uses slot s."""
        if inp.slots is None:
            n = inp.seq_lens.shape[0]
            if n > self.num_state_slots:
                raise ValueError(f"{n} sequences need a state slot each, the decoder has {self.num_state_slots}")
            inp.slots = torch.arange(n, dtype=torch.int32, device=self.device)
        return inp.slots

    # ---- the stream ---------------------------------------------------------------------------------------------
    def _embed_parallel(self, st):
        st.residual = ops.latent.embed_f32(st.inp.token_ids, self.w.embed)
        if self.cfg.loop is not None:
            C = self.cfg.hidden_size
            st.cat = torch.empty(st.residual.shape[0], 2 * C, dtype=self.act_dtype, device=self.device)
            par.residual_tanh(st.residual, dtype=self.act_dtype, out=st.cat[:, C:])

    def _op_loop_mix(self, st, li):
        C, w = self.cfg.hidden_size, self.w.loop
        par.residual_tanh(st.residual, dtype=self.act_dtype, out=st.cat[:, :C])
        y = ops.linear(st.cat, w.w_in, out_f32=True)
        st.residual, st.normed = par.residual_tanh(None, y, w.step[self.cfg.layers[li].loop_pass], self.w.layers[li].norm, self.act_dtype)

    def _op_tanh_norm(self, st, li):
        if st.normed is None:       # (else produced with the residual)
            _, st.normed = par.residual_tanh(st.residual, norm=self.w.layers[li].norm, dtype=self.act_dtype, want_x=False)

    def _op_parallel_in(self, st, li):
        lay, T = self.layouts[li], st.residual.shape[0]
        new = torch.zeros if lay.zero_fill else torch.empty
        st.qkv = new(T, lay.width, dtype=self.act_dtype, device=self.device)
        ops.linear(st.normed, self.w.layers[li].w_in, out=st.qkv[:, lay.in_first:], relu2_cols=lay.ff_cols)
        st.normed = None

    def _op_parallel_out(self, st, li):
        lay = self.layouts[li]
        st.residual = ops.linear(st.qkv[:, :lay.out_cols], self.w.layers[li].w_out, out=st.residual, residual=st.residual, out_f32=True)
        st.qkv = None
        if self.capture_hidden is not None:
            self.capture_hidden.append(st.residual.detach().clone().cpu())      # (the next layer adds in place)

    def _op_final_tanh_norm(self, st, _):
        _, st.normed = par.residual_tanh(st.residual, norm=self.w.final_norm, dtype=self.act_dtype, want_x=False)

    # ---- mixers -------------------------------------------------------------------------------------------------
    def _window_section(self, st, li):
        sec = self.layouts[li].part(WindowAttnSpec)
        a = sec.spec
        q, k, v = (st.qkv[:, sec.col[n]:sec.col[n] + rows] for n, rows in a.sections()[:3])
        return sec, a, q, k, v

    def _op_window_append(self, st, li):
        _, a, q, k, v = self._window_section(st, li)
        w, inp = self.w.layers[li].attn, st.inp
        args = (self.rope_tables[li], inp.positions, inp.seq_of_token, inp.block_table, self.kv[li], self.page_size, self.cfg.rms_norm_eps)
        if a.row_norm:
            par.window_append(q, k, v, w.q_norm, w.k_norm, a, *args)
        else:
            par.head_append(q, k, v, a, *args, w=w, mix=self._value_mix(st, a, v))

    def _value_mix(self, st, a, v):
        """The first mixing layer keeps its values for the step's later ones."""
        if not a.v_mix:
            return None
        keep = st.v_first is None
        if keep:
            st.v_first = torch.empty(v.shape, dtype=v.dtype, device=v.device)
        return par.ValueMix(st.v_first, keep)

    def _op_window_attention(self, st, li):
        sec, a, q, _, _ = self._window_section(st, li)
        gate = st.qkv[:, sec.col["g"]:sec.col["g"] + a.out_width] if a.gated else None
        par.window_attn(q, a, st.inp, self.kv[li], self.page_size, st.qkv[:, sec.out:sec.out + a.out_width], sec.scale,
                        par.HeadMix(self.w.layers[li].attn.lam, gate, self.cfg.rms_norm_eps, self.w.layers[li].attn.sinks))

    def _op_recurrence(self, st, li):
        sec, inp = self.layouts[li].part(RecurrentSpec), st.inp
        cols = rec.RecColumns.of(sec.spec, sec.col)
        args = (st.qkv, cols, sec.spec, self.w.layers[li].rec, self.rec_state[li], inp.positions, self._slots(inp))
        if self._decode_rows(inp):
            r, gate = sec.spec, None
            if r.corrects:
                gate = rec.HeadGate(self.w.layers[li].rec.norm, self._output_gate(st, sec), st.qkv[:, sec.out:sec.out + r.out_width],
                                    self.cfg.rms_norm_eps, sec.scale, sigmoid=r.kind == "channel_delta")
            st.attn = rec.rec_step(*args, gate=gate, step=st.dense)
        else:
            st.attn = rec.rec_chunk(*args, inp.seq_of_token, inp.q_start, inp.q_len, inp.max_q_len, step=st.dense)
        st.dense = None

    @staticmethod
    def _output_gate(st, sec):
        """Inputs of a recurrence's output gate: columns of the row, or the product behind a bottleneck."""
        r = sec.spec
        if r.kind == "channel_delta":
            return st.cat
        g = sec.col["z" if r.kind == "ssd" else "g"]
        return st.qkv[:, g:g + r.out_width]

    def _op_gated_norm(self, st, li):
        if st.attn is None:
            return              # applied by the decode step's kernel
        sec = self.layouts[li].part(RecurrentSpec)
        r, w = sec.spec, self.w.layers[li].rec
        groups = {"ssd": r.norm_groups, "delta": r.heads, "channel_delta": r.heads, "lightning": 1}[r.kind]
        par.gated_norm(st.attn, self._output_gate(st, sec), w.norm, st.qkv[:, sec.out:sec.out + r.out_width], groups, self.cfg.rms_norm_eps,
                       gate_first=r.kind == "ssd", silu=r.kind in ("ssd", "delta"), scale=sec.scale)
        st.attn = None
