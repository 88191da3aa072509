"""Python faces of the row kernels of the layered decoders (csrc/k_rows*.cu, libsfb_rows.so).

Tensors are on the current CUDA device; activations are bf16 or float32 (the dtype of the first activation tensor chooses the
kernel), everything that is 32-bit by contract is float32.  Launches go to the current stream and raise on an error code.
"""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_int64, c_void_p

import torch

from .. import _lib
from ..runtime.segments import note
from .native import _check, _p, _stream

MAX_TAPS = 8
PAGE = 64                 # positions of a cache page (kv/paged.py)


def _fp32(t: torch.Tensor) -> c_int:
    return c_int(1 if t.dtype == torch.float32 else 0)


POST = {"layer": 0, "rms": 1, "scale": 2}


def seam(x, n, *, h=None, y=None, y2=None, merge_w=(None, None), post=(None, None), embed=None, tokens=None, from_embed=False, add_embed=False,
         step_vec=None, tap=None, norm=(None, None), row_map=None, conv=None, eps=1e-6, status=None, embed_scale=1.0, parts_w=None, post_kind="layer",
         norm_kind="layer"):
    """x += LN(y; post) (y and y2: half the sum of their RMS norms), + embedding * embed_scale, + step_vec; h = LN(x; norm), or x itself.
    ``post_kind``: layer norm, "rms" norm or "scale" (y * post[0]); ``norm_kind``: "layer" or "rms".  ``parts_w`` [n, parts]: y is [n, parts, d]
    and its weighted sum over the parts is the output.
    ``conv``: (weight [taps, d], history, src, dst) applies h + conv(h) on a step of single-row segments."""
    rms = norm_kind == "rms"
    act = h if h is not None else (y if y is not None else embed)
    cw, hist, src, dst = conv if conv is not None else (None, None, None, None)
    _check(_lib.rows().sfb_rows_seam(_p(x), _p(y), _p(y2), _p(merge_w[0]), _p(merge_w[1]), _p(parts_w), _p(post[0]), _p(post[1]), _p(embed), _p(tokens),
                                     _p(step_vec), _p(tap), _p(norm[0]), _p(norm[1]), _p(h), _p(row_map), _p(cw), _p(hist), _p(src), _p(dst),
                                     c_int(from_embed), c_int(add_embed), c_int(cw.shape[0] if cw is not None else 0),
                                     c_int(parts_w.shape[1] if parts_w is not None else 0), c_int(POST[post_kind]), c_int(rms), c_int(n), c_int(x.shape[1]),
                                     c_int(embed.shape[0] if embed is not None else 0), c_float(eps), c_float(embed_scale), _fp32(act), _p(status), _stream()), "rows_seam")


MAX_STREAMS = 8


def stream_seam(x, n, *, h, norm, y=None, parts_w=None, mix=None, out=None, into=None, embed=None, tokens=None, embed_scale=1.0, tap=None, row_map=None, conv=None,
                keep=True, eps=1e-6, status=None):
    """Several residual streams x [rows, streams, d]: x_t = sum_s mix[s, t] x_s + out[t] y (y None: every stream is the scaled embedding), then
    h = RMS(sum_t into[t] x_t; norm) (``into`` None: ones).  ``parts_w`` [rows, parts]: y is [rows, parts, d] and its weighted sum the output.
    ``conv``: (weight [taps, d], history, src, dst) applies h + conv(h) on a step of single-row segments.  ``keep`` False: the streams end here."""
    cw, hist, src, dst = conv if conv is not None else (None, None, None, None)
    S, d = x.shape[1], x.shape[2]
    _check(_lib.rows().sfb_rows_streams(_p(x), _p(y), _p(parts_w), _p(mix), _p(out), _p(embed), _p(tokens), _p(tap), _p(into), _p(norm), _p(h), _p(row_map), _p(cw),
                                        _p(hist), _p(src), _p(dst), c_int(S), c_int(parts_w.shape[1] if parts_w is not None else 0),
                                        c_int(cw.shape[0] if cw is not None else 0), c_int(keep), c_int(n), c_int(d),
                                        c_int(embed.shape[0] if embed is not None else 0), c_float(eps), c_float(embed_scale), _fp32(h), _p(status), _stream()),
           "rows_streams")


CONV_PLAIN, CONV_RESIDUAL, CONV_SILU = 0, 1, 2


def conv(x, w, bias, y, hist, seg, n, mode=CONV_PLAIN):
    """y = causal depthwise convolution of x [n, C] over the step's segments (+ x, or followed by silu)."""
    _check(_lib.rows().sfb_rows_conv(_p(x), c_int64(x.stride(0)), _p(w), _p(bias), _p(y), _p(hist), _p(seg.row_seg), _p(seg.seg_row0), _p(seg.seg_len),
                                     _p(seg.seg_src), _p(seg.seg_dst), c_int(n), c_int(w.shape[1]), c_int(w.shape[0]), c_int(mode), _fp32(y),
                                     _stream()), "rows_conv")


def qk_append(proj, qw, kw, q, kpool, vpool, table, row_lane, row_pos, n, heads, eps, status):
    G, dim, vdim = kpool.shape[1], kpool.shape[3], vpool.shape[3]
    _check(_lib.rows().sfb_rows_qk_append(_p(proj), c_int64(proj.stride(0)), _p(qw), _p(kw), _p(q), _p(kpool), _p(vpool), _p(table), _p(row_lane),
                                          _p(row_pos), c_int(table.shape[1]), c_int(kpool.shape[0]), c_int(n), c_int(heads), c_int(G), c_int(dim),
                                          c_int(vdim), c_float(eps), _fp32(q), _p(status), _stream()), "rows_qk_append")


def head_append(proj, qw, kw, q, kpool, vpool, table, row_lane, row_pos, n, heads, eps, status):
    """q | k | v of ``proj``: RMS norm of every query and key head (weights [dim]), queries to ``q``, the rest to the pools."""
    G, dim, vdim = kpool.shape[1], kpool.shape[3], vpool.shape[3]
    _check(_lib.rows().sfb_rows_head_append(*_strides(proj), _p(qw), _p(kw), _p(q), _p(kpool), _p(vpool), _p(table), _p(row_lane), _p(row_pos),
                                            c_int(table.shape[1]), c_int(kpool.shape[0]), c_int(n), c_int(heads), c_int(G), c_int(dim), c_int(vdim),
                                            c_float(eps), _fp32(q), _p(status), _stream()), "rows_head_append")


def rot_append(proj, cs, dims, q, kpool, vpool, v_first, lam, table, row_lane, row_pos, n, heads, status):
    """q | k | v of ``proj``: queries and keys turned (cs [positions, dims / 2, 2]), values mixed with ``v_first`` by ``lam`` (None: left there,
    if given), queries to ``q``, the rest to the pools."""
    G, dim, vdim = kpool.shape[1], kpool.shape[3], vpool.shape[3]
    _check(_lib.rows().sfb_rows_rot_append(*_strides(proj), _p(cs), _p(q), _p(kpool), _p(vpool), _p(v_first), _p(lam), _p(table), _p(row_lane), _p(row_pos),
                                           c_int(table.shape[1]), c_int(kpool.shape[0]), c_int(n), c_int(heads), c_int(G), c_int(dim), c_int(vdim),
                                           c_int(dims), _fp32(q), _p(status), _stream()), "rows_rot_append")


def token_linear(x, w, table, col0, tokens, z, out, status):
    """out = gelu(x w^T) * table[token, col0 : col0 + dim]: one kernel for few rows, else a product to ``z`` and token_gate."""
    if _gemv_takes(x):
        _check(_lib.rows().sfb_rows_gemv_token(_p(w), _p(x), _p(out), *_strides(table), _p(tokens), c_int(col0), c_int(table.shape[0]), c_int(x.shape[0]),
                                               c_int(w.shape[0]), c_int(x.shape[1]), _p(status), _stream()), "rows_gemv")
        return out
    linear(x, w, None, z)
    token_gate(z, table, col0, tokens, out, x.shape[0], status)
    return out


def token_gate(z, table, col0, tokens, out, n, status):
    """out = gelu(z) * table[token, col0 : col0 + dim]."""
    _check(_lib.rows().sfb_rows_token_gate(_p(z), _p(table), _p(tokens), _p(out), c_int(n), c_int(z.shape[1]), c_int64(table.stride(0)), c_int(col0),
                                           c_int(table.shape[0]), _fp32(z), _p(status), _stream()), "rows_token_gate")


NO_WINDOW = 2 ** 31 - 1


def attn(q, kpool, vpool, table, row_lane, row_pos, rows, n_rows, bias, out, part, ml, heads, scale, splits, status, window=NO_WINDOW, vdim=None,
         compact=False, sink=None, cap=0.0):
    """Exact arm: one block per (row, group of heads, range of pages).  ``rows``: indices of the rows to run, or None for all.
    ``vpool`` None: values are the first ``vdim`` columns of the keys.  ``compact``: q and out hold only the rows of the launch.
    ``cap``: scores become cap tanh(score / cap), 0: not.  ``sink`` [heads]: logits that only the denominator sees."""
    _check(_lib.rows().sfb_rows_attn(_p(q), _p(kpool), _p(vpool), _p(table), _p(row_lane), _p(row_pos), _p(rows), _p(bias),
                                     c_int64(bias.shape[1] if bias is not None else 0), _p(sink), c_float(cap), _p(out), _p(part), _p(ml), c_int(table.shape[1]),
                                     c_int(kpool.shape[0]), c_int(n_rows), c_int(heads), c_int(kpool.shape[1]), c_int(kpool.shape[3]),
                                     c_int(vdim or vpool.shape[3]), c_int(splits), c_int(window), c_int(compact), c_float(scale), _fp32(q), _p(status), _stream()),
           "rows_attn")


def scan(gates, rb, ib, decay, u, y, out, S, sums, seg, n, bs):
    """Gated recurrence over the step's chunks; ``gates`` [parts, n, 2 bs] pre-activations (overwritten), y [n, width] view."""
    _check(_lib.rows().sfb_rows_scan(_p(gates), _p(rb), _p(ib), _p(decay), _p(u), _p(y), c_int64(y.stride(0)), _p(out), _p(S), _p(sums),
                                     _p(seg.chunk_seg), _p(seg.chunk_row0), _p(seg.chunk_rows), _p(seg.chunk_first), _p(seg.seg_src), _p(seg.seg_dst),
                                     _p(seg.seg_row0), _p(seg.seg_len), c_int(seg.chunks), c_int(seg.summaries), c_int(n), c_int(S.shape[1]), c_int(bs),
                                     _fp32(out), _stream()), "rows_scan")


def gated_step(x, y, cw, cb, hist, wg, rb, ib, decay, S, out, src, dst, n):
    """Convolution, gates, recurrence and output gate of single-row segments in one kernel."""
    _check(_lib.rows().sfb_rows_gated_step(_p(x), c_int64(x.stride(0)), _p(y), c_int64(y.stride(0)), _p(cw), _p(cb), _p(hist), _p(wg), _p(rb), _p(ib),
                                           _p(decay), _p(S), _p(out), _p(src), _p(dst), c_int(n), c_int(S.shape[1]), c_int(wg.shape[2]),
                                           c_int(cw.shape[0]), _fp32(out), _stream()), "rows_gated_step")


ACT = {"silu": 1, "gelu_tanh": 2, "clamp": 3}


def act_mul(gate_up, out, n, act="silu", alpha=0.0, limit=0.0):
    """out = act(gate) * up; "clamp": g sigmoid(alpha g) (u + 1) with g = min(gate, limit), u = up within +-limit."""
    _check(_lib.rows().sfb_rows_act_mul(_p(gate_up), *_strides(out), c_int(n), c_int(out.shape[1]), c_int(ACT[act]), c_float(alpha), c_float(limit), _fp32(out),
                                        _stream()), "rows_act_mul")


SINGLE_ACT = {"relu2": 4, "xielu": 5}          # activations of one input, with up to two numbers


def act_linear(x, w, out, act, a=0.0, b=0.0):
    """out = act(x w^T): one kernel for few rows, else a product and an element-wise pass over it."""
    if _gemv_takes(x):
        _gemv(x, w, None, out, SINGLE_ACT[act], a, b)
        return out
    linear(x, w, None, out)
    return act_rows(out, out, act, a, b)


def act_rows(z, out, act, a=0.0, b=0.0):
    _check(_lib.rows().sfb_rows_act(_p(z), _p(out), c_int64(out.numel()), c_int(SINGLE_ACT[act]), c_float(a), c_float(b), _fp32(out), _stream()), "rows_act")
    return out


def _strides(t) -> tuple:
    return (_p(t), c_int64(t.stride(0))) if t is not None else (None, c_int64(0))


def state_rows(q, k, v, dt, dt_bias, a, D, rot, rot_dims, k_scale, row_pos, y, S, N, groups, segs, n_segs, seg, conv=None,
               beta=None, q_scale=1.0, unit_eps=0.0):
    """S = a S + w k v^T, y = S^T q + D v, one block per (segment, head, tile of value dims); q, k, v, dt: [n, .] views.
    ``rot``: [positions, rot_dims / 2, 2] or None.  ``conv``: (weight [taps, C], bias, history, first channels of q, k, v) where every
    segment is one row and q, k, v are the inputs of a convolution with silu.  ``segs``: segments to run, or None for all.
    ``beta``: raw write strengths: the delta rule on unit vectors q (times ``q_scale``) and k."""
    _, H, P, Np = S.shape
    cw, cb, hist, ch = conv if conv is not None else (None, None, None, (0, 0, 0))
    _check(_lib.rows().sfb_rows_state(*_strides(q), *_strides(k), *_strides(v), *_strides(dt), _p(dt_bias), _p(a), _p(D), *_strides(beta), _p(rot), _p(row_pos), _p(y), _p(S),
                                      _p(cw), _p(cb), _p(hist), _p(segs), _p(seg.seg_row0), _p(seg.seg_len), _p(seg.seg_src), _p(seg.seg_dst),
                                      c_int(n_segs), c_int(rot_dims), c_int(cw.shape[0] if cw is not None else 0),
                                      c_int(cw.shape[1] if cw is not None else 0), *map(c_int, ch), c_int(H), c_int(groups), c_int(N), c_int(P),
                                      c_int(Np), c_float(k_scale), c_float(q_scale), c_float(unit_eps), _fp32(y), _stream()), "rows_state")


def state_tc_supports(dtype: torch.dtype, n: int, p: int, terms: int) -> bool:
    """Shapes the tensor-core arm of the matrix-state recurrence takes (csrc/k_rows_state_tc.cu)."""
    return dtype == torch.bfloat16 and n % 16 == 0 and n <= (128 if terms > 1 else 256) and p % 8 == 0


def state_turn(q, k, rot, rot_dims, k_scale, row_pos, out, n, heads, N):
    """Turned q and k of every row as two bf16 terms each: out [n, 4 heads N] = q hi | q lo | k hi | k lo."""
    _check(_lib.rows().sfb_rows_state_turn(*_strides(q), *_strides(k), _p(rot), _p(row_pos), _p(out), c_int(n), c_int(heads), c_int(N), c_int(rot_dims),
                                           c_float(k_scale), _stream()), "rows_state_turn")


def state_tc(qk, qk_cols, v, v_col, dt, dt_bias, log_a, D, S, sums, dec, rates, starts, y, N, groups, seg, terms, status):
    """Long segments in chunks of 128 rows.  ``qk``: [n, stride] tensor with the columns (q, k, distance to q's and to k's lower terms) of
    ``qk_cols``; ``v``: [n, stride] tensor with values from column ``v_col`` on; sums, dec, rates, starts: scratch of all chunks."""
    _, H, P, Np = S.shape
    mqk, mv = tensor_map(qk, qk.shape[1], 128), tensor_map(v, v.shape[1], 128)
    ms = tensor_map(starts, Np, 64)
    qc, kc, ql, kl = qk_cols
    _check(_lib.rows().sfb_rows_state_tc(mqk.ptr, mqk.ptr, mv.ptr, ms.ptr, _p(seg.long_row0), _p(seg.long_rows), _p(seg.long_seg), _p(seg.long_first),
                                         _p(seg.seg_src), _p(seg.seg_dst), *_strides(dt), _p(dt_bias), _p(log_a), _p(D), _p(S), _p(sums), _p(dec), _p(rates),
                                         _p(starts), _p(y), c_int(seg.nlong), c_int(seg.nchunks), c_int(H), c_int(groups), c_int(N), c_int(P), c_int(Np),
                                         c_int(terms), c_int(qc), c_int(kc), c_int(v_col), c_int(ql), c_int(kl), _p(status), _stream()), "rows_state_tc")


DELTA_RATES = 6           # numbers per (chunk, head) and row (csrc/k_rows_state_tc.cuh)


def delta_tc_supports(dtype: torch.dtype, n: int, p: int) -> bool:
    """Shapes the tensor-core arm of the delta rule takes (csrc/k_rows_delta_tc.cu)."""
    return dtype == torch.bfloat16 and n % 16 == 0 and n <= 128 and p % 8 == 0


def delta_tc(qkv, cols, dt, beta, dt_bias, log_a, S, rates, dec, inv, u, starts, y, N, groups, seg, q_scale, unit_eps, status):
    """Long segments in chunks of 128 rows.  ``qkv``: [n, stride] tensor with q, k, v from the columns ``cols`` on.  Scratch of all chunks: rates,
    dec (32-bit), inv [chunks, H, 2, 128, 128], starts [2, chunks, H, N, P] and u [2, chunks, H, 128, P] in bf16."""
    _, H, P, Np = S.shape
    mqk, mt, mt64 = tensor_map(qkv, qkv.shape[1], 128), tensor_map(inv, 128, 128), tensor_map(inv, 128, 64)
    mv, us, ss = tensor_map(qkv, qkv.shape[1], 128, box_cols=32), tensor_map(u, P, 128, box_cols=32), tensor_map(starts, P, N, box_cols=32)
    mu, ms, at = tensor_map(u, P, 128), tensor_map(starts, P, 64), [c_int(c) for c in cols]
    _check(_lib.rows().sfb_rows_delta_tc(mqk.ptr, mt.ptr, mt64.ptr, mv.ptr, us.ptr, ss.ptr, _p(seg.long_row0), _p(seg.long_rows), _p(seg.long_seg), _p(seg.long_first), _p(seg.seg_src),
                                         _p(seg.seg_dst), *_strides(qkv), *_strides(dt), *_strides(beta), _p(dt_bias), _p(log_a), _p(S), _p(rates), _p(dec),
                                         _p(inv), c_int(seg.nlong), c_int(seg.nchunks), c_int(H), c_int(groups), c_int(N),
                                         c_int(P), c_int(Np), *at, c_float(q_scale), c_float(unit_eps), _p(status), _stream()), "rows_delta_tc")
    _check(_lib.rows().sfb_rows_delta_out(mqk.ptr, mqk.ptr, mu.ptr, ms.ptr, _p(seg.long_row0), _p(seg.long_rows), _p(rates), _p(starts), _p(y),
                                          c_int(seg.nchunks), c_int(H), c_int(groups), c_int(N), c_int(P), at[0], at[1], _p(status),
                                          _stream()), "rows_delta_tc")


STATE_PADS = tuple(range(32, 257, 32)) + (384, 512)


def state_pad(n: int) -> int:
    """Length of a stored state column of ``n`` elements."""
    for p in STATE_PADS:
        if n <= p:
            return p
    raise ValueError(f"states of {n} rows are beyond the {STATE_PADS[-1]} implemented")


def gated_norm(y, gate, w, out, part, before, eps):
    """RMS norm of equal parts of a row, times silu(gate): ``before`` the norm, or after it; optional weight."""
    _check(_lib.rows().sfb_rows_gated_norm(_p(y), *_strides(gate), _p(w), _p(out), c_int(y.shape[0]), c_int(y.shape[1]), c_int(part), c_int(before),
                                           c_float(eps), _fp32(y), _stream()), "rows_gated_norm")


def latent_append(q, c, w, cs, pool, table, row_lane, row_pos, n, heads, dim, rot, rank, eps, status, halves=False, cq=None, wq=None, cq_out=None):
    """``c`` [n, stride] view of latent | shared key part: normed and turned into the pool [pages, 1, 64, rank + rot].  ``q`` [n, stride] view of the
    queries, turned in place, or None.  ``cq``, ``wq``: latent of the queries, a view with c's stride, normed to ``cq_out`` [n, q_rank].
    ``halves``: element i turns with i + rot / 2, else neighbours do."""
    _check(_lib.rows().sfb_rows_latent_append(*_strides(q), _p(c), _p(cq), _p(cq_out), c_int64(c.stride(0)), _p(w), _p(wq), _p(cs), _p(pool), _p(table), _p(row_lane), _p(row_pos),
                                              c_int(table.shape[1]), c_int(pool.shape[0]), c_int(n), c_int(heads), c_int(dim), c_int(rot), c_int(rank),
                                              c_int(wq.shape[0] if wq is not None else 0), c_int(halves), c_float(eps), _fp32(pool), _p(status), _stream()),
           "rows_latent_append")


def latent_turn(q, cs, row_pos, n, heads, dim, rot, halves):
    """The last ``rot`` of every head of q [n, heads (dim + rot)], turned in place (``halves``: element i with i + rot / 2, else neighbours)."""
    _check(_lib.rows().sfb_rows_latent_turn(*_strides(q), _p(cs), _p(row_pos), c_int(n), c_int(heads), c_int(dim), c_int(rot), c_int(halves), _fp32(q),
                                            _stream()), "rows_latent_turn")


def head_proj(x, x_head, w, out, out_head, n, rows=None, lists=0, tail=0, merge=None, turn=None, gate=None):
    """out[row][h] = x[row][h] w[h], w [heads, K, M]; heads ``x_head`` / ``out_head`` elements apart.  ``rows`` names rows of x (lists=1) or
    of out (lists=2); ``tail`` elements behind x's K are copied behind out's M, turned by ``turn`` = (cs, row_pos) (element i with i + tail / 2).
    ``merge``: (part, ml, parts, ctas) of latent_decode; x is then the merged attention output.  ``gate`` [rows of out, heads M]
    view: outputs are multiplied by its sigmoid."""
    part, ml, parts, most = merge or (None, None, None, 0)
    cs, pos = turn if turn is not None else (None, None)
    H, K, M = w.shape
    _check(_lib.rows().sfb_rows_head_proj(*_strides(x), c_int64(x_head), _p(w), *_strides(out), c_int64(out_head), _p(rows), c_int(lists if rows is not None else 0),
                                          _p(part), _p(ml), _p(parts), c_int(most), _p(pos), c_int(n), c_int(H), c_int(K), c_int(M), c_int(tail), _p(cs),
                                          *_strides(gate), _fp32(w), _stream()), "rows_head_proj")


def gather_pages(pool, pages, out, count, status):
    nbytes = pool.stride(0) * pool.element_size()
    _check(_lib.rows().sfb_rows_gather_pages(_p(pool), _p(pages), _p(out), c_int(count), c_int64(nbytes), c_int(pool.shape[0]), _p(status), _stream()),
           "rows_gather_pages")


def sample(logits, row_pos, temperature, seed, mask, best_val, best_id, n):
    _check(_lib.rows().sfb_sample(_p(logits), c_int64(logits.stride(0)), _p(row_pos), _p(temperature), _p(seed), _p(mask),
                                  c_int64(mask.stride(0) if mask is not None else 0), _p(best_val), _p(best_id), c_int(n), c_int(logits.shape[1]),
                                  c_int(0), _stream()), "sample")


GEMV_ROWS = 4


def _gemv_takes(x: torch.Tensor) -> bool:
    n, K = x.shape
    return x.dtype == torch.bfloat16 and n <= GEMV_ROWS and K % 8 == 0 and (n if n < 3 else 4) * K * 2 <= 200 * 1024


def _gemv(x, w, b, out, act: int = 0, alpha: float = 0.0, limit: float = 0.0) -> None:
    _check(_lib.rows().sfb_rows_gemv(_p(w), _p(x), _p(b), *_strides(out), c_int(x.shape[0]), c_int(out.shape[1]), c_int(x.shape[1]),
                                     c_int(out.dtype == torch.float32), c_int(act), c_float(alpha), c_float(limit), _stream()), "rows_gemv")


def linear(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor | None, out: torch.Tensor) -> torch.Tensor:
    """out = x w^T (+ b) with 32-bit accumulation: up to four bf16 rows by the streaming kernel, a library product otherwise."""
    if _gemv_takes(x):
        _gemv(x, w, b, out)
        return out
    if b is not None:
        torch.addmm(b, x, w.t(), out=out)
    else:
        torch.mm(x, w.t(), out=out)
    note("linear")
    return out


def gated_linear(x: torch.Tensor, w: torch.Tensor, scratch: torch.Tensor | None, out: torch.Tensor, act: str = "silu", alpha: float = 0.0,
                 limit: float = 0.0) -> torch.Tensor:
    """out = act(x wg^T) * (x wu^T), w = wg stacked on wu; ``scratch`` [n, 2 ff] holds both products where they are not fused."""
    if _gemv_takes(x):
        _gemv(x, w, None, out, ACT[act], alpha, limit)
        return out
    linear(x, w, None, scratch)
    act_mul(scratch, out, x.shape[0], act, alpha, limit)
    return out


class exact_matmul:
    """Library products inside keep 32-bit accumulation throughout: no TF32, no 16-bit partial sums in split reductions."""

    def __enter__(self):
        m = torch.backends.cuda.matmul
        self.saved = (m.allow_tf32, m.allow_bf16_reduced_precision_reduction)
        m.allow_tf32, m.allow_bf16_reduced_precision_reduction = False, False

    def __exit__(self, *exc):
        m = torch.backends.cuda.matmul
        m.allow_tf32, m.allow_bf16_reduced_precision_reduction = self.saved


def block_gates(u: torch.Tensor, wg: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Block-diagonal product with a 32-bit result: out [parts, n, 2 bs] = u's part k [n, bs] times wg[k] [2 bs, bs] transposed."""
    parts, _, bs = wg.shape
    x = u.view(u.shape[0], parts, bs).transpose(0, 1)
    if u.dtype == torch.float32:
        torch.bmm(x, wg.transpose(1, 2), out=out)
    else:
        torch.bmm(x, wg.transpose(1, 2), out_dtype=torch.float32, out=out)
    note("block_gates")
    return out


def head(x: torch.Tensor, embed: torch.Tensor, out: torch.Tensor, name: str = "head") -> torch.Tensor:
    """32-bit logits of x [rows, width] against the output table (or a router's)."""
    if _gemv_takes(x):
        _gemv(x, embed, None, out)
        return out
    if x.dtype == torch.float32:
        torch.mm(x, embed.t(), out=out)
    else:
        torch.mm(x, embed.t(), out_dtype=torch.float32, out=out)
    note(name)
    return out


def attn_blocks(heads: int, kv_heads: int) -> int:
    """Blocks the exact arm launches per row and range."""
    rep = heads // kv_heads
    r = 1 if rep <= 1 else 2 if rep <= 2 else 4 if rep <= 4 else 8
    return kv_heads * -(-rep // r)


STREAM_CTAS = 592          # most CTAs of the streaming arm (csrc/k_rows_attn_dec.cu)
STREAM_ROWS = 1024


def attn_stream_heads(heads: int, kv_heads: int, dim: int) -> int:
    """Query heads the streaming arm handles per pass over a key head's pages."""
    rep = heads // kv_heads
    r = 1 if rep <= 1 else 2 if rep <= 2 else 4
    return min(r, 2) if dim > 128 else r


def attn_stream_supports(dtype: torch.dtype, dim: int, vdim: int) -> bool:
    return dtype == torch.bfloat16 and dim in (32, 64, 96, 128, 256) and vdim % 32 == 0 and vdim <= 256


def attn_stream(q, kpool, vpool, table, row_lane, row_pos, rows, n_rows, bias, out, part, ml, heads, scale, page_bound, status,
                window=NO_WINDOW, sink=None, cap=0.0):
    """Single rows, bf16: the pages of all rows cut evenly over the machine.  ``page_bound``: at least the sum of the pages that rows see."""
    G, dim, vdim = kpool.shape[1], kpool.shape[3], vpool.shape[3]
    _check(_lib.rows().sfb_rows_attn_stream(_p(q), _p(kpool), _p(vpool), _p(table), _p(row_lane), _p(row_pos), _p(rows), _p(bias),
                                            c_int64(bias.shape[1] if bias is not None else 0), _p(sink), c_float(cap), c_int(window), _p(out), _p(part), _p(ml),
                                            c_int(table.shape[1]), c_int(kpool.shape[0]), c_int(n_rows), c_int(heads), c_int(G), c_int(dim), c_int(vdim),
                                            c_int(attn_stream_heads(heads, G, dim)), c_int(page_bound), c_float(scale), _p(status), _stream()),
           "rows_attn_stream")


def attn_tc_supports(dtype: torch.dtype, dim: int, vdim: int) -> bool:
    """Shapes the tensor-core arm takes (csrc/k_rows_attn_tc.cu)."""
    return dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and max(dim, vdim) <= 128


class TensorMap:
    """A 2-D TMA map over a bf16 tensor seen as [rows, cols] with rows ``stride`` elements apart (cols by default), from element
    ``first`` on; boxes of ``box_cols`` (64 or 32) columns x ``box`` rows."""

    def __init__(self, t: torch.Tensor, rows: int, cols: int, box: int, stride: int | None = None, first: int = 0, box_cols: int = 64):
        self._raw = (ctypes.c_uint8 * 192)()
        self.ptr = c_void_p((ctypes.addressof(self._raw) + 63) & ~63)
        rc = _lib.rows().sfb_rows_tmap(self.ptr, c_void_p(t.data_ptr() + 2 * first), c_int64(rows), c_int64(cols), c_int64((stride or cols) * 2), c_int(box),
                                       c_int(box_cols))
        if rc:
            raise RuntimeError(f"tensor map over [{rows}, {cols}]: error {rc}")


def attn_pools(kv, index: int, tc: bool):
    """(k pool, v pool, tensor maps of both for the tensor-core arm or None) of one attention layer run."""
    k, v = kv.k[index], kv.v[index]
    maps = None
    if tc and k.is_cuda:
        maps = tuple(TensorMap(t, t.shape[0] * t.shape[1] * t.shape[2], t.shape[3], 64) for t in (k, v))
    return k, v, maps


_maps: dict[tuple, TensorMap] = {}


def tensor_map(t: torch.Tensor, cols: int, box: int, stride: int | None = None, first: int = 0, box_cols: int = 64) -> TensorMap:
    """The map over all of ``t``'s storage, kept, so that one map serves every step over a scratch buffer (it is an address and a shape:
    memory that is allocated again at the same place may use it again)."""
    stride = stride or cols
    total = t.untyped_storage().nbytes() // 2
    key = (t.untyped_storage().data_ptr(), total, cols, box, stride, first, box_cols)
    m = _maps.get(key)
    if m is None:
        base = t if t.storage_offset() == 0 else torch.empty(0, dtype=t.dtype, device=t.device).set_(t.untyped_storage())
        m = _maps[key] = TensorMap(base, (total - first - cols) // stride + 1, cols, box, stride, first, box_cols)
    return m


def attn_tc(q, kv, table, row_lane, row_pos, tiles, n_tiles, bias, out, heads, scale, status, window=NO_WINDOW, sink=None, cap=0.0):
    """Tensor-core arm over runs of rows: ``tiles`` are (row0, rows <= 256) pairs, each inside one segment; kv from attn_pools."""
    k, v, (mk, mv) = kv
    mq = tensor_map(q, q.shape[1], 128)
    G = k.shape[1]
    _check(_lib.rows().sfb_rows_attn_tc(mq.ptr, mk.ptr, mv.ptr, None, _p(table), _p(row_lane), _p(row_pos), _p(tiles), None, c_int(n_tiles), _p(bias),
                                        c_int64(bias.shape[1] if bias is not None else 0), _p(sink), c_float(cap), _p(out), None, c_int64(0),
                                        c_int(table.shape[1]), c_int(k.shape[0]), c_int(heads), c_int(G), c_int(k.shape[3]), c_int(v.shape[3]), c_int(0), c_int(G * 64), c_int(64),
                                        c_int(window), c_float(scale), _p(status), _stream()), "rows_attn_tc")


def latent_tc_supports(dtype: torch.dtype, dim: int, rot: int, vdim: int, rank: int) -> bool:
    return attn_tc_supports(dtype, dim, vdim) and rot % 8 == 0 and 0 < rot <= 64 and rank % 8 == 0


def latent_decode_supports(dtype: torch.dtype, rot: int, rank: int) -> bool:
    """Shapes the tensor-core arm for single rows takes (csrc/k_rows_latent_dec.cu)."""
    return dtype == torch.bfloat16 and rot % 8 == 0 and 0 < rot <= 64 and rank % 8 == 0 and rank <= 512


LATENT_ROWS = 256          # most rows of a launch of latent_decode (csrc/k_rows_latent_dec.cu)
SMS = 148


def latent_ctas(heads: int, pages: int) -> int:
    """CTAs that share up to ``pages`` pages of a launch: at most one per SM over the groups of heads."""
    return max(1, min(SMS // -(-heads // (16 if heads <= 16 else 32)), pages if pages <= 64 else (pages + 1) // 2))


def latent_places(n: int, heads: int) -> int:
    """Partial results (a row, every head) that a launch of n rows leaves at most."""
    return SMS // -(-heads // (16 if heads <= 16 else 32)) + 1 + n


def latent_decode(q, pool, rank, rot, table, row_lane, row_pos, rows, n, heads, part, ml, parts, window, ctas, pages, scale, status):
    """Attention of single rows over the cached latents, the pages of all rows (``pages`` at most) shared equally among ``ctas``: (log2 maximum, sum, output) of every
    share of a row to ml and part, ctas + n places; a row's first place and number of places to parts [n, 2].  q: [n, heads (rank + rot)] of the
    launch's rows."""
    key, box = rank + rot, _lib.rows().sfb_rows_latent_heads(heads)
    maps = (tensor_map(q, rank, box, key), tensor_map(q, rot, box, key, rank), tensor_map(pool, rank, 64, key), tensor_map(pool, rot, 64, key, rank))
    _check(_lib.rows().sfb_rows_latent_decode(*(m.ptr for m in maps), _p(table), _p(row_lane), _p(row_pos), _p(rows), _p(part), _p(ml), _p(parts),
                                              c_int(table.shape[1]), c_int(pool.shape[0]), c_int(n), c_int(heads), c_int(rank), c_int(rot), c_int(window),
                                              c_int(ctas), c_int(pages), c_int(q.storage_offset() // key), c_float(scale), _p(status), _stream()), "rows_latent_decode")


def expand(c: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out [heads, rows, M] = c [rows, K] times w [heads, K, M] of every head."""
    torch.bmm(c.unsqueeze(0).expand(w.shape[0], -1, -1), w, out=out)
    note("linear")
    return out


def latent_attn_tc(q, q_stride, kx, vx, rows, rank, row_pos, tiles, offs, n_tiles, out, heads, dim, rot, vdim, window, scale, status, gate=None):
    """Tensor-core arm over keys kx [heads, m, dim] and values vx [heads, m, vdim] that were multiplied out, and the shared key part: the
    last columns of ``rows`` [m, rank + rot].  q: [n, q_stride] with a head's dim + rot columns side by side.
    ``gate`` [n, heads vdim] view: outputs are multiplied by its sigmoid."""
    m = kx.shape[1]
    mq, mk, mv = tensor_map(q, heads * (dim + rot), 128, q_stride, q.storage_offset()), tensor_map(kx, dim, 64), tensor_map(vx, vdim, 64)
    mr = tensor_map(rows, rot, 64, rank + rot, rank)
    _check(_lib.rows().sfb_rows_attn_tc(mq.ptr, mk.ptr, mv.ptr, mr.ptr, None, None, _p(row_pos), _p(tiles), _p(offs), c_int(n_tiles), None, c_int64(0), None, c_float(0.0),
                                        _p(out), *_strides(gate), c_int(0), c_int(m // 64), c_int(heads), c_int(heads), c_int(dim), c_int(vdim), c_int(rot), c_int(64),
                                        c_int(m), c_int(window), c_float(scale), _p(status), _stream()), "rows_attn_tc")


# ---- mixture of experts (csrc/k_rows_moe.cu, csrc/k_rows_moe_tc.cu) --------------------------------------------------------
MOE_TILE, MOE_TC_TILE = 32, 128          # pairs of a tile on CUDA cores, on the tensor cores
MOE_MAX_EXPERTS, MOE_MAX_TOP = 1024, 32


def moe_tiles(n: int, experts: int, top: int, tile: int) -> int:
    """Most tiles of a step of n rows."""
    return n * top // tile + min(experts, n * top)


class Choice:
    """How a row's experts are chosen and weighted.  ``corr`` None: the largest logits, the softmax over them.  Else s = sigmoid(logit): the largest
    s + corr [E] among the ``keep`` of ``groups`` groups of neighbours whose two largest sum highest, weighted by s over their sum, times ``scale``."""

    def __init__(self, corr=None, groups: int = 1, keep: int = 1, scale: float = 1.0):
        self.corr, self.groups, self.keep, self.scale = corr, groups, keep, scale

    def args(self) -> tuple:
        return _p(self.corr), c_int(self.groups), c_int(self.keep), c_float(self.scale)


SOFTMAX = Choice()
MOE_MAX_GROUPS = 256


def moe_route(z, ids, wts, experts, top, shared, choice=SOFTMAX):
    """Choices [n, top] and weights [n, top + shared] of logits z [n, >= experts + shared]."""
    _check(_lib.rows().sfb_rows_moe_route(*_strides(z), _p(ids), _p(wts), c_int(z.shape[0]), c_int(experts), c_int(top), c_int(shared), *choice.args(), _stream()),
           "rows_moe_route")


MOE_PLAN_ROWS = 128        # up to this many rows the plan makes the choice itself


def moe_plan(z, ids, wts, order, tiles, count, experts, top, shared, tile, choice=SOFTMAX):
    """``z``: logits (few rows: the choice is made here), or None: ``ids`` are there."""
    zp, ld = _strides(z)
    _check(_lib.rows().sfb_rows_moe_plan(zp, ld, _p(ids), _p(wts), _p(order), _p(tiles), _p(count), c_int(ids.shape[0]), c_int(experts), c_int(top),
                                         c_int(shared), c_int(tile), *choice.args(), _stream()), "rows_moe_plan")


MOE_ACT = {None: 0, "clamp": 3, **SINGLE_ACT}          # of an expert's first product: gated (gate and up stacked), or of one product; None: the second


def moe_tile(x, w, out, plan, M, top, slots, act, alpha=0.0, limit=0.0):
    """One product of every expert on its pairs; ``plan``: (order, tiles, count, most tiles).  ``act`` (see MOE_ACT): x [n, K], w [E, M, K] (gated:
    [E, 2 M, K]), out [pairs, M] in plan order; None: x [pairs, K], w [E, M, K], out [n, slots, M]."""
    order, tiles, count, most = plan
    _check(_lib.rows().sfb_rows_moe_tile(_p(x), _p(w), _p(out), _p(order), _p(tiles), _p(count), c_int(most), c_int(M), c_int(w.shape[2]), c_int(top),
                                         c_int(slots), c_int(MOE_ACT[act]), c_float(alpha), c_float(limit), _fp32(out), _stream()), "rows_moe_tile")


def moe_tc_supports(dtype: torch.dtype, width: int, ff: int, shared_ff: int) -> bool:
    """Shapes the tensor-core products take (csrc/k_rows_moe_tc.cu)."""
    return dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0 and shared_ff % 8 == 0


MOE_GATHER_ROWS = 256      # up to this many rows the product gathers its rows itself (csrc/k_rows_moe_tc.cu)


def moe_pick(x, order, out, top):
    """Rows x [n, K] in plan order: out [pairs, K]."""
    _check(_lib.rows().sfb_rows_moe_pick(_p(x), _p(order), _p(out), c_int(out.shape[0]), c_int(top), c_int(x.shape[1]), _stream()), "rows_moe_pick")


def moe_gemm(x, w, out, plan, shared, n, M, top, slots, act, status, alpha=0.0, limit=0.0, gather=False):
    """``moe_tile`` on the tensor cores (tiles of up to 128 pairs); w and out in bf16; x in plan order, or ``gather``: the layer's rows.
    ``shared``: (x, w, out, M, limit) of the shared expert, whose rows are done beside the pairs, or None."""
    order, tiles, count, most = plan
    sx, sw, sout, sm, sl = shared if shared is not None else (None, None, None, 0, 0.0)
    msx, msw = (tensor_map(sx, sx.shape[1], 128).ptr, tensor_map(sw, sw.shape[1], 128).ptr) if shared is not None else (None, None)
    mx, mw = tensor_map(x, x.shape[1], 1 if gather else 128), tensor_map(w, w.shape[2], 128)
    _check(_lib.rows().sfb_rows_moe_gemm(mx.ptr, mw.ptr, msx, msw, _p(order), _p(tiles), _p(count), _p(out), _p(sout), c_int(most), c_int(n), c_int(M),
                                         c_int(w.shape[2]), c_int(sm), c_int(sw.shape[1] if sw is not None else 0), c_int(top), c_int(slots), c_int(MOE_ACT[act]),
                                         c_int(gather), c_float(alpha), c_float(limit), c_float(sl), _p(status), _stream()), "rows_moe_gemm")


def moe_gemv_takes(x: torch.Tensor, ff: int, shared_ff: int) -> bool:
    n, K = x.shape
    return x.dtype == torch.bfloat16 and n <= GEMV_ROWS and K % 8 == 0 and ff % 8 == 0 and shared_ff % 8 == 0 and max(K, ff, shared_ff) * 2 <= 200 * 1024


def moe_gemv(z, ids, wts, x, w, out, shared, n, M, top, slots, act, alpha=0.0, limit=0.0, choice=SOFTMAX):
    """Few rows; ``z``: logits, the experts are chosen here and left in ``ids`` and ``wts``; None: ``ids`` are there.  ``shared``: (x, w, out, M,
    limit) of the shared expert or None."""
    sx, sw, sout, sm, sl = shared if shared is not None else (None, None, None, 0, 0.0)
    _check(_lib.rows().sfb_rows_moe_gemv(*_strides(z), c_int(w.shape[0]), _p(ids), _p(wts), *choice.args(), _p(x), _p(w), _p(out), _p(sx), _p(sw), _p(sout), c_int(ids.numel()), c_int(n), c_int(M), c_int(w.shape[2]),
                                         c_int(sm), c_int(sw.shape[1] if sw is not None else 0), c_int(top), c_int(slots), c_int(MOE_ACT[act]), c_float(alpha),
                                         c_float(limit), c_float(sl), _stream()), "rows_moe_gemv")
