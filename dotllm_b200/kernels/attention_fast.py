"""Dispatch to the tensor-core attention kernels for the sizes they take.

Decode steps (one new token per sequence) go to the stream-K kernel of csrc/attention_decode.cu,
which cuts the step's cache pages into equal shares per block on the device.  Its scratch (the
partial results of cut segments, two per block) is allocated once per step and shared by the
layers, which run one after another on one stream.
"""
from __future__ import annotations

import torch

from . import library as _library

_P, _I, _F = _library._P, _library._I, _library._F
_library.register_signatures({
    "dl_attention_decode_bf16": [_P, _I, _P, _I, _P, _P, _I, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _P, _F, _P, _P, _I, _I, _I,
                                 _P, _P, _I, _P, _I, _P, _P],
    "dl_attention_decode_fresh_bf16": [_P, _I, _P, _I, _P, _I, _P, _P, _I, _I, _P, _I, _P, _P, _I, _P, _P, _I, _I, _I, _I,
                                       _I, _F, _I, _I, _P, _P, _I, _P, _I, _P, _P],
    "dl_attention_decode_gated_bf16": [_P, _I, _P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _P, _I, _P, _F, _P, _I, _P, _I, _P, _P, _I, _P, _P, _I, _I,
                                       _I, _I, _I, _F, _I, _I, _P, _P, _I, _P, _I, _P, _P],
    "dl_attention_prefill_bf16": [_P, _I, _P, _I, _P, _P, _I, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I,
                                  _F, _I, _I, _P, _F, _P, _P, _I, _P, _P],
    "dl_attention_prefill_tc_bf16": [_P, _I, _I, _P, _I, _P, _P, _I, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _I,
                                     _F, _I, _I, _P, _F, _P, _P, _I, _P, _P],
})

PREFILL_ROWS = 128       # query rows per block of the mma.sync prefill kernel (AP_ROWS)
PREFILL_TC_ROWS = 256    # ... and of the tcgen05 one (PT_TILES * PT_ROWS)
PREFILL_TC_HEAD_DIMS = (64, 128)     # head sizes of the tcgen05 prefill kernel; others take the mma.sync one
PREFILL_TC = True        # False: always the mma.sync kernel (tests compare the two)
PREFILL_TC_SPECIAL = True    # False: prompts with kept first tokens or sinks take the mma.sync kernel at every head size

DECODE_HEAD_DIMS = (32, 64, 96, 128)
DECODE_SPECIAL = True    # False: decode steps with kept first tokens or sinks take the packed prefill kernel (tests compare the two)
DECODE_BLOCKS = 0        # > 0: persistent blocks of the decode kernel (tuning and tests); 0: one per multiprocessor


def decode_fits(group, head_dim):
    """Whether at least two ring stages and the merge buffers of the decode kernel fit in shared
    memory (it takes up to six stages when they fit)."""
    return 2 * 2 * 64 * head_dim * 2 + 4 * group * (head_dim + 4) * 4 + 4096 <= 227 * 1024


def decode_tiles(n_heads, n_kv_heads, split=True):
    """KV heads as the decode kernel counts them: a head of the pages whose group of query heads has more rows than a tile (16)
    is walked by several tiles of query heads, each of equally many (a group of a prime number of heads: one head a tile);
    without ``split`` such a group is not taken (0)."""
    group = n_heads // n_kv_heads
    if group > 16 and not split:
        return 0
    return n_kv_heads * next(p for p in range(1, group + 1) if group % p == 0 and group // p <= 16)


def _gate_args(gate):
    """(pointer, row stride) of a gate [T, n_heads], or of none."""
    if gate is None:
        return None, 0
    return gate.data_ptr(), gate.stride(0) if gate.shape[0] > 1 else max(gate.stride(0), gate.shape[1])


def _decode(q, q_stride, out, k_pool, v_pool, n_pages, block_table, n_heads, n_kv_heads, head_dim,
            scale, window, plan, keep_first=0, sinks=None, softcap=0.0, slopes=None, gate=None):
    B = plan.n_seqs
    tiles = decode_tiles(n_heads, n_kv_heads)
    group = n_heads // tiles
    part_o, part_ml, slots = _decode_scratch(plan, group, head_dim, q.device)
    counters = _pair_counters(q.device)
    _library.call("dl_attention_decode_bf16", q.data_ptr(), q_stride, out.data_ptr(), out.stride(0),
                  k_pool.data_ptr(), v_pool.data_ptr(), n_pages, plan.seq_total.data_ptr(),
                  block_table.data_ptr(), block_table.shape[1], B, n_heads, tiles, head_dim,
                  scale, window, int(keep_first), None if sinks is None else sinks.data_ptr(), float(softcap),
                  None if slopes is None else slopes.data_ptr(), *_gate_args(gate), n_kv_heads, DECODE_BLOCKS,
                  part_o.data_ptr(), part_ml.data_ptr(), slots, counters.data_ptr(), counters.numel(),
                  _library.status_word(q.device).data_ptr(), _library.current_stream())
    return True


_counters = {}


def _pair_counters(device):
    """Per device: one arrival counter per (sequence, KV head) of a decode step.  Zero at rest: the block
    that finishes a pair resets its counter.  Launches that share them must be on one stream."""
    key = device.index
    if key not in _counters:
        _counters[key] = torch.zeros(1 << 16, dtype=torch.int32, device=device)
        _library.register_counters(_counters[key])
    return _counters[key]


def _decode_scratch(plan, group, head_dim, device):
    slots = 2 * max(1, _library.library().dl_sm_count())
    key = ("decode", group, head_dim)
    if key not in plan.scratch:
        plan.scratch[key] = (torch.empty(slots * group * head_dim, dtype=torch.float32, device=device),
                             torch.empty(slots * group * 2, dtype=torch.float32, device=device))
    return plan.scratch[key] + (slots,)


FRESH_ROTATE_HEAD_DIMS = (64, 128)   # head sizes whose rotation the decode kernel does itself


def decode_fresh(q, k, v, cos, sin, rotary_dim, block_table, k_pool, v_pool, n_heads, n_kv_heads, head_dim,
                 scale, window, plan, biases=None, gate=None, sinks=None, softcap=0.0, split=False, slopes=None):
    """A decode step with the new token handled inside the attention kernel (rotation of q and k,
    cache write, attention): returns the output, or None when the sizes are not the kernel's.
    ``biases`` (q, k, v: float32 vectors or None) are added before the rotation and ``gate`` ([B, n_heads] logits of
    q's dtype, a column view is fine) multiplies each head's output by its sigmoid, both inside the kernel; with them
    k and v may be None (a layer that reads another's cache: only the queries are biased and rotated).  ``sinks``,
    ``softcap``, ``slopes`` and ``split`` as in ``run``."""
    tiles = decode_tiles(n_heads, n_kv_heads, split)
    if tiles == 0:
        return None
    group = n_heads // tiles
    if not (plan.all_single and q.shape[0] == plan.n_seqs and head_dim in DECODE_HEAD_DIMS
            and decode_fits(group, head_dim) and (rotary_dim == 0 or (rotary_dim == head_dim
                                                                      and head_dim in FRESH_ROTATE_HEAD_DIMS))):
        return None
    rows = lambda t: t.stride(0) if t.shape[0] > 1 else max(t.stride(0), t.shape[1])
    extras = biases is not None or gate is not None or sinks is not None or softcap > 0 or slopes is not None or tiles != n_kv_heads
    if k is None and not extras:
        return None
    qs = rows(q)
    ks, vs = (rows(k), rows(v)) if k is not None else (0, 0)
    if q.stride(1) != 1 or qs % 8 or q.data_ptr() % 16 or k_pool.dtype != q.dtype or v_pool.dtype != q.dtype:
        return None
    if k is not None and (k.stride(1) != 1 or v.stride(1) != 1 or ks % 4 or vs % 4 or k.data_ptr() % 8 or v.data_ptr() % 8
                          or k.dtype != q.dtype or v.dtype != q.dtype):
        return None
    if gate is not None and (gate.dtype != q.dtype or gate.stride(1) != 1 or gate.shape != (q.shape[0], n_heads)):
        return None
    if rotary_dim and (cos.dtype != torch.float32 or sin.dtype != torch.float32 or not cos.is_contiguous()
                       or not sin.is_contiguous() or cos.shape != sin.shape or cos.shape[1] != head_dim // 2
                       or cos.data_ptr() % 16 or sin.data_ptr() % 16):
        return None
    B = plan.n_seqs
    out = torch.empty((B, n_heads * head_dim), dtype=q.dtype, device=q.device)
    part_o, part_ml, slots = _decode_scratch(plan, group, head_dim, q.device)
    counters = _pair_counters(q.device)
    if extras:
        qb, kb, vb = biases if biases is not None else (None, None, None)
        ptr = lambda t: None if t is None else t.data_ptr()
        _library.call("dl_attention_decode_gated_bf16", q.data_ptr(), qs, ptr(k), ks, ptr(v), vs,
                      cos.data_ptr() if rotary_dim else None, sin.data_ptr() if rotary_dim else None,
                      cos.shape[0] if rotary_dim else 0, 1 if rotary_dim else 0, ptr(qb), ptr(kb) if k is not None else None,
                      ptr(vb) if k is not None else None, ptr(gate), rows(gate) if gate is not None else 0, ptr(sinks), float(softcap), ptr(slopes), n_kv_heads,
                      out.data_ptr(), out.stride(0), k_pool.data_ptr(), v_pool.data_ptr(), k_pool.shape[0],
                      plan.seq_total.data_ptr(), block_table.data_ptr(), block_table.shape[1], B, n_heads, tiles, head_dim,
                      scale, window, DECODE_BLOCKS, part_o.data_ptr(), part_ml.data_ptr(), slots, counters.data_ptr(),
                      counters.numel(), _library.status_word(q.device).data_ptr(), _library.current_stream())
        return out
    _library.call("dl_attention_decode_fresh_bf16", q.data_ptr(), qs, k.data_ptr(), ks, v.data_ptr(), vs,
                  cos.data_ptr() if rotary_dim else None, sin.data_ptr() if rotary_dim else None,
                  cos.shape[0] if rotary_dim else 0, 1 if rotary_dim else 0, out.data_ptr(), out.stride(0),
                  k_pool.data_ptr(), v_pool.data_ptr(), k_pool.shape[0], plan.seq_total.data_ptr(),
                  block_table.data_ptr(), block_table.shape[1], B, n_heads, n_kv_heads, head_dim, scale, window,
                  DECODE_BLOCKS, part_o.data_ptr(), part_ml.data_ptr(), slots, counters.data_ptr(), counters.numel(),
                  _library.status_word(q.device).data_ptr(), _library.current_stream())
    return out


def _prefill(q, q_stride, out, k_pool, v_pool, n_pages, block_table, n_heads, n_kv_heads, head_dim,
             scale, window, plan, keep_first=0, sinks=None, softcap=0.0, slopes=None, gate=None):
    tc = PREFILL_TC and head_dim in PREFILL_TC_HEAD_DIMS and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 \
        and (PREFILL_TC_SPECIAL or (not keep_first and sinks is None)) and (slopes is None or softcap <= 0)
    rows = PREFILL_TC_ROWS if tc else PREFILL_ROWS
    if ("prefill_tiles", rows) not in plan.scratch:
        # tiles that see the most keys first: the kernels start blocks in this order, and the short
        # ones at the end fill the multiprocessors' last gaps
        tiles = [(b, r0) for b, n in enumerate(plan.news) for r0 in range(0, n, rows)]
        tiles.sort(key=lambda t: -((plan.starts[t[0]] if plan.starts else 0) + min(plan.news[t[0]], t[1] + rows)))
        tile_seq, tile_row0 = [t[0] for t in tiles], [t[1] for t in tiles]
        host = torch.tensor(tile_seq + tile_row0, dtype=torch.int32).pin_memory()
        dev = host.to(q.device, non_blocking=True)
        # the pinned list stays with the plan: a captured step copies it again, from this memory, at every replay
        plan.scratch[("prefill_tiles", rows)] = (dev[:len(tile_seq)], dev[len(tile_seq):], len(tile_seq), host)
    tile_seq, tile_row0, n_tiles, _ = plan.scratch[("prefill_tiles", rows)]
    if tc:
        _library.call("dl_attention_prefill_tc_bf16", q.data_ptr(), q_stride, q.shape[0], out.data_ptr(), out.stride(0),
                      k_pool.data_ptr(), v_pool.data_ptr(), n_pages, tile_seq.data_ptr(), tile_row0.data_ptr(),
                      n_tiles, plan.seq_start.data_ptr(), plan.seq_new.data_ptr(), plan.cu_new.data_ptr(),
                      block_table.data_ptr(), block_table.shape[1], n_heads, n_kv_heads, head_dim, scale, window,
                      int(keep_first), None if sinks is None else sinks.data_ptr(), float(softcap),
                      None if slopes is None else slopes.data_ptr(), *_gate_args(gate), _library.status_word(q.device).data_ptr(), _library.current_stream())
        return True
    _library.call("dl_attention_prefill_bf16", q.data_ptr(), q_stride, out.data_ptr(), out.stride(0),
                  k_pool.data_ptr(), v_pool.data_ptr(), n_pages, tile_seq.data_ptr(), tile_row0.data_ptr(),
                  n_tiles, plan.seq_start.data_ptr(), plan.seq_new.data_ptr(), plan.cu_new.data_ptr(),
                  block_table.data_ptr(), block_table.shape[1], n_heads, n_kv_heads, head_dim, scale, window,
                  int(keep_first), None if sinks is None else sinks.data_ptr(), float(softcap),
                  None if slopes is None else slopes.data_ptr(), *_gate_args(gate), _library.status_word(q.device).data_ptr(), _library.current_stream())
    return True


def run(q, q_stride, out, k_pool, v_pool, n_pages, token_seq, token_pos, block_table,
        n_heads, n_kv_heads, head_dim, scale, window, plan, keep_first=0, sinks=None, softcap=0.0, split=False, slopes=None, gate=None):
    """Run a tensor-core kernel into ``out`` and return True, or return False to let the
    generic kernel take the call.  Kept first tokens and sinks are taken by the decode kernel (the kept pages join the
    step's list of pages; the sink's term enters where a head is normalised) and by both prefill kernels (the tcgen05 one
    walks the kept pages ahead of the window's, the mma.sync one lists them per tile).  ``softcap`` c > 0: scaled scores s
    become c tanh(s / c), in all three; then ``slopes`` add slope_h * (key - query), likewise (a prompt with both takes the mma.sync
    kernel); ``gate`` [T, n_heads] of q's dtype: a head's output times its sigmoid, where it is written.  ``split``: decode steps of more than 16 query heads a KV head run as several tiles of
    query heads over the same pages (otherwise they are the generic kernel's)."""
    if q.dtype != torch.bfloat16 or q_stride % 8 or q.data_ptr() % 16 or head_dim not in DECODE_HEAD_DIMS:
        return False
    special = bool(keep_first) or sinks is not None
    if special and (out.stride(0) % 2 or out.data_ptr() % 4):
        return False
    if plan.all_single and q.shape[0] == plan.n_seqs and (DECODE_SPECIAL or not special):
        tiles = decode_tiles(n_heads, n_kv_heads, split)
        if tiles == 0 or not decode_fits(n_heads // tiles, head_dim):
            return False
        return _decode(q, q_stride, out, k_pool, v_pool, n_pages, block_table, n_heads, n_kv_heads,
                       head_dim, scale, window, plan, keep_first, sinks, softcap, slopes, gate)
    if plan.news and q.shape[0] == sum(plan.news):
        return _prefill(q, q_stride, out, k_pool, v_pool, n_pages, block_table, n_heads, n_kv_heads,
                        head_dim, scale, window, plan, keep_first, sinks, softcap, slopes, gate)
    return False
