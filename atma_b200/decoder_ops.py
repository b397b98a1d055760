"""Python entry points of libatma_decoder.so: the operations of the configured decoder models.

Every function launches on the current CUDA stream, allocates only its result and never synchronises, so all of them
can be captured in a CUDA graph.  Activations, caches and weights are float32 or bfloat16; the residual stream, the
recurrent state and everything between a projection and the state are float32.
"""

import ctypes

import torch

from . import _lib


def _ptr(t):
    return None if t is None else ctypes.c_void_p(t.data_ptr())


def _check(rc):
    _lib.check(rc, _lib.load_decoder())


def _rows(t, what):
    if t.ndim != 2 or t.stride(1) != 1:
        raise ValueError(f"{what} must be a matrix with contiguous rows")
    return t


def embed_bigram(ids, prev, embed, bigram=None, mul_prev=0, mul_cur=0):
    """fp32 rows embed[id] + bigram[(prev * mul_prev + id * mul_cur) mod buckets]; prev < 0 takes the table's last row."""
    _lib.require_cuda(embed, "embed_bigram")
    n, D = ids.numel(), embed.shape[1]
    x = torch.empty((n, D), device=embed.device, dtype=torch.float32)
    buckets = 1 if bigram is None else bigram.shape[0] - 1
    _check(_lib.load_decoder().atma_embed_bigram(_ptr(ids), _ptr(prev), _ptr(embed), _ptr(bigram), _ptr(x), n, D, embed.shape[0],
                                                 int(mul_prev), int(mul_cur), buckets, _lib.dtype_code(embed), _lib.stream_ptr()))
    return x


def residual_norms(x, y, weights, eps, offset=1.0, dtype=None, in_place=True):
    """x (rows, D) fp32 becomes x + y (y in the activation dtype or None); for every weight of ``weights`` (one or two,
    None = skipped) the normalised row times (offset + weight).  Returns the list of normalised tensors."""
    _lib.require_cuda(x, "residual_norms")
    n, D = x.shape
    dtype = dtype or next(w.dtype for w in weights if w is not None)
    hs = [None if w is None else torch.empty((n, D), device=x.device, dtype=dtype) for w in weights]
    w1, w2 = (list(weights) + [None])[:2]
    h1, h2 = (hs + [None])[:2]
    x_out = x if (y is not None and in_place) else None
    _check(_lib.load_decoder().atma_residual_norms(_ptr(x), _ptr(y), _ptr(x_out), _ptr(w1), _ptr(h1), _ptr(w2), _ptr(h2), n, D,
                                                   float(eps), float(offset), _lib.DTYPE_CODE[dtype], _lib.stream_ptr()))
    return hs


def embed_position_norm(ids, positions, embed, pos, weight, eps, scale=1.0, offset=0.0):
    """Rows s = embed[id] * scale + pos[position] (pos None = no second term), divided by their root mean square, times
    (offset + weight).  Returns them in fp32 and in the tables' dtype (the same tensor for fp32)."""
    _lib.require_cuda(embed, "embed_position_norm")
    n, D = ids.numel(), embed.shape[1]
    x = torch.empty((n, D), device=embed.device, dtype=torch.float32)
    h = None if embed.dtype == torch.float32 else torch.empty((n, D), device=embed.device, dtype=embed.dtype)
    _check(_lib.load_decoder().atma_embed_position_norm(_ptr(ids), _ptr(positions), _ptr(embed), _ptr(pos), _ptr(weight), _ptr(x), _ptr(h),
                                                        n, D, embed.shape[0], 0 if pos is None else pos.shape[0], float(scale), float(eps),
                                                        float(offset), _lib.dtype_code(embed), _lib.stream_ptr()))
    return x, x if h is None else h


def residual_post_norm(x, y, weight, eps, bias=None, next_weight=None, offset=0.0, in_place=True):
    """Norm on a sublayer's output: t = y + bias; x (rows, D) fp32 becomes x + t / rms(t) * (offset + weight).  Returns
    the new x in y's dtype (x itself for fp32) or, with ``next_weight``, its own norm times (offset + next_weight); not
    ``in_place`` leaves x as it is."""
    _lib.require_cuda(x, "residual_post_norm")
    n, D = x.shape
    if y.shape != x.shape or not y.is_contiguous() or not x.is_contiguous():
        raise ValueError("x and y must be contiguous and of one shape")
    h = None
    if next_weight is not None or y.dtype != torch.float32 or not in_place:
        h = torch.empty((n, D), device=x.device, dtype=y.dtype)
    _check(_lib.load_decoder().atma_residual_post_norm(_ptr(x), _ptr(y), _ptr(bias), _ptr(weight), _ptr(x if in_place else None), _ptr(h),
                                                       _ptr(next_weight), n, D, float(eps), float(offset), _lib.dtype_code(y),
                                                       _lib.stream_ptr()))
    return x if h is None else h


def bias_squared_relu(z, bias, out):
    """out = relu(z + bias)^2 (bias None = none; rows may be strided; out may be z)."""
    _rows(z, "z"), _rows(out, "out")
    _check(_lib.load_decoder().atma_bias_squared_relu(_ptr(z), z.stride(0), _ptr(bias), _ptr(out), out.stride(0), z.shape[0], z.shape[1],
                                                      _lib.dtype_code(z), _lib.stream_ptr()))
    return out


def gelu_gate(gate, up, out):
    """out = gelu_tanh(gate) * up (rows may be strided)."""
    _rows(gate, "gate"), _rows(up, "up"), _rows(out, "out")
    _check(_lib.load_decoder().atma_gelu_gate(_ptr(gate), gate.stride(0), _ptr(up), up.stride(0), _ptr(out), out.stride(0),
                                              gate.shape[0], gate.shape[1], _lib.dtype_code(gate), _lib.stream_ptr()))
    return out


def head_norm_silu_gate(o, weight, gate, out, eps):
    """out = o / rms(o) * weight * silu(gate) per head; o (rows, H, vdim) dense, gate and out (rows, H*vdim)."""
    n, H, vdim = o.shape
    _rows(gate, "gate"), _rows(out, "out")
    _check(_lib.load_decoder().atma_head_norm_silu_gate(_ptr(o), _ptr(weight), _ptr(gate), gate.stride(0), _ptr(out), out.stride(0),
                                                        n, H, vdim, float(eps), _lib.dtype_code(o), _lib.stream_ptr()))
    return out


def rotary_store(z, positions, slot_mapping, table, k_cache, v_cache, *, heads, kv_heads, maps, dim, vdim, rot_dims):
    """Rotates q and k of the projection rows z = [q | k | v], stores k and v in the cache rows ``slot_mapping`` and
    returns q (rows, heads, maps, dim).  ``table`` (positions, rot_dims/2, 2) fp32 cos and sin."""
    _lib.require_cuda(z, "rotary_store")
    _rows(z, "z")
    n = z.shape[0]
    q = torch.empty((n, heads, maps, dim), device=z.device, dtype=z.dtype)
    _check(_lib.load_decoder().atma_rotary_store(_ptr(z), z.stride(0), _ptr(positions), _ptr(slot_mapping), _ptr(table),
                                                 0 if table is None else table.shape[0], _ptr(q), _ptr(k_cache), _ptr(v_cache), n, heads,
                                                 kv_heads, maps, dim, vdim, rot_dims, _lib.dtype_code(z), _lib.stream_ptr()))
    return q


def norm_store(z, slot_mapping, k_cache, v_cache, q_width, *, q_weight=None, k_weight=None, eps=0.0, v_first=None, lam=0.0):
    """Of the projection rows z = [q | k | v | ...]: q and k divided by their root mean square over the whole projection,
    times the weights (None = as they are); v or, with ``v_first``, (1 - lam) v + lam v_first.  k and v go to the cache
    rows ``slot_mapping``; returns q (rows, q_width)."""
    _lib.require_cuda(z, "norm_store")
    _rows(z, "z")
    n, nk, nv = z.shape[0], k_cache.shape[2] * k_cache.shape[3], v_cache.shape[2] * v_cache.shape[3]
    if q_width + nk + nv > z.shape[1] or (v_first is not None and v_first.shape != (n, nv)):
        raise ValueError("norm_store: z or v_first does not fit the cache")
    q = torch.empty((n, q_width), device=z.device, dtype=z.dtype)
    _check(_lib.load_decoder().atma_norm_store(_ptr(z), z.stride(0), _ptr(slot_mapping), _ptr(q_weight), _ptr(k_weight), _ptr(v_first),
                                               0 if v_first is None else _rows(v_first, "v_first").stride(0), float(lam), float(eps),
                                               _ptr(q), _ptr(k_cache), _ptr(v_cache), n, q_width, nk, nv, _lib.dtype_code(z),
                                               _lib.stream_ptr()))
    return q


NO_WINDOW = 2 ** 31 - 1


def _softmax_args(q, k_cache, v_cache, group, out, scale, lam=0.0, out_scale=1.0, eps=0.0, window=None, keep_first=0, sink=None, gate=None):
    n, H, maps, dim = q.shape
    _rows(out, "out")
    a = _lib.SoftmaxArgs()
    a.q, a.k_cache, a.v_cache = q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr()
    a.block_tables, a.bt_stride, a.max_blocks = group.block_tables.data_ptr(), group.block_tables.stride(0), group.block_tables.shape[1]
    a.cu_rows, a.start_pos = group.cu_rows.data_ptr(), group.start_pos.data_ptr()
    a.out, a.out_rs = out.data_ptr(), out.stride(0)
    a.n_seqs, a.max_rows, a.total_rows = group.n_seqs, group.max_rows, group.total_rows
    a.num_blocks, a.block_size, a.G, a.vdim = k_cache.shape[0], k_cache.shape[1], v_cache.shape[2], v_cache.shape[3]
    a.H, a.maps, a.dim, a.dtype = H, maps, dim, _lib.dtype_code(q)
    a.scale, a.lambda_, a.out_scale, a.eps = float(scale), float(lam), float(out_scale), float(eps)
    if gate is not None:
        a.gate, a.gate_rs = gate.data_ptr(), _rows(gate, "gate").stride(0)
    a.window, a.keep_first = NO_WINDOW if window is None else int(window), int(keep_first)
    a.sink = float("-inf") if sink is None else float(sink)
    return a


def softmax_prefill(q, k_cache, v_cache, group, out, **options):
    """Causal softmax attention of a group's rows over the paged cache; with two maps the differential combination.
    q (rows, H, maps, dim); caches (blocks, block_size, G, maps*dim | vdim); ``group``: an engine ``RowGroup``.
    Options: scale (needed); lam, out_scale, eps (two maps); window and keep_first (position i sees key j <= i if
    i - j < window or j < keep_first; None = every key); sink (score of an added key without a value, None = none);
    gate (rows, H*vdim): the result is multiplied by its sigmoid."""
    _lib.require_cuda(q, "softmax_prefill")
    a = _softmax_args(q, k_cache, v_cache, group, out, **options)
    if group.tile_seq is not None:
        a.tile_seq, a.tile_row, a.n_tiles = group.tile_seq.data_ptr(), group.tile_row.data_ptr(), group.tile_seq.numel()
    _check(_lib.load_decoder().atma_softmax_prefill(ctypes.byref(a), _lib.stream_ptr()))
    return out


def decode_key_ranges(n_seqs, heads, kv_heads, maps, max_keys):
    """Key ranges per sequence and group of query heads for ``softmax_decode`` (launch-time shapes only)."""
    from .polar import decode_num_splits
    per_cta = 8 // maps
    return decode_num_splits(n_seqs, kv_heads * -(-(heads // kv_heads) // per_cta), max_keys, min_keys=256)


def softmax_decode(q, k_cache, v_cache, group, out, *, n_splits=None, **options):
    """The same for one row per sequence."""
    _lib.require_cuda(q, "softmax_decode")
    lib = _lib.load_decoder()
    a = _softmax_args(q, k_cache, v_cache, group, out, **options)
    scratch = None
    if lib.atma_softmax_decode_path(ctypes.byref(a)):
        most = min(a.max_blocks * a.block_size, a.window + a.keep_first)
        a.n_splits = n_splits or decode_key_ranges(a.n_seqs, a.H, a.G, a.maps, most)
        scratch = torch.empty(int(lib.atma_softmax_decode_scratch_floats(a.n_seqs, a.H, a.maps, a.vdim, a.n_splits)),
                              device=q.device, dtype=torch.float32)
        a.scratch = scratch.data_ptr()
    _check(lib.atma_softmax_decode(ctypes.byref(a), _lib.stream_ptr()))
    return out


class DeltaWeights:
    """What the delta rule needs besides its projections: conv_{q,k,v} (channels, taps) in the activation dtype, A_log
    and dt_bias (heads,) fp32, norm (vdim,) in the activation dtype, sizes and constants."""

    def __init__(self, conv_q, conv_k, conv_v, A_log, dt_bias, norm, *, heads, kv_heads, dim, vdim, unit_eps, q_scale):
        self.conv = [c.contiguous() for c in (conv_q, conv_k, conv_v)]
        self.A_log, self.dt_bias, self.norm = A_log.float().contiguous(), dt_bias.float().contiguous(), norm.contiguous()
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.taps = conv_q.shape[1]
        self.unit_eps, self.q_scale = unit_eps, q_scale
        self.channels = 2 * kv_heads * dim + heads * vdim

    def args(self, z, conv_table, state_table, group):
        _rows(z, "z")
        a = _lib.DeltaArgs()
        a.z, a.z_rs = z.data_ptr(), z.stride(0)
        a.conv_q, a.conv_k, a.conv_v = (c.data_ptr() for c in self.conv)
        a.A_log, a.dt_bias = self.A_log.data_ptr(), self.dt_bias.data_ptr()
        a.conv_table, a.conv_ss = conv_table.data_ptr(), conv_table.stride(0)
        a.state_table, a.state_ss = state_table.data_ptr(), state_table.stride(0)
        a.slots, a.cu_rows, a.start_pos = group.slots.data_ptr(), group.cu_rows.data_ptr(), group.start_pos.data_ptr()
        a.row_seq = None if group.row_seq is None else group.row_seq.data_ptr()
        a.n_seqs, a.total_rows = group.n_seqs, group.total_rows
        a.H, a.G, a.dim, a.vdim, a.taps, a.dtype = self.heads, self.kv_heads, self.dim, self.vdim, self.taps, _lib.dtype_code(z)
        a.unit_eps, a.q_scale = self.unit_eps, self.q_scale
        return a


class DeltaParts:
    """The two halves of ``delta_prefill`` on buffers of their own: ``prepare`` (convolutions, unit-norm factors, gates,
    convolution state) and ``scan`` (the recurrence; its result is ``o`` (rows, heads, vdim))."""

    def __init__(self, z, weights, conv_table, state_table, group):
        _lib.require_cuda(z, "delta_prefill")
        w, n, dev = weights, z.shape[0], z.device
        self.lib, self.keep = _lib.load_decoder(), (z, weights, conv_table, state_table, group)
        self.args = w.args(z, conv_table, state_table, group)
        self.q = torch.empty((n, w.kv_heads, w.dim), device=dev, dtype=z.dtype)
        self.k = torch.empty_like(self.q)
        self.v = torch.empty((n, w.heads, w.vdim), device=dev, dtype=z.dtype)
        self.inv = torch.empty((2, n, w.kv_heads), device=dev, dtype=torch.float32)
        self.gates = torch.empty((2, n, w.heads), device=dev, dtype=torch.float32)
        self.o = torch.empty_like(self.v)
        nbytes = int(self.lib.atma_delta_scan_scratch_bytes(ctypes.byref(self.args)))
        self.scratch = torch.empty(nbytes, device=dev, dtype=torch.uint8) if nbytes > 0 else None

    def _factors(self):
        return _ptr(self.inv[0]), _ptr(self.inv[1]), _ptr(self.gates[0]), _ptr(self.gates[1])

    def prepare(self):
        _check(self.lib.atma_delta_prepare(ctypes.byref(self.args), _ptr(self.q), _ptr(self.k), _ptr(self.v), *self._factors(), _lib.stream_ptr()))

    def scan(self):
        _check(self.lib.atma_delta_scan(ctypes.byref(self.args), _ptr(self.q), _ptr(self.k), _ptr(self.v), *self._factors(), _ptr(self.o),
                                        _ptr(self.scratch), _lib.stream_ptr()))


def delta_prefill(z, weights, conv_table, state_table, group, out, eps):
    """The delta mixer between its input and output projections for a group's rows: z rows [q | k | v | gate | a | b],
    conv_table (slots, taps, channels), state_table (slots, heads, dim, vdim) fp32, both updated in place; out
    (rows, heads*vdim)."""
    parts = DeltaParts(z, weights, conv_table, state_table, group)
    parts.prepare()
    parts.scan()
    g0 = weights.channels
    return head_norm_silu_gate(parts.o, weights.norm, z[:, g0:g0 + weights.heads * weights.vdim], out, eps)


def delta_step(z, weights, conv_table, state_table, group, out, eps):
    """The same for one row per sequence, in one launch."""
    _lib.require_cuda(z, "delta_step")
    _rows(out, "out")
    a = weights.args(z, conv_table, state_table, group)
    _check(_lib.load_decoder().atma_delta_step(ctypes.byref(a), _ptr(weights.norm), _ptr(out), out.stride(0), float(eps),
                                               _lib.stream_ptr()))
    return out


def linear(x, weight, out=None):
    """x @ weight.T in the activation dtype: the weight-streaming kernel for up to 16 16-bit rows, cuBLAS otherwise."""
    from .inference_ops import decode_linear, decode_linear_supported
    if decode_linear_supported(x, weight):
        return decode_linear(x, weight, out=out, lib=_lib.load_decoder())
    if out is None:
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out=out)


def squared_relu_linear(x, weight, bias=None):
    """relu(x @ weight.T + bias)^2."""
    from .inference_ops import decode_linear, decode_linear_supported
    if decode_linear_supported(x, weight):
        return decode_linear(x, weight, bias=bias, gated="plain_squared_relu", lib=_lib.load_decoder())
    z = torch.mm(x, weight.t())
    return bias_squared_relu(z, bias, z)


def gelu_gated_linear(x, weight, out):
    """out = gelu_tanh(x @ gate.T) * (x @ up.T) with weight = [gate; up]."""
    from .inference_ops import decode_linear, decode_linear_supported
    if decode_linear_supported(x, weight, gated=True):
        return decode_linear(x, weight, gated="gelu_tanh", out=out, lib=_lib.load_decoder())
    gu = torch.mm(x, weight.t())
    half = weight.shape[0] // 2
    return gelu_gate(gu[:, :half], gu[:, half:], out)


def linear_f32_out(x, weight):
    """x @ weight.T with an fp32 result (the LM head)."""
    if x.dtype == torch.float32:
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out_dtype=torch.float32)


def device_status():
    """Like ``atma_b200.device_status`` for this library's tensor-core kernels."""
    status = ctypes.c_int(-1)
    _check(_lib.load_decoder().atma_decoder_device_status(ctypes.byref(status)))
    return status.value
