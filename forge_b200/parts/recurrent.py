"""Mixers that carry a matrix of state per head from token to token instead of a cache of keys and values.

Both have N heads of K channels, keep S [K, K] per head and request in 32-bit (a row of the layer's state tensor per
request slot, zero at admission), make their decay from a low-rank projection, x = W2 tanh(W1 .) + w0, divide every head's
output by its root mean square, multiply by a weight per channel and by a gate, and project back to the model's width.

"wkv" (decay and bonus, with a look at the previous token):
    each of r, k, v, g, w reads h + (h_prev - h) * mu_s;  w_t = exp(-exp(x_t));  gate = silu(g)
    o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T          (the previous token's h is state too)
"general_delta" (generalized delta rule):
    w_t = exp(-exp(-1/2) sigmoid(x_t));  a_t = sigmoid(Wa h + b);  n_t = k_t / sqrt(|k_t|^2 + 1e-6);  gate = sigmoid(g)
    S <- diag(w_t) S - (a_t * n_t)(n_t^T S) + k_t v_t^T;   o_t = S^T r_t

The rank of the decay's projection is read from the file's tensors (``rank`` is only what random weights take).

"gated_write" (HGRN2; N heads of K key and V value channels, state [K, V], no key and no low-rank decay):
    q_t = silu(Wq h);  f_t = l + (1 - l) sigmoid(Wf h + b)  (l: a lower bound per channel);  v_t = Wv h
    S <- diag(f_t) S + (1 - f_t) v_t^T;   o_t = S^T q_t;   every head's o divided by its root mean square, times a weight per
    value channel that the heads share; projected back.  ``out_scale`` multiplies the mixer's output.

"retention" (N heads of K key and V value channels, state [K, V], one fixed decay g_n per head, no softmax, no denominator):
    q_t, k_t rotated by the position (a position part with ``inv_freq``; channel i paired with i + half), k_t times K^-1/2
    S <- g_n S + k_t v_t^T;   o_t = S^T q_t;   every head's o divided by its root mean square (no weight), times silu(Wg h);
    projected back.

"gated_linear" (gated linear attention; N heads of K key and V value channels, state [K, V], no softmax, no denominator):
    a_t = sigmoid(Wa2 (Wa1 h) + b)^(1/tau)  (a decay per key channel; the hidden layer's size is read from the file)
    S <- diag(a_t) S + k_t v_t^T;   o_t = K^-1/2 S^T q_t;   every head's o divided by its root mean square, times a weight per value
    channel that the heads share, times silu(Wg h); projected back.

"gated_delta" (gated delta rule; N heads of K key and V value channels, state [K, V]; groups of heads share one q and k):
    q, k, v each pass a short causal convolution over time (a filter per channel) and silu; q and k become unit vectors per head, q times K^-1/2
    g_t = exp(-exp(A) softplus(Wa h + dt)),  beta_t = sigmoid(Wb h)  (one of each per head)
    S <- g_t S;   S <- S + k_t (beta_t (v_t - S^T k_t))^T;   o_t = S^T q_t;   every head's o divided by its root mean square, times a weight
    per value channel that the heads share, times silu(Wg h); projected back.  The convolutions' last inputs are state too.

"lightning" (linear attention with one fixed decay per head; N heads of K key and V value channels, state [K, V]):
    q, k, v = silu(Wq h), silu(Wk h), silu(Wv h);   S <- g_n S + k_t v_t^T;   o_t = S^T q_t;   all of a token's heads together divided by their
    root mean square, times a weight per channel, times sigmoid(Wg h); projected back.
"""
import torch

from .. import kernels
from ..config.base import ConfigError
from ..weights.loader import TensorSpec
from .base import Part, StateSpec, register_part
from .linear import Linear


class _StateMixer(Part):
    graph_safe = True       # request boundaries and state rows come from the batch's device tensors (q_start, slots)
    MATRICES = ()

    def __init__(self, rt, hidden_size, num_heads, head_dim, eps, rank=16, names=None, prefix="mix."):
        if head_dim > 128:
            raise ConfigError(f"state mixers take heads of up to 128 channels, not {head_dim}")
        self.rt, self.hidden_size, self.num_heads, self.head_dim = rt, hidden_size, num_heads, head_dim
        self.eps, self.rank, self.prefix = float(eps), int(rank), prefix
        self.names = dict(names or {})

    def _n(self, short):
        return self.names.get(short, self.prefix + short)

    def _common_specs(self):
        W, NK = self.hidden_size, self.num_heads * self.head_dim
        specs = {self._n(m): TensorSpec((NK, W)) for m in self.MATRICES}
        specs.update({self._n("w1"): TensorSpec((-1, W), default_shape=(self.rank, W)),
                      self._n("w2"): TensorSpec((NK, -1), default_shape=(NK, self.rank)),
                      self._n("w0"): TensorSpec((NK,), role="bias"), self._n("norm"): TensorSpec((NK,), role="norm"),
                      self._n("o"): TensorSpec((W, NK))})
        return specs

    def _bind_common(self, tensors):
        w1, w2 = tensors[self._n("w1")], tensors[self._n("w2")]
        if w1.shape[0] != w2.shape[1]:
            from ..weights.loader import WeightError
            raise WeightError(self._n("w1"), wrong=[f"{self._n('w1')} has {w1.shape[0]} rows, {self._n('w2')} {w2.shape[1]} columns"])
        self.w2 = Linear(self._matrix(w2), None, self.rt)
        self.w0 = self._vector_f32(tensors[self._n("w0")])
        self.norm = self._vector_f32(tensors[self._n("norm")])
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)
        return w1

    def _decay_input(self, hidden):
        """hidden: (fp32 matrix, first column) of W1's product; returns fp32 [T, N*K], W2 tanh(.) (w0 is added where
        the decay is made)."""
        return self.w2.forward(kernels.tanh_rows(hidden, self.rt.dtype, n=self.w2.in_features))


class WKVMixer(_StateMixer):
    MATRICES = ("r", "k", "v", "g")
    SHIFTED = ("r", "k", "v", "g", "w")

    def tensor_specs(self):
        specs = self._common_specs()
        specs.update({self._n("mu." + s): TensorSpec((self.hidden_size,), role="fraction") for s in self.SHIFTED})
        specs[self._n("u")] = TensorSpec((self.num_heads, self.head_dim), role="bias")
        return specs

    def bind(self, tensors):
        self.w1 = Linear(self._matrix(self._bind_common(tensors)), None, self.rt)
        self.lin = {m: Linear(self._matrix(tensors[self._n(m)]), None, self.rt) for m in self.MATRICES}
        self.mu = torch.stack([self._vector_f32(tensors[self._n("mu." + s)]) for s in self.SHIFTED]).contiguous()
        self.bonus = self._vector_f32(tensors[self._n("u")]).reshape(-1).contiguous()

    def cache_spec(self):
        n = self.num_heads * self.head_dim * self.head_dim
        return StateSpec((n + self.hidden_size,), torch.float32)      # the heads' matrices, then the previous token's input

    def forward(self, x, batch, cache, residual):
        N, K = self.num_heads, self.head_dim
        prev_off = N * K * K
        shifted = kernels.token_shift(x, cache.state, prev_off, batch, self.mu)            # [5, T, W]
        r, k, v, g = (self.lin[m].forward(shifted[i]) for i, m in enumerate(self.MATRICES))
        decay_in = self._decay_input((self.w1.forward(shifted[4]), 0))
        o = kernels.state_scan("decay_bonus", (r, 0), (k, 0), (v, 0), (decay_in, 0), self.w0, cache.state, batch, N, K,
                               bonus=self.bonus, last_in=x, prev_off=prev_off)
        y = kernels.head_finish(o, self.norm, (g, 0), N, K, self.eps, "silu", self.rt.dtype)
        self.o.forward(y, accumulate_into=residual)


class GeneralDeltaMixer(_StateMixer):
    MATRICES = ("r", "k", "v", "g", "a")

    def tensor_specs(self):
        specs = self._common_specs()
        specs[self._n("a.b")] = TensorSpec((self.num_heads * self.head_dim,), role="bias")
        return specs

    def bind(self, tensors):
        w1 = self._bind_common(tensors)
        # r, k, v, g, a and the decay's first matrix read the same input: one product
        self.proj = Linear(self._matrix(torch.cat([tensors[self._n(m)] for m in self.MATRICES] + [w1], dim=0)), None, self.rt)
        self.a0 = self._vector_f32(tensors[self._n("a.b")])

    def cache_spec(self):
        return StateSpec((self.num_heads * self.head_dim * self.head_dim,), torch.float32)

    def forward(self, x, batch, cache, residual):
        N, K = self.num_heads, self.head_dim
        NK = N * K
        p = self.proj.forward(x)                                     # fp32 [T, 5*N*K + rank]: r | k | v | g | a | hidden
        decay_in = self._decay_input((p, 5 * NK))
        o = kernels.state_scan("delta", (p, 0), (p, NK), (p, 2 * NK), (decay_in, 0), self.w0, cache.state, batch, N, K,
                               y=(p, 4 * NK), a0=self.a0)
        y = kernels.head_finish(o, self.norm, (p, 3 * NK), N, K, self.eps, "sigmoid", self.rt.dtype)
        self.o.forward(y, accumulate_into=residual)


class GatedWriteMixer(Part):
    graph_safe = True       # request boundaries and state rows come from the batch's device tensors (q_start, slots)

    def __init__(self, rt, hidden_size, num_heads, head_dim, eps, v_head_dim=None, out_scale=1.0, prefix="mix."):
        if head_dim > 256:
            raise ConfigError(f"the gated-write mixer takes heads of up to 256 key channels, not {head_dim}")
        self.rt, self.hidden_size, self.num_heads, self.head_dim = rt, hidden_size, num_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.eps, self.out_scale, self.prefix = float(eps), float(out_scale), prefix

    def _n(self, short):
        return self.prefix + short

    def tensor_specs(self):
        W, NK, NV = self.hidden_size, self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return {self._n("q"): TensorSpec((NK, W)), self._n("f"): TensorSpec((NK, W)), self._n("f.b"): TensorSpec((NK,), role="bias"),
                self._n("lower"): TensorSpec((NK,), role="fraction"), self._n("v"): TensorSpec((NV, W)),
                self._n("norm"): TensorSpec((self.v_head_dim,), role="norm"), self._n("o"): TensorSpec((W, NV))}

    def bind(self, tensors):
        # q, f and v read the same input: one product
        self.proj = Linear(self._matrix(torch.cat([tensors[self._n(m)] for m in ("q", "f", "v")], dim=0)), None, self.rt)
        self.f_bias = self._vector_f32(tensors[self._n("f.b")])
        self.lower = self._vector_f32(tensors[self._n("lower")])
        self.norm = self._vector_f32(tensors[self._n("norm")])
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)

    def cache_spec(self):
        return StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def in_width(self):
        return self.num_heads * (2 * self.head_dim + self.v_head_dim)

    def out_width(self):
        return self.num_heads * self.v_head_dim

    def mix(self, p, col, batch, cache, out=None):
        """p fp32 [T, >= col + in_width]: [q | f | v] from column ``col`` (q and f are overwritten); returns the normed heads
        [T, N*V] (or writes them into ``out`` = (matrix, first column))."""
        N, K, V = self.num_heads, self.head_dim, self.v_head_dim
        NK = N * K
        o = kernels.state_scan("gated_write", (p, col), None, (p, col + 2 * NK), (p, col + NK), self.f_bias, cache.state, batch, N, K,
                               a0=self.lower, KV=V)
        return kernels.head_finish(o, self.norm, None, N, V, self.eps, "none", self.rt.dtype, scale=self.out_scale, out=out)

    def forward(self, x, batch, cache, residual):
        y = self.mix(self.proj.forward(x), 0, batch, cache)          # the projection: fp32 [T, 2*N*K + N*V]
        self.o.forward(y, accumulate_into=residual)


class RetentionMixer(Part):
    graph_safe = True       # positions, request boundaries and state rows come from the batch's device tensors

    def __init__(self, rt, hidden_size, num_heads, head_dim, decay, eps, position, v_head_dim=None, prefix="mix."):
        from .base import build_part
        if head_dim > 256:
            raise ConfigError(f"the retention mixer takes heads of up to 256 key channels, not {head_dim}")
        if len(decay) != num_heads:
            raise ConfigError(f"retention: {len(decay)} decays for {num_heads} heads")
        self.rt, self.hidden_size, self.num_heads, self.head_dim = rt, hidden_size, num_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.eps, self.prefix = float(eps), prefix
        self.decay = torch.tensor([float(g) for g in decay], dtype=torch.float64).to(torch.float32).to(rt.device)
        self.position = build_part("position", position, rt)
        if not hasattr(self.position, "inv_freq"):
            raise ConfigError("retention rotates inside its own scan and needs a position part with 'inv_freq'")
        self.ones = torch.ones(self.v_head_dim, dtype=torch.float32, device=rt.device)       # the head norm has no weight

    def sub_parts(self):
        return [self.position]

    def _n(self, short):
        return self.prefix + short

    def tensor_specs(self):
        W, NK, NV = self.hidden_size, self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return {self._n("q"): TensorSpec((NK, W)), self._n("k"): TensorSpec((NK, W)), self._n("v"): TensorSpec((NV, W)),
                self._n("g"): TensorSpec((NV, W)), self._n("o"): TensorSpec((W, NV))}

    def bind(self, tensors):
        # q, k, v and the gate read the same input: one product
        self.proj = Linear(self._matrix(torch.cat([tensors[self._n(m)] for m in ("q", "k", "v", "g")], dim=0)), None, self.rt)
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)

    def cache_spec(self):
        return StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def forward(self, x, batch, cache, residual):
        """Adds the mixer's output into ``residual``, or (``residual`` None) returns it as a new fp32 [T, W]."""
        N, K, V = self.num_heads, self.head_dim, self.v_head_dim
        NK, NV = N * K, N * V
        p = self.proj.forward(x)                                     # fp32 [T, 2*N*K + 2*N*V]: q | k | v | g
        freq = self.position.inv_freq
        o = kernels.retention_scan((p, 0), (p, NK), (p, 2 * NK), batch, freq if freq.numel() else None, K ** -0.5, self.decay,
                                   cache.state, N, K, V)
        y = kernels.head_finish(o, self.ones, (p, 2 * NK + NV), N, V, self.eps, "silu", self.rt.dtype)
        return self.o.forward(y, accumulate_into=residual)


class GatedLinearMixer(Part):
    graph_safe = True       # request boundaries and state rows come from the batch's device tensors (q_start, slots)

    def __init__(self, rt, hidden_size, num_heads, head_dim, tau, eps, v_head_dim=None, rank=16, prefix="mix."):
        if head_dim > 256:
            raise ConfigError(f"the gated linear mixer takes heads of up to 256 key channels, not {head_dim}")
        if not tau > 0.0:
            raise ConfigError(f"the gated linear mixer's decays are a sigmoid to the power 1/tau with a positive tau, not {tau}")
        self.rt, self.hidden_size, self.num_heads, self.head_dim = rt, hidden_size, num_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.tau, self.eps, self.rank, self.prefix = float(tau), float(eps), int(rank), prefix

    def _n(self, short):
        return self.prefix + short

    def tensor_specs(self):
        W, NK, NV = self.hidden_size, self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return {self._n("q"): TensorSpec((NK, W)), self._n("k"): TensorSpec((NK, W)), self._n("v"): TensorSpec((NV, W)),
                self._n("g"): TensorSpec((NV, W)), self._n("a1"): TensorSpec((-1, W), default_shape=(self.rank, W)),
                self._n("a2"): TensorSpec((NK, -1), default_shape=(NK, self.rank)), self._n("a2.b"): TensorSpec((NK,), role="bias"),
                self._n("norm"): TensorSpec((self.v_head_dim,), role="norm"), self._n("o"): TensorSpec((W, NV))}

    def bind(self, tensors):
        a1, a2 = tensors[self._n("a1")], tensors[self._n("a2")]
        if a1.shape[0] != a2.shape[1]:
            from ..weights.loader import WeightError
            raise WeightError(self._n("a1"), wrong=[f"{self._n('a1')} has {a1.shape[0]} rows, {self._n('a2')} {a2.shape[1]} columns"])
        self.rank = int(a1.shape[0])
        # q, k, v, the gate and the decay's hidden layer read the same input: one product
        self.proj = Linear(self._matrix(torch.cat([tensors[self._n(m)] for m in ("q", "k", "v", "g")] + [a1], dim=0)), None, self.rt)
        self.a2t = self._vector_f32(a2.t())                          # fp32 [rank, N*K]
        self.a_bias = self._vector_f32(tensors[self._n("a2.b")])
        self.norm = self._vector_f32(tensors[self._n("norm")])
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)

    def cache_spec(self):
        return StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), torch.float32)

    def in_width(self):
        return 2 * self.num_heads * (self.head_dim + self.v_head_dim) + self.rank

    def out_width(self):
        return self.num_heads * self.v_head_dim

    def mix(self, p, col, batch, cache, out=None):
        """p fp32 [T, >= col + in_width]: [q | k | v | g | hidden] from column ``col``; returns the gated heads [T, N*V] (or writes them
        into ``out`` = (matrix, first column))."""
        N, K, V = self.num_heads, self.head_dim, self.v_head_dim
        NK, NV = N * K, N * V
        q, k, v, g, hidden = (p, col), (p, col + NK), (p, col + 2 * NK), (p, col + 2 * NK + NV), (p, col + 2 * NK + 2 * NV)
        if kernels.gla_token_supports(batch, N, K, V, self.rank):        # a step of single tokens: one kernel
            return kernels.gla_token(q, k, v, g, hidden, self.rank, self.a2t, self.a_bias, self.tau, batch, cache.state, N, K, V, self.norm,
                                     self.eps, self.rt.dtype, out=out)
        o = kernels.gla_scan(q, k, v, hidden, self.rank, self.a2t, self.a_bias, self.tau, batch, cache.state, N, K, V)
        return kernels.head_finish(o, self.norm, g, N, V, self.eps, "silu", self.rt.dtype, out=out)

    def forward(self, x, batch, cache, residual):
        """Adds the mixer's output into ``residual``, or (``residual`` None) returns it as a new fp32 [T, W]."""
        return self.o.forward(self.mix(self.proj.forward(x), 0, batch, cache), accumulate_into=residual)


class GatedDeltaMixer(Part):
    graph_safe = True       # positions, request boundaries and state rows come from the batch's device tensors
    ROW_MULTIPLE = 8        # the projection's rows are filled up to a multiple of this: aligned rows of its result

    def __init__(self, rt, hidden_size, num_heads, head_dim, taps, eps, num_qk_heads=None, v_head_dim=None, prefix="mix."):
        """``num_qk_heads``: heads of q and k, each shared by num_heads / num_qk_heads neighbouring heads; ``taps``: tokens that the
        convolutions look at (the current one and taps - 1 before it)."""
        num_qk_heads = num_heads if num_qk_heads is None else num_qk_heads
        if head_dim > 256:
            raise ConfigError(f"the gated delta mixer takes heads of up to 256 key channels, not {head_dim}")
        if num_qk_heads < 1 or num_heads % num_qk_heads:
            raise ConfigError(f"gated delta rule: {num_heads} heads cannot share {num_qk_heads} query/key heads")
        if taps < 1:
            raise ConfigError(f"gated delta rule: a convolution over {taps} tokens")
        self.rt, self.hidden_size, self.num_heads, self.num_qk_heads, self.head_dim = rt, hidden_size, num_heads, num_qk_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.taps, self.eps, self.prefix = int(taps), float(eps), prefix

    def _n(self, short):
        return self.prefix + short

    def _conv_channels(self):
        return 2 * self.num_qk_heads * self.head_dim + self.num_heads * self.v_head_dim

    def tensor_specs(self):
        W, N, QK, NV = self.hidden_size, self.num_heads, self.num_qk_heads * self.head_dim, self.num_heads * self.v_head_dim
        specs = {}
        for m, rows in (("q", QK), ("k", QK), ("v", NV)):
            specs.update({self._n(m): TensorSpec((rows, W)), self._n(m + ".conv"): TensorSpec((rows, self.taps), role="filter")})
        specs.update({self._n("b"): TensorSpec((N, W)), self._n("A_log"): TensorSpec((N,), role="bias"),
                      self._n("norm"): TensorSpec((self.v_head_dim,), role="norm"), self._n("a"): TensorSpec((N, W)),
                      self._n("dt_bias"): TensorSpec((N,), role="bias"), self._n("g"): TensorSpec((NV, W)), self._n("o"): TensorSpec((W, NV))})
        return specs

    def bind(self, tensors):
        # everything that reads h is one product: q, k, v, the gate, the write strengths and the decays (and rows of zeros at the end)
        rows = torch.cat([tensors[self._n(m)] for m in ("q", "k", "v", "g", "b", "a")], dim=0)
        pad = -rows.shape[0] % self.ROW_MULTIPLE
        self.proj = Linear(self._matrix(torch.cat([rows, rows.new_zeros(pad, rows.shape[1])], dim=0)), None, self.rt)
        # [taps, channels], the current token's weights first: neighbouring threads read neighbouring channels
        self.conv = self._vector_f32(torch.cat([tensors[self._n(m + ".conv")] for m in "qkv"], dim=0).flip(1).t())
        self.decay_rate = self._vector_f32(torch.exp(tensors[self._n("A_log")].to(torch.float64)))
        self.dt = self._vector_f32(tensors[self._n("dt_bias")])
        self.norm = self._vector_f32(tensors[self._n("norm")])
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)

    def cache_spec(self):
        n = self.num_heads * self.head_dim * self.v_head_dim + self.taps * self._conv_channels()
        return StateSpec((n + -n % 4,), torch.float32)              # the heads' matrices, then the ring of the convolutions' last inputs

    def in_width(self):
        n = self._conv_channels() + self.num_heads * (self.v_head_dim + 2)
        return n + -n % self.ROW_MULTIPLE

    def out_width(self):
        return self.num_heads * self.v_head_dim

    def mix(self, p, col, batch, cache, out=None):
        """p fp32 [T, >= col + in_width]: [q | k | v | g | b | a] from column ``col``; returns the gated heads [T, N*V] (or writes them into
        ``out`` = (matrix, first column))."""
        N, M, K, V = self.num_heads, self.num_qk_heads, self.head_dim, self.v_head_dim
        g_col = col + self._conv_channels()
        b_col, a_col = g_col + N * V, g_col + N * V + N
        if kernels.token_state_supports(batch, K, V, True):            # a step of single tokens: one kernel
            return kernels.gated_delta_token(p, col, g_col, b_col, a_col, self.conv, self.decay_rate, self.dt, batch, cache.state, N, M, K, V,
                                             self.norm, self.eps, self.rt.dtype, out=out)
        qkv, g, beta = kernels.gated_delta_prepare(p, col, b_col, a_col, self.conv, self.decay_rate, self.dt, batch, cache.state, N, M, K, V)
        o = kernels.gated_delta_scan(qkv, g, beta, batch, cache.state, N, M, K, V)
        return kernels.head_finish(o, self.norm, (p, g_col), N, V, self.eps, "silu", self.rt.dtype, out=out)

    def forward(self, x, batch, cache, residual):
        """Adds the mixer's output into ``residual``, or (``residual`` None) returns it as a new fp32 [T, W]."""
        return self.o.forward(self.mix(self.proj.forward(x), 0, batch, cache), accumulate_into=residual)


class LightningMixer(Part):
    graph_safe = True       # request boundaries and state rows come from the batch's device tensors (q_start, slots)

    def __init__(self, rt, hidden_size, num_heads, head_dim, decay, eps, v_head_dim=None, prefix="mix."):
        """``decay``: one number per head."""
        if head_dim > 256:
            raise ConfigError(f"the lightning mixer takes heads of up to 256 key channels, not {head_dim}")
        if len(decay) != num_heads:
            raise ConfigError(f"lightning attention: {len(decay)} decays for {num_heads} heads")
        self.rt, self.hidden_size, self.num_heads, self.head_dim = rt, hidden_size, num_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.eps, self.prefix = float(eps), prefix
        self.decay = torch.tensor([float(g) for g in decay], dtype=torch.float64).to(torch.float32).to(rt.device)

    def _n(self, short):
        return self.prefix + short

    def tensor_specs(self):
        W, NK, NV = self.hidden_size, self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return {self._n("q"): TensorSpec((NK, W)), self._n("k"): TensorSpec((NK, W)), self._n("v"): TensorSpec((NV, W)),
                self._n("g"): TensorSpec((NV, W)), self._n("o"): TensorSpec((W, NV)), self._n("norm"): TensorSpec((NV,), role="norm")}

    def bind(self, tensors):
        # q, k, v and the gate read the same input: one product
        self.proj = Linear(self._matrix(torch.cat([tensors[self._n(m)] for m in ("q", "k", "v", "g")], dim=0)), None, self.rt)
        self.norm = self._vector_f32(tensors[self._n("norm")])
        self.o = Linear(self._matrix(tensors[self._n("o")]), None, self.rt)

    def cache_spec(self):
        n = self.num_heads * self.head_dim * self.v_head_dim
        return StateSpec((n + -n % 4,), torch.float32)

    def in_width(self):
        return 2 * self.num_heads * (self.head_dim + self.v_head_dim)

    def out_width(self):
        return self.num_heads * self.v_head_dim

    def mix(self, p, col, batch, cache, out=None):
        """p fp32 [T, >= col + in_width]: [q | k | v | g] from column ``col`` (portions: q, k, v are overwritten); returns the normed and
        gated heads [T, N*V] (or writes them into ``out`` = (matrix, first column))."""
        N, K, V = self.num_heads, self.head_dim, self.v_head_dim
        scan = kernels.lightning_token if kernels.token_state_supports(batch, K, V, False) else kernels.lightning_scan
        o = scan(p, col, self.decay, batch, cache.state, N, K, V)
        return kernels.gated_rows(o, self.norm, (p, col + N * (2 * K + V)), self.eps, self.rt.dtype, out=out)

    def forward(self, x, batch, cache, residual):
        """Adds the mixer's output into ``residual``, or (``residual`` None) returns it as a new fp32 [T, W]."""
        return self.o.forward(self.mix(self.proj.forward(x), 0, batch, cache), accumulate_into=residual)


register_part("mixer", "gated_delta", GatedDeltaMixer, replace=True)
register_part("mixer", "lightning", LightningMixer, replace=True)
register_part("mixer", "gated_linear", GatedLinearMixer, replace=True)
register_part("mixer", "retention", RetentionMixer, replace=True)
register_part("mixer", "gated_write", GatedWriteMixer, replace=True)
register_part("mixer", "wkv", WKVMixer, replace=True)
register_part("mixer", "general_delta", GeneralDeltaMixer, replace=True)
