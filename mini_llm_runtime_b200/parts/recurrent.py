"""Mixers that carry a matrix-valued state per head instead of a key/value cache.

Both keep, per request and head, a state S [dim, vdim] of 32-bit floats that starts at zero and is
advanced token by token; what enters the recurrence beside the projections (decays, gates, norms)
is 32-bit.  Projections leave as 32-bit rows so that nothing is rounded on the way into the
recurrence; the mixer's output projection leaves 32-bit rows for a 32-bit residual stream.

``wkv``    time mixing with a data-dependent per-channel decay and a bonus for the current token:
           every projection reads its own blend of the input with the previous token's input
           (coefficients ``mu.*``); w_t = exp(-exp(W2 tanh(W1 x_w) + w0));
           o_t = (S + diag(u) k_t v_t^T)^T r_t;  S <- diag(w_t) S + k_t v_t^T;
           out = Wo (o / rms(o) * norm * silu(Wg x_g)).
``state_space``  a selective state-space layer with a scalar decay per head (Mamba-2, "state-space
           duality"), see ``StateSpaceMixer``.
``matrix_memory``  a memory written with exponential gates and read through a normaliser, see
           ``MatrixMemoryMixer``.
``gated_delta_rule``  a delta rule with a scalar decay and step size per head, see ``DeltaRuleMixer``.
``hgrn2``  gated linear attention whose forget gate also sets what is written:
           f_t = l + (1 - l) sigmoid(Wf x + b);  S <- diag(f_t) S + (1 - f_t) v_t^T;
           o_t = S^T silu(Wq x);  out = Wo (o / rms(o) * norm).
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import Mixer, StateNeed, TensorSpec, build_part, register_part


def _float(tensor, device):
    return tensor.to(device=device, dtype=torch.float32).contiguous()


class WKVMixer(Mixer):
    graph_safe = True
    wants_float_input = True       # its own blends are taken of 32-bit rows

    BLENDS = ("r", "k", "v", "g", "w")

    def __init__(self, spec, compute_dtype):
        super().__init__(spec, compute_dtype)
        a = self.args
        self.hidden_size = int(a["hidden_size"])
        self.heads = int(a["heads"])
        self.dim = int(a["dim"])
        self.eps = float(a["eps"])
        self.inner = self.heads * self.dim
        # the decay's bottleneck width is whatever the checkpoint's w1/w2 have; random weights use this
        self.default_rank = int(a.get("decay_rank") or max(16, self.hidden_size // 16))
        # the blends with the previous token's input: a token shift with five coefficient vectors
        self.blend = build_part("shift", PartSpec("token_shift", {
            "hidden_size": self.hidden_size, "state": "previous_input",
            "tensors": tuple(self.prefix + "mu." + name for name in self.BLENDS)}), compute_dtype)
        self.w = {}
        self.decay_bias = self.bonus = self.norm = None

    def cache_need(self):
        return (StateNeed((self.heads, self.dim, self.dim), torch.float32, "state"), self.blend.state_need())

    def tensors(self):
        p, h, n = self.prefix, self.hidden_size, self.inner
        out = {p + name: TensorSpec((n, h)) for name in ("r", "k", "v", "g")}
        out[p + "o"] = TensorSpec((h, n))
        out[p + "w0"] = TensorSpec((n,), init="bias")
        out[p + "u"] = TensorSpec((self.heads, self.dim), init="bias")
        out[p + "norm"] = TensorSpec((n,), init="norm")
        out[p + "w1"] = TensorSpec((self.default_rank, h), flexible=(0,))
        out[p + "w2"] = TensorSpec((n, self.default_rank), flexible=(1,))
        out.update(self.blend.tensors())
        return out

    def load(self, tensors, device):
        p = self.prefix
        if tensors[p + "w1"].shape[0] != tensors[p + "w2"].shape[1]:
            raise ValueError(f"{p}w1 and {p}w2 disagree on the decay's bottleneck width")
        for name in ("r", "k", "v", "g", "o", "w1", "w2"):
            self.w[name] = self._to_compute(tensors[p + name], device)
        self.decay_bias = _float(tensors[p + "w0"], device)
        self.bonus = _float(tensors[p + "u"], device).reshape(-1)
        self.norm = _float(tensors[p + "norm"], device)
        self.blend.load(tensors, device)

    def forward(self, x, ctx, view, writes_cache):
        k = ops.current()
        xr, xk, xv, xg, xw = self.blend.forward(x, ctx, view)
        f32 = torch.float32
        r = k.linear(xr, self.w["r"], out_dtype=f32)
        key = k.linear(xk, self.w["k"], out_dtype=f32)
        value = k.linear(xv, self.w["v"], out_dtype=f32)
        gate = k.linear(xg, self.w["g"], out_dtype=f32)
        decay = k.linear(k.tanh_(k.linear(xw, self.w["w1"])), self.w["w2"], out_dtype=f32)
        mixed = k.bonus_recurrence(r, key, value, decay, gate, self.decay_bias, self.bonus, self.norm, self.eps,
                                   view.states["state"], ctx, self.heads, self.dim, self.compute_dtype)
        return k.linear(mixed, self.w["o"], out_dtype=f32)


class HGRN2Mixer(Mixer):
    graph_safe = True

    def __init__(self, spec, compute_dtype):
        super().__init__(spec, compute_dtype)
        a = self.args
        self.hidden_size = int(a["hidden_size"])
        self.heads = int(a["heads"])
        self.dim = int(a["dim"])
        self.vdim = int(a["vdim"])
        self.eps = float(a["eps"])
        self.w_qfv = self.w_o = self.forget_bias = self.lower = self.norm = None

    def cache_need(self):
        return StateNeed((self.heads, self.dim, self.vdim), torch.float32, "state")

    def tensors(self):
        p, h, n = self.prefix, self.hidden_size, self.heads * self.dim
        return {p + "q": TensorSpec((n, h)), p + "f": TensorSpec((n, h)), p + "f.b": TensorSpec((n,), init="bias"),
                p + "lower": TensorSpec((n,), init="unit"), p + "v": TensorSpec((self.heads * self.vdim, h)),
                p + "norm": TensorSpec((self.vdim,), init="norm"), p + "o": TensorSpec((h, self.heads * self.vdim))}

    def load(self, tensors, device):
        p = self.prefix
        # one product yields [q | f | v]
        self.w_qfv = self._to_compute(torch.cat([tensors[p + "q"], tensors[p + "f"], tensors[p + "v"]], dim=0), device)
        self.w_o = self._to_compute(tensors[p + "o"], device)
        self.forget_bias = _float(tensors[p + "f.b"], device)
        self.lower = _float(tensors[p + "lower"], device)
        self.norm = _float(tensors[p + "norm"], device)

    def forward(self, x, ctx, view, writes_cache):
        k = ops.current()
        n = self.heads * self.dim
        qfv = k.linear(x, self.w_qfv, out_dtype=torch.float32)
        mixed = k.forget_gate_recurrence(qfv[:, :n], qfv[:, n:2 * n], qfv[:, 2 * n:], self.forget_bias, self.lower,
                                         self.norm, self.eps, view.states["state"], ctx, self.heads, self.dim,
                                         self.vdim, self.compute_dtype)
        return k.linear(mixed, self.w_o, out_dtype=torch.float32)


class StateSpaceMixer(Mixer):
    """Selective state-space layer with a scalar decay per head.

    With inner = heads * vdim, N = ``state`` and G = ``groups``, one product W_in x yields
    [z: inner | x: inner | B: G N | C: G N | dt: heads].  x, B and C together pass a causal convolution
    per channel (``conv`` [channels, taps], last column the current token's, bias ``conv.b``, zeros before
    the request's start) and silu.  dt <- softplus(dt + dt_bias).  Per head h, reading group
    h // (heads / G):  S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T  (S: N x vdim),
    y_t = S_t^T C_t + D_h x_t.  Then y * silu(z), an RMS norm in ``norm_groups`` equal parts (each by its
    own root mean square) times ``norm``, and W_o.

    Per request the layer carries S (32-bit, kept transposed: [heads, vdim, N]) and the convolution's
    last taps - 1 inputs.  Everything between the in-projection and W_o is 32-bit."""

    graph_safe = True

    def __init__(self, spec, compute_dtype):
        super().__init__(spec, compute_dtype)
        a = self.args
        self.hidden_size = int(a["hidden_size"])
        self.heads = int(a["heads"])
        self.vdim = int(a["vdim"])
        self.n = int(a["state"])
        self.groups = int(a.get("groups", 1))
        self.taps = int(a["conv"])
        self.norm_groups = int(a.get("norm_groups", 1))
        self.eps = float(a["eps"])
        self.inner = self.heads * self.vdim
        self.channels = self.inner + 2 * self.groups * self.n
        if self.heads % self.groups or self.inner % self.norm_groups or self.taps < 2:
            raise ValueError("heads must divide into the groups, the inner width into the norm's parts, and the "
                             "convolution needs at least two taps")
        self.w_in = self.w_o = self.conv = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.norm = None

    def cache_need(self):
        return (StateNeed((self.heads, self.vdim, self.n), torch.float32, "state"),
                StateNeed((self.taps - 1, self.channels), torch.float32, "conv"))

    def tensors(self):
        p, h = self.prefix, self.hidden_size
        return {p + "in": TensorSpec((2 * self.inner + 2 * self.groups * self.n + self.heads, h)),
                p + "conv": TensorSpec((self.channels, self.taps), init="bias"),
                p + "conv.b": TensorSpec((self.channels,), init="bias"),
                p + "dt_bias": TensorSpec((self.heads,), init="bias"),
                p + "A_log": TensorSpec((self.heads,), init="bias"),
                p + "D": TensorSpec((self.heads,), init="norm"),
                p + "norm": TensorSpec((self.inner,), init="norm"),
                p + "o": TensorSpec((h, self.inner))}

    def load(self, tensors, device):
        p = self.prefix
        self.w_in = self._to_compute(tensors[p + "in"], device)
        self.w_o = self._to_compute(tensors[p + "o"], device)
        self.conv = _float(tensors[p + "conv"], device)
        self.conv_bias = _float(tensors[p + "conv.b"], device)
        self.dt_bias = _float(tensors[p + "dt_bias"], device)
        self.a_log = _float(tensors[p + "A_log"], device)
        self.skip = _float(tensors[p + "D"], device)
        self.norm = _float(tensors[p + "norm"], device)

    def forward(self, x, ctx, view, writes_cache):
        k = ops.current()
        inner, gn = self.inner, self.groups * self.n
        projected = k.linear(x, self.w_in, out_dtype=torch.float32)
        mixed = k.causal_conv(projected[:, inner:inner + self.channels], self.conv, self.conv_bias, view.states["conv"],
                              ctx, "silu")
        y = k.state_space_scan(mixed[:, :inner], mixed[:, inner:inner + gn], mixed[:, inner + gn:],
                               projected[:, inner + self.channels:], self.dt_bias, self.a_log, self.skip,
                               view.states["state"], ctx, self.heads, self.vdim, self.n, self.groups)
        gated = k.gated_group_norm(y, projected[:, :inner], self.norm, self.eps, self.norm_groups, self.compute_dtype)
        return k.linear(gated, self.w_o, out_dtype=torch.float32)


class DeltaRuleMixer(Mixer):
    """Gated delta rule: a recurrence that writes, per head and token, the difference between the value and
    what the state already answers to the key.

    q = Wq x and k = Wk x [kv_heads * dim], v = Wv x [heads * vdim] each pass a causal convolution per channel
    (``<name>.conv`` [channels, taps], last column the current token's, zeros before the request's start) and
    silu; head h reads the q and k of head h // (heads / kv_heads).  k and q are divided by sqrt(sum of squares
    + ``unit_eps``), q also multiplied by dim^-0.5.  Per head g = exp(-exp(A_log) softplus(Wa x + dt_bias)),
    beta = sigmoid(Wb x) and, on a state S [dim, vdim],
    S_t = g_t S_{t-1} + k_t u_t^T with u_t = beta_t (v_t - g_t S_{t-1}^T k_t), and o_t = S_t^T q_t.
    Every head's o is divided by its root mean square over vdim, times ``norm`` [vdim] (shared by the heads),
    times silu(Wg x); then Wo.

    Per request the layer carries S (32-bit, kept transposed: [heads, vdim, dim]) and the convolution's last
    taps - 1 inputs.  Everything between the projections and Wo is 32-bit."""

    graph_safe = True

    def __init__(self, spec, compute_dtype):
        super().__init__(spec, compute_dtype)
        a = self.args
        self.hidden_size = int(a["hidden_size"])
        self.heads = int(a["heads"])
        self.kv_heads = int(a.get("kv_heads", self.heads))
        self.dim = int(a["dim"])
        self.vdim = int(a["vdim"])
        self.taps = int(a["conv"])
        self.eps = float(a["eps"])
        self.unit_eps = float(a["unit_eps"])
        if self.heads % self.kv_heads or self.taps < 1:
            raise ValueError("heads must be divisible by kv_heads, and the convolution needs at least one tap")
        self.qk, self.inner = self.kv_heads * self.dim, self.heads * self.vdim
        self.channels = 2 * self.qk + self.inner
        self.w_in = self.w_o = self.conv = self.dt_bias = self.a_log = self.norm = None

    def cache_need(self):
        return (StateNeed((self.heads, self.vdim, self.dim), torch.float32, "state"),
                StateNeed((self.taps - 1, self.channels), torch.float32, "conv"))

    def tensors(self):
        p, h = self.prefix, self.hidden_size
        sizes = {"q": self.qk, "k": self.qk, "v": self.inner}
        out = {p + name: TensorSpec((rows, h)) for name, rows in sizes.items()}
        out.update({p + name + ".conv": TensorSpec((rows, self.taps), init="bias") for name, rows in sizes.items()})
        out.update({p + "g": TensorSpec((self.inner, h)), p + "a": TensorSpec((self.heads, h)),
                    p + "b": TensorSpec((self.heads, h)), p + "A_log": TensorSpec((self.heads,), init="bias"),
                    p + "dt_bias": TensorSpec((self.heads,), init="bias"),
                    p + "norm": TensorSpec((self.vdim,), init="norm"), p + "o": TensorSpec((h, self.inner))})
        return out

    def load(self, tensors, device):
        p = self.prefix
        # one product yields [q | k | v | g | a | b], filled up with zeros so that its rows start at 16-byte boundaries
        rows = [tensors[p + name] for name in ("q", "k", "v", "g", "a", "b")]
        fill = -(2 * self.inner + 2 * self.qk + 2 * self.heads) % 8
        if fill:
            rows.append(torch.zeros((fill, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = self._to_compute(torch.cat(rows, dim=0), device)
        self.w_o = self._to_compute(tensors[p + "o"], device)
        self.conv = _float(torch.cat([tensors[p + name + ".conv"] for name in "qkv"], dim=0), device)
        self.dt_bias = _float(tensors[p + "dt_bias"], device)
        self.a_log = _float(tensors[p + "A_log"], device)
        self.norm = _float(tensors[p + "norm"], device)

    def forward(self, x, ctx, view, writes_cache):
        k = ops.current()
        qk, channels, inner = self.qk, self.channels, self.inner
        projected = k.linear(x, self.w_in, out_dtype=torch.float32)
        mixed = k.causal_conv(projected[:, :channels], self.conv, None, view.states["conv"], ctx, "silu")
        at = channels + inner
        y = k.delta_rule_scan(mixed[:, :qk], mixed[:, qk:2 * qk], mixed[:, 2 * qk:], projected[:, at:at + self.heads],
                              projected[:, at + self.heads:at + 2 * self.heads], self.dt_bias, self.a_log,
                              view.states["state"], ctx, self.heads, self.kv_heads, self.dim, self.vdim, self.unit_eps)
        gated = k.gated_head_norm(y, projected[:, channels:at], self.norm, self.eps, self.heads, self.compute_dtype)
        return k.linear(gated, self.w_o, out_dtype=torch.float32)


class MatrixMemoryMixer(Mixer):
    """Matrix memory with exponential gates (the mLSTM of xLSTM).

    q = Wq x * dim^-0.5 and k = Wk x [heads * dim], v = Wv x [heads * vdim].  Per head and token a logarithm of the
    input gate i = cap tanh((Wi x + bi) / cap) and one of the forget gate f = logsigmoid(cap tanh((Wf x + bf) /
    cap)), cap = ``gate_cap``.  The memory S [dim, vdim] and its normaliser n [dim] are kept relative to the
    exponential of a running maximum m, so that no gate overflows:  m_t = max(f + m_{t-1}, i),  S_t = e^(f + m_{t-1} -
    m_t) S_{t-1} + e^(i - m_t) k v^T,  n_t likewise with k alone,  o = S_t^T q / (max(|n_t . q|, e^(-m_t)) +
    ``guard``).  Every head's o is divided by its root mean square, the heads together are multiplied by ``norm``
    [heads * vdim] and by sigmoid(Wg x); then Wo.

    Per request the layer carries, in 32-bit, S with n behind it (kept transposed, n as one more value channel:
    [heads, vdim + 1, dim]) and m; all start at zero.  Everything between the projections and Wo is 32-bit."""

    graph_safe = True
    NAMES = ("q", "k", "v", "g", "i", "f")

    def __init__(self, spec, compute_dtype):
        super().__init__(spec, compute_dtype)
        a = self.args
        self.hidden_size = int(a["hidden_size"])
        self.heads = int(a["heads"])
        self.dim = int(a["dim"])
        self.vdim = int(a["vdim"])
        self.eps = float(a["eps"])
        self.gate_cap = float(a["gate_cap"])
        self.guard = float(a.get("guard", 1e-6))
        self.qk, self.inner = self.heads * self.dim, self.heads * self.vdim
        self.w_in = self.w_o = self.input_bias = self.forget_bias = self.norm = None

    def cache_need(self):
        return (StateNeed((self.heads, self.vdim + 1, self.dim), torch.float32, "state"),
                StateNeed((self.heads,), torch.float32, "maximum"))

    def _sizes(self):
        return dict(zip(self.NAMES, (self.qk, self.qk, self.inner, self.inner, self.heads, self.heads)))

    def tensors(self):
        p, h = self.prefix, self.hidden_size
        out = {p + name: TensorSpec((rows, h)) for name, rows in self._sizes().items()}
        out.update({p + "i.b": TensorSpec((self.heads,), init="bias"), p + "f.b": TensorSpec((self.heads,), init="bias"),
                    p + "norm": TensorSpec((self.inner,), init="norm"), p + "o": TensorSpec((h, self.inner))})
        return out

    def load(self, tensors, device):
        p = self.prefix
        # one product yields [q | k | v | g | i | f], filled up with zeros so that its rows start at 16-byte boundaries
        rows = [tensors[p + name] for name in self.NAMES]
        fill = -sum(part.shape[0] for part in rows) % 8
        if fill:
            rows.append(torch.zeros((fill, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = self._to_compute(torch.cat(rows, dim=0), device)
        self.w_o = self._to_compute(tensors[p + "o"], device)
        self.input_bias = _float(tensors[p + "i.b"], device)
        self.forget_bias = _float(tensors[p + "f.b"], device)
        self.norm = _float(tensors[p + "norm"], device)

    def forward(self, x, ctx, view, writes_cache):
        k = ops.current()
        projected = k.linear(x, self.w_in, out_dtype=torch.float32)
        parts, at = {}, 0
        for name, width in self._sizes().items():
            parts[name] = projected[:, at:at + width]
            at += width
        mixed = k.matrix_memory(parts["q"], parts["k"], parts["v"], parts["i"], parts["f"], self.input_bias,
                                self.forget_bias, self.gate_cap, self.guard, parts["g"], self.norm, self.eps,
                                view.states["state"], view.states["maximum"], ctx, self.heads, self.dim, self.vdim,
                                self.compute_dtype)
        return k.linear(mixed, self.w_o, out_dtype=torch.float32)


register_part("mixer", "wkv", WKVMixer)
register_part("mixer", "matrix_memory", MatrixMemoryMixer)
register_part("mixer", "gated_delta_rule", DeltaRuleMixer)
register_part("mixer", "state_space", StateSpaceMixer)
register_part("mixer", "hgrn2", HGRN2Mixer)
