"""CPU oracle for the Suvapel decoder -- TEST INFRASTRUCTURE ONLY (plain, slow, one function per mechanism).

Suvapel is a decoder-only model whose layer list comes from config.json.  A layer reads ONE Dynamic-Tanh norm of the stream; its
mixer and its feed-forward both start from it and are added back together, then a token's own embedding for that layer joins:

  h = dyt(x);   x <- x + m (mixer(h) + ff(h));   x <- x + m rms(P (gelu_tanh(G x) * e[token, layer])) w_side

Notation (weights W are [out, in], applied as W x; m = residual_mult):
  dyt(x)        = tanh(alpha x) * w + b
  rms(y)        = y / sqrt(mean(y^2) + eps);   unit(y) = y / sqrt(sum(y^2) + 1e-6)
  conv(u)       : per channel, y_t = sum_j w[j] u_(t - taps + 1 + j), zeros before the sequence
  delta rule    : per head  S <- decay * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
                  q = unit(silu(conv(W_q h))) / sqrt(dim), k = unit(silu(conv(W_k h))), v = silu(conv(W_v h)), beta = sigmoid(W_b h)
  mixer delta   : decay = exp(-exp(A_h) softplus(W_a h + t_h)) per head;  W_o (rms(o) w_norm * silu(W_g h))
  mixer parallel: left_scale * left + right_scale * right
    left        : q, k, v = conv of the projections; rotation of the first `dims` dimensions of q and k (halves paired, YaRN
                  frequencies); softmax over the keys j <= i with i - j < size or j < keep_first; head h times sigmoid(W_g h)_h; W_o
    right       : delta rule with a decay per head and key channel, exp(-exp(A_h) softplus(W_a2 W_a1 h + t));
                  W_o (rms(o) w_norm * sigmoid(W_g2 W_g1 h))
  feed-forward  : W_down (silu(W_gate h + b) * (W_up h + b)) + b
  head          : W_head dyt(x)

Everything runs in the dtype of the weights handed in (float64 in the tests), whole prompts or token by token; `State` makes the
two forms comparable.
"""
from __future__ import annotations

import math

import numpy as np
import torch


# ---------------------------------------------------------------------------------------------- mechanisms
def dyt(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def rms(y, eps):
    return y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)


def unit(y):
    return y / torch.sqrt(y.pow(2).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.nn.functional.softplus(z, threshold=1e9)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(u, w, before):
    """u [S, C] the new inputs, before [taps - 1, C] the inputs ahead of them (zeros at a sequence's start), w [C, taps] with the
    last column on the current token -> (conv [S, C], the last taps - 1 inputs)."""
    taps = w.shape[1]
    full = torch.cat([before, u], 0)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            out[t] = out[t] + w[:, j] * full[t + j]
    return out, full[full.shape[0] - (taps - 1):].clone()


def rotation(rot):
    """-> (radians per position of every pair, factor on cosines and sines)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):          # the (real-valued) pair index that turns `turns` times over the original context
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [S, heads, d]: dimension i turns together with dimension i + dims / 2."""
    f, mag = rotation(rot)
    half = rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        a = pos.to(x.dtype) * f[i]
        c, s = (torch.cos(a) * mag)[:, None], (torch.sin(a) * mag)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def visible(p, mask):
    """Positions a row at position p sees: all earlier ones and itself, or with a mask its window and the first keep_first tokens."""
    j = torch.arange(p + 1)
    if not mask:
        return j
    return j[(p - j < mask["size"]) | (j < mask.get("keep_first", 0))]


def attend(q, k, v, q_pos, scale, mask):
    """Softmax attention of rows q [S, H, d] at positions q_pos over the keys k [n, G, d] / values v [n, G, dv]."""
    S, H, _ = q.shape
    G, dv = v.shape[1], v.shape[2]
    group = torch.arange(H) // (H // G)          # key / value head of every query head
    out = torch.zeros(S, H, dv, dtype=q.dtype)
    for i in range(S):
        js = visible(int(q_pos[i]), mask)
        p = torch.softmax((k[js][:, group] * q[i]).sum(-1) * scale, 0)          # [keys, H]
        out[i] = (p[:, :, None] * v[js][:, group]).sum(0)
    return out


def delta_rule(q, k, v, beta, decay, S0):
    """One head.  q, k, decay [S, d]; v [S, dv]; beta [S]; S0 [d, dv] -> (o [S, dv], S_end)."""
    S = S0.clone()
    o = torch.zeros(v.shape, dtype=v.dtype)
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def feed_forward(h, p, pre):
    a = silu(h @ p[pre + "gate"].T + p[pre + "gate.b"]) * (h @ p[pre + "up"].T + p[pre + "up.b"])
    return a @ p[pre + "down"].T + p[pre + "down.b"]


# ---------------------------------------------------------------------------------------------- the model
class State:
    """What a sequence carries: per layer the keys and values (attention), the windows of the convolutions and the delta rule's
    memory per head."""

    def __init__(self, config):
        n = len(config["layers"])
        self.k = [None] * n
        self.v = [None] * n
        self.win = [dict() for _ in range(n)]
        self.mem = [None] * n
        self.len = 0


def _grow(old, new):
    return new if old is None else torch.cat([old, new], 0)


def _conv_projection(h, p, name, windows):
    u, w = h @ p[name].T, p[name + ".conv"]
    before = windows.get(name)
    if before is None:
        before = torch.zeros(w.shape[1] - 1, w.shape[0], dtype=h.dtype)
    y, windows[name] = causal_conv(u, w, before)
    return y


def window_attention(h, pos, p, pre, mc, state, li):
    H, G, d, dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    S = h.shape[0]
    q = _conv_projection(h, p, pre + "q", state.win[li]).reshape(S, H, d)
    k = _conv_projection(h, p, pre + "k", state.win[li]).reshape(S, G, d)
    v = _conv_projection(h, p, pre + "v", state.win[li]).reshape(S, G, dv)
    q, k = rotate(q, pos, mc["rot"]), rotate(k, pos, mc["rot"])
    state.k[li], state.v[li] = _grow(state.k[li], k), _grow(state.v[li], v)
    o = attend(q, state.k[li], state.v[li], pos, mc["scale"], mc.get("mask"))
    o = o * torch.sigmoid(h @ p[pre + "g"].T)[:, :, None]
    return o.reshape(S, H * dv) @ p[pre + "o"].T


def delta_mixer(h, p, pre, mc, eps, state, li, per_channel):
    H, Hk, d, dv = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    S = h.shape[0]
    q = unit(silu(_conv_projection(h, p, pre + "q", state.win[li])).reshape(S, Hk, d)) * d ** -0.5
    k = unit(silu(_conv_projection(h, p, pre + "k", state.win[li])).reshape(S, Hk, d))
    v = silu(_conv_projection(h, p, pre + "v", state.win[li])).reshape(S, H, dv)
    beta = torch.sigmoid(h @ p[pre + "b"].T)
    rate = torch.exp(p[pre + "A_log"])
    if per_channel:
        z = ((h @ p[pre + "a1"].T) @ p[pre + "a2"].T + p[pre + "dt_bias"]).reshape(S, H, d)
        decay = torch.exp(-rate[None, :, None] * softplus(z))
        gate = torch.sigmoid((h @ p[pre + "g1"].T) @ p[pre + "g2"].T)
    else:
        z = h @ p[pre + "a"].T + p[pre + "dt_bias"]
        decay = torch.exp(-rate[None, :] * softplus(z))[:, :, None].expand(S, H, d)
        gate = silu(h @ p[pre + "g"].T)
    if state.mem[li] is None:
        state.mem[li] = [torch.zeros(d, dv, dtype=h.dtype) for _ in range(H)]
    o = torch.zeros(S, H, dv, dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // Hk)
        o[:, hh], state.mem[li][hh] = delta_rule(q[:, g], k[:, g], v[:, hh], beta[:, hh], decay[:, hh], state.mem[li][hh])
    o = rms(o, eps) * p[pre + "norm"]
    return (o.reshape(S, H * dv) * gate) @ p[pre + "o"].T


def token_side(x, ids, p, pre, part, eps):
    """part: this layer's columns of the side embedding."""
    g = gelu_tanh(x @ p[pre + "side.gate"].T) * p["side.embed"][ids][:, part]
    return rms(g @ p[pre + "side.proj"].T, eps) * p[pre + "side.norm"]


def forward(config, p, tokens, state=None, trace=None):
    """tokens: the next tokens of one sequence -> logits [S, vocab].  `p`: name -> tensor.  `trace`, a list, receives the
    stream after every layer."""
    state = state or State(config)
    eps, m, sd = config["norm"]["eps"], config["residual_mult"], config["token_side"]["dim"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    pos = torch.arange(state.len, state.len + ids.numel())
    x = p["embed"][ids]
    for li, lc in enumerate(config["layers"]):
        pre, mc = f"l{li}.", lc["mixer"]
        h = dyt(x, p[pre + "norm1.alpha"], p[pre + "norm1"], p[pre + "norm1.b"])
        if lc["type"] == "parallel":
            y = mc["left_scale"] * window_attention(h, pos, p, pre + "mix.left.", mc["left"], state, li) \
                + mc["right_scale"] * delta_mixer(h, p, pre + "mix.right.", mc["right"], eps, state, li, True)
        elif lc["type"] == "delta":
            y = delta_mixer(h, p, pre + "mix.", mc, eps, state, li, False)
        else:
            raise ValueError(lc["type"])
        if lc.get("mlp"):
            y = y + feed_forward(h, p, pre + "mlp.")
        x = x + m * y
        x = x + m * token_side(x, ids, p, pre, slice(li * sd, (li + 1) * sd), eps)
        if trace is not None:
            trace.append(x.clone())
    state.len += ids.numel()
    return dyt(x, p["final.norm.alpha"], p["final.norm"], p["final.norm.b"]) @ p["head"].T


# ---------------------------------------------------------------------------------------------- random models for tests
def tensor_shapes(config):
    """`a_rank` / `g_rank` of a right mixer (default 12) are read here only: the engine takes the ranks from the tensors."""
    W, V, sd = config["width"], config["vocab"], config["token_side"]["dim"]
    out = {"embed": (V, W), "side.embed": (V, sd * len(config["layers"])), "final.norm": (W,), "final.norm.b": (W,), "final.norm.alpha": (), "head": (V, W)}

    def delta(pre, m, per_channel):
        H, Hk, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        out.update({pre + "q": (Hk * d, W), pre + "q.conv": (Hk * d, taps), pre + "k": (Hk * d, W), pre + "k.conv": (Hk * d, taps),
                    pre + "v": (H * dv, W), pre + "v.conv": (H * dv, taps), pre + "b": (H, W), pre + "A_log": (H,), pre + "norm": (dv,), pre + "o": (W, H * dv)})
        if per_channel:
            ra, rg = m.get("a_rank", 12), m.get("g_rank", 12)
            out.update({pre + "a1": (ra, W), pre + "a2": (H * d, ra), pre + "dt_bias": (H * d,), pre + "g1": (rg, W), pre + "g2": (H * dv, rg)})
        else:
            out.update({pre + "a": (H, W), pre + "dt_bias": (H,), pre + "g": (H * dv, W)})

    for i, lc in enumerate(config["layers"]):
        m, pre = lc["mixer"], f"l{i}."
        out.update({pre + "norm1": (W,), pre + "norm1.b": (W,), pre + "norm1.alpha": ()})
        if lc["type"] == "parallel":
            a = m["left"]
            H, G, d, dv, taps = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"]
            L = pre + "mix.left."
            out.update({L + "q": (H * d, W), L + "k": (G * d, W), L + "v": (G * dv, W), L + "q.conv": (H * d, taps), L + "k.conv": (G * d, taps),
                        L + "v.conv": (G * dv, taps), L + "g": (H, W), L + "o": (W, H * dv)})
            delta(pre + "mix.right.", m["right"], True)
        else:
            delta(pre + "mix.", m, False)
        if lc.get("mlp"):
            F = lc["mlp"]["ff"]
            M = pre + "mlp."
            out.update({M + "gate": (F, W), M + "gate.b": (F,), M + "up": (F, W), M + "up.b": (F,), M + "down": (W, F), M + "down.b": (W,)})
        out.update({pre + "side.gate": (sd, W), pre + "side.proj": (W, sd), pre + "side.norm": (W,)})
    return out


def random_weights(config, seed=0):
    """bf16-representable float64 tensors: projections ~ 1/sqrt(in), norms around one, decays spread over a few orders."""
    g = torch.Generator().manual_seed(seed)
    p = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        if name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g)
        elif last == "alpha":
            t = 0.5 + torch.rand(shape, generator=g) * 0.5
        elif last in ("norm1", "norm"):
            t = 1.0 + torch.randn(shape, generator=g) * 0.1
        elif last == "conv":
            t = torch.randn(shape, generator=g) * 0.4
            t[:, -1] += 0.7
        elif last == "A_log":
            t = torch.log(torch.rand(shape, generator=g) * 3.0 + 0.05)
        elif last == "dt_bias":
            t = torch.log(torch.expm1(torch.rand(shape, generator=g) * 0.2 + 0.005))
        elif last == "b" and len(shape) == 1:
            t = torch.randn(shape, generator=g) * 0.3
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        p[name] = t.to(torch.bfloat16).to(torch.float64)
    return p


def to_numpy_bf16_bits(t):
    return t.to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16)
