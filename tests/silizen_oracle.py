"""Silizen in float64, one plain function per mechanism, written from the equations; it shares no code with the package.

Notation: T tokens, W width.  unit(x) = x / sqrt(mean(x^2) + eps) over the last axis; ln(x) = g (x - mean) / sqrt(mean((x -
mean)^2) + eps) + b.  Everything runs token after token with explicit states.

  embedding     x = E[token];  x0 denotes this x
  runs          the layer list with the slice [start, stop) repeated `times` times in a row, every repetition with caches and
                states of its own; ahead of every repetition x <- W_in [x | x0]
  layer         h = ln(x);  x <- x + mixer(h) + ff(h)
  parallel      s_l left(h) + s_r right(h)
    left        q, k, v = projections; every q and k head: g * unit(.), then rotary (pairs i, i + n/2) on its first n = rot.dims;
                s = cap(scale q_h . k_c(h)), cap(z) = c tanh(z / c);  p_j = e^s_j / (1 + sum e^s);  o_h = sum_j p_j v_j;
                W_o concat(o_h sigmoid(W_g h)_h)
    right       q = W_q h / sqrt(d), k, v;  f = sigmoid(W_a2 W_a1 h + b)^(1/tau) per head and channel;
                S <- diag(f) S + k v^T;  o = S^T q;  W_o (concat(g * unit(o)) * silu(W_g h))
  parallel_2    (g_l * unit(left(h)) + g_r * unit(right(h))) / 2
    left        q, k, v = projections with biases; every q and k head: unit(.);  s = scale q_h . k_c(h) - 2^(-8 (h + 1) / H) (i - j);
                visible 0 <= i - j < size;  p, o and gates as in parallel
    right       q, k, v = silu(causal convolution(projection));  q <- q / sqrt(sum q^2 + 1e-6) / sqrt(d), k <- k / sqrt(sum k^2 + 1e-6);
                b = sigmoid(W_b h);  f = exp(-e^A_h softplus(W_a2 W_a1 h + dt)) per head and channel;
                S <- diag(f) S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q;
                W_o (concat(g * unit(o)) * sigmoid(W_g2 W_g1 h))
  wkv           y_s = h + (h_prev - h) mu_s for s in r, k, v, g, w;  r, k, v = projections of theirs;
                f = exp(-exp(W_w2 tanh(W_w1 y_w) + w0));  o = S^T r + (sum r u k) v;  S <- diag(f) S + k v^T;
                W_o (concat(unit(o)) * g * silu(W_g y_g))
  ff            W_down (gelu(W_gate h) * W_up h), gelu(z) = z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
  output        logits = scale E ln(x)
"""
import math

import torch

F64 = torch.float64


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return w * c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) + b


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def scaled_frequencies(base, dims, scaling):
    """f_i = base^(-2 i / dims); with scaling, by wavelength: long ones divided by factor, short ones kept, a blend between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            ratio = scaling["original"] / (2 * math.pi / f)              # original context over wavelength
            if ratio < scaling["low"]:
                f = f / scaling["factor"]
            elif ratio <= scaling["high"]:
                s = (ratio - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_half_pairs(x, positions, freqs):
    """x [T, heads, size]: dimension i < n / 2 turns with i + n / 2 by position * freqs[i] (n = 2 len(freqs)); the rest passes."""
    n = 2 * len(freqs)
    a = positions.to(F64)[:, None] * freqs[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def sink_attention_rows(q, k, v, scale, softcap=0.0, window=0, slopes=None, first=0):
    """q [T, H, d] and k [S, G, d] as they meet, v [S, G, dv]; query row t sits at position first + t.  The softmax's
    denominator has one more term exp(0)."""
    T, H, _ = q.shape
    S, G, dv = v.shape
    i, j = first + torch.arange(T)[:, None], torch.arange(S)[None, :]
    seen = (j <= i) & (i - j < window) if window else j <= i
    out = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if slopes is not None:
            s = s - slopes[h] * (i - j)
        s = torch.where(seen, s, torch.tensor(-math.inf, dtype=F64))
        m = s.amax(-1, keepdim=True).clamp(min=0.0)
        e = torch.exp(s - m)
        out[:, h] = (e / (torch.exp(-m) + e.sum(-1, keepdim=True))) @ v[:, g]
    return out


def distance_slopes(H):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=F64)


def head_gated(o, gate):
    """o [T, H, dv], gate [T, H]."""
    return (o * sigmoid(gate)[:, :, None]).reshape(o.shape[0], -1)


def full_attention_branch(t, p, m, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    fr = scaled_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    pos = torch.arange(T)
    q = rotate_half_pairs(t[p + "q.norm"] * unit((h @ t[p + "q"].T).reshape(T, H, d), eps), pos, fr)
    k = rotate_half_pairs(t[p + "k.norm"] * unit((h @ t[p + "k"].T).reshape(T, G, d), eps), pos, fr)
    o = sink_attention_rows(q, k, (h @ t[p + "v"].T).reshape(T, G, dv), m["scale"], softcap=m["softcap"])
    return head_gated(o, h @ t[p + "g"].T) @ t[p + "o"].T


def window_attention_branch(t, p, m, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[p + n].T + t[p + n + ".b"] for n in "qkv")
    o = sink_attention_rows(unit(q.reshape(T, H, d), eps), unit(k.reshape(T, G, d), eps), v.reshape(T, G, dv), m["scale"],
                            window=m["mask"]["size"], slopes=distance_slopes(H))
    return head_gated(o, h @ t[p + "g"].T) @ t[p + "o"].T


def gated_rows(q, k, v, f, S=None):
    """q, k, f [T, H, d], v [T, H, dv]:  S <- diag(f) S + k v^T,  o = S^T q.  Returns (o [T, H, dv], S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        S = f[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = (q[i][:, None, :] @ S)[:, 0]
    return out, S


def root_sigmoid(z, tau):
    return torch.exp(-softplus(-z) / tau)


def gla_branch(t, p, m, h, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[p + "q"].T).reshape(T, H, d) * d ** -0.5, (h @ t[p + "k"].T).reshape(T, H, d), (h @ t[p + "v"].T).reshape(T, H, dv)
    f = root_sigmoid(h @ t[p + "a1"].T @ t[p + "a2"].T + t[p + "a2.b"], m["tau"]).reshape(T, H, d)
    o, _ = gated_rows(q, k, v, f)
    return ((t[p + "norm"] * unit(o, eps)).reshape(T, H * dv) * silu(h @ t[p + "g"].T)) @ t[p + "o"].T


def causal_conv_rows(x, w):
    """x [T, C], w [C, taps]: tap j meets the input taps - 1 - j tokens back, nothing ahead of the first token."""
    T, taps = x.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F64), x], 0)
    return sum(w[:, j] * pad[j:j + T] for j in range(taps))


def length_one(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rows(q, k, v, f, beta, S=None):
    """q, k, f [T, H, d], v [T, H, dv], beta [T, H]:  S <- diag(f) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T, H, d = f.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        S = f[i][:, :, None] * S
        u = beta[i][:, None] * (v[i] - (k[i][:, None, :] @ S)[:, 0])
        S = S + k[i][:, :, None] * u[:, None, :]
        out[i] = (q[i][:, None, :] @ S)[:, 0]
    return out, S


def delta_decay(z, A_log):
    """z [T, H, d] (bias included), A_log [H]."""
    return torch.exp(-torch.exp(A_log)[None, :, None] * softplus(z))


def delta_branch(t, p, m, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv_rows(h @ t[p + n].T, t[p + n + ".conv"])) for n in "qkv")
    rep = H // G
    q = (length_one(q.reshape(T, G, d)) * d ** -0.5).repeat_interleave(rep, 1)
    k = length_one(k.reshape(T, G, d)).repeat_interleave(rep, 1)
    f = delta_decay((h @ t[p + "a1"].T @ t[p + "a2"].T + t[p + "dt_bias"]).reshape(T, H, d), t[p + "A_log"])
    o, _ = delta_rows(q, k, v.reshape(T, H, dv), f, sigmoid(h @ t[p + "b"].T))
    return ((t[p + "norm"] * unit(o, eps)).reshape(T, H * dv) * sigmoid(h @ t[p + "g1"].T @ t[p + "g2"].T)) @ t[p + "o"].T


def wkv_rows(r, k, v, f, u, S=None):
    """r, k, f [T, H, d], v [T, H, dv], u [H, d]:  o = S^T r + (r . u k) v;  S <- diag(f) S + k v^T."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        out[i] = (r[i][:, None, :] @ S)[:, 0] + (r[i] * u * k[i]).sum(-1, keepdim=True) * v[i]
        S = f[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
    return out, S


def token_shift(h, mu, before=None):
    prev = torch.cat([torch.zeros(1, h.shape[1], dtype=F64) if before is None else before[None], h[:-1]], 0)
    return h + (prev - h) * mu


def wkv_mixer(t, p, m, h, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    y = {s: token_shift(h, t[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((y[s] @ t[p + s].T).reshape(T, H, d) for s in "rkv")
    f = torch.exp(-torch.exp(torch.tanh(y["w"] @ t[p + "w1"].T) @ t[p + "w2"].T + t[p + "w0"])).reshape(T, H, d)
    o, _ = wkv_rows(r, k, v, f, t[p + "u"])
    return (unit(o, eps).reshape(T, H * d) * t[p + "norm"] * silu(y["g"] @ t[p + "g"].T)) @ t[p + "o"].T


def gated_ff(t, p, h):
    return (gelu_tanh(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def run_order(n_layers, loop):
    """[(layer, whether it opens a repetition)] in the order the layers run."""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    out = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        out += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return out + [(i, False) for i in range(loop["stop"], n_layers)]


def mixer_out(t, p, l, h, eps):
    m = l["mixer"]
    if l["type"] == "wkv":
        return wkv_mixer(t, p, m, h, eps)
    if l["type"] == "parallel":
        return m["left_scale"] * full_attention_branch(t, p + "left.", m["left"], h, eps) + m["right_scale"] * gla_branch(t, p + "right.", m["right"], h, eps)
    left, right = window_attention_branch(t, p + "left.", m["left"], h, eps), delta_branch(t, p + "right.", m["right"], h, eps)
    return (t[p + "left.out"] * unit(left, eps) + t[p + "right.out"] * unit(right, eps)) / 2


def model_logits(tensors, cfg, tokens, residual_out=None):
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = t["embed"][torch.tensor(tokens)]
    for i, opens in run_order(len(cfg["layers"]), cfg.get("loop")):
        l, p = cfg["layers"][i], f"l{i}."
        if opens:
            x = torch.cat([x, x0], -1) @ t["loop.in"].T
        h = layer_norm(x, t[p + "norm1"], t[p + "norm1.b"], eps)
        y = mixer_out(t, p + "mix.", l, h, eps)
        if l.get("mlp"):
            y = y + gated_ff(t, p + "mlp.", h)
        x = x + y
        if residual_out is not None:
            residual_out.append(x.clone())
    return layer_norm(x, t["final.norm"], t["final.norm.b"], eps) @ t["embed"].T * cfg["logit_scale"]


def logit_error(got, want):
    """Per row: root mean square of the difference with its mean taken off, over the root mean square of the wanted row."""
    d = got.to(F64) - want.to(F64)
    d = d - d.mean(-1, keepdim=True)
    w = want.to(F64) - want.to(F64).mean(-1, keepdim=True)
    return torch.sqrt((d * d).mean(-1)) / torch.sqrt((w * w).mean(-1))
