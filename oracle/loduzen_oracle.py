"""Plain, slow restatement of the Loduzen decoder-only language model (test infrastructure only).

Torch on the CPU, one function per mechanism, whole sequences at once, no cache and no carried state: every position
is recomputed from the start of its sequence, and every recurrence is an explicit loop over time.  Nothing here is
imported by the product path and nothing of the product path is imported here.  The arithmetic type is the type of the
tensors handed in (float64 gives a reference whose own rounding is negligible).

Notation: matrices are ``[out, in]`` and applied as ``W @ x``; ``p`` maps the short tensor names of one mixer, feed-forward
or token input (``left.q.norm``, ``right.a2.b``, ``conv``, ``gate`` ...) to tensors, ``m`` is the matching dictionary of
the configuration.

The model: x = embed[token]; per layer x += mixer(rms(x) w_1), x += ff(rms(x) w_2), x += rms(proj(gelu(gate x) * e)) w_s
with e the layer's slice of a second embedding table; logits = embed @ (rms(x) w_f).
"""

from __future__ import annotations

import math

import torch


# ---- elementwise pieces ---------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu(z):
    """The tanh form."""
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u, w, b):
    """y[t, c] = b[c] + sum_j w[c, j] u[t - (taps - 1) + j, c], zeros before the start; the last tap is the current token's."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        y[t] = b
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * u[s]
    return y


# ---- rotary positions -------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(angle per position of every pair, multiplier of cosine and sine).  With scaling, a pair's rate is blended between
    the full rate and 1 / factor of it along a ramp over the pair's index, whose ends are where a pair makes ``fast`` and
    ``slow`` turns over the original length."""
    base, dims, sc = float(rot["base"]), int(rot["dims"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    factor, orig = float(sc["factor"]), float(sc["original"])

    def index_of(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """Turns the first ``dims`` channels of x [T, heads, n] (pairs 2i, 2i + 1) by position x rate; the others pass."""
    if not rot or rot["dims"] == 0:
        return x
    f, amp = frequencies(rot)
    dims = int(rot["dims"])
    ang = positions.to(x.dtype)[:, None, None] * torch.tensor(f, dtype=torch.float64).to(x.dtype)[None, None, :]
    cs, sn = torch.cos(ang) * amp, torch.sin(ang) * amp
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * cs - b * sn
    out[..., 1:dims:2] = b * cs + a * sn
    return out


# ---- mixers -----------------------------------------------------------------------------------------------------------
def visible(i, j, window):
    """Key j is seen from query i when it is not in the future and less than ``window`` tokens back (None: all)."""
    return 0 <= i - j and (window is None or i - j < window)


def window_attention(h, p, m, eps, positions=None, sink=True):
    """Grouped-query softmax attention whose values are the projected keys (before norm and rotation), per-head RMS norms of
    q and k, rotary positions, a sliding window, and one more unit in the softmax's denominator."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G = m.get("kv_heads") or H
    pos = torch.arange(T) if positions is None else positions
    window = m["mask"]["size"] if m.get("mask") else None
    k_raw = (h @ p["k"].T).reshape(T, G, d)
    q = rotate(rms_unit((h @ p["q"].T).reshape(T, H, d), eps) * p["q.norm"], pos, m.get("rot"))
    k = rotate(rms_unit(k_raw, eps) * p["k.norm"], pos, m.get("rot"))
    gap = pos[:, None] - pos[None, :]                                  # the rule of `visible`, for all pairs at once
    seen = (gap >= 0) & (gap < (window if window is not None else T + 1))
    out = torch.zeros((T, H, d), dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)    # the unit is exp(0): it belongs to the maximum
        e = torch.exp(s - top)
        out[:, hh] = (e / (e.sum(dim=-1, keepdim=True) + (torch.exp(-top) if sink else 0.0))) @ k_raw[:, g]
    return out.reshape(T, H * d) @ p["o"].T


def gated_linear_attention(h, p, m, eps):
    """Per head S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with a decay per key channel,
    alpha = sigmoid(a2 a1 h + b)^(1 / tau); o / rms(o) x w, x silu(gate), output projection."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ p["k"].T).reshape(T, H, d)
    v = (h @ p["v"].T).reshape(T, H, dv)
    z = (h @ p["a1"].T) @ p["a2"].T + p["a2.b"]
    alpha = torch.exp(-softplus(-z) / m["tau"]).reshape(T, H, d)
    out = torch.zeros((T, H, dv), dtype=h.dtype)
    for hh in range(H):
        S = torch.zeros((d, dv), dtype=h.dtype)
        for t in range(T):
            S = alpha[t, hh][:, None] * S + torch.outer(k[t, hh], v[t, hh])
            out[t, hh] = S.T @ q[t, hh]
    out = rms_unit(out, eps) * p["norm"]
    return (out.reshape(T, H * dv) * silu(h @ p["g"].T)) @ p["o"].T


def part(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def parallel(h, p, m, eps, positions=None):
    """Two mixers side by side on the same input, their outputs added with a weight each."""
    return (m["left_scale"] * window_attention(h, part(p, "left."), m["left"], eps, positions)
            + m["right_scale"] * gated_linear_attention(h, part(p, "right."), m["right"], eps))


def mamba2(h, p, m, eps):
    """State-space duality: one projection [z | x | B | C | dt]; x, B, C pass a short causal convolution with bias and silu;
    dt = softplus(dt + bias); per head S_t = exp(-exp(A) dt) S_(t-1) + dt B_t x_t^T, y_t = S_t^T C_t + D x_t (B, C shared by
    the heads of a group); y silu(z), RMS-normed in equal parts, x w, output projection."""
    T = h.shape[0]
    H, N, G, dv = m["heads"], m["state"], m["groups"], m["vdim"]
    inner = H * dv
    proj = h @ p["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, p["conv"], p["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + p["dt_bias"])                                   # [T, H]
    decay = torch.exp(-torch.exp(p["A_log"]) * dt)
    y = torch.zeros((T, H, dv), dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        S = torch.zeros((N, dv), dtype=h.dtype)
        for t in range(T):
            S = decay[t, hh] * S + dt[t, hh] * torch.outer(B[t, g], x[t, hh])
            y[t, hh] = S.T @ C[t, g] + p["D"][hh] * x[t, hh]
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms_unit(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * p["norm"]
    return y @ p["o"].T


# ---- feed-forward and token input ---------------------------------------------------------------------------------------
def dense_ff(h, p):
    return (gelu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def token_input(x, e, p, eps):
    """What a layer adds for the token itself: e [T, dim] is the layer's slice of the second embedding table."""
    y = (gelu(x @ p["gate"].T) * e) @ p["proj"].T
    return rms_unit(y, eps) * p["norm"]


# ---- the model --------------------------------------------------------------------------------------------------------
MIXERS = {"parallel": parallel, "mamba2": mamba2}


def forward(cfg: dict, w: dict, tokens, keep_layers: bool = False, dtype=torch.float64):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    w = {k: v.to(dtype) for k, v in w.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens]
    side = cfg.get("token_side")
    kept = []
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[lc["type"]](rms_unit(x, eps) * w[p + "norm1"], part(w, p + "mix."), lc["mixer"], eps)
        if lc.get("mlp"):
            x = x + dense_ff(rms_unit(x, eps) * w[p + "norm2"], part(w, p + "mlp."))
        if side:
            n = side["dim"]
            x = x + token_input(x, w["side.embed"][tokens][:, i * n:(i + 1) * n], part(w, p + "side."), eps)
        kept.append(x)
    logits = (rms_unit(x, eps) * w["final.norm"]) @ w["embed"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def greedy(cfg: dict, w: dict, prompt, n_new: int):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def random_weights(cfg: dict, seed: int, spread: float = 1.0, rank: int = 12) -> dict:
    """Random float32 tensors that bfloat16 holds exactly, under the checkpoint's names.  ``rank``: inner size of the
    two-step decay projections."""
    g = torch.Generator().manual_seed(seed)
    D, w = cfg["width"], {}

    def mat(n_out, n_in, gain=1.0):
        return (torch.randn((n_out, n_in), generator=g) * (gain * spread / math.sqrt(n_in))).to(torch.bfloat16).float()

    def vec(n, mean=0.0, dev=0.1):
        return (mean + dev * torch.randn((n,), generator=g)).to(torch.bfloat16).float()

    w["embed"] = (torch.randn((cfg["vocab"], D), generator=g) * spread).to(torch.bfloat16).float()
    w["final.norm"] = vec(D, 1.0)
    side = cfg.get("token_side")
    if side:
        w["side.embed"] = torch.randn((cfg["vocab"], side["dim"] * len(cfg["layers"])), generator=g).to(torch.bfloat16).float()
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        w[p + "norm1"] = vec(D, 1.0)
        if lc["type"] == "parallel":
            a, q = m["left"], p + "mix.left."
            H, G, d = a["heads"], a.get("kv_heads") or a["heads"], a["dim"]
            w[q + "q"], w[q + "k"], w[q + "o"] = mat(H * d, D), mat(G * d, D, 1.5), mat(D, H * d)
            w[q + "q.norm"], w[q + "k.norm"] = vec(d, 1.5, 0.4), vec(d, 1.5, 0.4)
            r, q = m["right"], p + "mix.right."
            H, d, dv = r["heads"], r["dim"], r["vdim"]
            w[q + "q"], w[q + "k"], w[q + "v"], w[q + "g"] = mat(H * d, D, 1.5), mat(H * d, D, 1.5), mat(H * dv, D), mat(H * dv, D, 1.5)
            w[q + "a1"], w[q + "a2"], w[q + "a2.b"] = mat(rank, D), mat(H * d, rank, 2.0), vec(H * d, 1.0, 1.0)
            w[q + "norm"], w[q + "o"] = vec(dv, 1.0), mat(D, H * dv)
        else:
            H, N, G, dv = m["heads"], m["state"], m["groups"], m["vdim"]
            inner, C = H * dv, H * dv + 2 * G * N
            q = p + "mix."
            w[q + "in"] = mat(inner + C + H, D, 1.5)
            w[q + "conv"] = (torch.randn((C, m["conv"]), generator=g) * 0.6).to(torch.bfloat16).float()
            w[q + "conv.b"] = vec(C, 0.0, 0.3)
            w[q + "dt_bias"], w[q + "A_log"], w[q + "D"] = vec(H, -2.0, 1.0), vec(H, 0.0, 0.7), vec(H, 1.0, 0.5)
            w[q + "norm"], w[q + "o"] = vec(inner, 1.0), mat(D, inner)
        f = lc.get("mlp")
        if f:
            w[p + "norm2"] = vec(D, 1.0)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(f["ff"], D, 1.5), mat(f["ff"], D, 1.5), mat(D, f["ff"])
        if side:
            w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = mat(side["dim"], D), mat(D, side["dim"]), vec(D, 0.6)
    return w
