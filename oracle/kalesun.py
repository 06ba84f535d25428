"""Plain numpy (float64) statement of the Kalesun architecture, one function per mechanism: the yardstick the GPU kernels
and the engine are tested against.  It shares no code with the product path: no paging, no packing of projections, no
chunked recurrences, no grouping of tokens by expert.  Every sequence is walked token by token; attention keeps an explicit
list of what it caches, the recurrent mixers their state matrices.

Notation: W x for a weight stored [out, in]; positions start at 0 in every sequence; rms(v) = v / sqrt(mean(v^2) + eps).
  embedding:  x = E[tok]
  layer:      x <- rms(alpha x + mixer(x)) w1;   x <- rms(alpha x + ff(x)) w2      (norm after the sum; ff may be absent)
  attention:  q, k, v = Wq x, Wk x, Wv x; every q head is rms(q) wq and every k head rms(k) wk, THEN rotated on its first
              rot.dims values (value i with i + dims / 2, angle pos * f_i); s = q.k * scale over the keys j <= i with
              i - j < size or j < keep_first; softmax whose denominator also holds exp(sink_h); the head's output times
              sigmoid(Wg x)_h; Wo.  f_i = base^(-2i / dims), stretched by wavelength (see scaled_frequency).
              v_mix layers other than the first such layer cache v <- (1 - l) v + l v_first, v_first = the first such
              layer's values of the same token.
  delta:      q, k, v = silu(conv(Wq x)), silu(conv(Wk x)), silu(conv(Wv x)), conv over the last taps tokens per channel;
              q, k unit vectors per head, q also times dim^-1/2; beta = sigmoid(Wb x) and g = exp(-exp(A_log) softplus(
              Wa x + dt_bias)), one number per head each; S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q;
              rms(o) w silu(Wg x) per head; Wo
  gla:        q = Wq x dim^-1/2, k, v; decay per key channel sigmoid(Wa2 Wa1 x + b)^(1 / tau); S <- diag(decay) S + k v^T;
              o = S^T q; rms(o) w silu(Wg x) per head; Wo
  ff:         Wd glu(Wg x, Wu x) with glu(a, b) = a' sigmoid(1.702 a') (b' + 1), a' = min(a, limit), b' = b clamped to
              [-limit, limit]; or a mixture of experts of that kind: z = Wr x + b, the `top` largest, weights softmax over
              those alone
  output:     logits = E (rms(x) w_final)
"""
import math

import numpy as np


def bf16_round(a):
    """Nearest-even rounding of float values to bfloat16, returned as float64."""
    u = np.asarray(a, np.float32).view(np.uint32)
    u = (u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) & np.uint32(0xFFFF0000)
    return u.view(np.float32).astype(np.float64)


def to_bf16_bits(a):
    """bf16-representable float values -> uint16 bit patterns."""
    return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> np.uint32(16)).astype(np.uint16)


# ---- configuration / weights --------------------------------------------------------------------------------------------
def attention_mixer(heads=4, kv_heads=2, dim=8, vdim=6, size=9, keep_first=3, rot_dims=4, rot_base=100.0, scaling=(3.0, 1.0, 4.0, 60), scale=0.4,
                    v_mix=False):
    """size=None: no mask entry (causal); scaling=None: plain rotary, else (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": rot_base, "dims": rot_dims}, "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep_first}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def delta_mixer(heads=4, kv_heads=2, dim=6, vdim=5, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def gla_mixer(heads=3, dim=6, vdim=5, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def dense_mlp(ff=24, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def expert_mlp(ff=8, experts=5, top=2, limit=0.9):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def make_config(layers, vocab=80, width=24, eps=1e-5, alpha=1.7):
    """layers: list of (type, mixer dict, mlp dict or None)."""
    return {"architecture": "Kalesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}


def tensor_shapes(cfg, low_rank=4):
    """low_rank: inner size of the gla layers' decay projections (the tensors decide; an int, or a dict layer -> size)."""
    W, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m, q = "l%d." % i, l["mixer"], "l%d.mix." % i
        out[p + "norm1"] = (W,)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        if l["type"] == "attention":
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "g"] = (H * D, W), (G * D, W), (G * V, W), (H, W)
            out[q + "q.norm"] = out[q + "k.norm"] = (D,)
            out[q + "sink"] = (H,)
            if m["v_mix"]:
                out[q + "vmix"] = ()
        elif l["type"] == "delta":
            out[q + "q"], out[q + "k"], out[q + "v"] = (G * D, W), (G * D, W), (H * V, W)
            for n in ("q", "k", "v"):
                out[q + n + ".conv"] = (out[q + n][0], m["conv"])
            out[q + "a"] = out[q + "b"] = (H, W)
            out[q + "A_log"] = out[q + "dt_bias"] = (H,)
            out[q + "norm"], out[q + "g"] = (V,), (H * V, W)
        elif l["type"] == "gla":
            r = low_rank[i] if isinstance(low_rank, dict) else low_rank
            out[q + "q"], out[q + "k"], out[q + "v"], out[q + "g"] = (H * D, W), (H * D, W), (H * V, W), (H * V, W)
            out[q + "a1"], out[q + "a2"], out[q + "a2.b"] = (r, W), (H * D, r), (H * D,)
            out[q + "norm"] = (V,)
        else:
            raise ValueError(l["type"])
        out[q + "o"] = (W, H * V)
        f = l["mlp"]
        if f is not None:
            out[p + "norm2"] = (W,)
            if f["kind"] == "dense":
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (f["ff"], W)
                out[p + "mlp.down"] = (W, f["ff"])
            else:
                E, ff = f["router"]["experts"], f["expert"]["ff"]
                out[p + "mlp.router"], out[p + "mlp.router.b"] = (E, W), (E,)
                for e in range(E):
                    out[p + "mlp.e%d.gate" % e] = out[p + "mlp.e%d.up" % e] = (ff, W)
                    out[p + "mlp.e%d.down" % e] = (W, ff)
    out["final.norm"] = (W,)
    return out


def random_weights(cfg, rng, low_rank=4):
    """bf16-representable float64 arrays."""
    W, out = cfg["width"], {}
    for name, shape in tensor_shapes(cfg, low_rank).items():
        fan_in = shape[-1] if len(shape) == 2 else W
        last = name.split(".")[-1]
        if "norm" in last:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "conv":
            a = 0.6 * rng.standard_normal(shape)
        elif last == "vmix":
            a = np.asarray(0.2 + 0.6 * rng.random())
        elif last in ("A_log", "dt_bias"):
            a = -1.0 + 0.5 * rng.standard_normal(shape)
        elif last == "sink":
            a = rng.standard_normal(shape)
        elif last == "b" and len(shape) == 1:
            a = 0.5 * rng.standard_normal(shape)
        elif last in ("gate", "up"):
            a = 1.5 / np.sqrt(fan_in) * rng.standard_normal(shape)      # pre-activations that reach the clamps
        elif name == "embed":
            a = 0.5 * rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / np.sqrt(fan_in)
        out[name] = bf16_round(a)
    return out


# ---- mechanisms --------------------------------------------------------------------------------------------------------
def rms(v, eps):
    v = np.asarray(v, np.float64)
    return v / np.sqrt(np.mean(v * v) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, np.float64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, np.float64))


def sum_norm(x, y, alpha, w, eps):
    """The residual step with the norm after the sum."""
    return rms(alpha * x + y, eps) * w


def scaled_frequency(f, scaling):
    """A rotary frequency under wavelength-dependent scaling: waves shorter than original / high keep it, waves longer than
    original / low turn `factor` times slower, a linear ramp in original / wavelength joins the two."""
    if scaling is None:
        return f
    turns = scaling["original"] * f / (2.0 * math.pi)           # how often the wave turns within the original context
    if turns > scaling["high"]:
        return f
    if turns < scaling["low"]:
        return f / scaling["factor"]
    s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
    return (1.0 - s) * f / scaling["factor"] + s * f


def rotate_halves(x, pos, dims, base, scaling=None):
    """Rotary positions on the first `dims` values of x: value i is paired with i + dims / 2."""
    y = np.array(x, np.float64)
    hf = dims // 2
    for i in range(hf):
        a = pos * scaled_frequency(float(base) ** (-2.0 * i / dims), scaling)
        c, s = math.cos(a), math.sin(a)
        u, v = x[i], x[i + hf]
        y[i], y[i + hf] = u * c - v * s, v * c + u * s
    return y


def visible_keys(pos, mask):
    """The keys a position sees: the last `size` ones and the first `keep_first` ones of the sequence (no mask: all)."""
    if not mask or not mask.get("size"):
        return list(range(pos + 1))
    return [j for j in range(pos + 1) if pos - j < mask["size"] or j < mask.get("keep_first", 0)]


def sink_softmax(scores, sink):
    """Weights of a softmax whose denominator also holds exp(sink); the sink has no value."""
    s = np.asarray(scores, np.float64)
    mx = max(float(np.max(s)), float(sink))
    e = np.exp(s - mx)
    return e / (np.sum(e) + math.exp(sink - mx))


def glu(a, b, limit):
    a = np.minimum(a, limit)
    return a * sigmoid(1.702 * a) * (np.clip(b, -limit, limit) + 1.0)


def gated_ff(w, p, x, limit):
    return w[p + "down"] @ glu(w[p + "gate"] @ x, w[p + "up"] @ x, limit)


def route(z, top):
    """The `top` largest entries of z (ties: lowest index) and the softmax over those entries alone."""
    order = sorted(range(len(z)), key=lambda e: (-z[e], e))[:top]
    e = np.exp(np.array([z[i] for i in order]) - z[order[0]])
    return order, e / np.sum(e)


def expert_ff(w, p, f, x):
    chosen, wts = route(w[p + "mlp.router"] @ x + w[p + "mlp.router.b"], f["router"]["top"])
    y = np.zeros(len(x))
    for e, g in zip(chosen, wts):
        y += g * gated_ff(w, p + "mlp.e%d." % e, x, f["expert"]["limit"])
    return y


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


class KeyValueList:
    """What an attention layer caches for one sequence: one (keys, values) pair of [kv_heads, *] arrays per position."""

    def __init__(self):
        self.k, self.v = [], []


def attention_step(w, q_, m, eps, st, x, pos, v_first):
    """v_first: the first value-mixing layer's values of this token ([kv_heads, vdim]), or None where nothing is mixed in.
    Returns (output, the layer's own values before mixing)."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    dims, base, scaling = m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling")
    q = (w[q_ + "q"] @ x).reshape(H, D)
    k = (w[q_ + "k"] @ x).reshape(G, D)
    own = (w[q_ + "v"] @ x).reshape(G, V)
    st.k.append(np.stack([rotate_halves(rms(k[g], eps) * w[q_ + "k.norm"], pos, dims, base, scaling) for g in range(G)]))
    st.v.append(own if v_first is None else mix_values(own, v_first, float(np.asarray(w[q_ + "vmix"]).reshape(-1)[0])))
    gate = sigmoid(w[q_ + "g"] @ x)
    see = visible_keys(pos, m.get("mask"))
    out = np.zeros((H, V))
    for h in range(H):
        g = h // (H // G)
        qh = rotate_halves(rms(q[h], eps) * w[q_ + "q.norm"], pos, dims, base, scaling)
        pr = sink_softmax([float(qh @ st.k[j][g]) * m["scale"] for j in see], w[q_ + "sink"][h])
        for p, j in zip(pr, see):
            out[h] += p * st.v[j][g]
        out[h] *= gate[h]
    return w[q_ + "o"] @ out.reshape(-1), own


class DeltaState:
    """The state matrices [heads, dim, vdim] and the last taps - 1 inputs of the three convolutions."""

    def __init__(self, m):
        H, G, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        self.S = np.zeros((H, D, V))
        self.hist = {n: np.zeros((T - 1, c)) for n, c in (("q", G * D), ("k", G * D), ("v", H * V))}


def short_conv(w_conv, hist, x):
    """Causal convolution over the last taps tokens (last column: the current one); returns (output, new history)."""
    win = np.vstack([hist, x[None, :]])                     # [taps, channels], oldest first
    return (win.T * w_conv).sum(1), win[1:]


def unit(v):
    return v / np.sqrt(np.sum(v * v) + 1e-6)


def head_decay(raw, a_log, dt_bias):
    """One decay per head."""
    return np.exp(-np.exp(a_log) * softplus(raw + dt_bias))


def delta_rule(S, q, k, v, beta, g):
    """One token of the gated delta rule for one head.  S: [dim, vdim]; g: one number."""
    S = g * S
    u = beta * (v - S.T @ k)
    S = S + np.outer(k, u)
    return S, S.T @ q


def delta_step(w, q_, m, eps, st, x):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    z = {}
    for n in ("q", "k", "v"):
        y, st.hist[n] = short_conv(w[q_ + n + ".conv"], st.hist[n], w[q_ + n] @ x)
        z[n] = silu(y)
    q, k, v = z["q"].reshape(G, D), z["k"].reshape(G, D), z["v"].reshape(H, V)
    beta = sigmoid(w[q_ + "b"] @ x)
    g = head_decay(w[q_ + "a"] @ x, w[q_ + "A_log"], w[q_ + "dt_bias"])
    gate = silu(w[q_ + "g"] @ x).reshape(H, V)
    out = np.zeros((H, V))
    for h in range(H):
        gg = h // (H // G)
        st.S[h], o = delta_rule(st.S[h], unit(q[gg]) * D ** -0.5, unit(k[gg]), v[h], beta[h], g[h])
        out[h] = rms(o, eps) * w[q_ + "norm"] * gate[h]
    return w[q_ + "o"] @ out.reshape(-1)


class MatrixState:
    def __init__(self, m):
        self.S = np.zeros((m["heads"], m["dim"], m["vdim"]))


def channel_decay(z, tau):
    """One decay per key channel."""
    return sigmoid(z) ** (1.0 / tau)


def gla_rule(S, q, k, v, decay):
    """One token of gated linear attention for one head: the decay acts on the rows of S."""
    S = decay[:, None] * S + np.outer(k, v)
    return S, S.T @ q


def gla_step(w, q_, m, eps, st, x):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (w[q_ + "q"] @ x).reshape(H, D) * D ** -0.5
    k, v = (w[q_ + "k"] @ x).reshape(H, D), (w[q_ + "v"] @ x).reshape(H, V)
    a = channel_decay(w[q_ + "a2"] @ (w[q_ + "a1"] @ x) + w[q_ + "a2.b"], m["tau"]).reshape(H, D)
    gate = silu(w[q_ + "g"] @ x).reshape(H, V)
    out = np.zeros((H, V))
    for h in range(H):
        st.S[h], o = gla_rule(st.S[h], q[h], k[h], v[h], a[h])
        out[h] = rms(o, eps) * w[q_ + "norm"] * gate[h]
    return w[q_ + "o"] @ out.reshape(-1)


# ---- the model ---------------------------------------------------------------------------------------------------------
class Sequence:
    """Everything one sequence carries from token to token."""

    def __init__(self, cfg):
        make = {"attention": lambda m: KeyValueList(), "delta": DeltaState, "gla": MatrixState}
        self.pos, self.layers = 0, [make[l["type"]](l["mixer"]) for l in cfg["layers"]]


def token_step(cfg, w, seq, tok, taps=None):
    """Runs one token; returns the logits.  taps (a list): receives the residual stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][tok]
    v_first = None
    for i, l in enumerate(cfg["layers"]):
        p, q_, m = "l%d." % i, "l%d.mix." % i, l["mixer"]
        if l["type"] == "attention":
            mixes = m.get("v_mix", False)
            y, own = attention_step(w, q_, m, eps, seq.layers[i], x, seq.pos, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        elif l["type"] == "delta":
            y = delta_step(w, q_, m, eps, seq.layers[i], x)
        else:
            y = gla_step(w, q_, m, eps, seq.layers[i], x)
        x = sum_norm(x, y, alpha, w[p + "norm1"], eps)
        f = l["mlp"]
        if f is not None:
            y = gated_ff(w, p + "mlp.", x, f["limit"]) if f["kind"] == "dense" else expert_ff(w, p, f, x)
            x = sum_norm(x, y, alpha, w[p + "norm2"], eps)
        if taps is not None:
            taps.append(x.copy())
    seq.pos += 1
    return w["embed"] @ (rms(x, eps) * w["final.norm"])


def run_sequence(cfg, w, tokens, want=None, layer_taps=False):
    """Logits [len(want), vocab] of one sequence walked token by token (want: positions, default all)."""
    seq = Sequence(cfg)
    want = range(len(tokens)) if want is None else want
    wanted, out, taps_all = set(want), {}, []
    for t, tok in enumerate(tokens):
        taps = [] if layer_taps else None
        lg = token_step(cfg, w, seq, int(tok), taps)
        if t in wanted:
            out[t] = lg
        if layer_taps:
            taps_all.append(np.stack(taps))
    logits = np.stack([out[t] for t in want]) if len(out) else np.zeros((0, cfg["vocab"]))
    if layer_taps:
        return logits, np.stack(taps_all, axis=1)          # [layers, tokens, width]
    return logits
