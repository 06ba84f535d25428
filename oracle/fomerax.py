"""Plain numpy (float64) statement of the Fomerax architecture, one function per mechanism: the yardstick the GPU kernels
and the engine are tested against.  It shares no code with the product path: no paging, no packed projections, no key map
folded into the queries, no grouping of tokens by expert.  Every sequence is walked token by token; an attention layer keeps
the list of what it caches.

Notation: W x for a weight stored [out, in]; positions start at 0 in every sequence; rms(v) = v / sqrt(mean(v^2) + eps).
  embedding:  x = E[tok]
  layer:      x += rms(mixer(rms(x) w1)) w1b;   x += rms(ff(rms(x) w2)) w2b        (ff may be absent)
              then the token's row of this layer: e = part i of the token's row of the side table, g = gelu(Wsg x) * e,
              x += rms(Wsp g) ws          (reads the stream itself, not a norm of it)
  attention:  q, k, v = Wq x, Wk x, Wv x, no rotation; q times a temperature that grows with the position; the score is
              capped, THEN lowered by slope_h per token of distance; causal softmax; output times sigmoid(Wg x) per value; Wo
  latent:     q = Wuq (rms(Wdq x) wdq), per head [unrotated | rotated]; Wdkv x = [latent | shared rotated key part]; the
              cache row is c = rms(latent) wdkv and the rotated part; per head k = [Wuk c | rotated part], v = Wuv c;
              softmax over the last `size` keys; output times sigmoid(Wg x) per value; Wo.  Rotary: neighbouring pairs,
              frequencies and amplitude as in yarn_frequencies
  ff:         Wd (gelu(Wg x) * (Wu x)), or a mixture of experts Wd (silu(Wg y) * (Wu y)): s = sigmoid(Wr x), the `top`
              largest are used, each on the INPUT y = s x, and their outputs are summed as they are
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
def attention_mixer(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, softcap=3.0, coef=0.3, every=5):
    """softcap=None: scores are not capped; coef=None: no query temperature."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return m


def latent_mixer(heads=3, dim=6, rot_dim=4, vdim=5, q_rank=10, kv_rank=7, size=9, scale=0.4, base=100.0, scaling=(3.0, 4.0, 1.0, 60)):
    """size=None: no mask entry (causal); scaling=None: plain rotary, else (factor, fast, slow, original)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        m["mask"] = {"size": size}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "fast", "slow", "original"), scaling))
    return m


def dense_mlp(ff=24):
    return {"kind": "dense", "ff": ff}


def expert_mlp(ff=8, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def make_config(layers, vocab=80, width=24, eps=1e-5, side_dim=5):
    """layers: list of (type, mixer dict, mlp dict or None)."""
    return {"architecture": "Fomerax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side_dim},
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}


def tensor_shapes(cfg):
    W, d, out = cfg["width"], cfg["token_side"]["dim"], {}
    out["embed"] = (cfg["vocab"], W)
    out["side.embed"] = (cfg["vocab"], d * len(cfg["layers"]))
    for i, l in enumerate(cfg["layers"]):
        p, m, q = "l%d." % i, l["mixer"], "l%d.mix." % i
        H, D, V = m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = out[p + "norm1b"] = (W,)
        if l["type"] == "attention":
            G = m["kv_heads"]
            out[q + "q"], out[q + "k"], out[q + "v"] = (H * D, W), (G * D, W), (G * V, W)
        elif l["type"] == "latent_attention":
            R, rd, QR = m["kv_rank"], m["rot_dim"], m["q_rank"]
            out[q + "dq"], out[q + "dq.norm"], out[q + "uq"] = (QR, W), (QR,), (H * (D + rd), QR)
            out[q + "dkv"], out[q + "dkv.norm"] = (R + rd, W), (R,)
            out[q + "uk"], out[q + "uv"] = (H * D, R), (H * V, R)
        else:
            raise ValueError(l["type"])
        out[q + "g"], out[q + "o"] = (H * V, W), (W, H * V)
        f = l["mlp"]
        if f is not None:
            out[p + "norm2"] = out[p + "norm2b"] = (W,)
            if f["kind"] == "dense":
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (f["ff"], W)
                out[p + "mlp.down"] = (W, f["ff"])
            else:
                E, ff = f["router"]["experts"], f["expert"]["ff"]
                out[p + "mlp.router"] = (E, W)
                for e in range(E):
                    out[p + "mlp.e%d.gate" % e] = out[p + "mlp.e%d.up" % e] = (ff, W)
                    out[p + "mlp.e%d.down" % e] = (W, ff)
        out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (d, W), (W, d), (W,)
    out["final.norm"] = (W,)
    return out


def random_weights(cfg, rng):
    """bf16-representable float64 arrays."""
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if "norm" in last:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "embed":
            a = rng.standard_normal(shape) * (0.5 if name == "embed" else 1.0)
        else:
            a = (1.5 if last in ("gate", "up", "q", "k", "uq", "uk") else 1.0) * rng.standard_normal(shape) / np.sqrt(shape[-1])
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


def gelu_tanh(z):
    z = np.asarray(z, np.float64)
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softmax(s):
    e = np.exp(np.asarray(s, np.float64) - np.max(s))
    return e / np.sum(e)


def yarn_frequencies(base, dims, scaling):
    """(frequencies of the dims / 2 pairs, factor on cos and sin).  With scaling, a pair's share of the slowed-down frequency
    grows linearly with its index between the two indices at which a wave turns `fast` and `slow` times in `original`."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if scaling is None:
        return f, 1.0
    index_at = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_at(scaling["fast"])), 0)
    hi = min(math.ceil(index_at(scaling["slow"])), dims - 1)
    share = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * share + f * (1.0 - share), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, pos, base, scaling=None):
    """Rotary positions on all of x: value 2i is paired with 2i + 1."""
    f, amp = yarn_frequencies(base, len(x), scaling)
    c, s = np.cos(pos * f) * amp, np.sin(pos * f) * amp
    y = np.array(x, np.float64)
    y[0::2], y[1::2] = x[0::2] * c - x[1::2] * s, x[1::2] * c + x[0::2] * s
    return y


def query_temperature(pos, q_temp):
    if not q_temp:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log((pos + 1) // q_temp["every"] + 1)


def head_slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def capped_scores(raw, softcap, slope, distance):
    """The cap first, the distance's share taken off what it leaves."""
    s = softcap * np.tanh(raw / softcap) if softcap else np.asarray(raw, np.float64)
    return s - slope * distance


def window_start(pos, mask):
    """First key a position sees (no mask: 0)."""
    return max(0, pos - mask["size"] + 1) if mask and mask.get("size") else 0


def gelu_ff(w, p, x):
    return w[p + "down"] @ (gelu_tanh(w[p + "gate"] @ x) * (w[p + "up"] @ x))


def silu_ff(w, p, x):
    return w[p + "down"] @ (silu(w[p + "gate"] @ x) * (w[p + "up"] @ x))


def route(z, top):
    """The `top` largest scores (ties: lowest index), as they are."""
    s = sigmoid(z)
    order = sorted(range(len(s)), key=lambda e: (-s[e], e))[:top]
    return order, np.array([s[e] for e in order])


def expert_ff(w, p, f, x):
    """The score multiplies what an expert reads, not what it returns."""
    y = np.zeros(len(x))
    for e, s in zip(*route(w[p + "mlp.router"] @ x, f["router"]["top"])):
        y += silu_ff(w, p + "mlp.e%d." % e, s * x)
    return y


def token_input(w, p, x, row, eps):
    """The layer's own part of the token's side row, gated by the stream; returns what the stream gains."""
    g = gelu_tanh(w[p + "side.gate"] @ x) * row
    return rms(w[p + "side.proj"] @ g, eps) * w[p + "side.norm"]


class Cached:
    """What a layer caches for one sequence, one entry per position (keys and values, or latents and rotated key parts)."""

    def __init__(self):
        self.a, self.b = [], []


def attention_step(w, q_, m, eps, st, x, pos):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (w[q_ + "q"] @ x).reshape(H, D) * query_temperature(pos, m.get("q_temp"))
    st.a.append((w[q_ + "k"] @ x).reshape(G, D))
    st.b.append((w[q_ + "v"] @ x).reshape(G, V))
    keys, vals = np.stack(st.a), np.stack(st.b)
    dist = pos - np.arange(pos + 1)
    out = np.zeros((H, V))
    for h in range(H):
        g = h // (H // G)
        out[h] = softmax(capped_scores(keys[:, g] @ q[h] * m["scale"], m.get("softcap"), head_slope(h, H), dist)) @ vals[:, g]
    return w[q_ + "o"] @ (out.reshape(-1) * sigmoid(w[q_ + "g"] @ x))


def latent_step(w, q_, m, eps, st, x, pos):
    H, D, rd, V, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base, scaling = m["rot"]["base"], m["rot"].get("scaling")
    q = (w[q_ + "uq"] @ (rms(w[q_ + "dq"] @ x, eps) * w[q_ + "dq.norm"])).reshape(H, D + rd)
    z = w[q_ + "dkv"] @ x
    st.a.append(rms(z[:R], eps) * w[q_ + "dkv.norm"])
    st.b.append(rotate_pairs(z[R:], pos, base, scaling))
    lo = window_start(pos, m.get("mask"))
    c, kr = np.stack(st.a[lo:]), np.stack(st.b[lo:])
    out = np.zeros((H, V))
    for h in range(H):
        k = c @ w[q_ + "uk"][h * D:(h + 1) * D].T
        s = (k @ q[h, :D] + kr @ rotate_pairs(q[h, D:], pos, base, scaling)) * m["scale"]
        out[h] = softmax(s) @ (c @ w[q_ + "uv"][h * V:(h + 1) * V].T)
    return w[q_ + "o"] @ (out.reshape(-1) * sigmoid(w[q_ + "g"] @ x))


# ---- the model ---------------------------------------------------------------------------------------------------------
class Sequence:
    """Everything one sequence carries from token to token."""

    def __init__(self, cfg):
        self.pos, self.layers = 0, [Cached() for _ in cfg["layers"]]


STEPS = {"attention": attention_step, "latent_attention": latent_step}


def token_step(cfg, w, seq, tok, taps=None):
    """Runs one token; returns the logits.  taps (a list): receives the residual stream after every layer."""
    eps, d = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    x = w["embed"][tok]
    for i, l in enumerate(cfg["layers"]):
        p, f = "l%d." % i, l["mlp"]
        y = STEPS[l["type"]](w, p + "mix.", l["mixer"], eps, seq.layers[i], rms(x, eps) * w[p + "norm1"], seq.pos)
        x = x + rms(y, eps) * w[p + "norm1b"]
        if f is not None:
            h = rms(x, eps) * w[p + "norm2"]
            y = gelu_ff(w, p + "mlp.", h) if f["kind"] == "dense" else expert_ff(w, p, f, h)
            x = x + rms(y, eps) * w[p + "norm2b"]
        x = x + token_input(w, p, x, w["side.embed"][tok, i * d:(i + 1) * d], eps)
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
