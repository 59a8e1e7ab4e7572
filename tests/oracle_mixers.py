"""Plain, slow restatement of the sequence-mixer models (test infrastructure): numpy in double
precision, one function per mechanism, whole sequences at a time, no cache.  It shares no code with
the product path; a test compares the framework's kernels, cache and steps with it.

Weights are a dict of arrays under the checkpoint's tensor names; a configuration is the parsed
config.json dict.  Vectors are rows: ``x`` is [tokens, width]."""

import math

import numpy as np
from math import erf

_erf = np.vectorize(erf, otypes=[np.float64])


def f64(array):
    return np.asarray(array, dtype=np.float64)


# ---- pointwise ------------------------------------------------------------------------------
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# Set by ``rounding_error`` while it measures what rounding alone does: applied to every matrix product.
_disturb = None


def linear(x, weight, bias=None):
    y = f64(x) @ f64(weight).T
    y = y if bias is None else y + f64(bias)
    return y if _disturb is None else _disturb(y)


def rms(x, eps):
    """x over the root of its mean square, eps inside the root, along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


# ---- rotary positions -----------------------------------------------------------------------
def rotary_frequencies(rot):
    """(frequency per pair, magnitude of cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    index = np.arange(dims // 2, dtype=np.float64)
    frequency = base ** (-2.0 * index / dims)
    scaling = rot.get("scaling")
    if not scaling:
        return frequency, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dimension(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(dimension(scaling["fast"])), 0)
    high = min(math.ceil(dimension(scaling["slow"])), dims - 1)
    ramp = np.clip((index - low) / max(high - low, 0.001), 0.0, 1.0)
    return frequency / factor * ramp + frequency * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """x [tokens, heads, dim]: neighbouring dimensions 2i, 2i + 1 turn by position * frequency_i."""
    frequency, magnitude = rotary_frequencies(rot)
    angle = f64(positions)[:, None, None] * frequency[None, None, :]
    cosine, sine = magnitude * np.cos(angle), magnitude * np.sin(angle)
    out = x.copy()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * cosine - v * sine
    out[..., 1:rot["dims"]:2] = v * cosine + u * sine
    return out


# ---- attention ------------------------------------------------------------------------------
def sink_attention(q, k, v, scale):
    """Causal; q [T, H, dim], k [T, G, dim], v [T, G, vdim].  The denominator counts one more term
    exp(0) that carries no value."""
    tokens, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((tokens, heads, v.shape[2]))
    visible = np.tril(np.ones((tokens, tokens), bool))
    for h in range(heads):
        score = np.where(visible, (q[:, h] @ k[:, h // group].T) * scale, -np.inf)
        top = np.maximum(score.max(axis=1, keepdims=True), 0.0)
        weight = np.exp(score - top)
        out[:, h] = (weight / (np.exp(-top) + weight.sum(axis=1, keepdims=True))) @ v[:, h // group]
    return out


def attention_mixer(h, w, prefix, size, eps):
    tokens = h.shape[0]
    project = lambda name: linear(h, w[f"{prefix}.{name}"], w[f"{prefix}.{name}.b"])
    q = project("q").reshape(tokens, size["heads"], size["dim"])
    k = project("k").reshape(tokens, size["kv_heads"], size["dim"])
    v = project("v").reshape(tokens, size["kv_heads"], size["vdim"])
    positions = np.arange(tokens)
    q = rotate(rms(q, eps) * f64(w[f"{prefix}.q.norm"]), positions, size["rot"])
    k = rotate(rms(k, eps) * f64(w[f"{prefix}.k.norm"]), positions, size["rot"])
    out = sink_attention(q, k, v, size["scale"]).reshape(tokens, -1)
    return linear(out, w[f"{prefix}.o"], w[f"{prefix}.o.b"])


# ---- gated delta rule -----------------------------------------------------------------------
def short_conv(x, taps):
    """Causal per-channel convolution, x [tokens, channels], taps [channels, n], the last tap on the
    current token, then silu."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return silu(sum(padded[j:j + x.shape[0]] * f64(taps)[:, j] for j in range(n)))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_scan(q, k, v, decay, beta, state=None):
    """q, k [T, H, dim], v [T, H, vdim], decay and beta [T, H]; returns (o, final state)."""
    tokens, heads, dim = q.shape
    state = np.zeros((heads, dim, v.shape[2])) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(tokens):
        for h in range(heads):
            state[h] *= decay[t, h]
            update = beta[t, h] * (v[t, h] - state[h].T @ k[t, h])
            state[h] += np.outer(k[t, h], update)
            out[t, h] = state[h].T @ q[t, h]
    return out, state


def delta_mixer(h, w, prefix, size, eps):
    tokens, heads, kv_heads, dim, vdim = h.shape[0], size["heads"], size["kv_heads"], size["dim"], size["vdim"]
    conv = lambda name: short_conv(linear(h, w[f"{prefix}.{name}"]), w[f"{prefix}.{name}.conv"])
    q = unit(conv("q").reshape(tokens, kv_heads, dim)) * dim ** -0.5
    k = unit(conv("k").reshape(tokens, kv_heads, dim))
    v = conv("v").reshape(tokens, heads, vdim)
    which = np.arange(heads) // (heads // kv_heads)
    beta = sigmoid(linear(h, w[f"{prefix}.b"]))
    step = softplus(linear(h, w[f"{prefix}.a"]) + f64(w[f"{prefix}.dt_bias"]))
    decay = np.exp(-np.exp(f64(w[f"{prefix}.A_log"])) * step)
    o, _ = delta_scan(q[:, which], k[:, which], v, decay, beta)
    gate = silu(linear(h, w[f"{prefix}.g"])).reshape(tokens, heads, vdim)
    o = rms(o, eps) * f64(w[f"{prefix}.norm"]) * gate
    return linear(o.reshape(tokens, -1), w[f"{prefix}.o"])


def parallel_mixer(h, w, prefix, size, eps):
    left = attention_mixer(h, w, f"{prefix}.left", size["left"], eps)
    right = delta_mixer(h, w, f"{prefix}.right", size["right"], eps)
    return 0.5 * (rms(left, eps) * f64(w[f"{prefix}.left.out"]) + rms(right, eps) * f64(w[f"{prefix}.right.out"]))


# ---- matrix memory --------------------------------------------------------------------------
def matrix_memory_scan(q, k, v, log_input, log_forget, state=None):
    """q, k [T, H, dim], v [T, H, vdim], log gates [T, H]; state (S, n, m)."""
    tokens, heads, dim = q.shape
    if state is None:
        state = (np.zeros((heads, dim, v.shape[2])), np.zeros((heads, dim)), np.zeros(heads))
    memory, norm, top = (part.copy() for part in state)
    out = np.zeros_like(v)
    for t in range(tokens):
        for h in range(heads):
            kept = log_forget[t, h] + top[h]
            top[h] = max(kept, log_input[t, h])
            keep, write = math.exp(kept - top[h]), math.exp(log_input[t, h] - top[h])
            memory[h] = keep * memory[h] + write * np.outer(k[t, h], v[t, h])
            norm[h] = keep * norm[h] + write * k[t, h]
            out[t, h] = memory[h].T @ q[t, h] / (max(abs(norm[h] @ q[t, h]), math.exp(-top[h])) + 1e-6)
    return out, (memory, norm, top)


def matrix_memory_mixer(h, w, prefix, size, eps):
    tokens, heads, dim, vdim, cap = h.shape[0], size["heads"], size["dim"], size["vdim"], size["gate_cap"]
    q = linear(h, w[f"{prefix}.q"]).reshape(tokens, heads, dim) * dim ** -0.5
    k = linear(h, w[f"{prefix}.k"]).reshape(tokens, heads, dim)
    v = linear(h, w[f"{prefix}.v"]).reshape(tokens, heads, vdim)
    log_input = cap * np.tanh(linear(h, w[f"{prefix}.i"], w[f"{prefix}.i.b"]) / cap)
    log_forget = log_sigmoid(cap * np.tanh(linear(h, w[f"{prefix}.f"], w[f"{prefix}.f.b"]) / cap))
    o, _ = matrix_memory_scan(q, k, v, log_input, log_forget)
    o = rms(o, eps).reshape(tokens, -1) * f64(w[f"{prefix}.norm"]) * sigmoid(linear(h, w[f"{prefix}.g"]))
    return linear(o, w[f"{prefix}.o"])


MIXERS = {"mlstm": matrix_memory_mixer, "mlstm_2": matrix_memory_mixer, "parallel": parallel_mixer}


# ---- the decoder ----------------------------------------------------------------------------
def token_side(x, ids, index, w, prefix, dim, eps):
    e = f64(w["side.embed"])[ids, index * dim:(index + 1) * dim]
    y = linear(gelu_tanh(linear(x, w[f"{prefix}.side.gate"])) * e, w[f"{prefix}.side.proj"])
    return rms(y, eps) * f64(w[f"{prefix}.side.norm"])


def forward(config, w, tokens, per_layer=None):
    """Logits [tokens, vocab]; ``per_layer`` (a list) collects the residual after every layer."""
    return FORWARD[config["architecture"]](config, w, tokens, per_layer)


def forward_post_norm(config, w, tokens, per_layer=None):
    ids, eps = np.asarray(tokens), config["norm"]["eps"]
    x = f64(w["embed"])[ids]
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}"
        x = x + rms(MIXERS[layer["type"]](x, w, f"{p}.mix", layer["mixer"], eps), eps) * (1.0 + f64(w[f"{p}.norm1"]))
        if layer.get("mlp"):
            y = linear(gelu_erf(linear(x, w[f"{p}.mlp.up"])), w[f"{p}.mlp.down"])
            x = x + rms(y, eps) * (1.0 + f64(w[f"{p}.norm2"]))
        if config.get("token_side"):
            x = x + token_side(x, ids, index, w, p, config["token_side"]["dim"], eps)
        if per_layer is not None:
            per_layer.append(x.copy())
    return linear(rms(x, eps) * (1.0 + f64(w["final.norm"])), w["head"])


# ---- tanh norms before and after each sublayer, windowed attention, routed experts -----------
def tanh_norm(x, w, name):
    return np.tanh(f64(w[f"{name}.alpha"]).reshape(()) * x) * f64(w[name]) + f64(w[f"{name}.b"])


def sinusoids(positions, width):
    """Neighbouring entries 2i, 2i + 1: sine and cosine of position * 10000^(-2i / width)."""
    column = np.arange(width)
    angle = f64(positions)[:, None] * 10000.0 ** (-2.0 * (column // 2) / width)
    return np.where(column % 2 == 0, np.sin(angle), np.cos(angle))


def visible_keys(queries, keys, mask):
    """[queries, keys] positions: not in the future, and near enough or among the first."""
    distance = queries[:, None] - keys[None, :]
    seen = distance >= 0
    if mask:
        seen &= (distance < mask["size"]) | (keys[None, :] < mask.get("keep_first", 0))
    return seen


def capped(score, cap):
    return cap * np.tanh(score / cap) if cap else score


def masked_attention(q, k, v, seen, scale, cap=None):
    """q [T, H, dim], k [S, G, dim], v [S, G, vdim], seen [T, S]."""
    group = q.shape[1] // k.shape[1]
    out = np.zeros((*q.shape[:2], v.shape[2]))
    for h in range(q.shape[1]):
        score = np.where(seen, capped((q[:, h] @ k[:, h // group].T) * scale, cap), -np.inf)
        weight = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, h] = weight / weight.sum(axis=1, keepdims=True) @ v[:, h // group]
    return out


def windowed_mixer(h, w, prefix, size, kept):
    """``kept``: the keys and values of earlier layers by index; returns (output, own keys and values)."""
    tokens = h.shape[0]
    q = linear(h, w[f"{prefix}.q"]).reshape(tokens, size["heads"], size["dim"])
    if size.get("kv_from") is not None:
        k, v = kept[size["kv_from"]]
    else:
        k = linear(h, w[f"{prefix}.k"]).reshape(tokens, size["kv_heads"], size["dim"])
        v = linear(h, w[f"{prefix}.v"]).reshape(tokens, size["kv_heads"], size["vdim"])
    places = np.arange(tokens)
    out = masked_attention(q, k, v, visible_keys(places, places, size.get("mask")), size["scale"], size.get("softcap"))
    out = out.reshape(tokens, -1) * sigmoid(linear(h, w[f"{prefix}.g"]))
    return linear(out, w[f"{prefix}.o"]), (k, v)


def gated_feed_forward(x, w, prefix):
    return linear(silu(linear(x, w[f"{prefix}.gate"])) * linear(x, w[f"{prefix}.up"]), w[f"{prefix}.down"])


def chosen_experts(scores, top):
    """[tokens, top] indices of the largest scores, the lower index first among equals."""
    return np.argsort(-scores, axis=1, kind="stable")[:, :top]


# (layer prefix -> choices) while ``rounding_error`` runs: its disturbed passes keep the undisturbed choices.
_choices = None


def routed_experts(h, w, prefix, router, margins=None):
    z = linear(h, w[f"{prefix}.router"])
    scores = sigmoid(z)
    chosen = chosen_experts(z, router["top"])
    if _choices is not None:
        chosen = _choices.setdefault(prefix, chosen)
    if margins is not None and router["top"] < router["experts"]:
        ranked = -np.sort(-z, axis=1)
        margins.append((ranked[:, router["top"] - 1] - ranked[:, router["top"]]) / z.std())
    out = np.zeros_like(h)
    for expert in range(router["experts"]):
        for place in range(router["top"]):
            rows = np.nonzero(chosen[:, place] == expert)[0]
            if len(rows):
                out[rows] += gated_feed_forward(scores[rows, expert][:, None] * h[rows], w, f"{prefix}.e{expert}")
    return out


def forward_sandwich(config, w, tokens, per_layer=None, margins=None):
    """``margins`` (a list) collects, per routed layer, how far each token's last chosen expert is ahead of the next."""
    ids, kept = np.asarray(tokens), {}
    x = f64(w["embed"])[ids] + sinusoids(np.arange(len(ids)), config["width"])
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}"
        y, kept[index] = windowed_mixer(tanh_norm(x, w, f"{p}.norm1"), w, f"{p}.mix", layer["mixer"], kept)
        x = x + tanh_norm(y, w, f"{p}.norm1b")
        mlp = layer.get("mlp")
        if mlp:
            h = tanh_norm(x, w, f"{p}.norm2")
            y = gated_feed_forward(h, w, f"{p}.mlp") if mlp["kind"] == "dense" else routed_experts(
                h, w, f"{p}.mlp", mlp["router"], margins)
            x = x + tanh_norm(y, w, f"{p}.norm2b")
        if per_layer is not None:
            per_layer.append(x.copy())
    return linear(tanh_norm(x, w, "final.norm"), w["embed"]) * config["logit_scale"]


FORWARD = {"Bizodra": forward_post_norm, "Dalorax": forward_sandwich}


def rounding_error(config, w, tokens, relative, draws=4):
    """Per position, the largest root-mean-square change of the centred logits over some draws of relative
    errors of size ``relative`` in every matrix product (and of that size times the row's scale): how much
    of a difference rounding alone explains.  Positions where a read-out nearly cancels stand out."""
    global _disturb, _choices
    _choices = {}
    base, worst = forward(config, w, tokens), None
    for draw in range(draws):
        rng = np.random.default_rng(draw)

        def disturb(y):
            scale = np.sqrt(np.mean(y * y, axis=-1, keepdims=True))
            return y + relative * (np.abs(y) * rng.uniform(-1, 1, y.shape) + 0.5 * scale * rng.uniform(-1, 1, y.shape))

        _disturb = disturb
        try:
            change = forward(config, w, tokens) - base
        finally:
            _disturb = None
        change -= change.mean(axis=-1, keepdims=True)
        error = np.sqrt((change ** 2).mean(axis=-1))
        worst = error if worst is None else np.maximum(worst, error)
    _choices = None
    return worst / np.sqrt(((base - base.mean(axis=-1, keepdims=True)) ** 2).mean())
