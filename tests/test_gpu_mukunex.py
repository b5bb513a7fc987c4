"""Mukunex on the GPU: each mechanism's kernels against the plain functions of `plain_mukunex`, and the
engine (step function, cache, scheduler, entry point) against the plain forward pass, on small
configurations that differ in every size, constant and in the order of their layers."""
import json

import numpy as np
import pytest
import torch

import plain_mukunex as PM
from helpers import TraceBuilder, random_tokens, rel_err, run_trace_engine

pytestmark = pytest.mark.gpu


def dense(ff):
    return {"kind": "dense", "ff": ff}


def rotation(base, dims, bands=None):
    rot = {"base": base, "dims": dims}
    if bands is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return rot


def parallel_layer(heads, kv_heads, dim, vdim, scale, rot, rheads, rdim, rvdim, decay, rrot, left_scale, right_scale, mlp):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot},
        "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay, "rot": rrot},
        "left_scale": left_scale, "right_scale": right_scale}}


def lru_layer(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def delta_layer(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank, mlp):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank, "gate_rank": gate_rank}}


# A: values of another size than keys (the row-wise attention), partly rotated heads, frequencies in bands, a recurrent unit wider
# than the model, two delta heads a key head.
# B: one head everywhere, filters of one weight (no history), one part, no scaling, layers without feed-forwards.
# C: keys and values of one size (the tensor-core attention in bfloat16), three query heads a kv head, a unit narrower than the
# model in parts of 8, long filters, scales of 1.
CONFIGS = {
    "A": ({"architecture": "Mukunex", "vocab": 131, "width": 64, "norm": {"eps": 1e-5}, "layers": [
        lru_layer(96, 4, 3, dense(88)),
        parallel_layer(6, 2, 16, 24, 0.3, rotation(500.0, 12, (4.0, 1.0, 4.0, 64)), 2, 24, 8, [0.9375, 0.99609375], rotation(90.0, 10), 0.7, 1.3, dense(72)),
        delta_layer(4, 2, 24, 16, 2, 7, 12, None),
        lru_layer(40, 5, 4, dense(24)),
    ]}, 41),
    "B": ({"architecture": "Mukunex", "vocab": 89, "width": 48, "norm": {"eps": 1e-6}, "layers": [
        delta_layer(1, 1, 16, 40, 1, 3, 5, dense(56)),
        parallel_layer(1, 1, 32, 8, 0.2, rotation(10000.0, 32), 1, 8, 40, [1.0], rotation(10000.0, 8), 1.0, 0.5, None),
        lru_layer(24, 1, 1, None),
    ]}, 42),
    "C": ({"architecture": "Mukunex", "vocab": 64, "width": 32, "norm": {"eps": 1e-5}, "layers": [
        parallel_layer(9, 3, 80, 80, 0.11, rotation(1000.0, 48, (2.0, 0.5, 8.0, 100)), 3, 40, 16, [0.5, 0.984375, 0.998046875], rotation(300.0, 40), 1.0, 1.0, dense(40)),
        lru_layer(16, 2, 7, None),
        delta_layer(3, 3, 8, 24, 4, 20, 1, dense(16)),
        parallel_layer(2, 1, 32, 32, 0.2, rotation(50.0, 2), 2, 16, 16, [0.75, 0.0], rotation(20.0, 4), -0.5, 1.5, None),
    ]}, 43),
}
# Largest difference of logits over the largest plain logit, row by row. The 32-bit runs see a few 1e-6 and every row is held to
# 1e-4. In bfloat16 (products and caches in bfloat16 under 32-bit norms, scores and recurrences) a row is held to 3e-1, the median
# row to 3e-2, and at most one row in twenty may be over 1e-1: a wrong key, a lost state or a forgotten sink moves every row by tenths.
TOL = {"float32": 1e-4, "bfloat16": 3e-1}


def check_rows(results, builder, plain_by_request, dtype, what=""):
    errs = []
    for step, rows in builder.rows.items():
        assert step in results, f"{what}: step {step} wrote no logits"
        got = results[step]
        assert got.shape[0] == len(rows), f"{what}: step {step}: {got.shape[0]} rows for {len(rows)} wanted"
        for i, (rid, pos) in enumerate(rows):
            err = rel_err(got[i], plain_by_request[rid][pos])
            assert err <= TOL[dtype], f"{what}: step {step}, request {rid}, position {pos}: relative error {err:.3e} > {TOL[dtype]:.1e}"
            errs.append(err)
    errs = np.asarray(errs)
    if dtype == "bfloat16":
        assert np.median(errs) < 3e-2 and (errs > 1e-1).sum() <= max(1, len(errs) // 20), f"{what}: median {np.median(errs):.2e}, {(errs > 1e-1).sum()} of {len(errs)} rows over 1e-1"
    return float(errs.max())


def make_folder(raw, seed, tmp):
    from kapel_b200.config import config_from_json
    from kapel_b200.weights import write_random_model

    return write_random_model(tmp, config_from_json(raw), seed)


def read_tensors(folder):
    """{name: float64 array} of a folder's model.safetensors, read with this file's own few lines."""
    blob = (folder / "model.safetensors").read_bytes()
    n = int.from_bytes(blob[:8], "little")
    header = json.loads(blob[8 : 8 + n])
    out = {}
    for name, rec in header.items():
        if name == "__metadata__":
            continue
        a, b = rec["data_offsets"]
        raw = np.frombuffer(blob[8 + n + a : 8 + n + b], dtype="<u2" if rec["dtype"] == "BF16" else "<f4")
        if rec["dtype"] == "BF16":
            raw = (raw.astype(np.uint32) << 16).view(np.float32)
        out[name] = raw.reshape(rec["shape"]).astype(np.float64)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (raw, seed) in CONFIGS.items():
        folder = make_folder(raw, seed, tmp_path_factory.mktemp(f"mukunex_{name}"))
        out[name] = (folder, raw, read_tensors(folder))
    return out


_PLAIN = {}


def plain(models, name, tokens):
    key = (name, tuple(tokens))
    if key not in _PLAIN:
        _, raw, t = models[name]
        _PLAIN[key] = PM.forward(raw, t, list(tokens))
    return _PLAIN[key]


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device="cuda").contiguous()


def bf16_round(a):
    return torch.tensor(np.asarray(a), dtype=torch.bfloat16).double().numpy()


def split_sum(rows):
    """A tensor as three split-K partial sums that add up to it exactly."""
    from kapel_b200 import kernels as K

    upper = (rows.view(torch.int32) & -4096).view(torch.float32)
    return K.SplitSum(torch.stack([upper, rows - upper, torch.zeros_like(rows)]).contiguous())


def batch_of(step):
    """(entry of every row, ranges, slots) on the device for a step [(name, slot, a, b)]."""
    from kapel_b200 import kernels as K

    entry = dev(np.concatenate([np.full(b - a, i) for i, (_, _, a, b) in enumerate(step)]), torch.int32)
    return entry, K.entry_ranges(entry, len(step)), dev([s for _, s, _, _ in step], torch.int32)


# The steps every stateful kernel below is walked through: three requests of unequal length; whole; then in portions down
# to two tokens beside each other's single tokens; a request that ends and whose slot the next one takes.
def walk(run, states, lengths):
    a, b, c = lengths["a"], lengths["b"], lengths["c"]
    run([("a", 1, 0, a), ("b", 2, 0, b)])
    for s in states:
        s.zero_()
    run([("a", 1, 0, 2), ("b", 2, 0, 30)])
    run([("b", 2, 30, 31), ("a", 1, 2, 99)])
    for i in range(6):
        run([("a", 1, 99 + 2 * i, 101 + 2 * i), ("b", 2, 31 + i, 32 + i)])
    for s in states:
        s[2].zero_()                                         # b is finished; c takes its slot
    run([("c", 2, 0, 3), ("a", 1, 111, a)])
    for i in range(3, c):
        run([("c", 2, i, i + 1)])


LENGTHS = {"a": 400, "b": 37, "c": 64}


def rows_of(data, step):
    rows = dev(np.concatenate([data[m][a:b] for m, _, a, b in step]))
    return split_sum(rows) if len(rows) <= 4 else rows


def compare(out, want, step, tol):
    at = 0
    for m, _, a, b in step:
        err = float(np.abs(out[at : at + b - a] - want[m][a:b]).max() / np.abs(want[m]).max())
        assert err < tol, f"{m}[{a}:{b}]: {err:.2e}"
        at += b - a


# -------------------------------------------------------------------------------------- attention with a sink
def paged(rng, n_tokens, page_size=16, spare=3):
    n_pages = -(-n_tokens // page_size)
    pages = rng.permutation(n_pages + spare)[:n_pages]
    lines = np.array([pages[p // page_size] * page_size + p % page_size for p in range(n_tokens)])
    return n_pages + spare, pages, lines


def plain_heads(q, k, v, scale, sinks, rows):
    """Rows `rows` of attention for q [len(rows), H, d] over k, v [T, G, .]: e^sink in every denominator."""
    H, per = q.shape[1], q.shape[1] // k.shape[1]
    out = np.zeros((len(rows), H, v.shape[2]))
    for i, r in enumerate(rows):
        for h in range(H):
            s = k[: r + 1, h // per] @ q[i, h] * scale
            top = max(s.max(), sinks[h])
            p = np.exp(s - top)
            out[i, h] = (p / (p.sum() + np.exp(sinks[h] - top))) @ v[: r + 1, h // per]
    return out


class Paged:
    """Keys and values of one request in shuffled pages, and the kernels' ways to attend to them."""

    def __init__(self, rng, k, v, dtype):
        self.n_pages, pages, lines = paged(rng, len(k))
        G, d, e = k.shape[1], k.shape[2], v.shape[2]
        self.kt = torch.zeros((self.n_pages, G, 16, d), dtype=dtype, device="cuda")
        self.vt = torch.zeros((self.n_pages, G, 16, e), dtype=dtype, device="cuda")
        where = torch.tensor(lines, device="cuda")
        self.kt[where // 16, :, where % 16] = dev(k, dtype)
        self.vt[where // 16, :, where % 16] = dev(v, dtype)
        self.bt = dev(np.concatenate([pages, [-1]])[None, :], torch.int32)
        self.dtype, self.G = dtype, G

    def rows(self, q, rows, scale, sinks):
        from kapel_b200 import kernels as K

        counts = dev(np.array(rows) + 1, torch.int32)
        entry = torch.zeros(len(rows), dtype=torch.int32, device="cuda")
        slots = max(rows) // K.attention_chunk() + 1
        return K.paged_attention_rows(dev(q, self.dtype), self.kt, self.vt, self.bt, entry, counts, 16, None, scale, None, slots,
                                      sinks=dev(sinks)).float().cpu().numpy()

    def tiles(self, q, rows, scale, sinks, split=0):
        """A run of rows as one portion of a prompt (the prompt kernel), the keys whole or in slots of `split`."""
        from kapel_b200 import kernels as K
        from kapel_b200.engine.batch import cut_tiles

        assert rows == list(range(rows[0], rows[-1] + 1))
        counts = dev(np.array(rows) + 1, torch.int32)
        cut = tuple(dev(t, torch.int32) for t in cut_tiles(np.array([0]), np.array([len(rows)]), K.attention_mma_rows(False) // (q.shape[1] // self.G)))
        slots = rows[-1] // split + 1 if split else 1
        return K.paged_attention_mma(dev(q, self.dtype), self.kt, self.vt, self.bt, counts, cut, 16, None, scale, None, 0, split if slots > 1 else 0,
                                     slots, False, sinks=dev(sinks)).float().cpu().numpy()

    def decode(self, q, rows, scale, sinks, split=0):
        """Every row a request of its own that brings one token (all share the pages), the keys whole or in slots of `split`."""
        from kapel_b200 import kernels as K

        n, per = len(rows), q.shape[1] // self.G
        counts = dev(np.array(rows) + 1, torch.int32)
        tiles = (dev(np.arange(n), torch.int32), dev(np.arange(n), torch.int32), dev(np.ones(n), torch.int32))
        slots = max(rows) // split + 1 if split else 1
        return K.paged_attention_mma(dev(q, self.dtype), self.kt, self.vt, self.bt.repeat(n, 1).contiguous(), counts, tiles, 16, None, scale, None, per,
                                     split, slots, True, sinks=dev(sinks)).float().cpu().numpy()


WAYS = ["rows f32", "rows bf16", "prompt", "prompt in slots", "decode", "decode in slots", "decode in many slots"]


def attend(way, cache, q, rows, scale, sinks):
    if way.startswith("rows"):
        return np.concatenate([cache.rows(q[i : i + 1], [r], scale, sinks) for i, r in enumerate(rows)])
    if way == "prompt":
        return cache.tiles(q, rows, scale, sinks)
    if way == "prompt in slots":
        return cache.tiles(q, rows, scale, sinks, split=128)
    split = {"decode": 0, "decode in slots": 256, "decode in many slots": 64}[way]
    return np.concatenate([cache.decode(q[i : i + 8], rows[i : i + 8], scale, sinks, split) for i in range(0, len(rows), 8)])


@pytest.mark.parametrize("way", WAYS)
@pytest.mark.parametrize("H,G,d", [(9, 3, 80), (10, 2, 64), (4, 4, 128), (16, 1, 32), (3, 1, 48)])
def test_attention_with_a_sink_on_every_kernel(way, H, G, d):
    rng = np.random.default_rng(H * d)
    dtype = torch.float32 if way == "rows f32" else torch.bfloat16
    T = 700
    k, v = rng.standard_normal((T, G, d)), rng.standard_normal((T, G, d))
    rows = list(range(600, 700)) if way.startswith("prompt") else [0, 1, 15, 16, 63, 64, 255, 256, 511, 639, 640, 699]
    q = rng.standard_normal((len(rows), H, d))
    if dtype == torch.bfloat16:
        q, k, v = bf16_round(q), bf16_round(k), bf16_round(v)
    cache = Paged(rng, k, v, dtype)
    for sinks in (rng.standard_normal(H) * 2, np.full(H, 9.0), np.full(H, -40.0)):
        want = plain_heads(q, k, v, 0.2, sinks, rows)
        assert rel_err(attend(way, cache, q, rows, 0.2, sinks), want) < (1e-5 if dtype == torch.float32 else 2e-2), sinks
    if way.startswith("prompt"):                             # the first tokens of a sequence
        rows = list(range(40))
        q = bf16_round(rng.standard_normal((40, H, d)))
        assert rel_err(attend(way, cache, q, rows, 0.2, np.full(H, 0.5)), plain_heads(q, k, v, 0.2, np.full(H, 0.5), rows)) < 2e-2


@pytest.mark.parametrize("e", [8, 24, 100])
def test_attention_with_a_sink_and_values_of_another_size(e):
    rng = np.random.default_rng(e)
    H, G, d, T = 6, 2, 16, 530
    k, v = rng.standard_normal((T, G, d)), rng.standard_normal((T, G, e))
    rows = [0, 3, 15, 16, 255, 256, 300, 529]
    q, sinks = rng.standard_normal((len(rows), H, d)), rng.standard_normal(H)
    assert rel_err(Paged(rng, k, v, torch.float32).rows(q, rows, 0.3, sinks), plain_heads(q, k, v, 0.3, sinks, rows)) < 1e-5


@pytest.mark.parametrize("way", WAYS)
def test_a_far_key_and_a_sink_that_show(way):
    """One key stands out by 20 against a query and is found wherever it lies: at the start, at page and slot borders, hundreds
    of keys back. A sink that stands out by 20 silences the head; a sink as high as the one key halves it; a head whose sink is
    far below is what it is without one."""
    rng = np.random.default_rng(3)
    dtype, tol = (torch.float32, 1e-4) if way == "rows f32" else (torch.bfloat16, 3e-2)
    H, d, T = 2, 64, 720
    rows = list(range(690, 720)) if way.startswith("prompt") else [690, 703, 704, 719]
    for target in (0, 1, 15, 16, 127, 128, 255, 256, 511, 640, 690):
        k, v = bf16_round(rng.standard_normal((T, 1, d)) * 0.2), bf16_round(rng.standard_normal((T, 1, d)))
        k[:, 0, 0] = 0.0
        k[target, 0, 0] = 1.0
        q = bf16_round(rng.standard_normal((len(rows), H, d)) * 0.1)
        q[..., 0] = 20.0
        cache = Paged(rng, k, v, dtype)
        y = attend(way, cache, q, rows, 1.0, np.array([-30.0, 40.0]))
        assert np.abs(y[:, 0] - v[target, 0]).max() < tol * 3 and np.abs(y[:, 1]).max() < 1e-5, target
        k[target, 0, 1:] = 0.0
        cache = Paged(rng, k, v, dtype)
        y = attend(way, cache, q, rows, 1.0, np.array([20.0, -30.0]))
        assert np.abs(y[:, 0] - 0.5 * v[target, 0]).max() < tol * 3 and np.abs(y[:, 1] - v[target, 0]).max() < tol * 3, target


# -------------------------------------------------------------------------------------- the other kernels alone
def test_one_gate_a_head_a_scale_and_columns_of_a_wider_output():
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(2)
    rows, heads, e = 9, 3, 20
    y, z = rng.standard_normal((rows, heads, e)), rng.standard_normal((rows, 5 + heads))
    want = (y * PM.sigmoid(z[:, 5:])[..., None]).reshape(rows, -1)
    assert rel_err(K.head_gate(dev(y), dev(z), 5, None, False, 0.0, torch.float32, by_head=True).cpu().numpy(), want) < 1e-5
    assert rel_err(K.head_gate(dev(y), split_sum(dev(z)), 5, None, False, 0.0, torch.float32, by_head=True).cpu().numpy(), want) < 1e-5
    w = rng.standard_normal((rows, 4 + heads * e))
    unit = (PM.rms_unit(y, 1e-5).reshape(rows, -1) * PM.silu(w[:, 4:])) * -0.7
    out = torch.full((rows, 3 + heads * e + 6), 7.0, device="cuda")
    K.head_gate(dev(y), dev(w), 4, None, True, 1e-5, torch.float32, gate_act="silu", scale=-0.7, out=out, column=3, pad_to=heads * e + 2)
    got = out.cpu().numpy()
    assert rel_err(got[:, 3 : 3 + heads * e], unit) < 1e-5
    assert (got[:, :3] == 7).all() and (got[:, -4:] == 7).all() and (got[:, 3 + heads * e : 5 + heads * e] == 0).all()
    with pytest.raises(K.KernelError):
        K.head_gate(dev(y), dev(z), 5, None, False, 0.0, torch.float32, by_head=True, out=out, column=12)


def test_columns_of_a_product():
    from kapel_b200 import kernels as K

    x = np.random.default_rng(1).standard_normal((7, 30))
    got = K.take_cols(dev(x), 11, 5, torch.float32, 8).cpu().numpy()
    assert np.array_equal(got[:, :5], x[:, 11:16].astype(np.float32)) and (got[:, 5:] == 0).all()
    assert rel_err(K.take_cols(split_sum(dev(x)), 25, 5, torch.bfloat16).float().cpu().numpy(), bf16_round(x[:, 25:])) < 1e-2


@pytest.mark.parametrize("channels,taps", [(40, 4), (7, 1), (1030, 2), (24, 16)])
def test_convolution_with_biases_before_and_after(channels, taps):
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(channels)
    bias, after, conv = rng.standard_normal(channels), rng.standard_normal(channels), rng.standard_normal((channels, taps))
    data = {n: rng.standard_normal((T, 3 + channels)) for n, T in LENGTHS.items()}
    want = {n: PM.short_conv(x[:, 3:] + bias, conv) + after for n, x in data.items()}
    state = torch.zeros((3, K.conv_history_floats(channels, taps)), dtype=torch.float32, device="cuda")

    def run(step):
        entry, ranges, slots = batch_of(step)
        out = K.conv_rows(rows_of(data, step), 3, channels, dev(bias), dev(conv), dev(after), state, entry, ranges, slots, len(step), taps).cpu().numpy()
        compare(out, want, step, 1e-5)

    walk(run, [state], LENGTHS)
    before = state.clone()                                   # rows of no request: zeros before them, nothing kept
    entry = dev([0, 1], torch.int32)
    out = K.conv_rows(dev(data["a"][:2]), 3, channels, dev(bias), dev(conv), dev(after), state, entry, K.entry_ranges(entry, 2), dev([0, 0], torch.int32), 2, taps)
    assert rel_err(out.cpu().numpy(), (data["a"][:2, 3:] + bias) * conv[:, -1] + after) < 1e-5 and torch.equal(before, state)


@pytest.mark.parametrize("w_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("blocks,part", [(4, 24), (1, 7), (3, 88), (2, 128), (5, 130), (30, 1)])
def test_recurrent_units_gates_in_true_32_bit(blocks, part, w_dtype):
    """Few rows and many; the weights in both dtypes, the inputs never rounded."""
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(part)
    n = blocks * part
    ra, ri = (bf16_round(rng.standard_normal((blocks, part, part)) * 2 * part ** -0.5) for _ in range(2))
    rab, rib, lam = rng.standard_normal(n), rng.standard_normal(n), rng.standard_normal(n) * 3 - 3
    for rows in (1, 3, 9, 64, 65, 200):
        u = rng.standard_normal((rows, n))
        r, i = PM.lru_gates(u, ra, rab.reshape(blocks, part), ri, rib.reshape(blocks, part))
        x = np.expm1(-8.0 * r * PM.softplus(lam))
        push = np.sqrt(-x * (x + 2.0)) * i * u
        got = K.lru_gates(dev(u), dev(ra, w_dtype), dev(ri, w_dtype), dev(rab), dev(rib), dev(lam), 8.0).cpu().numpy()
        assert np.abs(got[..., 0] / x - 1.0).max() < 2e-5, rows                          # a - 1 keeps its own precision however small it is
        assert rel_err(got[..., 1], push) < 5e-6, rows


@pytest.mark.parametrize("width", [40, 16, 7, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrent_unit_in_portions_and_token_by_token(width, dtype):
    """Runs of rows side by side (more than one round of them), a few rows one by one, portions down to two tokens, slots used again."""
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(width)
    yb, lam = rng.standard_normal(width), rng.standard_normal(width) * 2 - 4
    data, want, steps = {}, {}, {}
    for name, T in LENGTHS.items():
        u, r, i = rng.standard_normal((T, width)), rng.uniform(0, 1, (T, width)), rng.uniform(0, 1, (T, width))
        x = np.expm1(-8.0 * r * PM.softplus(lam))
        steps[name] = np.stack([x, np.sqrt(-x * (x + 2.0)) * i * u], axis=-1)
        data[name] = rng.standard_normal((T, 2 + width))
        want[name] = PM.lru_recurrence(u, r, i, lam) * PM.gelu_tanh(data[name][:, 2:] + yb)
    state = torch.zeros((3, width), dtype=torch.float32, device="cuda")

    def run(step):
        entry, ranges, slots = batch_of(step)
        ab = dev(np.concatenate([steps[m][a:b] for m, _, a, b in step]))
        longest = max(b - a for _, _, a, b in step)
        out = K.lru_scan(ab, rows_of(data, step), 2, dev(yb), state, ranges, slots, len(step), longest, dtype, pad_to=width + 3).float().cpu().numpy()
        assert np.abs(out[:, width:]).max() == 0.0
        compare(out[:, :width], want, step, 1e-5 if dtype == torch.float32 else 1e-2)

    walk(run, [state], LENGTHS)
    before = state.clone()
    for n in (3, 40):                                        # rows of no request
        entry = dev(np.zeros(n), torch.int32)
        out = K.lru_scan(dev(steps["a"][:n]), dev(data["a"][:n]), 2, dev(yb), state, K.entry_ranges(entry, 1), dev([0], torch.int32), 1, n, dtype)
        assert float(out.abs().max()) == 0.0 and torch.equal(before, state)


def test_recurrent_unit_with_a_memory_of_thousands_of_rows():
    """Decays within 1e-4 of one: after 5,000 rows the state is right to 32-bit rounding, walked in runs and row by row."""
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(4)
    T, width = 5000, 16
    x = -rng.uniform(1e-5, 1e-4, (T, width)).astype(np.float32).astype(np.float64)
    b = (np.sqrt(-x * (x + 2.0)) * rng.uniform(0.0, 2.0, (T, width))).astype(np.float32).astype(np.float64)
    S, want = np.zeros(width), np.zeros((T, width))
    for t in range(T):
        S = S + (x[t] * S + b[t])
        want[t] = S
    big = 30.0                                               # gelu(30) = 30
    for cut in (T, 9):
        state = torch.zeros((2, width), dtype=torch.float32, device="cuda")
        outs = []
        for at in range(0, T, cut):
            n = min(cut, T - at)
            ranges = K.entry_ranges(dev(np.zeros(n), torch.int32), 1)
            outs.append(K.lru_scan(dev(np.stack([x[at : at + n], b[at : at + n]], -1)), dev(np.zeros((n, width))), 0, dev(np.full(width, big)), state,
                                   ranges, dev([1], torch.int32), 1, n, torch.float32).cpu().numpy())
        assert rel_err(np.concatenate(outs) / big, want) < 1e-5, cut


@pytest.fixture
def scan_columns(request):
    from kapel_b200 import kernels as K

    K.decay_scan_columns(request.param)
    yield request.param
    K.decay_scan_columns(0)


@pytest.fixture
def chunk_rows(request):
    from kapel_b200 import kernels as K

    K.retention_chunk_rows(request.param)
    yield request.param
    K.retention_chunk_rows(-1)


# row by row with 1, 2 and 4 columns of the memory a warp; by chunks whatever a portion's length; the launchers' own choices
@pytest.mark.parametrize("scan_columns,chunk_rows", [(1, 0), (2, 0), (4, 0), (0, 1), (0, -1)], indirect=True)
@pytest.mark.parametrize("H,d,e,rotary", [(2, 24, 8, 24), (1, 8, 40, 2), (3, 40, 16, 10), (2, 130, 5, 130), (4, 48, 64, 0), (2, 128, 128, 64), (3, 64, 200, 64)])
def test_retention_in_portions_and_token_by_token(H, d, e, rotary, scan_columns, chunk_rows):
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(d + e)
    nq, nv = H * d, H * e
    decay = ([0.998046875, 0.75, 1.0, 0.0])[:H] if H > 1 else [0.984375]
    rot = {"base": 70.0, "dims": rotary}
    data, want = {}, {}
    for name, T in LENGTHS.items():
        x = rng.standard_normal((T, 3 + 2 * nq + nv))
        data[name] = x
        q, k = x[:, 3 : 3 + nq].reshape(T, H, d), x[:, 3 + nq : 3 + 2 * nq].reshape(T, H, d)
        if rotary:
            q, k = (PM.rotate_halves(z, np.arange(T), rot) for z in (q, k))
        v = x[:, 3 + 2 * nq :].reshape(T, H, e)
        want[name] = np.stack([PM.retention_recurrence(q[:, h], k[:, h] * d ** -0.5, v[:, h], decay[h]) for h in range(H)], axis=1)
    state = torch.zeros((3, nq * e), dtype=torch.float32, device="cuda")

    def run(step):
        entry, ranges, slots = batch_of(step)
        positions = dev(np.concatenate([np.arange(a, b) for _, _, a, b in step]), torch.int32)
        table = K.rope_table(positions, rotary, 70.0) if rotary else None
        out = K.retention_scan(rows_of(data, step), 3, 3 + nq, 3 + 2 * nq, dev(decay), table, rotary, d ** -0.5, state, ranges, slots, len(step),
                               max(b - a for _, _, a, b in step), H, d, e).cpu().numpy()
        compare(out, want, step, 5e-5)

    walk(run, [state], LENGTHS)
    before = state.clone()                                   # rows of no request
    entry = dev(np.zeros(70), torch.int32)
    table = K.rope_table(dev(np.arange(70), torch.int32), rotary, 70.0) if rotary else None
    out = K.retention_scan(dev(data["a"][:70]), 3, 3 + nq, 3 + 2 * nq, dev(decay), table, rotary, d ** -0.5, state, K.entry_ranges(entry, 1),
                           dev([0], torch.int32), 1, 70, H, d, e)
    assert float(out.abs().max()) == 0.0 and torch.equal(before, state)


@pytest.mark.parametrize("scan_columns", [0, 1, 2, 4], indirect=True)
@pytest.mark.parametrize("H,G,d,e,taps,rank", [(4, 2, 24, 16, 2, 7), (1, 1, 16, 40, 1, 3), (3, 3, 8, 24, 4, 20), (2, 1, 130, 9, 16, 5), (4, 1, 64, 64, 4, 24)])
def test_delta_rule_with_a_decay_a_channel_in_portions_and_token_by_token(H, G, d, e, taps, rank, scan_columns):
    from kapel_b200 import kernels as K

    rng = np.random.default_rng(d)
    nq, nv, n = G * d, H * e, H * d
    channels = 2 * nq + nv
    a2, dt, alog, conv = rng.standard_normal((n, rank)), rng.standard_normal(n), rng.standard_normal(H), rng.standard_normal((channels, taps))
    data, want = {}, {}
    for name, T in LENGTHS.items():
        x = rng.standard_normal((T, 2 + channels + H + rank))
        data[name] = x
        c = PM.silu(PM.short_conv(x[:, 2 : 2 + channels], conv))
        q, k = PM.unit_vectors(c[:, :nq].reshape(T, G, d)) * d ** -0.5, PM.unit_vectors(c[:, nq : 2 * nq].reshape(T, G, d))
        v = c[:, 2 * nq :].reshape(T, H, e)
        beta = PM.sigmoid(x[:, 2 + channels : 2 + channels + H])
        g = np.exp(-np.exp(alog)[None, :, None] * PM.softplus(x[:, 2 + channels + H :] @ a2.T + dt).reshape(T, H, d))
        want[name] = np.stack([PM.channel_delta_recurrence(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], g[:, h], beta[:, h]) for h in range(H)], axis=1)
    history = torch.zeros((3, K.conv_history_floats(channels, taps)), dtype=torch.float32, device="cuda")
    memory = torch.zeros((3, n * e), dtype=torch.float32, device="cuda")

    def scan(rows, entry, ranges, slots, entries):
        return K.cdelta_scan(rows, 2, 2 + channels, 2 + channels + H, dev(a2.T), dev(dt), dev(alog), dev(conv), history, memory, entry, ranges, slots,
                             entries, H, G, d, e, taps, d ** -0.5, 1e-6)

    def run(step):
        entry, ranges, slots = batch_of(step)
        compare(scan(rows_of(data, step), entry, ranges, slots, len(step)).cpu().numpy(), want, step, 5e-5)

    walk(run, [history, memory], LENGTHS)
    before = history.clone(), memory.clone()                 # rows of no request
    entry = dev([0, 1, 2, 3], torch.int32)
    out = scan(dev(data["a"][:4]), entry, K.entry_ranges(entry, 4), dev([0, 0, 0, 0], torch.int32), 4)
    assert float(out.abs().max()) == 0.0 and torch.equal(before[0], history) and torch.equal(before[1], memory)


# -------------------------------------------------------------------------------------- the engine
def engine_for(models, name, dtype, **kw):
    from kapel_b200.engine import Engine

    kw.setdefault("max_tokens", 1024)
    kw.setdefault("max_sequences", 4)
    return Engine.from_dir(models[name][0], dtype=dtype, **kw)


def test_the_states_the_shared_product_and_the_sizes_the_tensors_give(models, tmp_path):
    import shutil
    from kapel_b200.engine import Engine

    eng = engine_for(models, "A", "float32")
    assert sorted(str(k) for k in eng.cache.states) == sorted(str(k) for k in (0, (0, "conv"), (1, "right"), 2, (2, "conv"), 3, (3, "conv")))
    mixer = eng.model.blocks[1].mixer                        # one product for both sides, one output product over both
    assert mixer.w_in.shape == (6 * 16 + 2 * 16 + 2 * 24 + 6 + 2 * 24 * 2 + 2 * 8 * 2, 64) and mixer.w_o.shape == (64, 6 * 24 + 2 * 8)
    folder = tmp_path / "bare"                               # a config.json without the ranks: the tensors' shapes have them
    shutil.copytree(models["A"][0], folder)
    raw = json.loads((folder / "config.json").read_text())
    for layer in raw["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    (folder / "config.json").write_text(json.dumps(raw))
    m = Engine.from_dir(folder, dtype="float32", max_tokens=256, max_sequences=2).config.layers[2].mixer
    assert (m.decay_rank, m.gate_rank) == (7, 12)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts_portions_and_decoding_against_plain(models, name, dtype):
    """A prompt whole; the same prompt in portions of changing size down to two tokens and then token by token (a long decoding that
    crosses pages); logits at every position."""
    raw = models[name][1]
    tokens = random_tokens(np.random.default_rng(7), 220, raw["vocab"])
    want = {"w": plain(models, name, tokens), "p": plain(models, name, tokens)}
    eng = engine_for(models, name, dtype)
    tb = TraceBuilder()
    tb.step([("w", tokens, range(len(tokens)))], end=["w"])
    at = 0
    for n in (2, 17, 3, 2, 40, 5, 65):
        tb.step([("p", tokens[at : at + n], range(n))])
        at += n
    while at < len(tokens):
        tb.step([("p", tokens[at : at + 1], [0])], end=(["p"] if at + 1 == len(tokens) else []))
        at += 1
    worst = check_rows(run_trace_engine(eng, tb.steps), tb, want, dtype, f"{name} {dtype}")
    print(f"mukunex {name} {dtype}: worst {worst:.2e}")
    assert eng.cache.free_pages() == eng.cache.total_pages() and eng.cache.free_slots() == 4


@pytest.mark.parametrize("name", ["A", "C"])
def test_the_residual_after_every_layer_against_plain(models, name):
    from kapel_b200.engine import StepEntry

    folder, raw, t = models[name]
    tokens = random_tokens(np.random.default_rng(1), 150, raw["vocab"])
    plain_runs = []
    PM.forward(raw, t, tokens, plain_runs)
    eng = engine_for(models, name, "float32")
    seen = []
    eng.model.tap = lambda i, x: seen.append(x.detach().cpu().numpy().copy())
    eng.step([StepEntry("r", tokens, [])])
    assert len(seen) == len(plain_runs) == 4
    for i, (got, want) in enumerate(zip(seen, plain_runs)):
        assert rel_err(got, want) < 2e-5, f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_mixed_batches_and_reused_slots_against_each_alone(models, name, dtype):
    """Up to four unequal requests a step, portions beside single tokens, a request left out of a step, requests that end
    and whose pages and slots the next ones take; a pool of few pages."""
    raw = models[name][1]
    rng = np.random.default_rng(8)
    reqs = {k: random_tokens(rng, n, raw["vocab"]) for k, n in dict(a=250, b=41, c=23, d=70, e=33, f=18).items()}
    want = {k: plain(models, name, v) for k, v in reqs.items()}
    eng = engine_for(models, name, dtype, max_tokens=64 * 3 + 256 + 64)
    tb = TraceBuilder()
    fed = {k: 0 for k in reqs}

    def take(k, n, want_all=True):
        a = fed[k]
        n = min(n, len(reqs[k]) - a)
        fed[k] += n
        return (k, reqs[k][a : a + n], list(range(n)) if want_all else [n - 1])

    done = lambda k: fed[k] == len(reqs[k])
    tb.step([take("a", 30), take("b", 2), take("c", 23)], end=["c"])
    tb.step([take("a", 1), take("b", 20), take("d", 17)])
    tb.step([take("b", 1), take("d", 2), take("e", 33, False)], end=["e"])            # a is left out of this step
    tb.step([take("d", 1), take("a", 190), take("b", 1), take("f", 5)])
    while not all(done(k) for k in "abdf"):
        entries = [take(k, 1) for k in "abdf" if not done(k)]
        tb.step(entries, end=[k for k, _, _ in entries if done(k)])
    worst = check_rows(run_trace_engine(eng, tb.steps), tb, want, dtype, f"{name} {dtype}")
    print(f"mukunex mixed {name} {dtype}: worst {worst:.2e}")
    eng.cache.check()
    assert eng.cache.free_pages() == eng.cache.total_pages() and eng.cache.free_slots() == 4


def test_recorded_passes_leave_the_state_as_eager_ones_do(models):
    """A prompt pass of a shape seen before and a decoding pass go through recordings, whose first eager run must not
    advance the memories, the unit's state or the convolutions' history a second time."""
    raw = models["C"][1]
    outs = []
    for graphs in (False, True):
        eng = engine_for(models, "C", "float32", graphs=graphs)
        tb = TraceBuilder()
        for k in ("x", "y", "z"):
            tokens = random_tokens(np.random.default_rng(ord(k)), 150, raw["vocab"])
            tb.step([(k, tokens[:140], [139])])
            for i in range(140, 150):
                tb.step([(k, tokens[i : i + 1], [0])], end=([k] if i == 149 else []))
        outs.append(run_trace_engine(eng, tb.steps))
        if graphs:
            assert eng.recorded_passes > 0
    for step in outs[0]:
        assert rel_err(outs[1][step], outs[0][step]) < 2e-6, f"step {step}"


ODD = {"architecture": "Mukunex", "vocab": 77, "width": 52, "norm": {"eps": 1e-6}, "layers": [
    lru_layer(33, 3, 5, dense(19)),
    parallel_layer(3, 1, 10, 7, 0.3, rotation(60.0, 6, (2.0, 1.0, 2.0, 30)), 3, 6, 11, [0.9, 0.5, 0.99], rotation(40.0, 2), 0.9, 1.2, None),
    delta_layer(3, 1, 10, 7, 3, 9, 3, dense(13)),
    parallel_layer(34, 2, 16, 16, 0.25, rotation(60.0, 16), 1, 9, 5, [0.95], rotation(40.0, 8), 1.5, 0.3, dense(21))]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_no_multiples_of_eight(dtype, tmp_path):
    """Nor anything else; and 17 query heads a kv head, more than the tensor-core attention takes."""
    from kapel_b200.engine import Engine

    folder = make_folder(ODD, 6, tmp_path)
    t = read_tensors(folder)
    eng = Engine.from_dir(folder, dtype=dtype, max_tokens=512, max_sequences=4)
    tokens = random_tokens(np.random.default_rng(3), 165, ODD["vocab"])
    want = {"a": PM.forward(ODD, t, tokens)}
    tb = TraceBuilder()
    tb.step([("a", tokens[:140], range(140))])
    tb.step([("a", tokens[140:143], range(3))])
    for i in range(143, 165):
        tb.step([("a", tokens[i : i + 1], [0])], end=(["a"] if i == 164 else []))
    check_rows(run_trace_engine(eng, tb.steps), tb, want, dtype, f"odd {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_prompt_longer_than_the_attention_kernels_chunks(models, dtype):
    """700 tokens: the row-wise kernel's and the tensor-core kernels' key slots are merged with the sink; portions that start in the
    middle of a chunk; then single tokens beside another request."""
    raw = models["C"][1]
    tokens = random_tokens(np.random.default_rng(12), 700, raw["vocab"])
    short = random_tokens(np.random.default_rng(13), 30, raw["vocab"])
    want = {"a": plain(models, "C", tokens), "b": plain(models, "C", short)}
    eng = engine_for(models, "C", dtype)
    tb = TraceBuilder()
    tb.step([("a", tokens[:300], [0, 1, 63, 64, 255, 256, 299])])
    tb.step([("b", short[:20], [19]), ("a", tokens[300:690], [0, 29, 211, 212, 389])])
    for i in range(690, 700):
        tb.step([("a", tokens[i : i + 1], [0]), ("b", short[i - 670 : i - 669], [0])], end=(["a", "b"] if i == 699 else []))
    check_rows(run_trace_engine(eng, tb.steps), tb, want, dtype, "long")


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_through_the_entry_point_and_scheduler(models, name):
    import kapel_b200

    folder, raw, t = models[name]
    rng = np.random.default_rng(10)
    prompts = [random_tokens(rng, n, raw["vocab"]) for n in (3, 29, 75)]

    def plain_greedy(prompt, n):
        seq, margins = list(prompt), []
        for _ in range(n):
            row = PM.forward(raw, t, seq)[-1]
            order = np.argsort(row)
            margins.append(float(row[order[-1]] - row[order[-2]]))
            seq.append(int(order[-1]))
        return seq[len(prompt):], margins

    want = [plain_greedy(p, 12) for p in prompts]
    model = kapel_b200.Model(str(folder), dtype="f32", max_tokens_cached=1024, max_sequences=4, max_pass_tokens=32)
    for p, (tokens, margins) in zip(prompts, want):
        safe = next((i for i, m in enumerate(margins) if m < 1e-3), len(margins))
        assert model.generate(p, max_tokens=12)[:safe] == tokens[:safe]
    together = model.generate_batch(prompts, max_tokens=12)
    for got, (tokens, margins) in zip(together, want):
        safe = next((i for i, m in enumerate(margins) if m < 1e-3), len(margins))
        assert got[:safe] == tokens[:safe]
    assert model.engine.cache.free_pages() == model.engine.cache.total_pages()


def test_replay_program_and_command_line(models, tmp_path):
    import subprocess
    import sys

    import kapel_b200
    from helpers import ROOT

    folder, raw, _ = models["A"]
    tokens = random_tokens(np.random.default_rng(4), 40, raw["vocab"])
    want = plain(models, "A", tokens)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": tokens[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": tokens[33:35], "want": []}], "end": []},
             {"step": 5, "entries": [{"id": "q", "tokens": tokens[35:], "want": [4]}], "end": ["q"]}]
    out = tmp_path / "logits"
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(x) + "\n" for x in steps), capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == ["done 0", "done 1", "done 5"]
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, raw["vocab"])
    last = np.fromfile(out / "5.f32", dtype="<f4").reshape(1, raw["vocab"])
    assert rel_err(first, want[[0, 32]]) < TOL["float32"] and rel_err(last, want[[39]]) < TOL["float32"]

    model = kapel_b200.Model(str(folder), dtype="f32", max_tokens_cached=256, max_sequences=2)
    expect = model.generate(tokens[:9], max_tokens=6)
    r = subprocess.run([sys.executable, "-m", "kapel_b200", "run", str(folder), "--tokens", ",".join(map(str, tokens[:9])), "--max-tokens", "6",
                        "--greedy", "--dtype", "f32"], capture_output=True, text=True, timeout=900, cwd=str(ROOT))
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.strip().splitlines()[0].split(",")] == expect
