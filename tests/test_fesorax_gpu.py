"""The Fesorax design in the engine against its plain implementation (tests/plain/fesorax_plain.py).

First every mechanism alone through its kernels (attention over a window beside which the first tokens stay visible, with a
bias by distance and a gate per head; the norm of q and k without a weight; the matrix memory token by token and in
chunks, its state in slots; logistic routing and gated experts weighed at their input), with inputs made so that a key one
position off, a lost state or a weight in the wrong place shows; then whole models of six small configurations that
differ in every size, order and option, cut and batched in every way, in both number formats.
"""
import json
import os
import random

import numpy as np
import pytest
import torch

from helpers import batch_index, rel_error
from plain import fesorax_plain as plain

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KERNEL_TOL = {"float32": 2e-5, "bfloat16": 2e-2}
MODEL_TOL = {"float32": 3e-5, "bfloat16": 4e-2}


def _att(heads, kv_heads, dim, vdim, scale, bias_max, mask=None, kv_from=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max}
    if mask is not None:
        out["mask"] = {"size": mask[0], "keep_first": mask[1]}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return {"type": "attention", "mixer": out}


def _mem(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _moe(ff, limit, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def _config(vocab, width, eps, alpha, layers, scale=None):
    out = {"architecture": "Fesorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
           "layers": [{**mixer, "mlp": mlp} for mixer, mlp in layers]}
    if scale is not None:
        out["embedding"] = {"scale": scale}
    return out


def _configs():
    return {
        # a reader whose window and kept tokens reach further than those of the layer whose keys it reads, one without
        # any mask, a layer without feed-forward
        "A": _config(210, 96, 1e-5, 1.7, [
            (_att(6, 3, 16, 24, 0.5, 70.0, mask=(40, 5)), _moe(32, 1.5, 6, 2, shared=(48, 0.9))),
            (_mem(4, 32, 48, 9.0), _moe(32, 2.5, 6, 2, shared=(48, 1.1))),
            (_att(9, 3, 16, 24, 0.4, 33.0, mask=(90, 21), kv_from=0), _moe(40, 1.2, 5, 3, shared=(24, 3.0))),
            (_att(2, 1, 48, 16, 0.2, 100.0), None),
            (_att(3, 1, 48, 16, 0.2, 50.0, mask=(25, 0), kv_from=3), _moe(24, 0.8, 4, 1)),
            (_mem(2, 16, 64, 5.0), None)], scale=3.0),
        # what other models keep apart is equal or 1 here: as many kv heads as heads, keys as large as values, one expert
        # chosen, no kept tokens, a window of one page, no shared expert, alpha 1, no embedding scale
        "B": _config(128, 64, 1e-6, 1.0, [
            (_att(2, 2, 32, 32, 0.18, 33.0, mask=(64, 0)), _moe(64, 7.0, 2, 1)),
            (_mem(1, 16, 16, 15.0), _moe(64, 7.0, 1, 1)),
            (_att(2, 2, 32, 32, 0.18, 33.0, mask=(64, 0), kv_from=0), _moe(32, 7.0, 3, 3))]),
        # nothing a multiple of 8
        "C": _config(97, 100, 2e-5, 2.2, [
            (_mem(5, 12, 10, 7.5), _moe(18, 1.3, 5, 2, shared=(30, 2.0))),
            (_att(3, 1, 20, 12, 0.3, 17.5, mask=(17, 3)), _moe(22, 0.9, 7, 3, shared=(14, 1.0))),
            (_att(5, 1, 20, 12, 0.35, 40.0, mask=(31, 7), kv_from=1), _moe(18, 1.1, 5, 4)),
            (_mem(3, 21, 17, 4.0), _moe(18, 1.3, 5, 1, shared=(31, 2.0)))], scale=1.3),
        # heads of 64 (the kernels fed by TMA and the tcgen05 ones), large memories, many experts
        "D": _config(300, 128, 1e-6, 2.0, [
            (_att(8, 2, 64, 64, 0.15, 200.0, mask=(96, 33)), _moe(64, 2.0, 24, 4, shared=(64, 1.0))),
            (_mem(4, 128, 128, 12.0), _moe(64, 2.0, 24, 4, shared=(64, 1.0))),
            (_att(8, 2, 64, 64, 0.15, 60.0, mask=(70, 130), kv_from=0), _moe(64, 2.0, 16, 2, shared=(64, 1.0)))], scale=2.0),
        # many query heads to a kv head, head sizes that only the mma.sync kernels take, two readers of one layer
        "E": _config(250, 160, 1e-6, 3.0, [
            (_att(16, 2, 96, 80, 0.08, 40.0, mask=(50, 20)), _moe(40, 1.5, 32, 6, shared=(56, 1.5))),
            (_att(8, 2, 96, 80, 0.1, 90.0, mask=(128, 64), kv_from=0), _moe(40, 1.5, 32, 6, shared=(56, 1.5))),
            (_mem(2, 64, 96, 10.0), _moe(40, 1.5, 32, 6, shared=(56, 1.5))),
            (_att(4, 2, 96, 80, 0.1, 64.0, mask=(1, 1), kv_from=0), None)], scale=0.9),
        # heads of 128, a window of a few positions over many kept ones, memories with long keys and short values
        "F": _config(150, 96, 1e-5, 1.5, [
            (_att(4, 1, 128, 128, 0.08, 100.0, mask=(9, 140)), _moe(48, 1.0, 8, 2, shared=(32, 1.0))),
            (_mem(2, 200, 24, 6.0), _moe(48, 1.0, 8, 2, shared=(32, 1.0)))], scale=1.1),
    }


CONFIGS = _configs()
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64, "E": 65, "F": 66}


@pytest.fixture(scope="module")
def ops():
    from aegean_tge_b200 import ops as module
    module.core()
    return module


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from aegean_tge_b200 import write_random_model
    out = {}
    for name, config in CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"fesorax_{name}")
        write_random_model(str(folder), config, seed=SEEDS[name], dtype="float32")
        out[name] = str(folder)
    return out


def _read_weights(folder):
    with open(os.path.join(folder, "model.safetensors"), "rb") as handle:
        size = int.from_bytes(handle.read(8), "little")
        header = json.loads(handle.read(size))
        data = handle.read()
    out = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        assert entry["dtype"] == "F32", (name, entry["dtype"])
        begin, end = entry["data_offsets"]
        out[name] = np.frombuffer(data[begin:end], dtype="<f4").reshape(entry["shape"]).copy()
    return out


def _to_bfloat16(array):
    return torch.from_numpy(np.ascontiguousarray(array)).to(torch.bfloat16).float().numpy()


_WEIGHTS = {}


def _weights(folders, name, dtype):
    if (name, dtype) not in _WEIGHTS:
        from aegean_tge_b200 import architecture_of
        arch = architecture_of(CONFIGS[name])
        matrices = {tensor for tensor, _shape, role, _draw in arch.random_plan(arch.parse_config(CONFIGS[name])) if role == "matrix"}
        w = _read_weights(folders[name])
        if dtype == "bfloat16":         # matrices are held in bfloat16, vectors (taps, biases, tables, norms) in float32
            w = {k: (_to_bfloat16(v) if k in matrices else v) for k, v in w.items()}
        _WEIGHTS[(name, dtype)] = {k: v.astype(np.float64) for k, v in w.items()}
    return _WEIGHTS[(name, dtype)]


@pytest.fixture(scope="module")
def oracle(folders):
    """oracle(name, dtype, tokens) -> logits; oracle.margin(name, dtype, tokens) -> [T], every row's smallest distance
    from another choice of experts over all routed layer runs."""
    cache = {}

    def both(name, dtype, tokens, config=None):
        key = (name, dtype, tuple(tokens), json.dumps(config, sort_keys=True) if config else "")
        if key not in cache:
            margins = []
            logits = plain.forward(config or CONFIGS[name], _weights(folders, name, dtype), list(tokens), margins=margins)
            smallest = np.min(np.stack(margins), axis=0) if margins else np.full(len(tokens), np.inf)
            cache[key] = (torch.from_numpy(logits).float(), smallest)
        return cache[key]

    def get(name, dtype, tokens, config=None):
        return both(name, dtype, tokens, config)[0]
    get.margin = lambda name, dtype, tokens: both(name, dtype, tokens)[1]

    def following(name, dtype, tokens, choices):
        margins = []
        logits = plain.forward(CONFIGS[name], _weights(folders, name, dtype), list(tokens), margins=margins, choices=choices)
        worst = min((float(m.min()) for m in margins), default=0.0)
        assert worst > -CLOSE_CALL, (name, dtype, "an expert was chosen whose logit lies far below another's", worst)
        return torch.from_numpy(logits).float()
    get.following = following
    return get


# In bfloat16 a rounding can send a row to other experts when two router logits lie close together.  So the engine's
# choices are recorded (``_Run``) and the oracle takes the same experts, with its own scores; a choice that is not the
# oracle's own must have been a close call.
CLOSE_CALL = 0.1


def _agree(got, oracle, name, dtype, tokens, rows=None, where="", choices=None):
    """``got``: logits of ``rows`` (default: all) of the sequence ``tokens``; ``choices``: the experts the engine took."""
    ref = oracle(name, dtype, tokens) if choices is None else oracle.following(name, dtype, tokens, choices)
    rows = list(range(len(tokens))) if rows is None else list(rows)
    scale = float(ref.abs().max())
    ref = ref[rows]
    got = got.detach().float().cpu()
    assert got.shape == ref.shape and torch.isfinite(got).all()
    error = (got - ref).abs().max(dim=1).values / scale
    if dtype == "bfloat16" and choices is None:
        # nothing was recorded: rows before the request's first close call must agree
        close = np.nonzero(oracle.margin(name, dtype, tokens) < 3e-2)[0]
        error = error[[n for n, r in enumerate(rows) if not len(close) or r < close[0]]]
        if not len(error):
            return
    assert float(error.max()) < MODEL_TOL[dtype], (name, dtype, where, int(error.argmax()), float(error.max()))


class _Run:
    """An engine's step function, with the experts every request was sent to.  Recording needs steps that are not replayed
    from a graph; in float32 nothing is recorded and graphs are used."""

    def __init__(self, engine, dtype):
        self.engine, self.record, self.taken = engine, dtype == "bfloat16", {}
        if self.record:
            engine.runner.use_graphs = False

    def step(self, portions):
        """portions: [(request, tokens)] -> logits of every token"""
        from aegean_tge_b200.parts.routed_mlp import RoutedExperts
        seen, route = [], RoutedExperts.route

        def recording(part, h):
            chosen = route(part, h)
            seen.append(chosen[0].cpu().numpy())
            return chosen
        if self.record:
            RoutedExperts.route = recording
        try:
            logits = self.engine.runner.step([_portion(r, tokens) for r, tokens in portions])
        finally:
            RoutedExperts.route = route
        at = 0
        for r, tokens in portions:
            self.taken.setdefault(r, []).append([ids[at:at + len(tokens)] for ids in seen])
            at += len(tokens)
        return logits

    def choices(self, request):
        if not self.record:
            return None
        return [np.concatenate(layer) for layer in zip(*self.taken[request])]


def _tokens(name, count, salt=0):
    rnd = random.Random(SEEDS[name] * 1000 + salt)
    return [rnd.randrange(CONFIGS[name]["vocab"]) for _ in range(count)]


def _engine(folders, name, dtype, **kw):
    from aegean_tge_b200 import Engine
    kw.setdefault("context", 512)
    kw.setdefault("max_tokens", 1024)
    kw.setdefault("max_requests", 8)
    return Engine(folders[name], dtype=dtype, **kw)


def _portion(request, tokens, want=None):
    from aegean_tge_b200.engine import Portion
    return Portion(request, tokens, list(range(len(tokens))) if want is None else want)


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _f32(array):
    return torch.from_numpy(np.ascontiguousarray(array, dtype=np.float32)).to(DEV)


# ---------------------------------------------------------------------------
# mechanisms, one by one
def _scattered(lengths, kv_heads, dim, vdim, page, dtype, seed):
    """Random keys and values of requests of the given lengths on shuffled pages: (k pages, v pages, table, k list, v list)."""
    gen = torch.Generator().manual_seed(seed)
    need = [-(-n // page) for n in lengths]
    order = torch.randperm(sum(need) + 3, generator=gen).tolist()
    k_pages = torch.randn(sum(need) + 3, kv_heads, page, dim, generator=gen).to(dtype)
    v_pages = torch.randn(sum(need) + 3, kv_heads, page, vdim, generator=gen).to(dtype)
    table = torch.full((len(lengths), max(need)), -1, dtype=torch.int32)
    ks, vs = [], []
    for s, n in enumerate(lengths):
        k = torch.randn(n, kv_heads, dim, generator=gen).to(dtype)
        v = torch.randn(n, kv_heads, vdim, generator=gen).to(dtype)
        for j in range(need[s]):
            table[s, j] = order.pop()
            part = slice(j * page, min((j + 1) * page, n))
            k_pages[table[s, j], :, :part.stop - part.start] = k[part].transpose(0, 1)
            v_pages[table[s, j], :, :part.stop - part.start] = v[part].transpose(0, 1)
        ks.append(k)
        vs.append(v)
    return k_pages.to(DEV), v_pages.to(DEV), table.to(DEV), ks, vs


def _hide(table, s, start, page, window, keep):
    """Takes the pages away that no query at position ``start`` or later may read."""
    for j in range(table.shape[1]):
        if j * page >= keep and (j + 1) * page <= start - window + 1:
            table[s, j] = -1


SHAPES = [(16, 24, 16), (64, 64, 64), (64, 64, 16), (128, 128, 64), (128, 128, 32), (48, 48, 16), (96, 80, 64), (256, 256, 64), (20, 12, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim,page", SHAPES)
@pytest.mark.parametrize("window,keep", [(40, 5), (70, 64), (1, 1), (64, 100), (17, 0), (130, 33), (500, 20)])
def test_window_with_kept_tokens_bias_and_gate(ops, dtype, dim, vdim, page, window, keep):
    """Prompts, single tokens and mixed steps, keys cut into runs or not, pages behind the window taken away: every kernel
    that attends, against the plain softmax.  The bias's rows differ by several units, so a distance one off shows."""
    from aegean_tge_b200.parts.attention import GQAttention
    heads, kv_heads, scale, rows, far = 6, 2, 2.0 * dim ** -0.5, 16, 90.0
    rng = np.random.default_rng(dim + window)
    rel = rng.permutation(rows * heads).reshape(rows, heads).astype(np.float64) * 0.15
    table_bias = GQAttention.expand_distance_bias(torch.from_numpy(rel).float(), far).to(DEV)
    lengths = [275, 41, 150]
    k_pages, v_pages, full_table, ks, vs = _scattered(lengths, kv_heads, dim, vdim, page, TORCH[dtype], seed=dim + window)
    gate_all = [torch.randn(n, heads + 2, generator=torch.Generator().manual_seed(n)).to(TORCH[dtype]) for n in lengths]
    q_all = [torch.randn(n, heads * dim, generator=torch.Generator().manual_seed(7 + n)).to(TORCH[dtype]) for n in lengths]
    refs = []
    for s, n in enumerate(lengths):
        a = plain.attend(q_all[s].double().numpy().reshape(n, heads, dim), ks[s].double().numpy(), vs[s].double().numpy(), scale,
                         rel, far, window, keep)
        refs.append((a * plain.sigmoid(gate_all[s][:, :heads].double().numpy())[:, :, None]).reshape(n, -1))
    steps = [(lengths, 0), ([1, 1, 1], 0), ([60, 2, 1], 0), ([1, 1, 1], 64), ([33, 40, 3], 128), ([1, 1, 1], 128)]
    for new, split in steps:
        starts = [n - m for n, m in zip(lengths, new)]
        table = full_table.clone()
        for s in range(3):
            _hide(table, s, starts[s], page, window, keep)
        positions, seq, q_start, start_pos = batch_index(new, starts, DEV)
        q = torch.cat([q_all[s][starts[s]:] for s in range(3)]).to(DEV)
        gate = torch.cat([gate_all[s][starts[s]:] for s in range(3)]).to(DEV)[:, :heads]
        got = ops.attention(q, k_pages, v_pages, table, q_start, start_pos, positions, seq, 3, max(new), max(lengths), heads, kv_heads,
                            dim, scale, window=window, keep_first=keep, split_tokens=split, dist_bias=table_bias, gate=gate)
        ref = np.concatenate([refs[s][starts[s]:] for s in range(3)])
        assert rel_error(got, torch.from_numpy(ref)) < KERNEL_TOL[dtype], (new, split)
    # leading single tokens beside a portion take the decode kernel
    new = [1] * 40 + [200]
    lengths2 = [100 + 3 * i for i in range(40)] + [260]
    k_pages, v_pages, table, ks, vs = _scattered(lengths2, kv_heads, dim, vdim, page, TORCH[dtype], seed=1)
    starts = [n - m for n, m in zip(lengths2, new)]
    positions, seq, q_start, start_pos = batch_index(new, starts, DEV)
    q = torch.randn(sum(new), heads * dim, generator=torch.Generator().manual_seed(9)).to(TORCH[dtype])
    got = ops.attention(q.to(DEV), k_pages, v_pages, table, q_start, start_pos, positions, seq, len(new), 200, max(lengths2), heads,
                        kv_heads, dim, scale, window=window, keep_first=keep, dist_bias=table_bias, decode_prefix=40)
    for s in (0, 21, 39):
        full = np.zeros((lengths2[s], heads, dim))
        full[-1] = q[s].double().numpy().reshape(heads, dim)
        ref = plain.attend(full, ks[s].double().numpy(), vs[s].double().numpy(), scale, rel, far, window, keep)[-1]
        assert rel_error(got[s], torch.from_numpy(ref.reshape(-1))) < KERNEL_TOL[dtype], s


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,page", [(32, 16), (64, 64), (128, 16)])
def test_one_key_just_inside_or_outside_what_is_seen(ops, dtype, dim, page):
    """A key made to dominate its query sits at the last kept token, the first one not kept, the window's oldest position and
    the one before it: the row is that key's value exactly if it is seen, decoded alone and as the end of a portion."""
    heads, kv_heads, n, window, keep = 2, 1, 300, 75, 21
    flat = torch.zeros(heads, 1, device=DEV)
    for place, seen in ((0, True), (keep - 1, True), (keep, False), (150, False), (n - window - 1, False), (n - window, True), (n - 1, True)):
        for new in (1, 2, 150):
            k_pages, v_pages, table, ks, vs = _scattered([n], kv_heads, dim, dim, page, TORCH[dtype], seed=place)
            key = ks[0][place, 0].float()
            q = torch.zeros(new, heads * dim)
            q[-1] = (key * (60.0 / float(key @ key))).repeat(heads)
            positions, seq, q_start, start_pos = batch_index([new], [n - new], DEV)
            got = ops.attention(q.to(TORCH[dtype]).to(DEV), k_pages, v_pages, table, q_start, start_pos, positions, seq, 1, new, n, heads,
                                kv_heads, dim, 1.0, window=window, keep_first=keep, dist_bias=flat)
            error = rel_error(got[-1].float().cpu().reshape(heads, dim), vs[0][place, 0].float().repeat(heads, 1))
            assert (error < 2 * KERNEL_TOL[dtype]) == seen, (place, new, error)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,pad", [(4, 2, 16, 24, 8), (3, 1, 20, 12, 1), (28, 4, 128, 128, 4), (9, 3, 48, 80, 16), (6, 0, 64, 32, 2),
                                                        (5, 0, 20, 12, 0)])
def test_norm_without_a_weight_and_store(ops, dtype, heads, kv_heads, dim, vdim, pad):
    """q and k over their root mean square per head, keys and values into their pages; no kv heads: queries alone.  What
    lies behind them in the rows stays."""
    rng = np.random.default_rng(dim)
    page, n, first = 16, 37, 59
    width = heads * dim + kv_heads * (dim + vdim) + pad
    rows = torch.from_numpy(rng.standard_normal((n, width)) * 2).to(TORCH[dtype])
    raw = rows.double().numpy()
    ones = torch.ones(dim, device=DEV)
    pages = 8
    k_pages = torch.zeros(pages, max(kv_heads, 1), page, dim, dtype=TORCH[dtype], device=DEV)
    v_pages = torch.zeros(pages, max(kv_heads, 1), page, vdim, dtype=TORCH[dtype], device=DEV)
    table = _i32([[5, 2, 7, 0, 3, 1, 6]])
    positions, seq = _i32(list(range(first, first + n))), _i32([0] * n)
    got = rows.to(DEV).clone()
    stored = kv_heads > 0
    ops.qk_norm_kv_store(got, ones, ones if stored else None, 1e-5, True, positions, seq, table if stored else None,
                         k_pages if stored else None, v_pages if stored else None, heads, kv_heads, dim, vdim)
    q = plain.unit_rms(raw[:, :heads * dim].reshape(n, heads, dim), 1e-5)
    assert rel_error(got[:, :heads * dim], torch.from_numpy(q.reshape(n, -1))) < KERNEL_TOL[dtype]
    tail = heads * dim + kv_heads * dim
    assert torch.equal(got[:, tail:].cpu(), rows[:, tail:])
    if stored:
        k = plain.unit_rms(raw[:, heads * dim:tail].reshape(n, kv_heads, dim), 1e-5)
        order = table[0].tolist()
        for t in range(n):
            p = first + t
            assert rel_error(k_pages[order[p // page], :, p % page], torch.from_numpy(k[t])) < KERNEL_TOL[dtype]
            assert torch.equal(v_pages[order[p // page], :, p % page].cpu(), rows[t, tail:tail + kv_heads * vdim].reshape(kv_heads, vdim))


def _memory_inputs(rng, total, heads, dim, vdim, dtype, forget=2.0, write=0.0):
    rows = torch.from_numpy(rng.standard_normal((total, 2 * heads * (dim + vdim)))).to(TORCH[dtype])
    gates = torch.from_numpy(np.concatenate([rng.standard_normal((total, heads)) * 2 + write,
                                             rng.standard_normal((total, heads)) * 2 + forget], axis=1)).float()
    return rows, gates, torch.from_numpy(rng.uniform(0.5, 1.5, heads * vdim)).float()


def _memory_reference(rows, gates, norm_w, heads, dim, vdim, cap, eps):
    r, z = rows.double().numpy(), gates.double().numpy()
    n = r.shape[0]
    cut = [heads * dim, 2 * heads * dim, 2 * heads * dim + heads * vdim]
    q, k, v, g = (part.reshape(n, heads, -1) for part in np.split(r, cut, axis=1))
    i = plain.soft_cap(z[:, :heads], cap)
    f = plain.log_sigmoid(plain.soft_cap(z[:, heads:], cap))
    o = np.stack([plain.mlstm_memory(q[:, h] * dim ** -0.5, k[:, h], v[:, h], i[:, h], f[:, h]) for h in range(heads)], axis=1)
    return plain.unit_rms(o, eps).reshape(n, -1) * norm_w.double().numpy() * plain.sigmoid(g.reshape(n, -1))


class _Memory:
    """State of a few requests in slots out of order, every other slot full of junk."""

    def __init__(self, ops, heads, dim, vdim, requests, cap=6.0, eps=1e-5):
        self.ops, self.heads, self.dim, self.vdim, self.cap, self.eps = ops, heads, dim, vdim, cap, eps
        slots = requests + 3
        self.slot_of = {r: (2 * r + 1) % slots for r in range(requests)}
        self.state = torch.full((slots, heads, dim, vdim), 7.5, device=DEV)
        self.normaliser = torch.full((slots, heads, dim), 7.5, device=DEV)
        self.maximum = torch.full((slots, heads), 7.5, device=DEV)
        for slot in self.slot_of.values():
            for t in (self.state, self.normaliser, self.maximum):
                t[slot].zero_()

    def run(self, parts, norm_w):
        """parts: [(request, rows, gates)] -> the readout of the step"""
        counts = [p[1].shape[0] for p in parts]
        q_start = _i32(np.concatenate([[0], np.cumsum(counts)]).tolist())
        slots = _i32([self.slot_of[p[0]] for p in parts])
        return self.ops.mlstm(torch.cat([p[1] for p in parts]).to(DEV), torch.cat([p[2] for p in parts]).to(DEV), self.heads, self.dim,
                              self.vdim, norm_w.to(DEV), self.state, self.normaliser, self.maximum, slots, q_start, counts, self.cap,
                              self.dim ** -0.5, self.eps).float().cpu()

    def junk_untouched(self):
        free = [s for s in range(self.state.shape[0]) if s not in self.slot_of.values()]
        return all(bool((t[free] == 7.5).all()) for t in (self.state, self.normaliser, self.maximum))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(4, 32, 48), (3, 12, 10), (2, 128, 128), (1, 200, 24), (2, 8, 8), (6, 48, 48), (2, 64, 96), (1, 256, 120),
                                           (2, 40, 200), (1, 17, 33)])
def test_matrix_memory_in_portions_batches_and_slots(ops, dtype, heads, dim, vdim):
    """Portions of one to 200 tokens, so that both ways through (token by token, chunks) and their borders are met in one
    request, batched with others, in slots out of order."""
    rng = np.random.default_rng(dim * 10 + vdim)
    lengths = [330, 23, 150]
    cap, eps = 6.0, 1e-5
    data = [_memory_inputs(rng, n, heads, dim, vdim, dtype) for n in lengths]
    norm_w = data[0][2]
    memory = _Memory(ops, heads, dim, vdim, 3, cap, eps)
    cuts = [[(0, 70), (1, 1), (2, 17)], [(2, 1), (0, 1), (1, 2)], [(1, 20), (0, 16)], [(2, 65), (0, 200)], [(0, 2), (2, 2)],
            [(0, 40), (2, 64)], [(0, 1), (2, 1)]]
    got, done = [[] for _ in lengths], [0] * 3
    for step in cuts:
        out = memory.run([(r, data[r][0][done[r]:done[r] + n], data[r][1][done[r]:done[r] + n]) for r, n in step], norm_w)
        at = 0
        for r, n in step:
            got[r].append(out[at:at + n])
            at += n
            done[r] += n
    assert done == lengths and memory.junk_untouched()
    for r in range(3):
        ref = _memory_reference(data[r][0], data[r][1], norm_w, heads, dim, vdim, cap, eps)
        assert rel_error(torch.cat(got[r]), torch.from_numpy(ref)) < (1e-4 if dtype == "float32" else 1e-2), r


def test_chunks_and_single_tokens_leave_the_same_state(ops):
    """The same tokens in one portion (chunks) and one by one: state, normaliser and maximum agree to float32 rounding, so
    the chunk kernels' products lose nothing of the 32-bit factors and states; gates from wide open to nearly shut."""
    heads, dim, vdim, n = 3, 64, 72, 300
    for forget, write in ((6.0, 0.0), (0.0, 3.0), (-5.0, -8.0)):
        rng = np.random.default_rng(5)
        rows, gates, norm_w = _memory_inputs(rng, n, heads, dim, vdim, "bfloat16", forget, write)
        whole, single = _Memory(ops, heads, dim, vdim, 1), _Memory(ops, heads, dim, vdim, 1)
        a = whole.run([(0, rows, gates)], norm_w)
        b = torch.cat([single.run([(0, rows[t:t + 1], gates[t:t + 1])], norm_w) for t in range(n)])
        slot = whole.slot_of[0]
        for name in ("state", "normaliser", "maximum"):
            assert rel_error(getattr(whole, name)[slot], getattr(single, name)[slot]) < 3e-6, (name, forget)
        assert rel_error(a, b) < 6e-3, forget


def test_a_portion_longer_than_the_scratch_memory_holds(ops):
    """More chunks than are worked on at a time, beside a short portion and a second long one."""
    heads, dim, vdim = 1, 16, 16
    lengths = [64 * (ops.MLSTM_WAVE + 7) + 5, 3, 700]
    rng = np.random.default_rng(3)
    data = [_memory_inputs(rng, n, heads, dim, vdim, "bfloat16", forget=4.0) for n in lengths]
    memory = _Memory(ops, heads, dim, vdim, 3)
    got = memory.run([(r, data[r][0], data[r][1]) for r in range(3)], data[0][2])
    at = 0
    for r, n in enumerate(lengths):
        ref = _memory_reference(data[r][0], data[r][1], data[0][2], heads, dim, vdim, memory.cap, memory.eps)
        assert rel_error(got[at:at + n], torch.from_numpy(ref)) < 1e-2, r
        at += n
    assert memory.junk_untouched()


@pytest.mark.parametrize("dtype", DTYPES)
def test_memory_keeps_what_no_gate_closes(ops, dtype):
    """Forget gates wide open: a value written under its own key at the first token is read back 400 tokens later, through
    chunks and single tokens; with its input gate shut it is not."""
    heads, dim, vdim, n = 1, 32, 16, 400
    for write, found in ((5.0, True), (-20.0, False)):
        rng = np.random.default_rng(8)
        rows, gates, norm_w = _memory_inputs(rng, n, heads, dim, vdim, dtype)
        key, value = torch.zeros(dim), torch.linspace(-1.0, 1.0, vdim)
        key[0] = 4.0
        rows[:, dim] = 0.0                                     # no other key has this component
        rows[0, dim:2 * dim] = key
        rows[0, 2 * dim:2 * dim + vdim] = value
        rows[n - 1, :dim] = 20.0 * key
        rows[:, 2 * dim + vdim:] = 30.0                        # the output gate is open
        gates[:, 1] = 40.0                                     # so are the forget gates
        gates[:, 0] = -20.0                                    # and every other input gate is shut
        gates[0, 0] = write
        memory = _Memory(ops, heads, dim, vdim, 1, cap=30.0)
        memory.run([(0, rows[:300], gates[:300])], torch.ones(vdim))
        for t in range(300, n):
            last = memory.run([(0, rows[t:t + 1], gates[t:t + 1])], torch.ones(vdim))
        want = value / (value.pow(2).mean() + 1e-5).sqrt()
        assert (rel_error(last[0], want) < 1e-2) == found, write


@pytest.mark.parametrize("tokens,outputs,top", [(5, 8, 1), (130, 24, 4), (3, 3, 3), (9, 1, 1), (40, 100, 7)])
def test_logistic_router(ops, tokens, outputs, top):
    rng = np.random.default_rng(outputs)
    z = rng.standard_normal((tokens, outputs)) * 3
    z[0] += 40.0                                               # scores that are 1 in float32: the logits still order them
    ids, w = ops.router_topk(_f32(z), None, top, logistic=True, over_sum=False)
    order = np.argsort(-z.astype(np.float32), axis=-1, kind="stable")[:, :top]
    assert ids.cpu().numpy().tolist() == order.tolist()
    assert rel_error(w, torch.from_numpy(plain.sigmoid(np.take_along_axis(z, order, axis=-1)))) < KERNEL_TOL["float32"]
    ids2, w2 = ops.router_topk(_f32(z), None, top, logistic=True)
    assert torch.equal(ids, ids2) and rel_error(w2.sum(dim=1), torch.ones(tokens)) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,ff,experts,top,shared", [(1, 64, 48, 8, 2, 32), (7, 100, 18, 5, 1, None), (16, 128, 64, 8, 4, 64),
                                                             (64, 96, 35, 6, 3, 50), (300, 128, 64, 24, 4, 64), (290, 100, 22, 7, 7, None),
                                                             (40, 64, 32, 64, 1, 16)])
def test_gated_experts_weighed_at_their_input(ops, dtype, tokens, width, ff, experts, top, shared):
    """The three ways through the experts (pair by pair, all experts at once, grouped), against the plain mixture; the
    weight in front of the gate's nonlinearity, not behind it."""
    from aegean_tge_b200.config import PartSpec
    from aegean_tge_b200.parts import FEED_FORWARDS, build_part
    from aegean_tge_b200.parts.base import BuildEnv, StepContext
    rng = np.random.default_rng(tokens + ff)
    W = {"m.router": rng.standard_normal((experts, width)) * 2 * width ** -0.5}
    for name, inner in [(f"e{e}", ff) for e in range(experts)] + ([("shared", shared)] if shared else []):
        W[f"m.{name}.gate"] = rng.standard_normal((inner, width)) * 2 * width ** -0.5
        W[f"m.{name}.up"] = rng.standard_normal((inner, width)) * 2 * width ** -0.5
        W[f"m.{name}.down"] = rng.standard_normal((width, inner)) * inner ** -0.5
    h = rng.standard_normal((tokens, width))
    rounded = (lambda a: torch.from_numpy(a).to(TORCH[dtype]).double().numpy())
    W, h = {k: rounded(v) for k, v in W.items()}, rounded(h)
    mlp = {"expert": {"ff": ff, "limit": 1.3}, "router": {"experts": experts, "top": top}}
    part_shared = None
    if shared:
        mlp["shared"] = {"ff": shared, "limit": 0.8}
        part_shared = PartSpec("clamped_glu", {"hidden_size": width, "intermediate_size": shared, "limit": 0.8})
    env = BuildEnv(dtype=TORCH[dtype], device=DEV, hidden_size=width, max_positions=64, page_size=16, ops=ops)
    params = {"hidden_size": width, "intermediate_size": ff, "experts": experts, "top": top, "activation": "clamped_glu", "limit": 1.3,
              "correction": False, "score": "logistic", "weights_over_sum": False, "weigh": "input", "shared": part_shared}
    part = build_part(FEED_FORWARDS, PartSpec("routed_experts", params), env)
    mine = {"router.weight": W["m.router"]}
    for e in range(experts):
        mine.update({f"experts.{e}.{t}.weight": W[f"m.e{e}.{t}"] for t in ("gate", "up", "down")})
    if shared:
        mine.update({f"shared.{t}.weight": W[f"m.shared.{t}"] for t in ("gate", "up", "down")})
    assert set(mine) == set(part.param_specs())
    part.load({k: torch.from_numpy(v).to(DEV, TORCH[dtype]) for k, v in mine.items()})
    ctx = StepContext(num_tokens=tokens, num_seqs=1, token_ids=None, positions=None, seq_of_token=None, q_start=None, start_pos=None,
                      ctx_len=None, slots=None, block_tables=[], max_q_len=tokens, max_ctx_len=tokens)
    margins = []
    ref = plain.moe_ff(h, W, "m.", mlp, margins)
    got = part.forward_f32(torch.from_numpy(h).to(DEV, TORCH[dtype]), ctx).cpu()
    clear = margins[0] > (1e-4 if dtype == "float32" else 1e-3)        # a choice that rounding cannot turn
    assert clear.any()
    assert rel_error(got[clear], torch.from_numpy(ref[clear])) < 1.5 * KERNEL_TOL[dtype]
    behind = sum(w[:, None] * plain.expert(h, W, f"m.e{0}.", 1.3) for w in [np.full(tokens, 0.5)])
    before = plain.expert(h * 0.5, W, "m.e0.", 1.3)
    assert rel_error(torch.from_numpy(behind), torch.from_numpy(before)) > 0.05          # the place of the weight matters


# ---------------------------------------------------------------------------
# whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_and_first_tokens(folders, oracle, ops, name, dtype):
    engine = _engine(folders, name, dtype)
    run = _Run(engine, dtype)
    for length in (1, 2, 3, 7, 16, 33, 64, 65, 150, 300):
        tokens = _tokens(name, length, salt=500 + length)
        logits = run.step([(length, tokens)])
        engine.runner.finish(length)
        _agree(logits, oracle, name, dtype, tokens, where=length, choices=run.choices(length))
    ops.check_status()
    engine.cache.check()


def _without(config, change):
    altered = json.loads(json.dumps(config))
    change(altered)
    return altered


def test_each_mechanism_changed_would_show(oracle):
    """The oracle with one mechanism changed differs from itself by far more than the tolerance: so the whole-model
    tests would see a kernel that got that mechanism wrong."""
    tokens = _tokens("A", 150, salt=3)
    ref = oracle("A", "float32", tokens)
    def wider_window(c): c["layers"][0]["mixer"]["mask"]["size"] = 41
    def narrower_reader(c): c["layers"][2]["mixer"]["mask"]["size"] = 89
    def one_kept_more(c): c["layers"][0]["mixer"]["mask"]["keep_first"] = 6
    def one_kept_less(c): c["layers"][2]["mixer"]["mask"]["keep_first"] = 20
    def other_far(c): c["layers"][2]["mixer"]["bias_max"] = 38.0
    def other_scale(c): c["layers"][3]["mixer"]["scale"] *= 1.3
    def other_cap(c): c["layers"][1]["mixer"]["gate_cap"] = 5.0
    def other_limit(c): c["layers"][0]["mlp"]["expert"]["limit"] = 1.0
    def other_shared_limit(c): c["layers"][0]["mlp"]["shared"]["limit"] = 1.5
    def other_top(c): c["layers"][1]["mlp"]["router"]["top"] = 3
    def other_alpha(c): c["postln_alpha"] = 1.8
    def no_embedding_scale(c): del c["embedding"]
    for change in (wider_window, narrower_reader, one_kept_more, one_kept_less, other_far, other_scale, other_cap, other_limit,
                   other_shared_limit, other_top, other_alpha, no_embedding_scale):
        assert rel_error(oracle("A", "float32", tokens, config=_without(CONFIGS["A"], change)), ref) > 1e-3, change.__name__


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prefill_against_token_by_token_decoding(folders, oracle, name, dtype):
    tokens = _tokens(name, 110, salt=1)
    engine = _engine(folders, name, dtype)
    run = _Run(engine, dtype)
    rows = [run.step([("r", tokens[:68])])]
    for t in range(68, len(tokens)):
        rows.append(run.step([("r", tokens[t:t + 1])]))
    got = torch.cat(rows)
    _agree(got, oracle, name, dtype, tokens, choices=run.choices("r"))
    if dtype == "float32":
        assert engine.runner.graph_replays > 0
        whole = _engine(folders, name, dtype).runner.step([_portion("w", tokens)])
        assert float((got - whole).abs().max()) <= 2e-5 * float(whole.abs().max())


@pytest.mark.parametrize("name", ["A", "D"])
def test_decode_graphs_give_what_single_steps_give(folders, name):
    """In bfloat16: four requests decoded together, replayed from graphs and run kernel by kernel."""
    prompts = [_tokens(name, n, salt=70 + n) for n in (30, 5, 120, 64)]
    outputs = []
    for graphs in (True, False):
        engine = _engine(folders, name, "bfloat16")
        engine.runner.use_graphs = graphs
        engine.runner.step([_portion(r, p) for r, p in enumerate(prompts)])
        rows = [engine.runner.step([_portion(r, [(7 * t + r) % CONFIGS[name]["vocab"]]) for r in range(4)]) for t in range(20)]
        assert (engine.runner.graph_replays > 0) == graphs
        outputs.append(torch.cat(rows))
    assert rel_error(outputs[0], outputs[1]) < 1e-2      # keys are cut into other runs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("page_size", [16, 64])
def test_portions_down_to_two_tokens(folders, oracle, name, dtype, page_size):
    tokens = _tokens(name, 230, salt=2)
    engine = _engine(folders, name, dtype, page_size=page_size)
    cuts = [7, 2, 16, 3, 2, 30, 2, 17, 41, 1, 1, 26, 2, 64, 5, 2, 2, 7]
    assert sum(cuts) == len(tokens)
    run = _Run(engine, dtype)
    rows, pos = [], 0
    for count in cuts:
        rows.append(run.step([("r", tokens[pos:pos + count])]))
        pos += count
    _agree(torch.cat(rows), oracle, name, dtype, tokens, choices=run.choices("r"))
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("page_size,pool_tokens", [(16, 320), (64, 512)])
def test_unequal_requests_in_one_batch_on_pages_and_slots_that_are_used_again(folders, oracle, ops, name, dtype, page_size,
                                                                            pool_tokens):
    """Up to four live requests in four slots, portions of some beside single tokens of others, a pool so small that
    pages and slots of finished requests serve the next ones; every request's logits are those it gets alone."""
    lengths = {"a": 70, "b": 45, "c": 130, "d": 19, "e": 64, "f": 33, "g": 90}
    tokens = {r: _tokens(name, n, salt=ord(r)) for r, n in lengths.items()}
    engine = _engine(folders, name, dtype, max_tokens=pool_tokens, page_size=page_size, max_requests=4)
    recorder = _Run(engine, dtype)
    got, done = {r: [] for r in lengths}, {r: 0 for r in lengths}
    holders, slot_users = {}, {}

    def run(step):
        logits = recorder.step([(r, tokens[r][done[r]:done[r] + count]) for r, count in step])
        row = 0
        for r, count in step:
            got[r].append(logits[row:row + count])
            row += count
            done[r] += count
            slot_users.setdefault(engine.cache.slot_of(r), set()).add(r)
            for page in engine.cache.groups[0].tables[r]:
                if page >= 0:
                    holders.setdefault(page, set()).add(r)
            if done[r] == lengths[r]:
                engine.runner.finish(r)

    run([("a", 40), ("b", 3)])
    run([("a", 2), ("b", 40), ("c", 64), ("d", 1)])
    run([("a", 28), ("b", 2), ("c", 2), ("d", 16)])          # a and b end
    run([("c", 60), ("d", 2), ("e", 1), ("f", 30)])           # d ends; e and f take over pages and slots
    for _ in range(3):
        run([("c", 1), ("e", 1), ("f", 1)])                   # f ends
    run([("c", 1), ("e", 58), ("g", 2)])
    run([("e", 2), ("g", 64)])                                # c ended before; e ends
    run([("g", 24)])
    ops.check_status()
    engine.cache.check()
    assert any(len(who) > 1 for who in holders.values()) and any(len(who) > 1 for who in slot_users.values())
    assert not engine.cache.live_requests()
    for r in lengths:
        assert done[r] == lengths[r]
        _agree(torch.cat(got[r]), oracle, name, dtype, tokens[r], where=r, choices=recorder.choices(r))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C", "D", "F"])
def test_long_decoding(folders, oracle, name, dtype):
    """Three tokens of prompt, then 330 single tokens through the decode graphs: over many page borders, every window
    wholly past the kept tokens, pages given back behind it, and past the distance where the bias stops changing."""
    tokens = _tokens(name, 333, salt=5)
    engine = _engine(folders, name, dtype, page_size=16)
    run = _Run(engine, dtype)
    rows = [run.step([("r", tokens[:3])])]
    for t in range(3, len(tokens)):
        rows.append(run.step([("r", tokens[t:t + 1])]))
    _agree(torch.cat(rows), oracle, name, dtype, tokens, choices=run.choices("r"))
    if dtype == "float32":
        assert engine.runner.graph_replays > 0
    # pages behind every window were given back, those of the kept tokens were not
    for group in engine.cache.groups:
        if group.spec.window is None:
            continue
        table = group.tables["r"]
        kept, first = -(-group.spec.keep_first // 16), (len(tokens) - group.spec.window + 1) // 16
        assert all(page >= 0 for page in table[:kept]) and all(page >= 0 for page in table[first:])
        assert all(page < 0 for page in table[kept:first])
    engine.cache.check()


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, oracle, name):
    """``Engine.generate`` (scheduler, portions of 16, sampler, steps queued ahead) gives the plain model's greedy
    continuation."""
    engine = _engine(folders, name, "float32", chunk=16, max_batch_tokens=48)
    prompts = [_tokens(name, n, salt=40 + n) for n in (5, 37, 1, 70)]
    outputs = engine.generate(prompts, n=12)
    for prompt, produced in zip(prompts, outputs):
        sequence = list(prompt)
        for token in produced:
            logits = oracle(name, "float32", sequence)[-1]
            best = int(torch.argmax(logits))
            if token != best:          # only a tie within rounding may differ
                assert float(logits[best] - logits[token]) < 1e-4 * float(logits.abs().max()), (name, len(sequence))
            sequence.append(int(token))
        assert len(produced) == 12
    assert not engine.cache.live_requests()
    engine.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sampled_generation_with_requests_that_come_and_go(folders, dtype):
    """Twelve requests with samplers through six slots, then three: the same seeds give the same tokens whatever shared
    a step with what (no state leaks between a slot's users; steps queued ahead and dropped leave none)."""
    from aegean_tge_b200 import SamplingParams
    prompts = [_tokens("A", 3 + 11 * i, salt=300 + i) for i in range(12)]
    params = [SamplingParams(temperature=0.8, top_k=(0, 20, 50)[i % 3], top_p=(1.0, 0.9)[i % 2], seed=40 + i) for i in range(12)]
    outputs = []
    for slots, budget, chunk in ((6, 64, 16), (3, 256, 64)):
        engine = _engine(folders, "A", dtype, max_requests=slots, max_batch_tokens=budget, chunk=chunk, max_tokens=640)
        outputs.append(engine.generate(prompts, n=10, sampling=params))
        assert not engine.cache.live_requests()
        engine.cache.check()
    if dtype == "float32":
        assert outputs[0] == outputs[1]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_of_a_fesorax_model(folders, oracle, tmp_path, dtype):
    """bin/trace_run as a subprocess: two requests, portions and single tokens in one batch, slots given back."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    a, b = _tokens("A", 60, salt=90), _tokens("A", 9, salt=91)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:41], "want": [0]}, {"id": "b", "tokens": b[:7], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[7:], "want": [1]}, {"id": "a", "tokens": a[41:], "want": [18]}], "end": ["a", "b"]}]
    out = tmp_path / "out"
    run = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["A"], "--dtype", dtype,
                          "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    vocab = CONFIGS["A"]["vocab"]
    read = lambda step: torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, vocab))
    _agree(torch.cat([read(0), read(1), read(2)[1:]]), oracle, "A", dtype, a, rows=[0, 39, 40, 59])
    _agree(read(2)[:1], oracle, "A", dtype, b, rows=[8])


def test_command_line_serves_the_design(folders, capsys):
    from aegean_tge_b200.cli import main
    assert main(["generate", "--model", folders["D"], "--tokens", "5 17 3", "--n", "6", "--print-ids", "--context", "128"]) == 0
    out = capsys.readouterr().out
    assert len(out.split("ids      :")[1].split()) == 6
    common = ["--model", folders["D"], "--context", "512", "--max-requests", "12"]
    assert main(["bench", "decode", *common, "--batch", "3", "--prompt-len", "40", "--n", "4"]) == 0
    assert main(["bench", "prefill", *common, "--prompt-len", "100", "--repeat", "1"]) == 0
    assert main(["plan", "--model", folders["A"], "--context", "256", "--sessions", "2"]) == 0
    capsys.readouterr()
