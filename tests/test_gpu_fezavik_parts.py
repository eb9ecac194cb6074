"""Each mechanism of the Fezavik decoder alone, on the device, against its plain function: the norm behind a sublayer with the
residual sum and the next norm; queries and keys normed over their whole projections, neighbours rotated by stretched
frequencies and written to scattered slots; attention with a learned sink, a window and values of another width than keys, in
every kernel that computes it, with keys made to stand out just inside and just outside the window, far back, at page borders
and at the start, in prompts and in decoding; sinks and one gate per head in every form of latent attention; the recurrence
whose forget gate also writes, with its state carried between steps in portions down to one token, in batches of unequal
requests and in slots that are used again; the router with its correction and identity experts on each of the expert paths."""
import math
import types

import pytest
import torch

from helpers import rel_err
from plain import fezavik_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
DTYPES = [torch.float32, torch.bfloat16]


def _weights(part, dtype, std, seed, overrides=None):
    g = torch.Generator().manual_seed(seed)
    w = {}
    for t in part.tensor_specs():
        shape = t.concrete_shape()
        x = 0.95 * torch.rand(shape, generator=g) if t.init == "unit" else std * torch.randn(shape, generator=g)
        w[t.name] = (1.0 + x if t.init == "norm" else x).to(dtype)
    for k, v in (overrides or {}).items():
        w[k] = v.to(dtype)
    part.load({k: v.to(DEV) for k, v in w.items()})
    return {k: v.double() for k, v in w.items()}


# ----------------------------------------------------------------------------- norms

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [8, 33, 50, 320, 512, 1000, 2048, 4100, 8192, 10000, 20000])
def test_norm_behind_a_sublayer_sum_and_next_norm(dtype, H):
    from photon_infer_b200.parts.base import Normed
    from photon_infer_b200.parts.registry import create_part
    g = torch.Generator().manual_seed(H)
    norms, ws = [], []
    for eps in (1e-5, 1e-2):                                        # the two norms have an eps of their own
        norms.append(create_part("norm", "rms_norm", {"size": H, "eps": eps, "weight_name": "w"}))
        ws.append((1 + 0.3 * torch.randn(H, generator=g)).to(dtype))
        norms[-1].load({"w": ws[-1].to(DEV)})
    x, y = 2 * torch.randn(7, H, generator=g), (0.3 * torch.randn(7, H, generator=g)).to(dtype)
    y[2] = 0                                                        # a sublayer that says nothing: eps alone is in the root
    new = x.double() + plain.rms_norm(y.double(), ws[1].double(), 1e-2)
    want = plain.rms_norm(new, ws[0].double(), 1e-5)
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    res = x.to(DEV).clone()
    out = norms[0].add_forward(Normed(y.to(DEV), norms[1]), res, dtype)
    assert out.dtype == dtype and rel_err(out.float().cpu(), want) < tol and rel_err(res.cpu(), new) < 3e-6
    # chosen rows: nothing is written back
    res = x.to(DEV).clone()
    rows = norms[0].add_forward_rows(Normed(y.to(DEV), norms[1]), res, i32([5, 0, 5]), torch.float32)
    assert torch.equal(res.cpu(), x) and rel_err(rows.cpu(), want[[5, 0, 5]]) < (3e-6 if dtype == torch.float32 else 2e-5)
    # what a consumer without the fused kernel gets
    assert rel_err(Normed(y.to(DEV), norms[1]).materialize().cpu(), plain.rms_norm(y.double(), ws[1].double(), 1e-2)) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_layer_between_norms(dtype):
    """The block with a real mixer and feed-forward, and the same without a feed-forward."""
    from photon_infer_b200.parts.registry import create_part
    H, T = 40, 9
    cut = dict(hidden_size=H, heads=2, dim=12, vdim=8, eps=1e-5)
    for with_ff in (True, False):
        mix, names = create_part("mixer", "hgrn2", cut), ["norm1", "norm1b"] + (["norm2", "norm2b"] if with_ff else [])
        w = _weights(mix, dtype, 0.3, 1)
        norms = {n: create_part("norm", "rms_norm", {"size": H, "eps": 1e-5, "weight_name": n}) for n in names}
        nw = {n: _weights(p, dtype, 0.2, i)[n] for i, (n, p) in enumerate(norms.items())}
        ff = create_part("feed_forward", "gated", dict(hidden_size=H, intermediate_size=24, activation="silu", names=("gate", "up", "down"))) if with_ff else None
        fw = _weights(ff, dtype, 0.3, 2) if with_ff else None
        block = create_part("block", "sandwich", dict(norm1=norms["norm1"], mixer=mix, post1=norms["norm1b"], norm2=norms.get("norm2"), feed_forward=ff,
                                                      post2=norms.get("norm2b")))
        x = 2 * torch.randn(T, H, generator=torch.Generator().manual_seed(3))
        want = plain.sandwich(x.double(), lambda h: plain.hgrn2(h, w, dict(heads=2, dim=12, vdim=8), 1e-5), nw["norm1"], nw["norm1b"], 1e-5)
        if with_ff:
            dense = lambda h: ((h @ fw["gate"].T) * torch.sigmoid(h @ fw["gate"].T) * (h @ fw["up"].T)) @ fw["down"].T
            want = plain.sandwich(want, dense, nw["norm2"], nw["norm2b"], 1e-5)
        ctx, lc = _recurrent_step([T], [0], 1, mix, dtype)
        res, delta = block.forward(x.to(DEV), None, ctx, lc)
        assert rel_err((res + delta.materialize()).cpu(), want) < (1e-5 if dtype == torch.float32 else 2e-2)


# ----------------------------------------------------------------------------- queries and keys

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("whole_row", [True, False])
@pytest.mark.parametrize("nq,nkv,d,dv,rot", [(6, 2, 16, 12, 8), (5, 1, 10, 7, 6), (4, 4, 64, 128, 64), (32, 8, 128, 128, 32), (3, 3, 6, 6, 0), (2, 1, 12, 8, 12)])
def test_norm_rotation_and_cache_write(dtype, interleaved, whole_row, nq, nkv, d, dv, rot):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(nq * 100 + d)
    pos = torch.tensor([0, 1, 2, 15, 16, 17, 100, 599, 3000])
    T, page, eps = len(pos), 8, 1e-5
    q, k, v = nq * d, nkv * d, nkv * dv
    rows = (2 * torch.randn(T, q + k + v + 4, generator=g)).to(dtype)             # sections of wider rows
    rows[4] *= 1e-3                                                                # a token whose mean square is of the size of eps
    qw, kw = ((1 + 0.3 * torch.randn(n, generator=g)).to(dtype) for n in ((q, k) if whole_row else (d, d)))
    freqs = plain.frequencies(rot, 500.0, dict(factor=8.0, low=1.0, high=4.0, original=64.0)) if rot else []
    kc, vc = (torch.full((3, nkv, page, n), 7.0, dtype=dtype, device=DEV) for n in (d, dv))
    slots, err = [5, 0, 23, 8, 7, -1, 16, 1, 12], torch.zeros(4, dtype=torch.int32, device=DEV)
    out = torch.empty(T, q, dtype=dtype, device=DEV)
    r = rows.to(DEV)
    inv = torch.tensor(freqs, dtype=torch.float64, device=DEV) if rot else None
    ops.qk_norm_rope_write(r[:, :q], r[:, q:q + k], r[:, q + k:q + k + v], out, qw.to(DEV), kw.to(DEV), eps, pos.int().to(DEV), inv, rot, i32(slots),
                           kc, vc, nq, nkv, d, dv, err, whole_row=whole_row, interleaved=interleaved)
    x = rows.double()
    if whole_row:
        normed = lambda a, w, heads: plain.rms_norm(a, w.double(), eps).view(T, heads, d)
    else:
        normed = lambda a, w, heads: plain.rms_norm(a.view(T, heads, d), w.double(), eps)
    wq = plain.rotate(normed(x[:, :q], qw, nq), pos, freqs, interleaved)
    wk = plain.rotate(normed(x[:, q:q + k], kw, nkv), pos, freqs, interleaved)
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    assert rel_err(out.float().cpu(), wq.reshape(T, q)) < tol and err.cpu().tolist()[0] == 0
    for t, s in enumerate(slots):
        if s >= 0:
            assert rel_err(kc[s // page, :, s % page].float().cpu(), wk[t]) < tol
            assert torch.equal(vc[s // page, :, s % page].cpu(), rows[t, q + k:q + k + v].view(nkv, dv))
    for s in set(range(24)) - set(slots):
        assert torch.all(kc[s // page, :, s % page] == 7.0) and torch.all(vc[s // page, :, s % page] == 7.0)
    # queries alone, for an entry that reads another one's pages
    alone = torch.empty_like(out)
    ops.qk_norm_rope_write(r[:, :q], None, None, alone, qw.to(DEV), kw.to(DEV), eps, pos.int().to(DEV), inv, rot, None, None, None, nq, nkv, d, dv, err,
                           whole_row=whole_row, interleaved=interleaved)
    assert torch.equal(alone, out)


# ----------------------------------------------------------------------------- attention

def _oracle(q, k, v, pos, scale, window, sink):
    """q [n, H, d], k [L, G, d], v [L, G, dv] -> [n, H * dv]."""
    i, j = torch.tensor(pos)[:, None], torch.arange(k.shape[0])[None, :]
    ok = (j <= i) & (i - j < (window or 10 ** 9))
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("nhd,lhd->hnl", q, k.repeat_interleave(rep, 1)) * scale
    p = plain.sink_softmax(s, ok, sink) if sink is not None else torch.softmax(s.masked_fill(~ok[None], -math.inf), -1)
    return torch.einsum("hnl,lhv->nhv", p, v.repeat_interleave(rep, 1)).flatten(1)


class _Step:
    """Requests whose keys and values lie in a paged cache (pages scattered over the pool, stale numbers in unused slots,
    pages behind the window taken away), and a step that brings the last tokens of each."""

    def __init__(self, lengths, counts, nq, nkv, d, dv, page, dtype, seed, std=1.0):
        g = torch.Generator().manual_seed(seed)
        self.lengths, self.counts, self.page, self.dtype, self.dims = lengths, counts, page, dtype, (nq, nkv, d, dv)
        S, per = len(lengths), max(-(-L // page) for L in lengths) + 1
        self.order = torch.randperm(S * per, generator=g).view(S, per).tolist()
        self.k = [(std * torch.randn(L, nkv, d, generator=g)).to(dtype) for L in lengths]
        self.v = [torch.randn(L, nkv, dv, generator=g).to(dtype) for L in lengths]
        self.q = [(std * torch.randn(n, nq, d, generator=g)).to(dtype) for n in counts]
        self.kc, self.vc = ((100.0 * torch.randn(S * per, nkv, page, n, generator=g)).to(dtype) for n in (d, dv))
        self.starts = [L - n for L, n in zip(lengths, counts)]
        self.pos = [list(range(a, L)) for a, L in zip(self.starts, lengths)]

    def ctx(self, window):
        from photon_infer_b200.parts.base import GroupView, StepContext
        for s, L in enumerate(self.lengths):
            for p in range(L):
                self.kc[self.order[s][p // self.page], :, p % self.page] = self.k[s][p]
                self.vc[self.order[s][p // self.page], :, p % self.page] = self.v[s][p]
        self.kcd, self.vcd = self.kc.to(DEV), self.vc.to(DEV)
        table = []
        for s, L in enumerate(self.lengths):
            lo = 0 if not window else max(0, self.starts[s] + 1 - window) // self.page
            table.append([pg if lo <= i and i * self.page < L else -1 for i, pg in enumerate(self.order[s])])
        cu = [0]
        for n in self.counts:
            cu.append(cu[-1] + n)
        seq = [s for s, n in enumerate(self.counts) for _ in range(n)]
        return StepContext(cu[-1], len(self.lengths), self.dtype, i32([0] * cu[-1]), i32(sum(self.pos, [])), i32(seq), i32(cu), i32(self.lengths),
                           i32(list(range(len(self.lengths)))), [GroupView(i32(table), i32([0] * cu[-1]), self.page, self.kc.shape[0], len(table[0]))],
                           self.counts, self.lengths, self.starts, max(self.counts), max(self.lengths), torch.zeros(4, dtype=torch.int32, device=DEV))

    def want(self, scale, window, sink):
        return torch.cat([_oracle(self.q[s].double(), self.k[s].double(), self.v[s].double(), self.pos[s], scale, window, sink)
                          for s in range(len(self.lengths))])

    def run(self, kernel, scale, window, sink, splits=1):
        from photon_infer_b200.kernels import ops
        from photon_infer_b200.parts.attention import attend_tensor_cores
        from photon_infer_b200.parts.base import LayerCache
        nq, nkv, d, dv = self.dims
        ctx = self.ctx(window)
        q = torch.cat(self.q).reshape(-1, nq * d).to(DEV)
        out = torch.full((q.shape[0], nq * dv), float("nan"), dtype=self.dtype, device=DEV)
        sinks = sink.float().to(DEV) if sink is not None else None
        if kernel == "general":
            ops.paged_attention(q, out, self.kcd, self.vcd, ctx.groups[0].block_table, ctx.token_seq, ctx.positions, nq, nkv, d, window, scale,
                                ctx.error_flag, value_dim=dv, splits=splits, sink=sinks)
        else:
            mixer = types.SimpleNamespace(n_q=nq, n_kv=nkv, head_dim=d, value_dim=dv, window=window, scale=scale, _max_groups=None)
            attend_tensor_cores(mixer, q, out, ctx, LayerCache(group=0, k=self.kcd, v=self.vcd), sink=sinks)
        torch.cuda.synchronize()
        assert ctx.error_flag.cpu().tolist()[0] == 0
        return out.float().cpu()


def _sinks(n, seed=0):
    """Scores of the extra key from far below every other to far above them."""
    return torch.tensor([-3.0, 0.0, 2.5, 6.0, -40.0, 1.0, 4.0, 9.0])[torch.arange(n) % 8] + 0.1 * torch.randn(n, generator=torch.Generator().manual_seed(seed))


# a whole short prompt, the end of a long one, single decoded tokens near and far, two tokens
LENGTHS, COUNTS = [33, 150, 97, 200, 1, 300], [33, 50, 1, 2, 1, 1]


@pytest.mark.parametrize("window", [None, 1, 3, 40, 64, 130])
@pytest.mark.parametrize("heads", [(2, 1), (6, 2), (3, 3), (16, 1)])
@pytest.mark.parametrize("kernel,dtype,d,dv,page", [
    ("general", torch.float32, 10, 14, 8), ("general", torch.float32, 64, 48, 16), ("general", torch.bfloat16, 24, 40, 16),
    ("tensor", torch.bfloat16, 64, 64, 16), ("tensor", torch.bfloat16, 128, 128, 16), ("tensor", torch.bfloat16, 64, 32, 16),
    ("tensor", torch.bfloat16, 32, 64, 8), ("tensor", torch.bfloat16, 80, 112, 32), ("tensor", torch.bfloat16, 128, 16, 64),
    ("tensor", torch.bfloat16, 16, 128, 16), ("tensor", torch.bfloat16, 48, 80, 16), ("tensor", torch.bfloat16, 96, 48, 24)])
def test_sinks_windows_and_wide_values_in_every_kernel(window, heads, kernel, dtype, d, dv, page):
    """Pages of 24 fit no tile of the tcgen05 kernel: the other tensor-core kernel takes those portions."""
    nq, nkv = heads
    st = _Step(LENGTHS, COUNTS, nq, nkv, d, dv, page, dtype, seed=nq * 100 + d, std=1.0 if d < 64 else 0.5)
    sink = _sinks(nq)
    scale = 1.3 / math.sqrt(d)
    got, want = st.run(kernel, scale, window, sink), st.want(scale, window, sink.double())
    per_row = (got.double() - want).abs().amax(dim=1) / float(want.abs().max())
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    assert float(per_row.max()) < tol, f"rows off: {(per_row >= tol).nonzero().flatten().tolist()[:10]}, worst {float(per_row.max()):.3g}"


@pytest.mark.parametrize("kernel,d,dv", [("general", 24, 40), ("tensor", 64, 32), ("tensor", 32, 128)])
def test_decoded_tokens_whose_keys_are_shared_out(kernel, d, dv):
    """Long contexts, few requests: shares of a token's keys run in several blocks and are merged; the sink enters the merged
    denominator once."""
    st = _Step([2700, 1, 333, 5200], [1, 1, 1, 1], 4, 2, d, dv, 16, torch.bfloat16, seed=3)
    sink = _sinks(4)
    want = st.want(0.2, None, sink.double())
    for splits in ((1, 3, 64) if kernel == "general" else (1,)):
        assert rel_err(st.run(kernel, 0.2, None, sink, splits=splits), want) < 2e-2


@pytest.mark.parametrize("kernel,dtype,d,dv,page", [("general", torch.float32, 12, 20, 8), ("general", torch.bfloat16, 24, 24, 16),
                                                    ("tensor", torch.bfloat16, 64, 32, 16), ("tensor", torch.bfloat16, 128, 128, 32)])
@pytest.mark.parametrize("count", [1, 2, 40])
def test_keys_that_stand_out_at_every_edge(kernel, dtype, d, dv, page, count):
    """Random keys score about 0.  One key at a time scores high for the LAST token of 333 (decoded alone, or the end of a
    portion): far back and at the start (no window), the first key the window holds, the key just behind it, the token itself,
    keys at both sides of a page border.  Where the rules let the token see it the output is that key's value, less what the
    sink takes; where they do not, it is the oracle's."""
    L, window = 333, 96
    i = L - 1
    places = {"first": (0, None), "far": (1, None), "page_low": ((i - 200) // page * page - 1, None), "page_high": ((i - 200) // page * page, None),
              "window_first": (i - window + 1, window), "window_behind": (i - window, window), "self": (i, window), "before": (i - 1, window)}
    for name, (j, w) in places.items():
        st = _Step([L, 50], [count, 1], 2, 1, d, dv, page, dtype, seed=len(name), std=0.05)
        qdir = st.q[0][-1, 0].double()
        st.k[0][j, 0] = (qdir / qdir.norm() * 40.0).to(dtype)
        st.v[0][j, 0] = torch.full((dv,), 7.0).to(dtype)
        scale, sink = 1.0 / float(qdir.norm()), torch.tensor([math.log(math.exp(40.0) / 3), 0.0])      # score 40; the sink takes a quarter
        got, want = st.run(kernel, scale, w, sink), st.want(scale, w, sink.double())
        row, share = got[count - 1, :dv], want[count - 1, :dv]
        assert float((row - share).abs().max()) < (1e-4 if dtype == torch.float32 else 0.1), name
        assert rel_err(got, want) < (1e-4 if dtype == torch.float32 else 2e-2), name
        if w is None or i - j < w:
            assert float((row - 5.25).abs().max()) < 0.4, f"{name}: key {j} must be seen, the sink beside it"
        else:
            assert float(row.abs().max()) < 0.1, f"{name}: key {j} must not be seen, and the sink takes all"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,d,dv,rot,window", [(6, 2, 16, 32, 8, 40), (3, 3, 10, 7, 10, 5), (4, 1, 64, 16, 32, None), (2, 2, 24, 24, 0, 1)])
def test_the_attention_mixer_in_portions(dtype, heads, kv, d, dv, rot, window):
    """Two unequal requests in portions from 90 tokens down to one, against the whole sequences; the pages are used before."""
    from photon_infer_b200.parts.base import LayerCache
    from photon_infer_b200.parts.registry import create_part
    H = 48
    m = dict(heads=heads, kv_heads=kv, dim=d, vdim=dv, scale=0.9 * d ** -0.5)
    scaling = dict(factor=4.0, low=1.0, high=4.0, original=64.0)
    if rot:
        m["rot"] = dict(base=300.0, dims=rot, scaling=scaling)
    if window:
        m["mask"] = dict(size=window)
    att = create_part("mixer", "normed_attention", dict(
        hidden_size=H, n_q_heads=heads, n_kv_heads=kv, head_dim=d, value_dim=dv, eps=1e-5, scale=m["scale"], window=window, norm_weight=True, norm_scope="row",
        rot_dims=rot, rot_base=300.0, rot_interleaved=True, sink="learned", rot_scaling=dict(
            factor=4.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_position_embeddings=64.0)))
    w = _weights(att, dtype, 0.3, 5, {"sink": _sinks(heads)})
    _portions(att, dtype, H, window, lambda h, pos: plain.attention(h, w, m, pos, 1e-5), (kv, d, dv))


def _portions(att, dtype, H, window, oracle, kv=None):
    """``kv``: (heads, key width, value width) of a cache with two planes; None: one row per token."""
    from photon_infer_b200.parts.base import LayerCache
    lens, ps = [150, 77], 8
    g = torch.Generator().manual_seed(6)
    hs = [torch.randn(L, H, generator=g).to(dtype) for L in lens]
    want = [oracle(h.double(), torch.arange(len(h))) for h in hs]
    pages = Pages(2, 20, ps, kv or (1, att.width, None), dtype, seed=3)
    got, starts = [[], []], [0, 0]
    for k, cut in enumerate([(33, 2), (2, 40), (1, 1), (90, 3), (1, 1), (23, 30)]):
        order = [1, 0] if k % 2 else [0, 1]
        ctx = pages.context(cut, starts, dtype, window, order)
        out = att.forward(torch.cat([hs[r][starts[r]:starts[r] + cut[r]] for r in order]).to(DEV), ctx, LayerCache(group=0, k=pages.k, v=pages.v)).float().cpu()
        assert ctx.error_flag.cpu().tolist()[0] == 0
        a = 0
        for r in order:
            got[r].append(out[a:a + cut[r]])
            a += cut[r]
        starts = [starts[r] + cut[r] for r in range(2)]
    for r in range(2):
        assert rel_err(torch.cat(got[r]), want[r]) < (2e-5 if dtype == torch.float32 else 3e-2)


class Pages:
    """Scattered pages for several requests, in a pool that is filled with stale numbers."""

    def __init__(self, requests, each, page_size, widths, dtype, seed):
        g = torch.Generator().manual_seed(seed)
        heads, kw, vw = widths
        self.ps, self.n = page_size, requests * each
        self.perm = torch.randperm(self.n, generator=g).view(requests, each).tolist()
        pool = lambda w: (50 * torch.randn(self.n, heads, page_size, w, generator=g)).to(dtype).to(DEV)
        self.k, self.v = pool(kw), pool(vw) if vw else None

    def fill(self, request, rows):
        """Stores the rows (one head) of positions 0 .. of a request."""
        idx = torch.tensor([self.perm[request][p // self.ps] * self.ps + p % self.ps for p in range(len(rows))], device=DEV)
        self.k.view(-1, rows.shape[1])[idx] = rows.to(self.k.dtype).to(DEV)

    def context(self, cut, starts, dtype, window=None, order=None):
        from photon_infer_b200.parts.base import GroupView, StepContext
        order = list(range(len(cut))) if order is None else order
        pos, seq, sm, tables = [], [], [], []
        for s, r in enumerate(order):
            first = 0 if window is None else max(0, starts[r] + 1 - window) // self.ps
            tables.append([p if i >= first else -1 for i, p in enumerate(self.perm[r])])
            for p in range(starts[r], starts[r] + cut[r]):
                pos.append(p); seq.append(s); sm.append(self.perm[r][p // self.ps] * self.ps + p % self.ps)
        lens, st = [cut[r] for r in order], [starts[r] for r in order]
        ends = [a + b for a, b in zip(lens, st)]
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        return StepContext(sum(lens), len(lens), dtype, i32([0] * sum(lens)), i32(pos), i32(seq), i32(cu), i32(ends), i32(list(range(len(lens)))),
                           [GroupView(i32(tables), i32(sm), self.ps, self.n, len(tables[0]))], lens, ends, st, max(lens), max(ends),
                           torch.zeros(4, dtype=torch.int32, device=DEV))


# ----------------------------------------------------------------------------- latent attention

def _latent(dtype, heads, dim, rot, vdim, kv_rank, q_rank, window, H=48, base=300.0, rot_dims=None, seed=5, std=0.3):
    from photon_infer_b200.parts.registry import create_part
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=0.8 * (dim + rot) ** -0.5,
             rot=dict(base=base, dims=rot if rot_dims is None else rot_dims))
    if window:
        m["mask"] = dict(size=window)
    att = create_part("mixer", "latent_attention", dict(hidden_size=H, heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                                                        scale=m["scale"], eps=1e-5, rot_base=base, rot_dims=m["rot"]["dims"], window=window,
                                                        output_gate="head", sink=True))
    return att, m, _weights(att, dtype, std, seed, {"sink": _sinks(heads)})


SHAPES = [dict(heads=3, dim=16, rot=8, vdim=24, kv_rank=24, q_rank=40),            # general kernel
          dict(heads=5, dim=16, rot=16, vdim=24, kv_rank=32, q_rank=24),           # tensor-core decoding, half a tile of heads
          dict(heads=18, dim=8, rot=32, vdim=8, kv_rank=64, q_rank=16, rot_dims=20),   # more heads than a tile, part of the rotated part turns
          dict(heads=2, dim=7, rot=6, vdim=9, kv_rank=13, q_rank=11)]              # multiples of nothing


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [None, 1, 2, 33, 100])
@pytest.mark.parametrize("expand", [False, True])
def test_latent_attention_in_portions(monkeypatch, dtype, shape, window, expand):
    """Sinks and one gate per head in every form: the general kernel, tensor-core decoding, products and a softmax, and
    (``expand``) keys and values formed from the rows."""
    from photon_infer_b200.parts import latent_attention
    if expand and (dtype == torch.float32 or shape["vdim"] % 8 or shape["dim"] % 8):
        pytest.skip("only bfloat16 with sizes of 8s expands rows")
    if expand:
        def every_long(self, ctx, lens, dtype):
            starts = ctx.host_start_positions
            return {i: (starts[i], starts[i] + n - self._first_seen(starts[i])) for i, n in enumerate(lens) if n >= 32}
        monkeypatch.setattr(latent_attention.LatentAttention, "_expanded_requests", every_long)
    else:
        monkeypatch.setattr(latent_attention, "USE_EXPANDED_PROMPTS", False)
    att, m, w = _latent(dtype, window=window, **shape)
    _portions(att, dtype, 48, window, lambda h, pos: plain.latent_attention(h, w, m, pos, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 5, 64, 65, 129])
@pytest.mark.parametrize("count", [1, 3, 40])
def test_a_row_just_inside_and_just_outside_the_window(dtype, window, count):
    """One cached row fits every query, at each distance around the window's edge and with the asking token at several places
    of a page and of the kernels' tiles: inside it shares the weight with the sink, one further the sink has nearly all."""
    from photon_infer_b200.parts.base import LayerCache
    heads, kr, rot, ps, n = 4, 32, 16, 8, 330
    att, m, _ = _latent(dtype, heads, 16, rot, 16, kr, 24, window)
    att.scale = 1.0
    sink = torch.tensor([9.8, 9.0, 0.0, 12.0])
    att.sinks = sink.to(DEV)
    width = kr + rot
    g = torch.Generator().manual_seed(window)
    rows = torch.randn(n, width, generator=g)
    rows = 0.2 * rows / rows.norm(dim=1, keepdim=True)
    special = torch.randn(width, generator=g)
    special = special / special.norm()
    pages = Pages(1, 48, ps, (1, width, None), dtype, seed=window)
    for asking in (window + 3, 191, 192, 255, 256, 257, 300, 329):
        for back in sorted({0, 1, window - 1, window, window + 1}):
            target = asking - back
            if target < 0 or back < 0:
                continue
            keys = rows.clone()
            keys[target] = special
            first = max(0, asking + 1 - count)
            m1 = asking + 1 - first
            pages.fill(0, keys)
            ctx = pages.context([m1], [first], dtype, window)
            q = torch.zeros(m1, heads, width)
            q[-1] = 10.0 * special
            out = torch.empty(m1, heads * kr, dtype=dtype, device=DEV)
            att.attend(q.to(dtype).to(DEV), out, ctx, LayerCache(group=0, k=pages.k))
            assert ctx.error_flag.cpu().tolist()[0] == 0
            kd = keys.to(dtype).double()
            lo = max(0, asking + 1 - window)
            s = (q[-1].to(dtype).double() @ kd.T)[:, lo:asking + 1]
            p = plain.sink_softmax(s[:, None, :], torch.ones(1, s.shape[1], dtype=torch.bool), sink.double())[:, 0]
            want = p @ kd[lo:asking + 1, :kr]
            got = out[-1].float().cpu().view(heads, kr)
            assert float((got - want).abs().max()) < (2e-5 if dtype == torch.float32 else 1e-2) * 0.3, (asking, back)
            if back < window:
                assert 0.05 < float(p[0, target - lo]) < 0.6        # row and sink side by side


@pytest.mark.parametrize("sizes", [(64, 16, 64), (128, 64, 128), (16, 16, 24), (72, 8, 80)])
@pytest.mark.parametrize("window", [None, 1, 65, 200])
@pytest.mark.parametrize("gate_heads", [True, False])
def test_long_portions_over_expanded_rows(sizes, window, gate_heads):
    """The tcgen05 kernel alone: sinks from far below to far above the scores, a gate per head in a column of unaligned rows
    or a gate per number; for some queries one key stands out at the window's edges."""
    from photon_infer_b200.kernels import ops
    d, r, v = sizes
    heads = 5
    g = torch.Generator().manual_seed(d + (window or 0))
    reqs = [(40, 0), (300, 517), (129, 130)]                        # (tokens, position of the first)
    T = sum(n for n, _ in reqs)
    q = torch.randn(T, heads, d + r, generator=g)
    seqs, kus, krs, vs, t, row = [], [], [], [], 0, 0
    for n, start in reqs:
        base = 0 if window is None else max(0, start + 1 - window)
        L = start + n - base
        ku, kr, vv = 0.3 * torch.randn(L, heads, d, generator=g), 0.3 * torch.randn(L, r, generator=g), torch.randn(L, heads, v, generator=g)
        for i in range(0, n, 7):
            lo = 0 if window is None else max(0, start + i + 1 - window)
            k = start + i - [0, start + i - lo, start + i - lo + 1, (window or 40) - 1, (window or 40)][(i // 7) % 5] - base
            if 0 <= k < L:
                q[t + i, :, :d] = ku[k] / 0.3 * (5.0 / d ** 0.5)
                q[t + i, :, d:] = kr[k] / 0.3 * (5.0 / r ** 0.5)
        seqs.append((t, n, start, base, row))
        kus.append(ku.bfloat16()); krs.append(kr.bfloat16()); vs.append(vv.bfloat16())
        t += n
        row += L
    q = q.bfloat16()
    kv = torch.cat([torch.cat([a.reshape(len(a), -1), c.reshape(len(c), -1)], 1) for a, c in zip(kus, vs)])
    gw = heads if gate_heads else heads * v
    wide = (2 * torch.randn(T, gw + (3 if gate_heads else 16), generator=g)).bfloat16()
    gate = wide.to(DEV)[:, 3:] if gate_heads else wide.to(DEV)[:, 16:]
    sink = _sinks(heads)
    out = torch.empty(T, heads * v, dtype=torch.bfloat16, device=DEV)
    err = torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.latent_prompt_attention(q.reshape(T, -1).to(DEV), q[:, :, d:].contiguous().to(DEV), kv.to(DEV), torch.cat(krs).to(DEV), out, seqs, heads, d, r, v,
                                window, 0.8, err, gate=gate, sink=sink.to(DEV))
    assert err.cpu().tolist()[0] == 0
    out = out.float().cpu()
    for (t, n, start, base, row), ku, kr, vv in zip(seqs, kus, krs, vs):
        p, k = start + torch.arange(n)[:, None], base + torch.arange(len(ku))[None, :]
        ok = (k <= p) & (p - k < (window or 10 ** 9))
        qq = q[t:t + n].double()
        s = (torch.einsum("nhd,lhd->hnl", qq[..., :d], ku.double()) + torch.einsum("nhr,lr->hnl", qq[..., d:], kr.double())) * 0.8
        want = torch.einsum("hnl,lhv->nhv", plain.sink_softmax(s, ok, sink.double()), vv.double())
        want = want * torch.sigmoid(gate.double().cpu()[t:t + n]).view(n, heads, -1)
        assert rel_err(out[t:t + n].view(n, heads, v), want) < 1.5e-2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 3, 9, 16, 40])
def test_one_gate_per_head_behind_the_products(dtype, T):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(T)
    heads, K, N = 3, 40, 20
    x, w = torch.randn(T, heads, K, generator=g).to(dtype), (0.3 * torch.randn(heads, N, K, generator=g)).to(dtype)
    wide = (3 * torch.randn(T, heads + 2, generator=g)).to(dtype)
    out = torch.empty(T, heads, N, dtype=dtype, device=DEV)
    ops.head_linear(x.to(DEV), w.to(DEV), out, gate=wide.to(DEV)[:, 1:1 + heads])
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(wide[:, 1:1 + heads].double())[..., None]
    assert rel_err(out.float().cpu(), want) < (5e-6 if dtype == torch.float32 else 1e-2)
    y = torch.randn(T, heads * N, generator=g).to(dtype).to(DEV)
    want = y.double().cpu().view(T, heads, N) * torch.sigmoid(wide[:, 1:1 + heads].double())[..., None]
    ops.gate_mul(y, wide.to(DEV)[:, 1:1 + heads])
    assert rel_err(y.float().cpu().view(T, heads, N), want) < (3e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_softmax_rows_with_sinks(dtype):
    from photon_infer_b200.kernels import ops
    heads, tokens, first_pos, first_key, window = 5, 21, 40, 16, 19
    cols = first_pos + tokens - first_key + 3
    s = 3 * torch.randn(tokens * heads, cols, generator=torch.Generator().manual_seed(1))
    sink, probs = _sinks(heads), torch.full(s.shape, float("nan"), dtype=dtype, device=DEV)
    ops.causal_softmax_rows(s.to(DEV), probs, heads, first_pos, 0.7, first_key=first_key, window=window, sink=sink.to(DEV))
    p, k = first_pos + torch.arange(tokens)[:, None], first_key + torch.arange(cols)[None, :]
    ok = (k <= p) & (p - k < window)
    want = plain.sink_softmax(0.7 * s.double().view(tokens, heads, cols).transpose(0, 1), ok, sink.double()).transpose(0, 1).reshape(-1, cols)
    assert rel_err(probs.float().cpu(), want) < (3e-6 if dtype == torch.float32 else 5e-3)


# ----------------------------------------------------------------------------- recurrence

def _recurrent_step(counts, slots, num_slots, mixer, dtype, state=None):
    """A step of requests that bring ``counts`` tokens, in state slots ``slots``."""
    from photon_infer_b200.parts.base import LayerCache, StepContext
    cu = [0]
    for n in counts:
        cu.append(cu[-1] + n)
    seq = [s for s, n in enumerate(counts) for _ in range(n)]
    if state is None:
        state = torch.zeros((num_slots,) + tuple(mixer.state_spec().shape), device=DEV)
    ctx = StepContext(cu[-1], len(counts), dtype, i32([0] * cu[-1]), i32([0] * cu[-1]), i32(seq), i32(cu), i32(counts), i32(slots), [], counts, counts,
                      [0] * len(counts), max(counts), max(counts), torch.zeros(4, dtype=torch.int32, device=DEV), None, slots)
    return ctx, LayerCache(state=state)


GRN = [(1, 4, 3), (2, 12, 20), (3, 9, 33), (2, 48, 16), (1, 128, 128), (4, 64, 40), (1, 200, 17)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", GRN)
def test_forget_and_write_in_portions_and_batches(dtype, heads, dim, vdim):
    """Three unequal requests in portions (70 tokens down to one, gates formed in the kernel or in their own pass), states in
    slots in another order than the requests; some are left out of a step; then one ends and its slot, cleared, goes on with
    another request."""
    from photon_infer_b200.parts.registry import create_part
    H, eps = 40, 1e-5
    mix = create_part("mixer", "hgrn2", dict(hidden_size=H, heads=heads, dim=dim, vdim=vdim, eps=eps))
    m = dict(heads=heads, dim=dim, vdim=vdim)
    low = torch.rand(heads * dim, generator=torch.Generator().manual_seed(2)) * 0.99
    low[0] = 0.0
    w = _weights(mix, dtype, 0.4, dim, {"lower": low, "f.b": 2 * torch.randn(heads * dim, generator=torch.Generator().manual_seed(3))})
    g = torch.Generator().manual_seed(6)
    hs = [torch.randn(L, H, generator=g).to(dtype) for L in (120, 47, 66)]
    want = [plain.hgrn2(h.double(), w, m, eps) for h in hs]
    state = 30 * torch.randn((5,) + tuple(mix.state_spec().shape), generator=g).to(DEV)      # stale numbers in every slot
    slots, got, starts = [3, 0, 4], [[], [], []], [0, 0, 0]
    for s in slots:
        state[s] = 0
    kept = state[[1, 2]].clone()
    for cut in [(33, 2, 0), (2, 1, 5), (1, 30, 1), (70, 0, 16), (1, 1, 17), (13, 13, 27)]:
        live = [r for r in (1, 2, 0) if cut[r]]
        ctx, lc = _recurrent_step([cut[r] for r in live], [slots[r] for r in live], 5, mix, dtype, state)
        out = mix.forward(torch.cat([hs[r][starts[r]:starts[r] + cut[r]] for r in live]).to(DEV), ctx, lc).float().cpu()
        assert ctx.error_flag.cpu().tolist()[0] == 0
        a = 0
        for r in live:
            got[r].append(out[a:a + cut[r]])
            a += cut[r]
            starts[r] += cut[r]
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    for r in range(3):
        assert rel_err(torch.cat(got[r]), want[r]) < tol, r
    assert torch.equal(state[[1, 2]], kept)
    # the same request in one portion, token by token, and in the first one's slot: equal bits in float32
    state[3] = 0
    ctx, lc = _recurrent_step([47], [3], 5, mix, dtype, state)
    whole = mix.forward(hs[1].to(DEV), ctx, lc).float().cpu()
    state[4] = 0
    single = []
    for t in range(47):
        ctx, lc = _recurrent_step([1], [4], 5, mix, dtype, state)
        single.append(mix.forward(hs[1][t:t + 1].to(DEV), ctx, lc).float().cpu())
    if dtype == torch.float32:
        assert torch.equal(torch.cat(single), whole) and torch.equal(torch.cat(got[1]), whole) and torch.equal(state[3], state[4])
    else:
        assert rel_err(torch.cat(single), whole) < tol
    # a negative slot: from zero, nothing is stored
    before = state.clone()
    ctx, lc = _recurrent_step([47], [-1], 5, mix, dtype, state)
    assert torch.equal(mix.forward(hs[1].to(DEV), ctx, lc).float().cpu(), whole) and torch.equal(state, before)


def test_gates_close_to_their_bounds():
    """Gates that forget nothing (bounds close to 1, large biases) keep a first token's value over 600 tokens, and gates that
    forget all keep the last one alone; both without cancellation in 1 - f."""
    from photon_infer_b200.kernels import ops
    T, d, v = 600, 8, 5
    g = torch.Generator().manual_seed(1)
    q, z, val = torch.randn(T, d, generator=g), 0.5 * torch.randn(T, d, generator=g), torch.randn(T, v, generator=g)
    val[0] *= 300
    bias = torch.tensor([0.0, 9.0, 12.0, -20.0, 14.0, 5.0, -3.0, 30.0])
    low = torch.tensor([0.0, 0.0, 0.99, 0.0, 0.999, 0.5, 0.3, 0.0])
    f = (low + (1 - low) * torch.sigmoid(z.double() + bias.double()))[:, None]
    sq = (q * torch.sigmoid(q)).double()[:, None]
    want, S = plain.hgrn2_states(sq, f, val.double()[:, None])
    for prepared in (False, True):
        state, o = torch.zeros(1, d * v, device=DEV), torch.empty(T, v, device=DEV)
        qd, kd, b, l = q.to(DEV), z.to(DEV), bias.to(DEV), low.to(DEV)
        if prepared:
            y = torch.empty(T, 2 * d, device=DEV)
            ops.linrec_gates(qd, kd, b, l, y[:, :d], y[:, d:])
            qd, kd, b, l = y[:, :d], y[:, d:], None, None
        ops.linrec("forget_write", qd, kd, val.to(DEV), None, None, b, l, None, 0.0, 1.0, i32([0, T]), i32([0]), state, o, 1, 1, 1, d, v, None)
        assert rel_err(o.cpu(), want[:, 0]) < 3e-6
        per_row = (state.cpu().view(d, v).double() - S[0]).abs().amax(1) / S[0].abs().amax(1)
        assert float(per_row[:7].max()) < 2e-5                     # row 7 writes 1e-13 of every value: nothing to compare with


# ----------------------------------------------------------------------------- experts

@pytest.mark.parametrize("E,I,top", [(6, 2, 2), (8, 0, 1), (4, 4, 4), (12, 1, 5), (40, 0, 3), (64, 16, 8), (1, 3, 2), (300, 20, 6), (1, 0, 1), (3, 1, 4)])
@pytest.mark.parametrize("rows", [1, 5, 70])
def test_router_with_correction_and_identity_experts(E, I, top, rows):
    from photon_infer_b200.kernels import ops
    g = torch.Generator().manual_seed(E + rows)
    h, wr = torch.randn(rows, 48, generator=g), 0.3 * torch.randn(E + I, 48, generator=g)
    corr = torch.randn(E + I, generator=g) / (E + I)                # of the size of the scores: it changes many choices
    want_ids, want_w = plain.route(h.double(), dict(router=wr.double(), correction=corr.double()), top)
    ids, weights, counts = ops.moe_route(h.to(DEV), wr.to(DEV), None, top, "softmax_raw", correction=corr.to(DEV), identity=I)
    assert torch.equal(ids.cpu().long(), want_ids) and rel_err(weights.cpu(), want_w) < 1e-5
    every = torch.bincount(want_ids.flatten(), minlength=E + I)
    assert counts.cpu().tolist() == every[:E].tolist() + ([int(every[E:].sum())] if I else [])
    # without the correction the choice is the scores' own
    ids, weights, _ = ops.moe_route(h.to(DEV), wr.to(DEV), None, top, "softmax_raw", identity=I)
    want_ids, want_w = plain.route(h.double(), dict(router=wr.double(), correction=torch.zeros(E + I).double()), top)
    assert torch.equal(ids.cpu().long(), want_ids) and rel_err(weights.cpu(), want_w) < 1e-5


def test_equal_choice_scores_go_to_the_lower_index():
    from photon_infer_b200.kernels import ops
    h, wr = torch.ones(1, 8, device=DEV), torch.zeros(70, 8, device=DEV)
    corr = torch.zeros(70)
    corr[[66, 5, 33]] = 1.0
    ids, weights, _ = ops.moe_route(h, wr, None, 5, "softmax_raw", correction=corr.to(DEV))
    assert ids.cpu().tolist() == [[5, 33, 66, 0, 1]] and torch.allclose(weights.cpu(), torch.full((1, 5), 1 / 70))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,I,top,ff,H,rows", [(6, 2, 2, 32, 64, 5), (8, 0, 1, 24, 48, 3), (4, 4, 4, 14, 50, 40), (5, 2, 3, 64, 96, 400), (3, 1, 1, 40, 64, 90),
                                                (40, 9, 2, 16, 56, 200), (1, 1, 2, 128, 256, 1), (1, 7, 4, 16, 64, 300)])
def test_experts_with_identity(dtype, E, I, top, ff, H, rows):
    """Each of the expert paths (pair by pair, own grouped product, the library's grouped product), with few and with mostly
    identity experts chosen; the plain side gets the router's choice."""
    from photon_infer_b200.kernels import ops
    from photon_infer_b200.parts.registry import create_part
    part = create_part("feed_forward", "moe", dict(hidden_size=H, experts=E, top=top, expert_size=ff, router_bias=False, scoring="softmax_raw",
                                                   correction=True, identity=I))
    w = _weights(part, dtype, 0.3, E + rows)
    h = torch.randn(rows, H, generator=torch.Generator().manual_seed(rows)).to(dtype)
    chosen, route = [], ops.moe_route
    ops.moe_route = lambda *a, **k: chosen.append(route(*a, **k)) or chosen[-1]
    try:
        got = part.forward(h.to(DEV), None).float().cpu()
    finally:
        ops.moe_route = route
    ids = chosen[0][0].long().cpu()
    want = plain.moe_ff(h.double(), w, dict(router=dict(top=top, experts=E)), ids)
    assert rel_err(got, want) < (1e-5 if dtype == torch.float32 else 2.5e-2)
    if I and rows > 30:
        assert 0 < int((ids >= E).sum()) < ids.numel()              # both kinds occur


def test_a_step_whose_tokens_all_choose_identity_experts():
    """No row for any product on any path; the output is the row times its weights."""
    from photon_infer_b200.parts.registry import create_part
    for rows in (3, 40, 300):
        part = create_part("feed_forward", "moe", dict(hidden_size=64, experts=2, top=2, expert_size=16, router_bias=False, scoring="softmax_raw",
                                                       correction=True, identity=3))
        w = _weights(part, torch.bfloat16, 0.2, 1, {"correction": torch.tensor([-9.0, -9.0, 0.0, 0.0, 0.0])})
        h = torch.randn(rows, 64, generator=torch.Generator().manual_seed(rows)).bfloat16()
        got = part.forward(h.to(DEV), None).float().cpu()
        ids, weights = plain.route(h.double(), w, 2)
        assert int(ids.min()) >= 2 and rel_err(got, h.double() * weights.sum(1, keepdim=True)) < 1e-2
