"""Each mechanism of the bfloat16-weight decoders alone, through the C ABI, against the plain implementation in
tests/sonuzen_plain.py (float64)."""
import ctypes as C

import numpy as np
import pytest

import sonuzen_plain as sp
from conftest import load_pkg
from device_data import EPS, Dev, pad8, rel, weights

pytestmark = pytest.mark.gpu
pkg = load_pkg()


# ---- products --------------------------------------------------------------------------------

@pytest.mark.parametrize("rows,cols,batch", [(8, 8, 1), (7, 24, 1), (192, 256, 3), (333, 76, 1), (1000, 1544, 2), (333, 1032, 1), (35, 2200, 1), (7, 8456, 2), (64, 4300, 1), (1, 5000, 1)])
def test_gemv_bf16_is_exact_in_f32(gpu, rows, cols, batch):
    rng = np.random.default_rng(rows)
    w, x = weights(rng, rows, cols), rng.standard_normal((batch, pad8(cols))).astype(np.float32)
    with Dev(gpu) as d:
        out = d.zeros(batch * rows * 4)
        d.call("lv_gemv_bf16", out, rows, d.bf16(w), rows, pad8(cols), cols, d.f32(x), pad8(cols), batch, 0.75, 0)
        got = d.get(out, (batch, rows))
    want = 0.75 * x[:, :cols].astype(np.float64) @ w.T.astype(np.float64)
    assert rel(got, want) < 1e-6


@pytest.mark.parametrize("rows,cols,batch", [(64, 64, 2), (7, 24, 3), (200, 72, 17), (560, 264, 40), (128, 328, 64), (1000, 520, 300), (300, 40, 129),
                                             (96, 4096, 5)])
@pytest.mark.parametrize("out_bf16", [False, True])
def test_gemm_bf16(gpu, rows, cols, batch, out_bf16):
    rng = np.random.default_rng(rows + batch)
    w, x = weights(rng, rows, cols), weights(rng, batch, cols, scale=1.0)
    with Dev(gpu) as d:
        out = d.zeros(batch * rows * 4)
        d.call("lv_gemm_bf16", out, pkg.TYPE_BF16 if out_bf16 else pkg.TYPE_F32, rows, d.bf16(w), rows, pad8(cols), cols, d.bf16(x), pad8(cols), batch, 0.5, 0)
        got = d.get(out, (batch, rows), out_bf16)
    want = 0.5 * x.astype(np.float64) @ w.T.astype(np.float64)
    assert rel(got, want) < (3e-3 if out_bf16 else 2e-5)


def expert_args(d, w0, w1, rows, cols, table, ids, pos, vocab):
    n, top = w0.shape[0], table.shape[1]
    a = pkg.ExpertArgs()
    a.w0 = d.bf16(w0.reshape(-1, w0.shape[-1])).value
    a.w1 = d.bf16(w1.reshape(-1, w1.shape[-1])).value if w1 is not None else None
    a.ld, a.rows, a.cols, a.experts, a.top, a.vocab = pad8(cols), rows, cols, n, top, vocab
    a.table = d.u32(table).value
    a.token_log = d.u32(np.concatenate([np.full(pos, vocab - 1), ids])).value
    a.pos = d.u32([pos] * 4).value
    return a


def draw_table(rng, vocab, n, top):
    return np.stack([rng.permutation(n)[:top] for _ in range(vocab)]).astype(np.int32)


@pytest.mark.parametrize("width,ff,n,top,batch", [(64, 40, 5, 2, 1), (48, 96, 3, 1, 2), (136, 72, 9, 3, 23), (64, 200, 4, 4, 70), (96, 32, 70, 2, 300),
                                                  (64, 64, 3, 2, 290)])
def test_experts_chosen_by_token(gpu, width, ff, n, top, batch):
    rng = np.random.default_rng(width + batch)
    vocab, pos = 50, 3
    gate, up, down = weights(rng, n, ff, width), weights(rng, n, ff, width), weights(rng, n, width, ff)
    table, ids = draw_table(rng, vocab, n, top), rng.integers(0, vocab, batch)
    if batch > 100:
        ids[:80] = ids[0]                                  # one expert with many rows
    x = weights(rng, batch, width, scale=1.0)
    want = sp.table_moe(x.astype(np.float64), ids, table, [(gate[e].astype(np.float64), up[e].astype(np.float64), down[e].astype(np.float64)) for e in range(n)])
    with Dev(gpu) as d:
        gu = expert_args(d, gate, up, ff, width, table, ids, pos, vocab)
        dn = expert_args(d, down, None, width, ff, table, ids, pos, vocab)
        xp = np.zeros((batch, pad8(width)), np.float32)
        xp[:, :width] = x
        act, out = d.zeros(batch * top * pad8(ff) * 4), d.zeros(batch * top * width * 4)
        d.call("lv_gemv_bf16_expert_gate_up", act, pad8(ff), C.byref(gu), d.f32(xp), pad8(width), batch)
        d.call("lv_gemv_bf16_expert_down", out, width, C.byref(dn), act, pad8(ff), batch)
        assert rel(d.get(out, (batch, width)), want) < 2e-6
        if batch == 1:
            return
        max_tiles = gpu.lib.lv_expert_max_tiles(batch, top, n)
        index, tiles = d.zeros(batch * top * 4), d.zeros(max_tiles * 12)
        job = np.zeros(1, np.dtype([("table", "u8"), ("experts", "u4"), ("top", "u4"), ("index", "u8"), ("tiles", "u8"), ("max_tiles", "u4"), ("unused", "u4")]))
        job[0] = (gu.table, n, top, index.value, tiles.value, max_tiles, 0)
        d.call("lv_expert_route", d.up(job), 1, n, gu.token_log, gu.pos, vocab, batch)
        rows = gpu.download(index, np.uint32, batch * top).reshape(batch, top)
        assert sorted(rows.ravel()) == list(range(batch * top))
        listed = gpu.download(tiles, np.uint32, max_tiles * 3).reshape(-1, 3)
        assert listed[:, 2].sum() == batch * top and listed[:, 2].max() <= gpu.lib.lv_expert_tile_rows(batch, top, n)
        expert_of = np.full(batch * top, -1)
        for e, r0, k in listed:
            expert_of[r0:r0 + k] = e
        assert np.array_equal(expert_of[rows], table[ids])
        xs = np.zeros((batch * top, width), np.float32)
        for s in range(top):
            xs[rows[:, s]] = x
        act16 = d.zeros(batch * top * pad8(ff) * 2)
        d.call("lv_gemm_bf16_expert_gate_up", act16, pad8(ff), C.byref(gu), tiles, d.bf16(xs), pad8(width), batch)
        d.call("lv_gemm_bf16_expert_down", out, width, C.byref(dn), tiles, act16, pad8(ff), batch)
        got = d.get(out, (batch * top, width))[rows].mean(axis=1)
    assert rel(got, want) < 5e-3                            # the activations between the products are bfloat16


# ---- norm, residual and convolution -----------------------------------------------------------

@pytest.mark.parametrize("width,taps,cuts", [(64, 4, [1] * 9), (72, 4, [9]), (2056, 3, [2, 1, 5, 1]), (100, 6, [3, 2, 1, 1, 13]), (64, 1, [4, 1]),
                                             (40, 9, [2, 2, 1, 20]), (64, 2, [7])])
def test_norm_conv_in_portions(gpu, width, taps, cuts):
    rng = np.random.default_rng(width * taps)
    T = sum(cuts)
    vocab = 20
    embed, ids = weights(rng, vocab, width, scale=1.0), rng.integers(0, vocab, T)
    post, pre, pre2 = rng.standard_normal((3, width)).astype(np.float32) * 0.3
    step, conv, conv2 = rng.standard_normal(width).astype(np.float32), rng.standard_normal((width, taps)).astype(np.float32), rng.standard_normal((width, taps)).astype(np.float32)
    y = rng.standard_normal((2 * T, width)).astype(np.float32)      # two rows per token, in some order
    order = rng.permutation(2 * T).reshape(T, 2)
    mult = 0.37
    # plain
    x0 = embed[ids].astype(np.float64)
    x0s = x0 + step
    h0 = sp.norm_one_plus(x0s, pre.astype(np.float64), EPS)
    want0 = h0 + sp.causal_conv(h0, conv.astype(np.float64))
    ym = y[order].astype(np.float64).mean(axis=1)
    x1 = x0s + mult * sp.norm_one_plus(ym, post.astype(np.float64), EPS)
    h1 = sp.norm_one_plus(x1, pre2.astype(np.float64), EPS)
    want1 = h1 + sp.causal_conv(h1, conv2.astype(np.float64))
    with Dev(gpu) as d:
        log = d.u32(ids)
        keep = max(taps - 1, 1)
        garbage = np.full((keep, width), np.nan, np.float32)          # entries before the start must not be read
        hist, hist2 = d.f32(garbage), d.f32(garbage)
        emb, dpost, dpre, dpre2, dstep = d.bf16(embed), d.f32(post), d.f32(pre), d.f32(pre2), d.f32(step)
        dconv, dconv2 = d.f32(conv.T), d.f32(conv2.T)
        at = 0
        for n in cuts:
            pos = d.u32([at] * 4)
            xa, xb, tr = d.zeros(n * width * 4), d.zeros(n * width * 4), d.zeros(n * width * 4)
            out = d.zeros(n * pad8(width) * 4)
            a = pkg.NormConvArgs(embed=emb.value, embed_ld=pad8(width), vocab=vocab, token_log=log.value, pos=pos.value, eps=EPS, mult=mult, step=dstep.value,
                                 x_out=xa.value, row_factor=d.zeros(n * 4).value, pre_w=dpre.value, conv_w=dconv.value, history=hist.value, taps=taps, out=out.value, out_type=pkg.TYPE_F32,
                                 out_ld=pad8(width), width=width, batch=n, y_rows=1)
            d.call("lv_norm_conv", C.byref(a))
            assert rel(d.get(out, (n, pad8(width)))[:, :width], want0[at:at + n]) < 2e-6
            # second sublayer: two rows per token averaged, scattered bfloat16 output
            y_at = d.f32(y)
            index = d.u32(order[at:at + n])
            rows = rng.permutation(3 * n).reshape(n, 3)
            out16 = d.zeros(3 * n * pad8(width) * 2)
            b = pkg.NormConvArgs(x=xa.value, pos=pos.value, y=y_at.value, y_index=index.value, y_rows=2, post_w=dpost.value, eps=EPS, mult=mult, trace=tr.value,
                                 x_out=(xa if n == 1 else xb).value, row_factor=d.zeros(n * 4).value, pre_w=dpre2.value, conv_w=dconv2.value, history=hist2.value, taps=taps, out=out16.value,
                                 out_type=pkg.TYPE_BF16, out_ld=pad8(width), out_index=d.u32(rows).value, out_copies=3, width=width, batch=n)
            d.call("lv_norm_conv", C.byref(b))
            assert rel(d.get(tr, (n, width)), x1[at:at + n]) < 1e-6
            assert rel(d.get(xa if n == 1 else xb, (n, width)), x1[at:at + n]) < 1e-6
            got = d.get(out16, (3 * n, pad8(width)), True)[:, :width]
            for s in range(3):
                assert rel(got[rows[:, s]], want1[at:at + n]) < 3e-3
            at += n


def test_norm_without_convolution_of_the_last_row(gpu):
    rng = np.random.default_rng(5)
    n, width = 6, 96
    x, pre = rng.standard_normal((n, width)).astype(np.float32), rng.standard_normal(width).astype(np.float32)
    with Dev(gpu) as d:
        out = d.zeros(width * 4)
        a = pkg.NormConvArgs(x=d.f32(x).value, pos=d.u32([0] * 4).value, eps=0.3, pre_w=d.f32(pre).value, out=out.value, out_type=pkg.TYPE_F32, out_ld=width,
                             width=width, first=n - 1, batch=n, y_rows=1)
        d.call("lv_norm_conv", C.byref(a))
        want = sp.norm_one_plus(x[-1].astype(np.float64), pre.astype(np.float64), 0.3)
        assert rel(d.get(out, (width,)), want) < 1e-6


# ---- gated recurrence ------------------------------------------------------------------------

@pytest.mark.parametrize("width,channels,cuts", [(64, 40, [1] * 6), (48, 70, [50, 1, 2, 33]), (64, 33, [2, 100, 1, 1]), (32, 8, [700])])
def test_min_gru_steps_and_scan(gpu, width, channels, cuts):
    rng = np.random.default_rng(channels)
    T = sum(cuts)
    w = weights(rng, 3 * channels, width)
    w[:channels] *= 4                                     # gates from nearly closed to nearly open: long and short memory
    bz, bx = (rng.standard_normal((2, channels)) * 2).astype(np.float32)
    h = rng.standard_normal((T, width)).astype(np.float32)
    z, u, g = np.split(h.astype(np.float64) @ w.T.astype(np.float64), 3, axis=1)
    want = sp.min_gru(z + bz, u + bx, g)
    with Dev(gpu) as d:
        dw, dbz, dbx = d.bf16(w), d.f32(bz), d.f32(bx)
        state = d.f32(np.full(channels, np.nan))          # position 0 starts from zero whatever the memory holds
        ld, at = pad8(width), 0
        for n in cuts:
            pos = d.u32([at] * 4)
            hp = np.zeros((n, ld), np.float32)
            hp[:, :width] = h[at:at + n]
            x = d.f32(hp)
            out = d.zeros(n * pad8(channels) * 4)
            if n == 1:
                each = channels * ld * 2
                d.call("lv_gemv_bf16_mingru", out, dw, pkg.offset(dw, each), pkg.offset(dw, 2 * each), ld, channels, width, dbz, dbx, x, state, pos)
            else:
                raw = d.zeros(n * 3 * channels * 4)
                d.call("lv_gemv_bf16", raw, 3 * channels, dw, 3 * channels, ld, width, x, ld, n, 1.0, 0)
                d.call("lv_mingru_scan", out, pkg.TYPE_F32, pad8(channels), raw, 3 * channels, channels, dbz, dbx, state, pos, n)
            assert rel(d.get(out, (n, pad8(channels)))[:, :channels], want[at:at + n]) < 1e-5
            at += n


# ---- attention -------------------------------------------------------------------------------

class Attention:
    """One sequence through lv_qk_norm_append / lv_attention_gqa in portions."""

    def __init__(self, d, rng, H, G, dim, vdim, rows, f32, scale, sink=True):
        self.d, self.H, self.G, self.dim, self.vdim, self.rows, self.f32, self.scale, self.sink = d, H, G, dim, vdim, rows, f32, scale, sink
        self.qn, self.kn = (1 + 0.5 * rng.standard_normal((2, dim))).astype(np.float32)
        self.r1 = np.linspace(0.1, 1.3, H).astype(np.float32)
        self.r2 = np.geomspace(0.02, 2.0, H).astype(np.float32)
        item = 4 if f32 else 2
        self.kc = d.up(np.full(G * rows * pad8(dim) * item, 0xFF, np.uint8))      # NaNs: only rows up to the position may be read
        self.vc = d.up(np.full(G * rows * pad8(vdim) * item, 0xFF, np.uint8))
        self.weights = [d.f32(v) for v in (self.qn, self.kn, self.r1, self.r2)]
        self.ld = (H + G) * dim + G * vdim
        self.scratch = None

    def args(self, raw, pos, out, bf16_out=False):
        qn, kn, r1, r2 = self.weights
        t = pkg.TYPE_F32 if self.f32 else pkg.TYPE_BF16
        return pkg.GqaArgs(qkv=raw.value if raw else None, qkv_ld=self.ld, heads=self.H, kv_heads=self.G, dim=self.dim, vdim=self.vdim, scale=self.scale, eps=EPS,
                           q_norm=qn.value, k_norm=kn.value, r1=r1.value, r2=r2.value, sink=int(self.sink), k_cache=self.kc.value, v_cache=self.vc.value,
                           cache_type=t, ctx_rows=self.rows, pos=pos.value if pos else None, out=out.value if out else None,
                           out_type=pkg.TYPE_BF16 if bf16_out else pkg.TYPE_F32, out_ld=pad8(self.H * self.vdim))

    def run(self, raw, at, bf16_out=False):
        d, n = self.d, raw.shape[0]
        pos, dr, out = d.u32([at] * 4), d.f32(raw), d.zeros(n * pad8(self.H * self.vdim) * 4)
        a = self.args(dr, pos, out, bf16_out)
        if self.scratch is None:
            self.bytes = d.gpu.lib.lv_gqa_scratch_bytes(d.gpu.handle, C.byref(a), 512, self.rows)
            self.scratch = d.zeros(self.bytes)
        if n > 1:
            d.call("lv_qk_norm_append", C.byref(a), n)
        d.call("lv_attention_gqa", C.byref(a), self.scratch, self.bytes, n, self.rows, int(n == 1))
        return d.get(out, (n, pad8(self.H * self.vdim)), bf16_out)[:, :self.H * self.vdim]

    def plain(self, raw):
        T = raw.shape[0]
        r = raw.astype(np.float64)
        q = sp.norm_plain(r[:, :self.H * self.dim].reshape(T, self.H, self.dim), self.qn.astype(np.float64), EPS)
        k = sp.norm_plain(r[:, self.H * self.dim:(self.H + self.G) * self.dim].reshape(T, self.G, self.dim), self.kn.astype(np.float64), EPS)
        v = r[:, (self.H + self.G) * self.dim:].reshape(T, self.G, self.vdim)
        if self.sink:
            return sp.attention(q, k, v, self.r1.astype(np.float64), self.r2.astype(np.float64), self.scale)
        g = self.H // self.G
        s = np.einsum("ihd,jhd->hij", q, np.repeat(k, g, axis=1)) * self.scale - sp.distance_bias(self.r1.astype(np.float64), self.r2.astype(np.float64), T)
        s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
        p = np.exp(s - s.max(axis=-1, keepdims=True))
        return np.einsum("hij,jhd->ihd", p / p.sum(axis=-1, keepdims=True), np.repeat(v, g, axis=1)).reshape(T, -1)


@pytest.mark.parametrize("H,G,dim,vdim,cuts", [
    (4, 1, 72, 64, [1] * 12), (4, 4, 24, 40, [5, 1, 1, 9]), (6, 2, 48, 80, [130, 1, 2, 1, 127, 1]), (8, 1, 96, 32, [300, 1, 1]), (3, 1, 128, 128, [64, 65, 1]),
    (10, 1, 32, 16, [2, 2, 129, 1, 1, 1]), (16, 2, 20, 36, [40, 1, 30]), (2, 1, 256, 256, [20, 1, 3]), (4, 2, 160, 96, [40, 1, 90]), (66, 1, 16, 16, [5, 1, 70])])
@pytest.mark.parametrize("f32", [True, False])
def test_attention_in_portions(gpu, H, G, dim, vdim, cuts, f32):
    rng = np.random.default_rng(H * dim + vdim)
    T = sum(cuts)
    with Dev(gpu) as d:
        at = Attention(d, rng, H, G, dim, vdim, 512, f32, scale=1.7 / dim ** 0.5)
        raw = rng.standard_normal((T, at.ld)).astype(np.float32)
        want, done = at.plain(raw), 0
        for n in cuts:
            got = at.run(raw[done:done + n], done, bf16_out=not f32 and n > 1)
            assert rel(got, want[done:done + n]) < (3e-6 if f32 else 8e-3), (done, n)
            done += n


@pytest.mark.parametrize("sink", [True, False])
def test_the_first_token_sees_itself_and_the_sink(gpu, sink):
    rng = np.random.default_rng(3)
    with Dev(gpu) as d:
        at = Attention(d, rng, 2, 1, 16, 24, 128, True, scale=0.2, sink=sink)
        raw = rng.standard_normal((1, at.ld)).astype(np.float32)
        assert rel(at.run(raw, 0), at.plain(raw)) < 1e-6
        if not sink:
            assert rel(at.run(raw, 0), np.tile(raw[:, -24:], 2)) < 1e-6


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("n", [1, 3, 40])
def test_a_single_far_key_is_found(gpu, f32, n):
    """One key among several hundred stands out for the last queries; a key that is missed, doubled or shifted shows at once."""
    rng = np.random.default_rng(11)
    H, G, dim, vdim, T = 4, 2, 64, 48, 530
    for far in (0, 1, 127, 128, 129, 255, 256, 383, 384, T - n - 1):
        with Dev(gpu) as d:
            at = Attention(d, rng, H, G, dim, vdim, 640, f32, scale=1.0)
            raw = rng.standard_normal((T, at.ld)).astype(np.float32)
            mark = rng.standard_normal(dim)
            raw[far, H * dim:(H + G) * dim] = np.tile(mark, G) * 4
            for i in range(T - n, T):
                raw[i, :H * dim] = np.tile(mark, H) * 4
            want = at.plain(raw)
            at.run(raw[:T - n], 0)
            got = at.run(raw[T - n:], T - n)
            assert rel(got, want[T - n:]) < (1e-5 if f32 else 1e-2), far
            own = raw[far, (H + G) * dim:].reshape(G, vdim).repeat(H // G, axis=0).ravel()
            assert np.corrcoef(got[-1], own)[0, 1] > 0.9


def test_positions_outside_the_cache_are_refused_on_the_device(gpu):
    rng = np.random.default_rng(1)
    with Dev(gpu) as d:
        at = Attention(d, rng, 2, 1, 16, 16, 128, True, scale=1.0)
        raw = rng.standard_normal((1, at.ld)).astype(np.float32)
        with pytest.raises(pkg.LvError) as e:
            at.run(raw, 128)
        assert e.value.code == pkg.LV_ERR_DEVICE_WAIT


def test_bad_arguments_are_refused(gpu):
    lib, h = gpu.lib, gpu.handle
    bad = pkg.LV_ERR_BAD_ARGUMENTS
    with Dev(gpu) as d:
        b = d.zeros(1 << 16)
        assert lib.lv_gemm_bf16(h, b, pkg.TYPE_F32, 8, b, 8, 12, 12, b, 16, 2, 1.0, 0) == bad          # ld not a multiple of 8
        assert lib.lv_gemv_bf16(h, b, 4, b, 8, 16, 16, b, 16, 1, 1.0, 0) == bad                        # out_ld below the rows
        a = pkg.NormConvArgs(pos=b.value, pre_w=b.value, out=b.value, width=8, batch=1, out_type=pkg.TYPE_F32)
        assert lib.lv_norm_conv(h, C.byref(a)) == bad                                               # no stream
        g = pkg.GqaArgs(qkv=b.value, qkv_ld=4096, heads=3, kv_heads=2, dim=16, vdim=16)
        assert lib.lv_attention_gqa(h, C.byref(g), b, 1 << 16, 1, 128, 1) == bad                    # heads not a multiple of kv_heads
