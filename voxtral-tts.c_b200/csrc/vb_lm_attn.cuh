/*
 * vb_lm_attn.cuh - device helpers that the attention kernels of the decoder language models share
 * (vb_lm_attn.cu, vb_lm_latent.cu): cache elements, rotation angles, visible key tiles, warp-level
 * tensor-core pieces.
 */
#ifndef VB_LM_ATTN_CUH
#define VB_LM_ATTN_CUH

#include "vb_lm_kernels.cuh"

namespace vb {

/* ------------------------------------------------------------------ cache elements */
VB_DEVINL void hilo(float v, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi = __bfloat16_as_ushort(h);
    lo = __bfloat16_as_ushort(__float2bfloat16_rn(v - __bfloat162float(h)));
}
/* `head`: a head's part of a cache row, `size` elements in either form. */
VB_DEVINL void kv_put(float *head, int size, int d, float v, int split) {
    if (split) {
        uint32_t hi, lo;
        hilo(v, hi, lo);
        uint16_t *h = reinterpret_cast<uint16_t *>(head);
        h[d] = (uint16_t)hi;
        h[size + d] = (uint16_t)lo;
    } else {
        head[d] = v;
    }
}
VB_DEVINL void kv_put4(float *head, int size, int d, float4 v, int split) {
    if (split) {
        uint32_t h[4], l[4];
        hilo(v.x, h[0], l[0]); hilo(v.y, h[1], l[1]); hilo(v.z, h[2], l[2]); hilo(v.w, h[3], l[3]);
        uint16_t *p = reinterpret_cast<uint16_t *>(head);
        *reinterpret_cast<uint2 *>(p + d) = make_uint2(h[0] | (h[1] << 16), h[2] | (h[3] << 16));
        *reinterpret_cast<uint2 *>(p + size + d) = make_uint2(l[0] | (l[1] << 16), l[2] | (l[3] << 16));
    } else {
        *reinterpret_cast<float4 *>(head + d) = v;
    }
}
VB_DEVINL float kv_get(const float *head, int size, int d, int split) {
    if (!split) return __ldcg(head + d);
    const unsigned short *h = reinterpret_cast<const unsigned short *>(head);
    return __uint_as_float((uint32_t)__ldcg(h + d) << 16) + __uint_as_float((uint32_t)__ldcg(h + size + d) << 16);
}
template <bool SPLIT>
VB_DEVINL float4 kv_get4(const float *head, int size, int d) {
    if constexpr (!SPLIT) return vb_ldcg4(head + d);
    const uint16_t *h = reinterpret_cast<const uint16_t *>(head);
    const uint2 hi = __ldcg(reinterpret_cast<const uint2 *>(h + d)), lo = __ldcg(reinterpret_cast<const uint2 *>(h + size + d));
    return make_float4(vb_bf16_lo(hi.x) + vb_bf16_lo(lo.x), vb_bf16_hi(hi.x) + vb_bf16_hi(lo.x), vb_bf16_lo(hi.y) + vb_bf16_lo(lo.y),
                       vb_bf16_hi(hi.y) + vb_bf16_hi(lo.y));
}

/* Cosine and sine of pos * f: the angle to twice fp32's precision (f as a high and a low part), sine and cosine of its
 * leading part and the remainder as a first-order correction. */
VB_DEVINL void lm_angle(int pos, float f_hi, float f_lo, float mag, float *cos_out, float *sin_out) {
    const float p = (float)pos;
    const float hi = p * f_hi, lo = fmaf(p, f_hi, -hi) + p * f_lo;
    float s, c;
    sincosf(hi, &s, &c);
    *cos_out = (c - s * lo) * mag;
    *sin_out = (s + c * lo) * mag;
}

/* ------------------------------------------------------------------ which keys */
/* Keys that rows at positions [imin, imax] may see: [0, a_end) and [b0, b_end), in tiles of KT. */
struct KeyTiles {
    int a_end, b0, b_end, a_tiles, n_tiles;
};
template <int KT>
VB_DEVINL KeyTiles key_tiles(int imin, int imax, int window, int keep) {
    KeyTiles t;
    t.b_end = imax + 1;
    if (window <= 0) { t.a_end = 0; t.b0 = 0; }
    else {
        t.a_end = keep < t.b_end ? keep : t.b_end;
        t.b0 = imin - window + 1 > t.a_end ? imin - window + 1 : t.a_end;
    }
    t.a_tiles = (t.a_end + KT - 1) / KT;
    t.n_tiles = t.a_tiles + (t.b_end > t.b0 ? (t.b_end - t.b0 + KT - 1) / KT : 0);
    return t;
}
/* First key of tile t and how many keys it has. */
template <int KT>
VB_DEVINL void key_tile(const KeyTiles &k, int t, int *j0, int *n) {
    const bool first = t < k.a_tiles;
    const int s = first ? t * KT : k.b0 + (t - k.a_tiles) * KT, e = first ? k.a_end : k.b_end;
    *j0 = s;
    *n = e - s < KT ? e - s : KT;
}
VB_DEVINL bool key_seen(int i, int j, int window, int keep) {
    return j <= i && (window <= 0 || i - j < window || j < keep);
}

/* ------------------------------------------------------------------ warp-level tensor cores */
VB_DEVINL void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
VB_DEVINL void ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
VB_DEVINL void ldsm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
/* Byte offset of the 16-byte chunk `chunk` of key row `key` in a [keys][16 * STEPS] BF16 tile; chunks are
 * XOR-swizzled by the key so that eight rows of one chunk column hit eight different banks. */
template <int STEPS>
VB_DEVINL uint32_t tile_off(int key, int chunk) {
    return (uint32_t)(key * STEPS * 32 + (((chunk & ~7) | ((chunk ^ key) & 7)) << 4));
}

VB_DEVINL void lm_cp16(void *smem_dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(vb_smem_u32(smem_dst)), "l"(src) : "memory");
}
VB_DEVINL void lm_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
VB_DEVINL void lm_cp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

} // namespace vb

#endif
