// Host-side sizes of the NVFP4 scale-atom layout, shared by every kernel that reads or writes it.

extern "C" int telb_nvfp4_k64_pad(int k) { return ((k + 255) / 256) * 4; }

// Bytes of an atom-layout scale buffer for `rows` x `k`.
extern "C" long long telb_nvfp4_sf_bytes(long long rows, int k) {
    return ((rows + 127) / 128) * (long long)telb_nvfp4_k64_pad(k) * 512;
}
