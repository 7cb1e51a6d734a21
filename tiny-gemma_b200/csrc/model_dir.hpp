// A model folder: config.json and model.safetensors. Host only.
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstdint>
#include <cstring>
#include <map>
#include <string>
#include <vector>

#include "json.hpp"

namespace tg {

// model.safetensors, memory-mapped: an 8-byte little-endian header length, that many bytes of JSON
// (name -> dtype, shape, data_offsets), then the data.
class SafeTensors {
	int fd = -1;
	uint8_t *base = nullptr;
	size_t size = 0;

   public:
	struct Tensor {
		std::string dtype;
		std::vector<long long> shape;
		const uint8_t *data = nullptr;
		size_t count() const {
			size_t n = 1;
			for (long long d : shape) n *= size_t(d);
			return n;
		}
		float at(size_t i) const {  // BF16 or F32
			uint32_t b = 0;
			if (dtype == "BF16") {
				uint16_t h;
				std::memcpy(&h, data + 2 * i, 2);
				b = uint32_t(h) << 16;
			} else {
				std::memcpy(&b, data + 4 * i, 4);
			}
			float f;
			std::memcpy(&f, &b, 4);
			return f;
		}
	};
	std::map<std::string, Tensor> tensors;

	SafeTensors() = default;
	SafeTensors(const SafeTensors &) = delete;
	SafeTensors &operator=(const SafeTensors &) = delete;
	~SafeTensors() {
		if (base) munmap(base, size);
		if (fd >= 0) close(fd);
	}

	bool open(const std::string &path, std::string *err) {
		auto bad = [&](const std::string &what) {
			*err = path + ": " + what;
			return false;
		};
		fd = ::open(path.c_str(), O_RDONLY);
		if (fd < 0) {
			*err = "Could not open file. (" + path + ")";
			return false;
		}
		struct stat st;
		if (fstat(fd, &st) != 0 || st.st_size < 8) return bad("too short");
		size = size_t(st.st_size);
		void *p = mmap(nullptr, size, PROT_READ, MAP_PRIVATE, fd, 0);
		if (p == MAP_FAILED) return bad("cannot be mapped");
		base = static_cast<uint8_t *>(p);
		uint64_t hlen;
		std::memcpy(&hlen, base, 8);
		if (hlen > size - 8) return bad("header is longer than the file");
		json::Value head;
		std::string e;
		if (!json::parse(reinterpret_cast<const char *>(base) + 8, hlen, &head, &e) || head.kind != json::Value::OBJECT) return bad("bad header: " + e);
		const uint8_t *data = base + 8 + hlen;
		const size_t avail = size - 8 - hlen;
		for (const auto &m : head.members) {
			if (m.first == "__metadata__") continue;
			Tensor t;
			const json::Value *dt = m.second.find("dtype"), *sh = m.second.find("shape"), *off = m.second.find("data_offsets");
			if (!dt || !sh || !off || off->items.size() != 2) return bad("bad entry " + m.first);
			t.dtype = dt->str;
			size_t n = t.dtype == "BF16" || t.dtype == "F16" ? 2 : (t.dtype == "F32" || t.dtype == "I32" ? 4 : 0);
			for (const auto &d : sh->items) {
				if (d.num < 0 || d.num > 1e12) return bad("bad shape of " + m.first);
				t.shape.push_back((long long)d.num);
			}
			const double a = off->items[0].num, b = off->items[1].num;
			if (a < 0 || b < a || b > double(avail)) return bad("offsets of " + m.first + " lie outside the file");
			if (n && t.count() * n != size_t(b) - size_t(a)) return bad("size of " + m.first + " does not fit its shape");
			t.data = data + size_t(a);
			tensors[m.first] = t;
		}
		return true;
	}
};

}  // namespace tg
