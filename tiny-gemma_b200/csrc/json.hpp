// A small JSON reader for model folders (config.json, the header of a safetensors file). Host only.
#pragma once
#include <cstdio>
#include <cstdlib>
#include <string>
#include <utility>
#include <vector>

namespace json {

struct Value {
	enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
	bool b = false;
	double num = 0.0;
	std::string str;
	std::vector<Value> items;                            // ARRAY
	std::vector<std::pair<std::string, Value>> members;  // OBJECT

	const Value *find(const std::string &key) const {  // null if absent or JSON null
		for (const auto &m : members)
			if (m.first == key) return m.second.kind == NUL ? nullptr : &m.second;
		return nullptr;
	}
};

class Parser {
	const char *p, *end;
	std::string *err;
	int depth = 0;
	bool bad(const char *what) {
		if (err->empty()) *err = what;
		return false;
	}
	void ws() {
		while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
	}
	bool lit(const char *s) {
		const char *q = p;
		while (*s) {
			if (q == end || *q != *s) return bad("bad literal");
			q++;
			s++;
		}
		p = q;
		return true;
	}
	static void utf8(std::string *o, unsigned c) {
		if (c < 0x80) {
			o->push_back(char(c));
		} else if (c < 0x800) {
			o->push_back(char(0xC0 | (c >> 6)));
			o->push_back(char(0x80 | (c & 63)));
		} else {
			o->push_back(char(0xE0 | (c >> 12)));
			o->push_back(char(0x80 | ((c >> 6) & 63)));
			o->push_back(char(0x80 | (c & 63)));
		}
	}
	bool string(std::string *o) {
		if (p == end || *p != '"') return bad("expected a string");
		for (p++; p < end && *p != '"'; p++) {
			if (*p != '\\') {
				o->push_back(*p);
				continue;
			}
			if (++p == end) return bad("unterminated string");
			switch (*p) {
				case 'b': o->push_back('\b'); break;
				case 'f': o->push_back('\f'); break;
				case 'n': o->push_back('\n'); break;
				case 'r': o->push_back('\r'); break;
				case 't': o->push_back('\t'); break;
				case 'u': {
					if (end - p < 5) return bad("bad \\u escape");
					unsigned c = 0;
					for (int i = 1; i <= 4; i++) {
						const char h = p[i];
						const int v = h >= '0' && h <= '9' ? h - '0' : (h >= 'a' && h <= 'f' ? h - 'a' + 10 : (h >= 'A' && h <= 'F' ? h - 'A' + 10 : -1));
						if (v < 0) return bad("bad \\u escape");
						c = c * 16 + unsigned(v);
					}
					utf8(o, c);
					p += 4;
					break;
				}
				default: o->push_back(*p);
			}
		}
		if (p == end) return bad("unterminated string");
		p++;
		return true;
	}
	bool value(Value *v) {
		ws();
		if (p == end) return bad("unexpected end");
		if (++depth > 64) return bad("nested too deeply");
		bool ok = true;
		if (*p == '{') {
			v->kind = Value::OBJECT;
			p++;
			ws();
			if (p < end && *p == '}') {
				p++;
			} else {
				for (;;) {
					std::pair<std::string, Value> m;
					ws();
					if (!string(&m.first)) return false;
					ws();
					if (p == end || *p != ':') return bad("expected ':'");
					p++;
					if (!value(&m.second)) return false;
					v->members.push_back(std::move(m));
					ws();
					if (p < end && *p == ',') {
						p++;
						continue;
					}
					if (p < end && *p == '}') {
						p++;
						break;
					}
					return bad("expected ',' or '}'");
				}
			}
		} else if (*p == '[') {
			v->kind = Value::ARRAY;
			p++;
			ws();
			if (p < end && *p == ']') {
				p++;
			} else {
				for (;;) {
					v->items.emplace_back();
					if (!value(&v->items.back())) return false;
					ws();
					if (p < end && *p == ',') {
						p++;
						continue;
					}
					if (p < end && *p == ']') {
						p++;
						break;
					}
					return bad("expected ',' or ']'");
				}
			}
		} else if (*p == '"') {
			v->kind = Value::STRING;
			ok = string(&v->str);
		} else if (*p == 't' || *p == 'f') {
			v->kind = Value::BOOL;
			v->b = *p == 't';
			ok = lit(v->b ? "true" : "false");
		} else if (*p == 'n') {
			ok = lit("null");
		} else {
			const std::string tok(p, size_t(end - p < 64 ? end - p : 64));
			char *e = nullptr;
			v->kind = Value::NUMBER;
			v->num = std::strtod(tok.c_str(), &e);
			if (e == tok.c_str()) return bad("expected a value");
			p += e - tok.c_str();
		}
		depth--;
		return ok;
	}

   public:
	Parser(const char *s, size_t n, std::string *e) : p(s), end(s + n), err(e) {}
	bool document(Value *v) {
		if (!value(v)) return false;
		ws();
		return p == end ? true : bad("text after the document");
	}
};

inline bool parse(const char *s, size_t n, Value *v, std::string *err) {
	err->clear();
	return Parser(s, n, err).document(v);
}

inline bool parse_file(const std::string &path, Value *v, std::string *err) {
	FILE *f = std::fopen(path.c_str(), "rb");
	if (!f) {
		*err = "Could not open file. (" + path + ")";
		return false;
	}
	std::string text;
	char buf[65536];
	size_t n;
	while ((n = std::fread(buf, 1, sizeof(buf), f)) > 0) text.append(buf, n);
	std::fclose(f);
	std::string e;
	if (parse(text.data(), text.size(), v, &e)) return true;
	*err = path + ": " + e;
	return false;
}

}  // namespace json
